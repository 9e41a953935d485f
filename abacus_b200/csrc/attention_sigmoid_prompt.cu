// Attention without a softmax for whole prompts (attention_sigmoid.cu has the formulas): bfloat16, every sequence of the
// step from its first token, keys and values from the step's own rows.
//
// The heads' weights are mixed per (token, key), so a CTA needs every head's scores of a tile at once. It has 16 query rows,
// all heads' queries in shared memory, a warp to each of (up to 16) output heads, and walks tiles of 16 * KG keys:
//   scores    warp w multiplies heads w, w + NW, ... with the tile's keys (mma.sync), makes the weights and leaves them in
//             shared memory, by query row: [head][key], float32
//   mixing    a warp takes a query row's 16 keys: [16 heads out x heads in] x [heads in x 8 keys] on the tensor cores, the
//             weights as three bfloat16 parts that hold their 24 bits, the mixing matrix in bfloat16 (as stored). What
//             comes out is split into three parts again and put where the weights were
//   values    warp w adds the mixed weights of its head times the tile's values, the product taken three times, once a part
// With more than 16 heads a CTA has 16 of the output heads (blockIdx.y) and makes all heads' scores for itself.
//
// Queries, keys and values come in by TMA as boxes of 64 columns of one head (128-byte swizzle, zeros beyond a head's last
// column), keys and values through rings of one or two stages each.
//
// Runs of keys add up (nothing is normalized over them), so the tiles of a query row can be dealt to the CTAs of a
// cluster: each sums its tiles' contributions and they are added at the end through distributed shared memory, in rank
// order. A step with few query rows gets clusters of up to 8, so that it fills the GPU.
#define ABK_DEFINE_ERROR
#include "common.cuh"
#include "attention_sigmoid.cuh"
#include "mma_tiles.cuh"
#include "tc_common.cuh"
#include "tensor_map.cuh"

#define SP_ROWS 16
#define SP_MAX_KS 2    // heads / 16 that are mixed: up to 32 heads
#define SP_MAX_HEADS (16 * SP_MAX_KS)

struct SigmoidPrompt {
    __nv_bfloat16 *out;           // [tokens, n_heads * v_dim]
    int n_heads, n_kv_heads, head_dim, v_dim;
    float scale, softcap;
    const float *slopes, *shift;  // [n_heads] or null
    const float *mix;             // [n_heads, n_heads] (out, in), bfloat16 numbers, or null
    const int *seq_start;         // [n_seqs + 1]
    int n_seqs, tiles;            // tiles: the grid's query tiles
    int kv_block;                 // kv heads an output block's values come from, at most
    int k_stages, v_stages;       // 1 or 2
    int *status;
};

// Bytes of the parts of shared memory.
struct SigmoidPromptSmem {
    int k_boxes, v_boxes, q, k, v, chunk, total;
    __host__ __device__ SigmoidPromptSmem(int H, int G, int D, int VD, int kv_block, int NW, int KG, int k_stages, int v_stages) {
        const int keys = 16 * KG, heads_in = (H + 15) / 16 * 16;
        k_boxes = (D + 63) / 64, v_boxes = (VD + 63) / 64;
        q = H * k_boxes * SP_ROWS * 128, k = G * k_boxes * keys * 128, v = kv_block * v_boxes * keys * 128;  // (k, v: a stage)
        // a query row's weights of 16 keys: float32 [2 halves of 8 keys][heads][8 keys], later bfloat16
        // [3 parts][output heads][16 keys]; the 16 bytes more keep the rows of a fragment in different banks
        chunk = (heads_in * 64 > NW * 96 ? heads_in * 64 : NW * 96) + 16;
        total = 1024 + q + k_stages * k + v_stages * v + SP_ROWS * KG * chunk;
        const int fold = 1024 + NW * ((VD + 15) / 16 * 2) * 512;  // the CTAs' sums, at the end, from the memory's start
        if (total < fold) total = fold;
    }
};

template <int NW, int KG, int VT, bool CAP>
__global__ void __launch_bounds__(32 * NW, NW == 16 ? 1 : 2) attention_sigmoid_prompt_kernel(const __grid_constant__ CUtensorMap map_q,
                                                                                          const __grid_constant__ CUtensorMap map_k,
                                                                                          const __grid_constant__ CUtensorMap map_v,
                                                                                          SigmoidPrompt p) {
    constexpr int NK = 16 * KG;
    extern __shared__ uint8_t sp_raw[];
    uint8_t *const sp_smem = (uint8_t *)(((uintptr_t)sp_raw + 1023) & ~(uintptr_t)1023);
    __shared__ SigmoidHead head_s[SP_MAX_HEADS];
    __shared__ uint64_t k_full[2], v_full[2];
    __shared__ int k_failed, v_failed;  // (each is set and read on the two sides of one barrier)
    const int H = p.n_heads, G = p.n_kv_heads, D = p.head_dim, VD = p.v_dim, R = H / G;
    const SigmoidPromptSmem sm(H, G, D, VD, p.kv_block, NW, KG, p.k_stages, p.v_stages);
    const uint32_t q_s = tc::smem_addr(sp_smem), k_s = q_s + sm.q, v_s = k_s + p.k_stages * sm.k;
    uint8_t *const chunks = sp_smem + sm.q + p.k_stages * sm.k + p.v_stages * sm.v;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, r8 = lane >> 2, q2 = lane & 3;
    const int ranks = (int)tc::cluster_size(), rank = (int)tc::cluster_rank();
    const int h0 = blockIdx.y * NW, hout = h0 + warp;  // this CTA's output heads, this warp's
    const int kv0 = h0 / R, kv_n = (min(h0 + NW, H) - 1) / R - kv0 + 1, heads_in = (H + 15) / 16 * 16;
    if (threadIdx.x == 0) {
#pragma unroll
        for (int s = 0; s < 2; s++) tc::mbar_init(&k_full[s], 1), tc::mbar_init(&v_full[s], 1);
        k_failed = v_failed = 0;
        tc::mbar_init_fence();
        tc::tma_prefetch_map(&map_q), tc::tma_prefetch_map(&map_k), tc::tma_prefetch_map(&map_v);
    }
    // weights: ahead of the wait. The mixing matrix as row operand: output heads h0 + r8 and + 8, input heads 16 s + 2 q2, + 1,
    // + 8, + 9
    for (int h = threadIdx.x; h < H; h += 32 * NW)
        head_s[h] = sigmoid_head(p.scale, p.softcap, p.slopes ? p.slopes[h] : 0.0f, p.shift ? p.shift[h] : 0.0f);
    uint32_t ta[SP_MAX_KS][4];
#pragma unroll
    for (int s = 0; s < SP_MAX_KS; s++) {
#pragma unroll
        for (int f = 0; f < 4; f++) {
            const int ho = h0 + r8 + (f & 1) * 8, gi = 16 * s + 2 * q2 + (f >> 1) * 8;
            float a = 0.0f, b = 0.0f;
            if (ho < H && r8 + (f & 1) * 8 < NW) {
                if (gi < H) a = p.mix ? p.mix[(long long)ho * H + gi] : (ho == gi ? 1.0f : 0.0f);
                if (gi + 1 < H) b = p.mix ? p.mix[(long long)ho * H + gi + 1] : (ho == gi + 1 ? 1.0f : 0.0f);
            }
            ta[s][f] = pack_bf16(a, b);
        }
    }
    __syncthreads();
    pdl_wait();
    // which sequence and which of its tiles of 16 query rows this cluster has; the tiles that see the most keys come first
    int seq = -1, tile = p.tiles - 1 - (int)blockIdx.x / ranks, start = 0, n = 0;
    for (int s = 0; s < p.n_seqs; s++) {
        start = p.seq_start[s], n = p.seq_start[s + 1] - start;
        const int tiles = (n + SP_ROWS - 1) / SP_ROWS;
        if (tile < tiles) {
            seq = s;
            break;
        }
        tile -= tiles;
    }
    if (seq < 0) return;  // (the whole cluster)
    const int r0 = tile * SP_ROWS, r_last = min(r0 + SP_ROWS - 1, n - 1), key_tiles = r_last / NK + 1;
    const int my_tiles = rank < key_tiles ? (key_tiles - rank + ranks - 1) / ranks : 0;  // tiles rank, rank + ranks, ...

    // warp 0 asks for this CTA's i-th tile of keys (with the queries, the first time) and of values
    auto load_keys = [&](int i) {
        const int s = p.k_stages == 2 ? i & 1 : 0, z = start + (rank + i * ranks) * NK, box = NK * 128;
        if (lane == 0) tc::mbar_expect_tx(&k_full[s], sm.k + (i == 0 ? sm.q : 0));
        __syncwarp();
        if (i == 0)
            for (int e = lane; e < H * sm.k_boxes; e += 32)
                tc::tma_load_3d(q_s + e * (SP_ROWS * 128), &map_q, (e % sm.k_boxes) * 64, e / sm.k_boxes, start + r0, &k_full[s]);
        for (int e = lane; e < G * sm.k_boxes; e += 32)
            tc::tma_load_3d(k_s + s * sm.k + e * box, &map_k, (e % sm.k_boxes) * 64, e / sm.k_boxes, z, &k_full[s]);
    };
    auto load_values = [&](int i) {
        const int s = p.v_stages == 2 ? i & 1 : 0, z = start + (rank + i * ranks) * NK, box = NK * 128;
        if (lane == 0) tc::mbar_expect_tx(&v_full[s], kv_n * sm.v_boxes * box);
        __syncwarp();
        for (int e = lane; e < kv_n * sm.v_boxes; e += 32)
            tc::tma_load_3d(v_s + s * sm.v + e * box, &map_v, (e % sm.v_boxes) * 64, kv0 + e / sm.v_boxes, z, &v_full[s]);
    };
    int k_asked = 0, v_asked = 0;
    if (warp == 0) {
        for (; k_asked < my_tiles && k_asked < p.k_stages; k_asked++) load_keys(k_asked);
        for (; v_asked < my_tiles && v_asked < p.v_stages; v_asked++) load_values(v_asked);
    }

    float o[VT][4];
#pragma unroll
    for (int t = 0; t < VT; t++) o[t][0] = o[t][1] = o[t][2] = o[t][3] = 0.0f;
    const int n_vt = (VD + 15) / 16 * 2, mix_steps = heads_in / 16, d_steps = (D + 15) / 16;
    // a lane's place in fragments of 16 rows of 128 bytes under the swizzle: row operand (rows lane & 15, pieces of 16 bytes
    // lane >> 4), column operand of the scores (keys, pieces (lane >> 3) & 1), of the values (transposed)
    const uint32_t row_a = (lane & 15) * 128, x_a = ((lane >> 4) ^ (lane & 7)) << 4;
    const uint32_t row_k = ((lane & 7) + ((lane >> 4) << 3)) * 128, x_k = (((lane >> 3) & 1) ^ (lane & 7)) << 4;

    for (int it = 0; it < my_tiles; it++) {
        const int key0 = (rank + it * ranks) * NK;
        const int ks_ = p.k_stages == 2 ? it & 1 : 0, vs_ = p.v_stages == 2 ? it & 1 : 0;
        const bool clear = key0 + NK - 1 <= r0 && r0 + SP_ROWS <= n;
        if (!tc::mbar_wait(&k_full[ks_], (p.k_stages == 2 ? it >> 1 : it) & 1)) k_failed = 1;
        // scores and weights of this warp's heads
        for (int g = warp; g < H; g += NW) {
            float s[2 * KG][4];
#pragma unroll
            for (int t = 0; t < 2 * KG; t++) s[t][0] = s[t][1] = s[t][2] = s[t][3] = 0.0f;
            uint32_t qa = q_s + g * sm.k_boxes * (SP_ROWS * 128) + row_a, kb = k_s + ks_ * sm.k + (g / R) * sm.k_boxes * (NK * 128) + row_k;
            for (int left = d_steps; left > 0; left -= 4, qa += SP_ROWS * 128, kb += NK * 128) {
#pragma unroll
                for (int c4 = 0; c4 < 4; c4++) {
                    if (c4 < left) {
                        uint32_t a[4];
                        ldsm_x4(qa + (x_a ^ (c4 << 5)), a[0], a[1], a[2], a[3]);
#pragma unroll
                        for (int c = 0; c < KG; c++) {
                            uint32_t b0, b1, b2, b3;
                            ldsm_x4(kb + c * 2048 + (x_k ^ (c4 << 5)), b0, b1, b2, b3);
                            mma_bf16(s[2 * c], a, b0, b1);
                            mma_bf16(s[2 * c + 1], a, b2, b3);
                        }
                    }
                }
            }
            const SigmoidHead hd = head_s[g];
            const float back = (float)(r0 + r8 - key0 - 2 * q2);  // of this thread's first row and key
            const float away_a = fmaf(hd.slope, back, hd.base), away_b = fmaf(hd.slope, 8.0f, away_a);
            float *w = (float *)(chunks + r8 * sm.chunk) + ((g >> 1) + (g & 1) * (heads_in >> 1)) * 8 + 2 * q2;
#pragma unroll
            for (int t = 0; t < 2 * KG; t++) {
#pragma unroll
                for (int e = 0; e < 4; e++) {
                    const float far = (float)(t * 8 + (e & 1));
                    s[t][e] = sigmoid_of(CAP, hd, s[t][e], fmaf(-hd.slope, far, e < 2 ? away_a : away_b));
                }
            }
            if (!clear) {
#pragma unroll
                for (int t = 0; t < 2 * KG; t++) {
#pragma unroll
                    for (int e = 0; e < 4; e++) {
                        const int j = key0 + t * 8 + 2 * q2 + (e & 1), i = r0 + r8 + (e >> 1) * 8;
                        if (j > i || i >= n) s[t][e] = 0.0f;
                    }
                }
            }
#pragma unroll
            for (int t = 0; t < 2 * KG; t++) {
                float *at = w + (t >> 1) * (SP_ROWS * sm.chunk / 4) + (t & 1) * heads_in * 8;
                *(float2 *)at = make_float2(s[t][0], s[t][1]);
                *(float2 *)(at + 2 * sm.chunk) = make_float2(s[t][2], s[t][3]);  // 8 rows (chunks) further
            }
        }
        __syncthreads();  // every head's weights are there, the keys are done with
        if (k_failed) break;
        if (warp == 0 && k_asked < my_tiles) load_keys(k_asked), k_asked++;
        // mixing, a query row's 16 keys at a time
        for (int ch = warp; ch < SP_ROWS * KG; ch += NW) {
            const float *w = (const float *)(chunks + ch * sm.chunk) + q2 * 8 + r8;
            const int odd = heads_in * 4;  // from an even head's weights to the next head's
            float m[2][4];
#pragma unroll
            for (int half = 0; half < 2; half++) m[half][0] = m[half][1] = m[half][2] = m[half][3] = 0.0f;
#pragma unroll
            for (int s = 0; s < SP_MAX_KS; s++) {
                if (s < mix_steps) {
                    const int gi = 16 * s + 2 * q2;  // (heads that are not there hold nothing)
                    const bool in0 = gi < H, in1 = gi + 1 < H, in8 = gi + 8 < H, in9 = gi + 9 < H;
#pragma unroll
                    for (int half = 0; half < 2; half++) {
                        const float *at = w + half * heads_in * 8 + s * 64;
                        const float x0 = in0 ? at[0] : 0.0f, x1 = in1 ? at[odd] : 0.0f, x8 = in8 ? at[32] : 0.0f, x9 = in9 ? at[odd + 32] : 0.0f;
                        uint32_t b0[3], b1[3];
                        split3_pair(x0, x1, b0), split3_pair(x8, x9, b1);
#pragma unroll
                        for (int k = 2; k >= 0; k--) mma_bf16(m[half], ta[s], b0[k], b1[k]);
                    }
                }
            }
            __syncwarp();  // the row's weights are read: their place is the mixed weights' now
            uint8_t *to = chunks + ch * sm.chunk + r8 * 32 + q2 * 4;
#pragma unroll
            for (int half = 0; half < 2; half++) {
                uint32_t lo[3], hi[3];
                split3_pair(m[half][0], m[half][1], lo);
                if (NW == 16) split3_pair(m[half][2], m[half][3], hi);
#pragma unroll
                for (int k = 0; k < 3; k++) {
                    *(uint32_t *)(to + k * NW * 32 + half * 16) = lo[k];
                    if (NW == 16) *(uint32_t *)(to + k * NW * 32 + half * 16 + 8 * 32) = hi[k];
                }
            }
        }
        if (!tc::mbar_wait(&v_full[vs_], (p.v_stages == 2 ? it >> 1 : it) & 1)) v_failed = 1;
        if (key0 + NK > n) {  // rows beyond the sequence's last are another's, or nobody's: their weights are 0, their values count as 0
            const int first = n - key0, pieces = sm.v_boxes * 8;
            for (int e = threadIdx.x; e < kv_n * (NK - first) * pieces; e += 32 * NW) {
                const int row = e / pieces, c = e - row * pieces, g = row / (NK - first), key = first + row - g * (NK - first);
                *(uint4 *)(sp_smem + sm.q + p.k_stages * sm.k + vs_ * sm.v + (g * sm.v_boxes + (c >> 3)) * (NK * 128) + key * 128 + (c & 7) * 16) =
                    make_uint4(0, 0, 0, 0);
            }
        }
        __syncthreads();  // all mixed weights are there
        if (hout < H && !v_failed) {
            uint32_t vb = v_s + vs_ * sm.v + (hout / R - kv0) * sm.v_boxes * (NK * 128) + row_a;
            const uint32_t wb = tc::smem_addr(chunks) + (lane & 15) * sm.chunk + warp * 32 + (lane >> 4) * 16;
            uint32_t part[KG][3][4];
#pragma unroll
            for (int c = 0; c < KG; c++)
#pragma unroll
                for (int k = 0; k < 3; k++)
                    ldsm_x4(wb + c * SP_ROWS * sm.chunk + k * NW * 32, part[c][k][0], part[c][k][1], part[c][k][2], part[c][k][3]);
#pragma unroll
            for (int tp = 0; tp < VT / 2; tp++) {
                if (2 * tp < n_vt) {
#pragma unroll
                    for (int c = 0; c < KG; c++) {
                        uint32_t b0, b1, b2, b3;
                        ldsm_x4_t(vb + (tp >> 2) * (NK * 128) + c * 2048 + (x_a ^ ((tp & 3) << 5)), b0, b1, b2, b3);
#pragma unroll
                        for (int k = 0; k < 3; k++) {
                            mma_bf16(o[2 * tp], part[c][k], b0, b1);
                            mma_bf16(o[2 * tp + 1], part[c][k], b2, b3);
                        }
                    }
                }
            }
        }
        __syncthreads();  // the values and the mixed weights are done with
        if (v_failed) break;
        if (warp == 0 && v_asked < my_tiles) load_values(v_asked), v_asked++;
    }
    __syncthreads();
    if (k_failed | v_failed) {  // a copy did not come: report it, and let the copies still in flight land (or run out of time)
        if (threadIdx.x == 0) atomicOr(p.status + 2, 1);
        if (warp == 0) {
            for (int i = max(0, k_asked - p.k_stages); i < k_asked; i++) tc::mbar_wait(&k_full[p.k_stages == 2 ? i & 1 : 0], (p.k_stages == 2 ? i >> 1 : i) & 1);
            for (int i = max(0, v_asked - p.v_stages); i < v_asked; i++) tc::mbar_wait(&v_full[p.v_stages == 2 ? i & 1 : 0], (p.v_stages == 2 ? i >> 1 : i) & 1);
        }
        __syncthreads();
    }
    __nv_bfloat16 *out = p.out + (long long)(start + r0 + r8) * H * VD + (long long)hout * VD + 2 * q2;
    const bool in_a = r0 + r8 < n, in_b = r0 + r8 + 8 < n;
    if (ranks > 1) {
        // the CTAs' sums side by side in their own memory, then every CTA adds its share of the column tiles, in rank order
        float4 *mine = (float4 *)sp_smem + warp * n_vt * 32 + lane;
#pragma unroll
        for (int t = 0; t < VT; t++)
            if (t < n_vt) mine[t * 32] = make_float4(o[t][0], o[t][1], o[t][2], o[t][3]);
        tc::cluster_sync();
        if (hout < H) {
            for (int t = rank; t < n_vt; t += ranks) {
                const uint32_t at = q_s + ((warp * n_vt + t) * 32 + lane) * 16;
                float4 v[8], sum = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
#pragma unroll
                for (int c = 0; c < 8; c++) v[c] = c < ranks ? tc::ld_cluster_f4(tc::peer_smem(at, c)) : sum;
#pragma unroll
                for (int c = 0; c < 8; c++) sum.x += v[c].x, sum.y += v[c].y, sum.z += v[c].z, sum.w += v[c].w;
                if (8 * t + 2 * q2 < VD) {  // (v_dim is even)
                    if (in_a) *(__nv_bfloat162 *)(out + 8 * t) = __floats2bfloat162_rn(sum.x, sum.y);
                    if (in_b) *(__nv_bfloat162 *)(out + 8LL * H * VD + 8 * t) = __floats2bfloat162_rn(sum.z, sum.w);
                }
            }
        }
        tc::cluster_sync();  // nobody leaves while its sums may still be read
        return;
    }
    if (hout >= H) return;
#pragma unroll
    for (int t = 0; t < VT; t++) {
        if (t < n_vt && 8 * t + 2 * q2 < VD) {
            if (in_a) *(__nv_bfloat162 *)(out + 8 * t) = __floats2bfloat162_rn(o[t][0], o[t][1]);
            if (in_b) *(__nv_bfloat162 *)(out + 8LL * H * VD + 8 * t) = __floats2bfloat162_rn(o[t][2], o[t][3]);
        }
    }
}

struct SigmoidPromptPlan {
    int nw, kg, k_stages, v_stages, kv_block, blocks, smem;
};

// How a CTA is laid out for these sizes: 32 keys a tile and two stages where shared memory allows (twice an SM for up to 8
// heads), else less. False: the sizes are not taken.
static bool sp_plan(int n_heads, int n_kv_heads, int head_dim, int v_dim, SigmoidPromptPlan &plan) {
    if (n_kv_heads < 1 || n_heads < 1 || n_heads % n_kv_heads || n_heads > SP_MAX_HEADS) return false;
    if (head_dim % 8 || head_dim < 8 || v_dim % 8 || v_dim < 8 || v_dim > 128) return false;
    plan.nw = n_heads <= 8 ? 8 : 16, plan.blocks = (n_heads + plan.nw - 1) / plan.nw, plan.kv_block = 0;
    const int r = n_heads / n_kv_heads;
    for (int b = 0; b < plan.blocks; b++) {
        const int last = ((b + 1) * plan.nw < n_heads ? (b + 1) * plan.nw : n_heads) - 1, count = last / r - b * plan.nw / r + 1;
        if (count > plan.kv_block) plan.kv_block = count;
    }
    const int whole = 226 * 1024, half = 112 * 1024;
    const int tries[][3] = {{2, 2, 2}, {2, 1, 1}, {1, 2, 2}, {1, 1, 2}, {1, 1, 1}};
    for (int pass = plan.nw == 8 ? 0 : 1; pass < 2; pass++) {
        for (auto &t : tries) {
            plan.kg = t[0], plan.k_stages = t[1], plan.v_stages = t[2];
            plan.smem = SigmoidPromptSmem(n_heads, n_kv_heads, head_dim, v_dim, plan.kv_block, plan.nw, t[0], t[1], t[2]).total;
            if (plan.smem <= (pass ? whole : half)) return true;
        }
    }
    return false;
}

extern "C" int abk_attention_sigmoid_prompt_takes(int n_heads, int n_kv_heads, int head_dim, int v_dim) {
    SigmoidPromptPlan plan;
    return sp_plan(n_heads, n_kv_heads, head_dim, v_dim, plan);
}

template <int NW, int KG, int VT, bool CAP>
static int sp_launch(const CUtensorMap &mq, const CUtensorMap &mk, const CUtensorMap &mv, const SigmoidPrompt &p, int blocks, int ranks, int smem,
                     cudaStream_t s) {
    cudaError_t e = abk_allow_shared_memory((const void *)attention_sigmoid_prompt_kernel<NW, KG, VT, CAP>, smem);
    if (e != cudaSuccess) return (int)e;
    abk_launch_clusters(attention_sigmoid_prompt_kernel<NW, KG, VT, CAP>, dim3(p.tiles * ranks, blocks), dim3(32 * NW), (size_t)smem, s, ranks, mq, mk, mv, p);
    return ABK_LAUNCH_RESULT();
}

// qkv: n_rows rows of `row` elements, q heads, then (at k_off) k heads, then (at v_off) v heads. tiles: an upper bound of
// the step's tiles of 16 query rows, sum over its sequences of ceil(rows / 16). mix holds bfloat16 numbers (the tensor-core
// operand), as a bfloat16 model stores it. forced_ranks: 0, or the CTAs of a cluster (1, 2, 4, 8). status word 2 is set if
// a wait ran out.
extern "C" int abk_attention_sigmoid_prompt(const void *qkv, long long row, int n_rows, void *out, int n_heads, int n_kv_heads, int head_dim,
                                            int v_dim, int k_off, int v_off, float scale, float softcap, const float *slopes,
                                            const float *shift, const float *mix, const int *seq_start, int n_seqs, int tiles,
                                            int forced_ranks, int *status, void *stream) {
    if (n_seqs <= 0 || tiles <= 0 || n_rows <= 0) return 0;
    SigmoidPromptPlan plan;
    if (!sp_plan(n_heads, n_kv_heads, head_dim, v_dim, plan))
        ABK_REFUSE("attention_sigmoid_prompt: %d heads of %d over %d kv heads with values of %d", n_heads, head_dim, n_kv_heads, v_dim);
    if (row % 8 || k_off % 8 || v_off % 8 || ((uintptr_t)qkv & 15) || ((uintptr_t)out & 3))
        ABK_REFUSE("attention_sigmoid_prompt: rows of q, k and v are not 16-byte aligned");
    SigmoidPrompt p;
    p.out = (__nv_bfloat16 *)out, p.n_heads = n_heads, p.n_kv_heads = n_kv_heads;
    p.head_dim = head_dim, p.v_dim = v_dim, p.scale = scale, p.softcap = softcap, p.kv_block = plan.kv_block;
    p.slopes = slopes, p.shift = shift, p.mix = mix, p.seq_start = seq_start, p.n_seqs = n_seqs, p.tiles = tiles;
    p.k_stages = plan.k_stages, p.v_stages = plan.v_stages, p.status = status;
    CUtensorMap mq, mk, mv;
    const __nv_bfloat16 *base = (const __nv_bfloat16 *)qkv;
    int rc = tmap::bf16_heads(base, head_dim, n_heads, n_rows, row, SP_ROWS, &mq);
    if (!rc) rc = tmap::bf16_heads(base + k_off, head_dim, n_kv_heads, n_rows, row, 16 * plan.kg, &mk);
    if (!rc) rc = tmap::bf16_heads(base + v_off, v_dim, n_kv_heads, n_rows, row, 16 * plan.kg, &mv);
    if (rc) return rc;
    int ranks = 1;
    while (ranks < 8 && (long long)tiles * plan.blocks * ranks * 3 < 5LL * abk_sm_count() * (plan.nw == 8 ? 2 : 1)) ranks *= 2;
    if (forced_ranks == 1 || forced_ranks == 2 || forced_ranks == 4 || forced_ranks == 8) ranks = forced_ranks;
    if ((long long)tiles * ranks > 0x7fffffffLL || plan.blocks > 65535) ABK_REFUSE("attention_sigmoid_prompt: %d tiles are more than a grid takes", tiles);
    cudaStream_t s = (cudaStream_t)stream;
#define SP_BY_CAP(NW, KG, VT) \
    (softcap > 0.0f ? sp_launch<NW, KG, VT, true>(mq, mk, mv, p, plan.blocks, ranks, plan.smem, s) : sp_launch<NW, KG, VT, false>(mq, mk, mv, p, plan.blocks, ranks, plan.smem, s))
#define SP_BY_VT(NW, KG) (v_dim <= 64 ? SP_BY_CAP(NW, KG, 8) : SP_BY_CAP(NW, KG, 16))
    if (plan.nw == 16) return plan.kg == 2 ? SP_BY_VT(16, 2) : SP_BY_VT(16, 1);
    return plan.kg == 2 ? SP_BY_VT(8, 2) : SP_BY_VT(8, 1);
#undef SP_BY_VT
#undef SP_BY_CAP
}
