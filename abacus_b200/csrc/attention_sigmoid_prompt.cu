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
// Runs of keys add up (nothing is normalized over them), so the tiles of a query row can be dealt to the CTAs of a
// cluster: each sums its tiles' contributions and they are added at the end through distributed shared memory, in rank
// order. A step with few query rows gets clusters of up to 8, so that it fills the GPU.
//
// Keys come in by cp.async under mixing and values, values under the next tile's scores.
#define ABK_DEFINE_ERROR
#include "common.cuh"
#include "attention_sigmoid.cuh"
#include "mma_tiles.cuh"
#include "tc_common.cuh"

#define SP_ROWS 16
#define SP_MAX_VT 16   // value columns / 8 a warp accumulates: values of up to 128
#define SP_MAX_KS 2    // heads / 16 that are mixed: up to 32 heads

struct SigmoidPrompt {
    const __nv_bfloat16 *qkv;  // rows of `row` elements: q heads, then (at k_off) k heads, then (at v_off) v heads
    long long row;
    __nv_bfloat16 *out;        // [tokens, n_heads * v_dim]
    int n_heads, n_kv_heads, head_dim, v_dim, k_off, v_off;
    float scale, softcap;
    const float *slopes, *shift;  // [n_heads] or null
    const float *mix;             // [n_heads, n_heads] (out, in), bfloat16 numbers, or null
    const int *seq_start;         // [n_seqs + 1]
    int n_seqs, tiles;            // tiles: the grid's query tiles
    int kv_block;                 // kv heads an output block's values come from, at most
};

// Bytes of the parts of shared memory.
struct SigmoidPromptSmem {
    int pitch_k, pitch_v, q, k, v, chunk, total;
    __host__ __device__ SigmoidPromptSmem(int H, int G, int D, int VD, int kv_block, int NW, int KG) {
        const int keys = 16 * KG, heads_in = (H + 15) / 16 * 16;
        pitch_k = (D + 15) / 16 * 32 + 16, pitch_v = (VD + 15) / 16 * 32 + 16;
        q = H * SP_ROWS * pitch_k, k = G * keys * pitch_k, v = kv_block * keys * pitch_v;
        // a query row's weights of 16 keys: float32 [2 halves of 8 keys][heads][8 keys], later bfloat16
        // [3 parts][output heads][16 keys]; the 16 bytes more keep the rows of a fragment in different banks
        chunk = (heads_in * 64 > NW * 96 ? heads_in * 64 : NW * 96) + 16;
        total = q + k + v + SP_ROWS * KG * chunk;
        const int fold = NW * ((VD + 15) / 16 * 2) * 512;  // the CTAs' sums, at the end, from the memory's start
        if (total < fold) total = fold;
    }
};

__device__ __forceinline__ void sp_copy_16(uint32_t dst, const void *src, bool real) {
    const int bytes = real ? 16 : 0;  // 0: the 16 bytes are filled with zeros
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(bytes) : "memory");
}
__device__ __forceinline__ void sp_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void sp_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

// `rows` rows (first .., those from `limit` on as zeros) of `heads` heads of `size` elements, which lie side by side in a
// row, to dst[head][row][pitch]. A warp a row; a lane's pieces follow one another 32 pieces apart.
template <int NW>
__device__ __forceinline__ void sp_load(uint32_t dst, int pitch, const __nv_bfloat16 *src, long long row_pitch, int first, int limit,
                                        int rows, int heads, int size, int warp, int lane) {
    const int per = (pitch - 16) >> 4;  // 16-byte pieces of a head, the padding to whole fragments among them
    const int step_h = 32 / per, step_c = 32 - step_h * per, h0 = lane / per, c0 = lane - h0 * per;
    for (int r = warp; r < rows; r += NW) {
        const bool in = first + r < limit;
        const __nv_bfloat16 *from = src + (long long)(first + r) * row_pitch;
        int h = h0, c = c0;
        while (h < heads) {
            const bool real = in && c * 8 < size;
            sp_copy_16(dst + (h * rows + r) * pitch + c * 16, real ? from + h * size + c * 8 : src, real);
            h += step_h, c += step_c;
            if (c >= per) c -= per, h++;
        }
    }
}

template <int NW, int KG> __global__ void __launch_bounds__(32 * NW, NW == 16 ? 1 : 2) attention_sigmoid_prompt_kernel(SigmoidPrompt p) {
    constexpr int NK = 16 * KG;
    extern __shared__ __align__(16) uint8_t sp_smem[];
    const int H = p.n_heads, G = p.n_kv_heads, D = p.head_dim, VD = p.v_dim, R = H / G;
    const SigmoidPromptSmem sm(H, G, D, VD, p.kv_block, NW, KG);
    const uint32_t q_s = (uint32_t)__cvta_generic_to_shared(sp_smem), k_s = q_s + sm.q, v_s = k_s + sm.k, w_s = v_s + sm.v;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, r8 = lane >> 2, q2 = lane & 3;
    const int ranks = (int)tc::cluster_size(), rank = (int)tc::cluster_rank();
    const int h0 = blockIdx.y * NW, hout = h0 + warp;  // this CTA's output heads, this warp's
    const int kv0 = h0 / R, heads_in = (H + 15) / 16 * 16, mix_steps = heads_in / 16;
    const int kv_n = min(h0 + NW, H) > h0 ? (min(h0 + NW, H) - 1) / R - kv0 + 1 : 0;
    // the mixing matrix as row operand: output heads h0 + r8 and + 8, input heads 16 s + 2 q2, + 1, + 8, + 9 (a weight: ahead
    // of the wait)
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
    const __nv_bfloat16 *base = p.qkv + (long long)start * p.row;
    const __nv_bfloat16 *kg = base + p.k_off, *vg = base + p.v_off + (long long)kv0 * VD;

    float o[SP_MAX_VT][4];
#pragma unroll
    for (int t = 0; t < SP_MAX_VT; t++) o[t][0] = o[t][1] = o[t][2] = o[t][3] = 0.0f;
    const int n_vt = (VD + 15) / 16 * 2;

    if (rank < key_tiles) {
        sp_load<NW>(q_s, sm.pitch_k, base, p.row, r0, n, SP_ROWS, H, D, warp, lane);
        sp_load<NW>(k_s, sm.pitch_k, kg, p.row, rank * NK, n, NK, G, D, warp, lane);
        sp_commit();
        sp_load<NW>(v_s, sm.pitch_v, vg, p.row, rank * NK, n, NK, kv_n, VD, warp, lane);
        sp_commit();
        sp_wait<1>();
        __syncthreads();
    }
    for (int kt = rank; kt < key_tiles; kt += ranks) {
        const int key0 = kt * NK;
        const bool more = kt + ranks < key_tiles, clear = key0 + NK - 1 <= r0 && r0 + SP_ROWS <= n;
        // scores and weights of this warp's heads
        for (int g = warp; g < H; g += NW) {
            float s[2 * KG][4];
#pragma unroll
            for (int t = 0; t < 2 * KG; t++) s[t][0] = s[t][1] = s[t][2] = s[t][3] = 0.0f;
            const uint32_t qa = q_s + (g * SP_ROWS + (lane & 15)) * sm.pitch_k + (lane >> 4) * 16;
            const uint32_t kb = k_s + ((g / R) * NK + (lane & 7) + ((lane >> 4) << 3)) * sm.pitch_k + ((lane >> 3) & 1) * 16;
#pragma unroll 4
            for (int ks = 0; ks < (D + 15) / 16; ks++) {
                uint32_t a[4];
                ldsm_x4(qa + ks * 32, a[0], a[1], a[2], a[3]);
#pragma unroll
                for (int c = 0; c < KG; c++) {
                    uint32_t b0, b1, b2, b3;
                    ldsm_x4(kb + c * 16 * sm.pitch_k + ks * 32, b0, b1, b2, b3);
                    mma_bf16(s[2 * c], a, b0, b1);
                    mma_bf16(s[2 * c + 1], a, b2, b3);
                }
            }
            const SigmoidHead hd = sigmoid_head(p.scale, p.softcap, p.slopes ? p.slopes[g] : 0.0f, p.shift ? p.shift[g] : 0.0f);
            const float back = (float)(r0 + r8 - key0 - 2 * q2);  // of this thread's first row and key
            const float away_a = fmaf(hd.slope, back, hd.base), away_b = fmaf(hd.slope, back + 8.0f, hd.base);
            const int slot = (g >> 1) + (g & 1) * (heads_in >> 1);
            float *w = (float *)(sp_smem + (w_s - q_s) + r8 * sm.chunk) + slot * 8 + 2 * q2;
#pragma unroll
            for (int t = 0; t < 2 * KG; t++) {
#pragma unroll
                for (int e = 0; e < 4; e++) {
                    const float far = (float)(t * 8 + (e & 1));
                    s[t][e] = sigmoid_of(hd, s[t][e], fmaf(-hd.slope, far, e < 2 ? away_a : away_b));
                    if (!clear) {
                        const int j = key0 + t * 8 + 2 * q2 + (e & 1), i = r0 + r8 + (e >> 1) * 8;
                        if (j > i || i >= n) s[t][e] = 0.0f;
                    }
                }
                float *at = w + (t >> 1) * (SP_ROWS * sm.chunk / 4) + (t & 1) * heads_in * 8;
                *(float2 *)at = make_float2(s[t][0], s[t][1]);
                *(float2 *)(at + 2 * sm.chunk) = make_float2(s[t][2], s[t][3]);  // 8 rows (chunks) further
            }
        }
        __syncthreads();  // every head's weights are there, the keys are done with
        if (more) sp_load<NW>(k_s, sm.pitch_k, kg, p.row, key0 + ranks * NK, n, NK, G, D, warp, lane);
        sp_commit();
        // mixing, a query row's 16 keys at a time
        for (int ch = warp; ch < SP_ROWS * KG; ch += NW) {
            const float *w = (const float *)(sp_smem + (w_s - q_s) + ch * sm.chunk) + r8;
            float m[2][4];
#pragma unroll
            for (int half = 0; half < 2; half++) m[half][0] = m[half][1] = m[half][2] = m[half][3] = 0.0f;
#pragma unroll
            for (int s = 0; s < SP_MAX_KS; s++) {
                if (s < mix_steps) {
#pragma unroll
                    for (int half = 0; half < 2; half++) {
                        const float *at = w + (half * heads_in + 8 * s + q2) * 8;
                        const int odd = heads_in * 4, gi = 16 * s + 2 * q2;  // (heads that are not there hold nothing)
                        const float x0 = gi < H ? at[0] : 0.0f, x1 = gi + 1 < H ? at[odd] : 0.0f;
                        const float x8 = gi + 8 < H ? at[32] : 0.0f, x9 = gi + 9 < H ? at[odd + 32] : 0.0f;
                        uint32_t b0[3], b1[3];
                        split3_pair(x0, x1, b0), split3_pair(x8, x9, b1);
#pragma unroll
                        for (int k = 2; k >= 0; k--) mma_bf16(m[half], ta[s], b0[k], b1[k]);
                    }
                }
            }
            __syncwarp();  // the row's weights are read: their place is the mixed weights' now
            uint8_t *to = sp_smem + (w_s - q_s) + ch * sm.chunk + r8 * 32 + q2 * 4;
#pragma unroll
            for (int half = 0; half < 2; half++) {
                uint32_t lo[3], hi[3];
                split3_pair(m[half][0], m[half][1], lo), split3_pair(m[half][2], m[half][3], hi);
#pragma unroll
                for (int k = 0; k < 3; k++) {
                    if (NW >= 8 || r8 < NW) *(uint32_t *)(to + k * NW * 32 + half * 16) = lo[k];
                    if (NW == 16) *(uint32_t *)(to + k * NW * 32 + half * 16 + 8 * 32) = hi[k];
                }
            }
        }
        sp_wait<1>();     // the values are here (the next keys may still be on their way)
        __syncthreads();  // and so are all mixed weights
        if (hout < H) {
            const uint32_t vb = v_s + ((hout / R - kv0) * NK + (lane & 7) + ((lane >> 3) & 1) * 8) * sm.pitch_v + (lane >> 4) * 16;
            const uint32_t wb = w_s + (lane & 15) * sm.chunk + warp * 32 + (lane >> 4) * 16;
#pragma unroll
            for (int c = 0; c < KG; c++) {
                uint32_t part[3][4];
#pragma unroll
                for (int k = 0; k < 3; k++)
                    ldsm_x4(wb + c * SP_ROWS * sm.chunk + k * NW * 32, part[k][0], part[k][1], part[k][2], part[k][3]);
#pragma unroll
                for (int tp = 0; tp < SP_MAX_VT / 2; tp++) {
                    if (2 * tp < n_vt) {
                        uint32_t b0, b1, b2, b3;
                        ldsm_x4_t(vb + c * 16 * sm.pitch_v + tp * 32, b0, b1, b2, b3);
#pragma unroll
                        for (int k = 0; k < 3; k++) {
                            mma_bf16(o[2 * tp], part[k], b0, b1);
                            mma_bf16(o[2 * tp + 1], part[k], b2, b3);
                        }
                    }
                }
            }
        }
        if (more) {
            sp_wait<0>();     // the next keys are here
            __syncthreads();  // the values and the mixed weights are done with
            sp_load<NW>(v_s, sm.pitch_v, vg, p.row, key0 + ranks * NK, n, NK, kv_n, VD, warp, lane);
            sp_commit();
        }
    }
    __nv_bfloat16 *out = p.out + (long long)(start + r0 + r8) * H * VD + (long long)hout * VD + 2 * q2;
    const bool row_a = r0 + r8 < n, row_b = r0 + r8 + 8 < n;
    if (ranks > 1) {
        // the CTAs' sums side by side in their own memory, then every CTA adds its share of the column tiles, in rank order
        sp_wait<0>();
        __syncthreads();
        float4 *mine = (float4 *)sp_smem + warp * n_vt * 32 + lane;
#pragma unroll
        for (int t = 0; t < SP_MAX_VT; t++)
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
                    if (row_a) *(__nv_bfloat162 *)(out + 8 * t) = __floats2bfloat162_rn(sum.x, sum.y);
                    if (row_b) *(__nv_bfloat162 *)(out + 8LL * H * VD + 8 * t) = __floats2bfloat162_rn(sum.z, sum.w);
                }
            }
        }
        tc::cluster_sync();  // nobody leaves while its sums may still be read
        return;
    }
    if (hout >= H) return;
#pragma unroll
    for (int t = 0; t < SP_MAX_VT; t++) {
        if (t < n_vt && 8 * t + 2 * q2 < VD) {
            if (row_a) *(__nv_bfloat162 *)(out + 8 * t) = __floats2bfloat162_rn(o[t][0], o[t][1]);
            if (row_b) *(__nv_bfloat162 *)(out + 8LL * H * VD + 8 * t) = __floats2bfloat162_rn(o[t][2], o[t][3]);
        }
    }
}

template <int NW, int KG> static int sp_launch(const SigmoidPrompt &p, int blocks, int ranks, int smem, cudaStream_t s) {
    cudaError_t e = abk_allow_shared_memory((const void *)attention_sigmoid_prompt_kernel<NW, KG>, smem);
    if (e != cudaSuccess) return (int)e;
    abk_launch_clusters(attention_sigmoid_prompt_kernel<NW, KG>, dim3(p.tiles * ranks, blocks), dim3(32 * NW), (size_t)smem, s, ranks, p);
    return ABK_LAUNCH_RESULT();
}

// tiles: an upper bound of the step's tiles of 16 query rows, sum over its sequences of ceil(rows / 16).
// mix holds bfloat16 numbers (the tensor-core operand), as a bfloat16 model stores it. forced_ranks: 0, or the CTAs of a
// cluster (1, 2, 4, 8).
extern "C" int abk_attention_sigmoid_prompt(const void *qkv, long long row, void *out, int n_heads, int n_kv_heads, int head_dim,
                                            int v_dim, int k_off, int v_off, float scale, float softcap, const float *slopes,
                                            const float *shift, const float *mix, const int *seq_start, int n_seqs, int tiles,
                                            int forced_ranks, void *stream) {
    if (n_seqs <= 0 || tiles <= 0) return 0;
    if (n_kv_heads < 1 || n_heads < 1 || n_heads % n_kv_heads)
        ABK_REFUSE("attention_sigmoid_prompt: %d query heads do not divide into %d kv heads", n_heads, n_kv_heads);
    if (n_heads > 16 * SP_MAX_KS) ABK_REFUSE("attention_sigmoid_prompt: %d heads are more than %d", n_heads, 16 * SP_MAX_KS);
    if (head_dim % 8 || head_dim < 8 || v_dim % 8 || v_dim < 8 || v_dim > 8 * SP_MAX_VT)
        ABK_REFUSE("attention_sigmoid_prompt: heads of %d and values of %d are not multiples of 8 (values up to %d)", head_dim, v_dim, 8 * SP_MAX_VT);
    if (row % 8 || k_off % 8 || v_off % 8 || ((uintptr_t)qkv & 15) || ((uintptr_t)out & 3))
        ABK_REFUSE("attention_sigmoid_prompt: rows of q, k and v are not 16-byte aligned");
    SigmoidPrompt p;
    p.qkv = (const __nv_bfloat16 *)qkv, p.row = row, p.out = (__nv_bfloat16 *)out, p.n_heads = n_heads, p.n_kv_heads = n_kv_heads;
    p.head_dim = head_dim, p.v_dim = v_dim, p.k_off = k_off, p.v_off = v_off, p.scale = scale, p.softcap = softcap;
    p.slopes = slopes, p.shift = shift, p.mix = mix, p.seq_start = seq_start, p.n_seqs = n_seqs, p.tiles = tiles;
    const int nw = n_heads <= 4 ? 4 : n_heads <= 8 ? 8 : 16, blocks = (n_heads + nw - 1) / nw, r = n_heads / n_kv_heads;
    p.kv_block = 0;
    for (int b = 0; b < blocks; b++) {
        const int last = ((b + 1) * nw < n_heads ? (b + 1) * nw : n_heads) - 1, count = last / r - b * nw / r + 1;
        if (count > p.kv_block) p.kv_block = count;
    }
    // 32 keys a tile where shared memory allows (for up to 8 heads: twice an SM), else 16
    const int most = 227 * 1024;
    int kg = 2, smem = SigmoidPromptSmem(n_heads, n_kv_heads, head_dim, v_dim, p.kv_block, nw, 2).total;
    if (smem > (nw == 16 ? most : most / 2 - 1024)) kg = 1, smem = SigmoidPromptSmem(n_heads, n_kv_heads, head_dim, v_dim, p.kv_block, nw, 1).total;
    if (smem > most) ABK_REFUSE("attention_sigmoid_prompt: %d heads of %d over %d kv heads are more than a CTA holds", n_heads, head_dim, n_kv_heads);
    int ranks = 1;
    while (ranks < 8 && (long long)tiles * blocks * ranks < 3LL * abk_sm_count()) ranks *= 2;
    if (forced_ranks == 1 || forced_ranks == 2 || forced_ranks == 4 || forced_ranks == 8) ranks = forced_ranks;
    if ((long long)tiles * ranks > 0x7fffffffLL || blocks > 65535) ABK_REFUSE("attention_sigmoid_prompt: %d tiles are more than a grid takes", tiles);
    cudaStream_t s = (cudaStream_t)stream;
    if (nw == 16) return kg == 2 ? sp_launch<16, 2>(p, blocks, ranks, smem, s) : sp_launch<16, 1>(p, blocks, ranks, smem, s);
    if (nw == 8) return kg == 2 ? sp_launch<8, 2>(p, blocks, ranks, smem, s) : sp_launch<8, 1>(p, blocks, ranks, smem, s);
    return kg == 2 ? sp_launch<4, 2>(p, blocks, ranks, smem, s) : sp_launch<4, 1>(p, blocks, ranks, smem, s);
}
