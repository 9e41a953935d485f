// Attention without a softmax for whole prompts (attention_sigmoid.cu has the formulas): bfloat16, every sequence of the
// step from its first token, keys and values from the step's own rows.
//
// The heads' weights are mixed per (token, key), so every head's weights of a tile have to meet. A CTA has 16 query rows and
// up to 16 heads, whose queries stay in shared memory, 16 warps (a warp a head; two to a head for up to 8 heads), and walks
// tiles of 16 * WPH keys of the heads' kv heads:
//   scores    a warp multiplies its head with 16 keys (mma.sync), makes the weights and leaves them in shared memory, by
//             query row: [head][key], float32
//   mixing    a warp takes a query row's 16 keys: [16 heads out x heads in] x [heads in x 8 keys] on the tensor cores, the
//             weights as three bfloat16 parts that hold their 24 bits, the mixing matrix in bfloat16 (as stored). What
//             comes out is split into three parts again
//   values    a warp adds the mixed weights of its head times the tile's values, the product taken three times, once a part
// The next tile's scores are made beside this tile's values, so that between two barriers there is tensor work and weights
// to be made. With more than 16 heads (up to 32) two CTAs of a cluster have 16 heads each and leave their weights in both
// CTAs' shared memory.
//
// Queries, keys and values come in by TMA as boxes of 64 columns of one head (128-byte swizzle, zeros beyond a head's last
// column), keys through a ring of one or two stages.
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
#define SP_WARPS 16
#define SP_THREADS (32 * SP_WARPS)
#define SP_MAX_HEADS 32

struct SigmoidPrompt {
    __nv_bfloat16 *out;           // [tokens, n_heads * v_dim]
    int n_heads, n_kv_heads, head_dim, v_dim;
    float scale, softcap;
    const float *slopes, *shift;  // [n_heads] or null
    const float *mix;             // [n_heads, n_heads] (out, in), bfloat16 numbers, or null
    const int *seq_start;         // [n_seqs + 1]
    int n_seqs, tiles;            // tiles: the grid's query tiles
    int kv_block;                 // kv heads a CTA's heads have, at most
    int k_stages;                 // 1 or 2
    int *status;
};

// Bytes of the parts of shared memory.
struct SigmoidPromptSmem {
    int k_boxes, v_boxes, q, k, v, w_row, p_row, w, p, total;
    __host__ __device__ SigmoidPromptSmem(int H, int D, int VD, int kv_block, int WPH, int k_stages) {
        const int keys = 16 * WPH, heads_in = (H + 15) / 16 * 16, heads = SP_WARPS / WPH, mine = H < heads ? H : heads;
        k_boxes = (D + 63) / 64, v_boxes = (VD + 63) / 64;
        q = mine * k_boxes * SP_ROWS * 128, k = kv_block * k_boxes * keys * 128, v = kv_block * v_boxes * keys * 128;  // (k: a stage)
        // a query row's weights of 16 keys, float32 [2 halves of 8 keys][heads][8 keys], and mixed, bfloat16 [3 parts][this CTA's
        // heads][16 keys]; the 16 bytes more keep the rows of a fragment in different banks
        w_row = heads_in * 64 + 16, p_row = heads * 96 + 16;
        w = SP_ROWS * WPH * w_row * (H > 16 ? 2 : 1), p = SP_ROWS * WPH * p_row;  // (weights from another CTA: two buffers)
        total = 1024 + q + k_stages * k + v + w + p;
        const int fold = 1024 + SP_WARPS * (16 / WPH) * 512;  // the warps' sums, at the end, from the memory's start
        if (total < fold) total = fold;
    }
};

// ldmatrix and shared-memory accesses at a register's address plus a constant, which goes into the instruction: the inner
// loops' addresses differ by constants, and a warp's time is the instructions it waits for, one after the other.
template <int OFF> __device__ __forceinline__ void ldsm_at(uint32_t addr, uint32_t *r) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4+%5];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr), "n"(OFF));
}
template <int OFF> __device__ __forceinline__ void ldsm_t_at(uint32_t addr, uint32_t *r) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4+%5];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr), "n"(OFF));
}
template <int OFF> __device__ __forceinline__ float lds_at(uint32_t addr) {
    float v;
    asm volatile("ld.shared.f32 %0, [%1+%2];" : "=f"(v) : "r"(addr), "n"(OFF));
    return v;
}
template <int OFF> __device__ __forceinline__ void sts_at(uint32_t addr, uint32_t v) {
    asm volatile("st.shared.b32 [%0+%1], %2;" ::"r"(addr), "n"(OFF), "r"(v) : "memory");
}
// f(0), f(1), .. f(N - 1), each with its number as a constant (decltype(i)::value)
template <int I> struct Number {
    static constexpr int value = I;
};
template <int N, int I = 0, typename F> __device__ __forceinline__ void each(F &&f) {
    if constexpr (I < N) {
        f(Number<I>{});
        each<N, I + 1>(f);
    }
}

// WPH: warps a head. PAIR: more than 16 heads, two CTAs of the cluster side by side. EXACT: 16 / WPH heads a CTA, heads and
// values of 128: nothing in the inner loops depends on a size that is only known at run time.
template <int WPH, bool CAP, bool EXACT, bool PAIR>
__global__ void __launch_bounds__(SP_THREADS, 1) attention_sigmoid_prompt_kernel(const __grid_constant__ CUtensorMap map_q,
                                                                                 const __grid_constant__ CUtensorMap map_k,
                                                                                 const __grid_constant__ CUtensorMap map_v, SigmoidPrompt p) {
    constexpr int NK = 16 * WPH, HEADS = SP_WARPS / WPH, VT = 16 / WPH, BLOCKS = PAIR ? 2 : 1;  // VT: a warp's tiles of 8 value columns
    extern __shared__ uint8_t sp_raw[];
    uint8_t *const sp_smem = (uint8_t *)(((uintptr_t)sp_raw + 1023) & ~(uintptr_t)1023);
    __shared__ uint64_t k_full[2], v_full;
    __shared__ int failed[2];  // by the tile's parity: set before a barrier, read after it
    const int H = p.n_heads, D = p.head_dim, VD = p.v_dim, R = H / p.n_kv_heads;
    const SigmoidPromptSmem sm(H, D, VD, p.kv_block, WPH, p.k_stages);
    const uint32_t q_s = tc::smem_addr(sp_smem), k_s = q_s + sm.q, v_s = k_s + p.k_stages * sm.k, w_s = v_s + sm.v, p_s = w_s + sm.w;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, r8 = lane >> 2, q2 = lane & 3;
    const int in_cluster = (int)tc::cluster_rank(), ranks = (int)tc::cluster_size() / BLOCKS, rank = in_cluster / BLOCKS;
    const int h0 = PAIR ? (in_cluster & 1) * HEADS : 0, heads_n = min(HEADS, H - h0);  // this CTA's heads
    const int hl = warp / WPH, part = warp % WPH;  // this warp's head among them, and which of the head's warps it is
    const bool has_head = EXACT || hl < heads_n;
    const int kv0 = h0 / R, kv_n = (h0 + heads_n - 1) / R - kv0 + 1, heads_in = EXACT ? (PAIR ? 32 : 16) : (H + 15) / 16 * 16;
    if (threadIdx.x == 0) {
        tc::mbar_init(&k_full[0], 1), tc::mbar_init(&k_full[1], 1), tc::mbar_init(&v_full, 1);
        failed[0] = failed[1] = 0;
        tc::mbar_init_fence();
        tc::tma_prefetch_map(&map_q), tc::tma_prefetch_map(&map_k), tc::tma_prefetch_map(&map_v);
    }
    // weights: ahead of the wait. The mixing matrix as row operand: output heads h0 + r8 and + 8, input heads 16 s + 2 q2, + 1,
    // + 8, + 9
    uint32_t ta[BLOCKS][4];
#pragma unroll
    for (int s = 0; s < BLOCKS; s++) {
#pragma unroll
        for (int f = 0; f < 4; f++) {
            const int row = r8 + (f & 1) * 8, ho = h0 + row, gi = 16 * s + 2 * q2 + (f >> 1) * 8;
            float a = 0.0f, b = 0.0f;
            if (row < heads_n) {
                if (gi < H) a = p.mix ? p.mix[(long long)ho * H + gi] : (ho == gi ? 1.0f : 0.0f);
                if (gi + 1 < H) b = p.mix ? p.mix[(long long)ho * H + gi + 1] : (ho == gi + 1 ? 1.0f : 0.0f);
            }
            ta[s][f] = pack_bf16(a, b);
        }
    }
    const int hg = has_head ? h0 + hl : h0;
    const SigmoidHead hd = sigmoid_head(p.scale, p.softcap, p.slopes ? p.slopes[hg] : 0.0f, p.shift ? p.shift[hg] : 0.0f);
    __syncthreads();
    pdl_wait();
    // which sequence and which of its tiles of 16 query rows this cluster has; the tiles that see the most keys come first
    int seq = -1, tile = p.tiles - 1 - (int)blockIdx.x / (ranks * BLOCKS), start = 0, n = 0;
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
    // tiles rank, rank + ranks, ...; where CTAs meet at every tile all of the cluster's walk as many (a tile beyond the last
    // has no visible key)
    const int my_tiles = PAIR ? (key_tiles + ranks - 1) / ranks : rank < key_tiles ? (key_tiles - rank + ranks - 1) / ranks : 0;

    // This CTA's i-th tile of keys (with the queries, the first time) and of values: a warp asks for every 16th box, so that no
    // warp falls behind the others, and one thread says how many bytes are to come (some may have come by then).
    const int k_count = kv_n * sm.k_boxes, v_count = kv_n * sm.v_boxes, q_count = heads_n * sm.k_boxes;
    auto load_keys = [&](int i) {
        const int s = p.k_stages == 2 ? i & 1 : 0, z = start + (rank + i * ranks) * NK;
        if (threadIdx.x == 0) tc::mbar_expect_tx(&k_full[s], k_count * (NK * 128) + (i == 0 ? q_count * (SP_ROWS * 128) : 0));
        if (lane == 0) {
            if (i == 0)
                for (int e = warp; e < q_count; e += SP_WARPS)
                    tc::tma_load_3d(q_s + e * (SP_ROWS * 128), &map_q, (e % sm.k_boxes) * 64, h0 + e / sm.k_boxes, start + r0, &k_full[s]);
            for (int e = warp; e < k_count; e += SP_WARPS)
                tc::tma_load_3d(k_s + s * sm.k + e * (NK * 128), &map_k, (e % sm.k_boxes) * 64, kv0 + e / sm.k_boxes, z, &k_full[s]);
        }
        __syncwarp();
    };
    auto load_values = [&](int i) {
        const int z = start + (rank + i * ranks) * NK;
        if (threadIdx.x == 0) tc::mbar_expect_tx(&v_full, v_count * (NK * 128));
        if (lane == 0)
            for (int e = warp; e < v_count; e += SP_WARPS)
                tc::tma_load_3d(v_s + e * (NK * 128), &map_v, (e % sm.v_boxes) * 64, kv0 + e / sm.v_boxes, z, &v_full);
        __syncwarp();
    };
    int k_asked = 0, v_asked = 0;
    for (; k_asked < my_tiles && k_asked < p.k_stages; k_asked++) load_keys(k_asked);
    if (my_tiles > 0) load_values(0), v_asked = 1;

    float o[VT][4];
#pragma unroll
    for (int t = 0; t < VT; t++) o[t][0] = o[t][1] = o[t][2] = o[t][3] = 0.0f;
    const int n_vt = EXACT ? VT * WPH : (VD + 15) / 16 * 2, d_steps = (D + 15) / 16;  // (n_vt: tiles of a whole head)
    // a lane's place in fragments of 16 rows of 128 bytes under the swizzle: row operand (rows lane & 15, pieces of 16 bytes
    // lane >> 4) and the values (transposed); column operand of the scores (keys, pieces (lane >> 3) & 1)
    const uint32_t row_a = (lane & 15) * 128, x_a = ((lane >> 4) ^ (lane & 7)) << 4;
    const uint32_t row_k = ((lane & 7) + ((lane >> 4) << 3)) * 128, x_k = (((lane >> 3) & 1) ^ (lane & 7)) << 4;
    const int kv_of = hg / R - kv0;
    const uint32_t qa = q_s + (hg - h0) * sm.k_boxes * (SP_ROWS * 128) + row_a;
    const uint32_t kb = k_s + kv_of * sm.k_boxes * (NK * 128) + part * 2048 + row_k;
    const uint32_t vb = v_s + kv_of * sm.v_boxes * (NK * 128) + row_a;
    uint32_t qx4[4], xk4[4], vx4[4];  // the four places of 16 columns within a box
#pragma unroll
    for (int c4 = 0; c4 < 4; c4++) qx4[c4] = qa + (x_a ^ (c4 << 5)), xk4[c4] = x_k ^ (c4 << 5), vx4[c4] = vb + (x_a ^ (c4 << 5));
    const uint32_t pb = p_s + (lane & 15) * sm.p_row + hl * 32 + (lane >> 4) * 16;
    // this thread's weights: query row r8 of the warp's 16 keys, the two keys 2 q2, + 1
    const uint32_t wb = w_s + (part * SP_ROWS + r8) * sm.w_row + ((hg >> 1) + (hg & 1) * (heads_in >> 1)) * 32 + q2 * 8;
    const int buffer = PAIR ? sm.w / 2 : 0;
    const uint32_t wb_peer = PAIR ? tc::peer_smem(wb, in_cluster ^ 1) : 0;

    // scores and weights of tile i, into shared memory (PAIR: both CTAs')
    auto scores = [&](int i) {
        const int s = p.k_stages == 2 ? i & 1 : 0, key0 = (rank + i * ranks) * NK + part * 16;  // this warp's first key
        if (!tc::mbar_wait(&k_full[s], (p.k_stages == 2 ? i >> 1 : i) & 1)) failed[i & 1] = 1;
        if (!has_head) return;
        float c[2][4];
#pragma unroll
        for (int t = 0; t < 2; t++) c[t][0] = c[t][1] = c[t][2] = c[t][3] = 0.0f;
        uint32_t qx = qa, kx = kb + s * sm.k;
        if constexpr (EXACT) {
            each<8>([&](auto step) {
                constexpr int c4 = decltype(step)::value % 4, box = decltype(step)::value / 4;
                uint32_t a[4], b[4];
                ldsm_at<box * SP_ROWS * 128>(qx4[c4], a);
                ldsm_at<box * NK * 128>(kx + xk4[c4], b);
                mma_bf16(c[0], a, b[0], b[1]);
                mma_bf16(c[1], a, b[2], b[3]);
            });
        } else {
            for (int left = d_steps; left > 0; left -= 4, qx += SP_ROWS * 128, kx += NK * 128) {
#pragma unroll
                for (int c4 = 0; c4 < 4; c4++) {
                    if (c4 < left) {
                        uint32_t a[4], b0, b1, b2, b3;
                        ldsm_x4(qx + (x_a ^ (c4 << 5)), a[0], a[1], a[2], a[3]);
                        ldsm_x4(kx + (x_k ^ (c4 << 5)), b0, b1, b2, b3);
                        mma_bf16(c[0], a, b0, b1);
                        mma_bf16(c[1], a, b2, b3);
                    }
                }
            }
        }
        const int first_back = r0 + r8 - key0 - 2 * q2;
        const float back = (float)first_back;  // of this thread's first row and key
        const float away_a = fmaf(hd.slope, back, hd.base), away_b = fmaf(hd.slope, 8.0f, away_a);
#pragma unroll
        for (int t = 0; t < 2; t++) {
#pragma unroll
            for (int e = 0; e < 4; e++)
                c[t][e] = sigmoid_of(CAP, hd, c[t][e], fmaf(-hd.slope, (float)(t * 8 + (e & 1)), e < 2 ? away_a : away_b));
        }
        if (!(key0 + 15 <= r0 && r0 + SP_ROWS <= n)) {  // not every key is seen from every row
#pragma unroll
            for (int t = 0; t < 2; t++) {
#pragma unroll
                for (int e = 0; e < 4; e++) {
                    const int j = key0 + t * 8 + 2 * q2 + (e & 1), row = r0 + r8 + (e >> 1) * 8;
                    if (j > row || row >= n) c[t][e] = 0.0f;
                }
            }
        }
        const uint32_t at = (PAIR ? (i & 1) * buffer : 0);
#pragma unroll
        for (int t = 0; t < 2; t++) {
            const uint32_t to = at + t * heads_in * 32;
            asm volatile("st.shared.v2.f32 [%0], {%1, %2};" ::"r"(wb + to), "f"(c[t][0]), "f"(c[t][1]) : "memory");
            asm volatile("st.shared.v2.f32 [%0], {%1, %2};" ::"r"(wb + to + 8 * sm.w_row), "f"(c[t][2]), "f"(c[t][3]) : "memory");
            if (PAIR) {
                asm volatile("st.shared::cluster.v2.f32 [%0], {%1, %2};" ::"r"(wb_peer + to), "f"(c[t][0]), "f"(c[t][1]) : "memory");
                asm volatile("st.shared::cluster.v2.f32 [%0], {%1, %2};" ::"r"(wb_peer + to + 8 * sm.w_row), "f"(c[t][2]), "f"(c[t][3]) : "memory");
            }
        }
    };
    // tile i's weights mixed, a query row's 16 keys at a time (warp w has query row w, of the first 16 keys, then of the next)
    const uint32_t mix_from = w_s + warp * sm.w_row + q2 * 32 + r8 * 4, mix_to = p_s + warp * sm.p_row + r8 * 32 + q2 * 4;
    auto mixing = [&](int i) {
#pragma unroll
        for (int c = 0; c < WPH; c++) {
            const uint32_t w = mix_from + (PAIR ? (i & 1) * buffer : 0) + c * SP_WARPS * sm.w_row;
            const uint32_t w_odd = w + heads_in * 16;  // an odd head's weights
            float m[2][4];
#pragma unroll
            for (int half = 0; half < 2; half++) m[half][0] = m[half][1] = m[half][2] = m[half][3] = 0.0f;
            each<BLOCKS>([&](auto block) {
                constexpr int s = decltype(block)::value;
                const int gi = 16 * s + 2 * q2;   // (heads that are not there left nothing)
                const bool in0 = EXACT || gi < H, in1 = EXACT || gi + 1 < H;
                const bool in8 = EXACT ? WPH == 1 : gi + 8 < H, in9 = EXACT ? WPH == 1 : gi + 9 < H;
#pragma unroll
                for (int half = 0; half < 2; half++) {
                    const uint32_t even = w + half * heads_in * 32, uneven = w_odd + half * heads_in * 32;
                    const float x0 = in0 ? lds_at<s * 256>(even) : 0.0f, x1 = in1 ? lds_at<s * 256>(uneven) : 0.0f;
                    const float x8 = in8 ? lds_at<s * 256 + 128>(even) : 0.0f, x9 = in9 ? lds_at<s * 256 + 128>(uneven) : 0.0f;
                    uint32_t b0[3], b1[3];
                    split3_pair(x0, x1, b0), split3_pair(x8, x9, b1);
#pragma unroll
                    for (int k = 2; k >= 0; k--) mma_bf16(m[half], ta[s], b0[k], b1[k]);
                }
            });
            const uint32_t to = mix_to + c * SP_WARPS * sm.p_row;
            each<2>([&](auto which) {
                constexpr int half = decltype(which)::value;
                uint32_t lo[3], hi[3];
                split3_pair(m[half][0], m[half][1], lo);
                if (WPH == 1) split3_pair(m[half][2], m[half][3], hi);
                each<3>([&](auto piece) {
                    constexpr int k = decltype(piece)::value;
                    sts_at<k * HEADS * 32 + half * 16>(to, lo[k]);
                    if (WPH == 1) sts_at<k * HEADS * 32 + half * 16 + 8 * 32>(to, hi[k]);
                });
            });
        }
    };
    // every weight of tile i is there (PAIR: from both CTAs); its keys, and the values and mixed weights of the tile before, are
    // done with
    auto meet = [&]() {
        if (PAIR) tc::cluster_sync();
        else __syncthreads();
    };

    if (PAIR) tc::cluster_sync();  // (the other CTA has started: its memory may be written)
    bool bad = false;
    if (my_tiles > 0) {
        scores(0);
        meet();
        bad = failed[0];
        if (k_asked < my_tiles && !bad) load_keys(k_asked), k_asked++;
        mixing(0);
        __syncthreads();
    }
    for (int it = 0; it < my_tiles; it++) {
        const int key0 = (rank + it * ranks) * NK;
        if (it + 1 < my_tiles && !bad) scores(it + 1);
        if (!bad && !tc::mbar_wait(&v_full, it & 1)) failed[(it + 1) & 1] = 1;
        if (key0 + NK > n) {  // rows beyond the sequence's last are another's, or nobody's: their weights are 0, their values count as 0
            const int first = max(n - key0, 0), pieces = sm.v_boxes * 8;
            for (int e = threadIdx.x; e < kv_n * (NK - first) * pieces; e += SP_THREADS) {
                const int row = e / pieces, c = e - row * pieces, g = row / (NK - first), key = first + row - g * (NK - first);
                *(uint4 *)(sp_smem + (v_s - q_s) + (g * sm.v_boxes + (c >> 3)) * (NK * 128) + key * 128 + (c & 7) * 16) = make_uint4(0, 0, 0, 0);
            }
            __syncthreads();
        }
        if (has_head) {
#pragma unroll
            for (int c = 0; c < WPH; c++) {
                uint32_t a[3][4];
#pragma unroll
                for (int k = 0; k < 3; k++) ldsm_x4(pb + c * SP_ROWS * sm.p_row + k * HEADS * 32, a[k][0], a[k][1], a[k][2], a[k][3]);
                if constexpr (EXACT) {
                    const uint32_t base = c * 2048 + part * (VT / 8) * (NK * 128);  // (a warp's columns are whole boxes)
                    each<VT / 2>([&](auto tile) {
                        constexpr int tp = decltype(tile)::value;
                        uint32_t b[4];
                        ldsm_t_at<(tp >> 2) * NK * 128>(vx4[tp & 3] + base, b);
#pragma unroll
                        for (int k = 0; k < 3; k++) {
                            mma_bf16(o[2 * tp], a[k], b[0], b[1]);
                            mma_bf16(o[2 * tp + 1], a[k], b[2], b[3]);
                        }
                    });
                } else {
#pragma unroll
                    for (int tp = 0; tp < VT / 2; tp++) {
                        const int gt = part * (VT / 2) + tp;  // the pair of column tiles within the head
                        if (2 * gt < n_vt) {
                            uint32_t b0, b1, b2, b3;
                            ldsm_x4_t(vb + (gt >> 2) * (NK * 128) + c * 2048 + (x_a ^ ((gt & 3) << 5)), b0, b1, b2, b3);
#pragma unroll
                            for (int k = 0; k < 3; k++) {
                                mma_bf16(o[2 * tp], a[k], b0, b1);
                                mma_bf16(o[2 * tp + 1], a[k], b2, b3);
                            }
                        }
                    }
                }
            }
        }
        if (it + 1 == my_tiles) break;
        meet();
        bad = bad || failed[(it + 1) & 1];
        if (!bad) {
            load_values(v_asked), v_asked++;
            if (k_asked < my_tiles) load_keys(k_asked), k_asked++;
        }
        mixing(it + 1);
        __syncthreads();
    }
    __syncthreads();
    if (failed[0] | failed[1]) {  // a copy did not come: report it, and let the copies still in flight land (or run out of time)
        if (threadIdx.x == 0) atomicOr(p.status + 2, 1);
        if (warp == 0) {
            for (int i = max(0, k_asked - p.k_stages); i < k_asked; i++) tc::mbar_wait(&k_full[p.k_stages == 2 ? i & 1 : 0], (p.k_stages == 2 ? i >> 1 : i) & 1);
            if (v_asked > 0) tc::mbar_wait(&v_full, (v_asked - 1) & 1);
        }
        __syncthreads();
    }
    __nv_bfloat16 *out = p.out + (long long)(start + r0 + r8) * H * VD + (long long)hg * VD + 2 * q2;
    const bool in_a = r0 + r8 < n, in_b = r0 + r8 + 8 < n;
    if (ranks > 1) {
        // the CTAs' sums side by side in their own memory, then every CTA adds its share of the column tiles, in rank order
        float4 *mine = (float4 *)sp_smem + warp * VT * 32 + lane;
#pragma unroll
        for (int t = 0; t < VT; t++) mine[t * 32] = make_float4(o[t][0], o[t][1], o[t][2], o[t][3]);
        tc::cluster_sync();
        if (has_head) {
            for (int t = rank; t < VT; t += ranks) {
                const uint32_t at = q_s + ((warp * VT + t) * 32 + lane) * 16;
                float4 v[8], sum = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
#pragma unroll
                for (int c = 0; c < 8; c++) v[c] = c < ranks ? tc::ld_cluster_f4(tc::peer_smem(at, c * BLOCKS + (in_cluster & (BLOCKS - 1)))) : sum;
#pragma unroll
                for (int c = 0; c < 8; c++) sum.x += v[c].x, sum.y += v[c].y, sum.z += v[c].z, sum.w += v[c].w;
                const int col = 8 * (part * VT + t);
                if (col + 2 * q2 < VD) {  // (v_dim is even)
                    if (in_a) *(__nv_bfloat162 *)(out + col) = __floats2bfloat162_rn(sum.x, sum.y);
                    if (in_b) *(__nv_bfloat162 *)(out + 8LL * H * VD + col) = __floats2bfloat162_rn(sum.z, sum.w);
                }
            }
        }
        tc::cluster_sync();  // nobody leaves while its sums may still be read
        return;
    }
    if (has_head) {
#pragma unroll
        for (int t = 0; t < VT; t++) {
            const int col = 8 * (part * VT + t);
            if (col + 2 * q2 < VD) {
                if (in_a) *(__nv_bfloat162 *)(out + col) = __floats2bfloat162_rn(o[t][0], o[t][1]);
                if (in_b) *(__nv_bfloat162 *)(out + 8LL * H * VD + col) = __floats2bfloat162_rn(o[t][2], o[t][3]);
            }
        }
    }
    if (PAIR) tc::cluster_sync();  // (the other CTA's last weights have arrived: nobody leaves while it may still be written to)
}

struct SigmoidPromptPlan {
    int wph, k_stages, kv_block, pair, smem;
};

// How a CTA is laid out for these sizes: two warps a head for up to 8 heads where shared memory allows, two stages of keys where
// it allows. False: the sizes are not taken.
static bool sp_plan(int n_heads, int n_kv_heads, int head_dim, int v_dim, SigmoidPromptPlan &plan) {
    if (n_kv_heads < 1 || n_heads < 1 || n_heads % n_kv_heads || n_heads > SP_MAX_HEADS) return false;
    if (head_dim % 8 || head_dim < 8 || v_dim % 8 || v_dim < 8 || v_dim > 128) return false;
    const int r = n_heads / n_kv_heads;
    plan.pair = n_heads > 16, plan.kv_block = 0;
    for (int h = 0; h < n_heads; h += 16) {
        const int last = (h + 16 < n_heads ? h + 16 : n_heads) - 1, count = last / r - h / r + 1;
        if (count > plan.kv_block) plan.kv_block = count;
    }
    for (plan.wph = n_heads <= 8 ? 2 : 1; plan.wph >= 1; plan.wph--) {
        for (plan.k_stages = 2; plan.k_stages >= 1; plan.k_stages--) {
            plan.smem = SigmoidPromptSmem(n_heads, head_dim, v_dim, plan.kv_block, plan.wph, plan.k_stages).total;
            if (plan.smem <= 226 * 1024) return true;
        }
    }
    return false;
}

extern "C" int abk_attention_sigmoid_prompt_takes(int n_heads, int n_kv_heads, int head_dim, int v_dim) {
    SigmoidPromptPlan plan;
    return sp_plan(n_heads, n_kv_heads, head_dim, v_dim, plan);
}

template <int WPH, bool CAP, bool EXACT, bool PAIR>
static int sp_launch(const CUtensorMap &mq, const CUtensorMap &mk, const CUtensorMap &mv, const SigmoidPrompt &p, int cluster, int smem, cudaStream_t s) {
    cudaError_t e = abk_allow_shared_memory((const void *)attention_sigmoid_prompt_kernel<WPH, CAP, EXACT, PAIR>, smem);
    if (e != cudaSuccess) return (int)e;
    abk_launch_clusters(attention_sigmoid_prompt_kernel<WPH, CAP, EXACT, PAIR>, dim3(p.tiles * cluster), dim3(SP_THREADS), (size_t)smem, s, cluster, mq, mk, mv, p);
    return ABK_LAUNCH_RESULT();
}

// qkv: n_rows rows of `row` elements, q heads, then (at k_off) k heads, then (at v_off) v heads. tiles: an upper bound of
// the step's tiles of 16 query rows, sum over its sequences of ceil(rows / 16). mix holds bfloat16 numbers (the tensor-core
// operand), as a bfloat16 model stores it. forced_ranks: 0, or the CTAs a query tile's keys are dealt to (1, 2, 4, 8; at most 4
// with more than 16 heads). status word 2 is set if a wait ran out.
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
    p.k_stages = plan.k_stages, p.status = status;
    CUtensorMap mq, mk, mv;
    const __nv_bfloat16 *base = (const __nv_bfloat16 *)qkv;
    int rc = tmap::bf16_heads(base, head_dim, n_heads, n_rows, row, SP_ROWS, &mq);
    if (!rc) rc = tmap::bf16_heads(base + k_off, head_dim, n_kv_heads, n_rows, row, 16 * plan.wph, &mk);
    if (!rc) rc = tmap::bf16_heads(base + v_off, v_dim, n_kv_heads, n_rows, row, 16 * plan.wph, &mv);
    if (rc) return rc;
    const int blocks = plan.pair ? 2 : 1;
    int ranks = 1;
    while (ranks < 8 / blocks && (long long)tiles * blocks * ranks * 3 < 5LL * abk_sm_count()) ranks *= 2;
    if (forced_ranks == 1 || forced_ranks == 2 || forced_ranks == 4 || forced_ranks == 8) ranks = forced_ranks < 8 / blocks ? forced_ranks : 8 / blocks;
    if ((long long)tiles * ranks * blocks > 0x7fffffffLL) ABK_REFUSE("attention_sigmoid_prompt: %d tiles are more than a grid takes", tiles);
    cudaStream_t s = (cudaStream_t)stream;
    // the sizes of larger models have kernels of their own
    const bool exact = n_heads == 16 / plan.wph * blocks && head_dim == 128 && v_dim == 128;
#define SP_RUN(WPH, CAP, EXACT, PAIR) sp_launch<WPH, CAP, EXACT, PAIR>(mq, mk, mv, p, ranks * blocks, plan.smem, s)
#define SP_BY_SIZE(WPH, CAP, PAIR) (exact ? SP_RUN(WPH, CAP, true, PAIR) : SP_RUN(WPH, CAP, false, PAIR))
    if (plan.pair) return softcap > 0.0f ? SP_BY_SIZE(1, true, true) : SP_BY_SIZE(1, false, true);
    if (plan.wph == 1) return softcap > 0.0f ? SP_BY_SIZE(1, true, false) : SP_BY_SIZE(1, false, false);
    return softcap > 0.0f ? SP_BY_SIZE(2, true, false) : SP_BY_SIZE(2, false, false);
#undef SP_BY_SIZE
#undef SP_RUN
}
