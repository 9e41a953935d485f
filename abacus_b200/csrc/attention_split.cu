// Decode attention (one new token per sequence) over the paged cache with the general options (a window that also
// keeps the first keys, a sink, values of another size than keys, float32 softmax weights), split along the keys so
// that a handful of rows fills the GPU: a CTA takes 64 or 128 of a row's visible keys for all query heads of one kv head
// (each key and value row is read once for the group), and leaves, per head, the maximum, the sum and the
// unnormalised weighted values of its keys; a second kernel folds a row's parts, the sink among them.
//
//   key j is seen from position i when j <= i and (window == 0 or i - j < window or j < keep_first)
//                                             and (chunk == 0 or j / chunk == i / chunk)
//   p_j = exp(z_j - M) / (exp(sink - M) + sum_j exp(z_j - M)),  z_j = scale * (q . k_j),  out = sum_j p_j v_j
//   (with a cap c of the scores, z_j = c tanh(scale * (q . k_j) / c))
//
// Differential attention (maps 2): query heads in runs of two read the two halves of a key row, each a map of its own over
// the same values; the fold makes one head of the two (csrc/differential.cuh), so both maps' sums stay float32.
//
// A row's visible keys are numbered: first the kept first keys the window no longer reaches, then the window's
// (or all). Part t has numbers [P t, P t + P), P = 128, or 64 where parts of 128 are too few. All arithmetic is float32.
#define ABK_DEFINE_ERROR
#include "common.cuh"
#include "differential.cuh"
#include "mma_tiles.cuh"

#define AS_THREADS 128
#define AS_MAX_GROUP 16
#define AS_MAX_DIM 256

struct AttnSplit {
    const void *q;       // row t, head h at q + t * q_row + h * head_dim
    long long q_row;
    float *parts;        // [tokens, heads, n_parts, v_dim + 2]: weighted values, then maximum and sum
    void *out;           // [tokens, heads * v_dim]
    int n_heads, n_kv_heads, head_dim, v_dim;
    int maps;            // a key row holds maps * head_dim elements; query head h reads slice h % maps
    DifferentialHead diff;  // maps 2: what makes a head of its two maps (out is then [tokens, n_heads / 2 * v_dim])
    float scale;
    float softcap;       // > 0: z <- softcap * tanh(z / softcap), after the scale
    int window, keep_first;
    int chunk;           // > 0: key j is seen from i only if j / chunk == i / chunk
    const float *sink;
    const int *token_seq, *token_pos, *seq_slot;
    const void *k_pool, *v_pool;
    PagedCache cache, v_cache;
    int n_parts, part_keys;  // a row's parts have part_keys keys each (128, or 64)
    int values_in_keys;  // a value is the first v_dim elements of its key row (one pool)
    int runs;            // runs of query heads, a CTA each, that share a kv head of the cache; n_kv_heads counts the runs
    const void *gate;    // null, or a gate per token and head (of q's type, at gate + t * ldg + h): the head's output is
    long long ldg;       // multiplied by its sigmoid where the parts are folded
};

// (first key of the window, number of kept first keys before it, number of visible keys) of a token at pos
__device__ __forceinline__ void visible_keys(const AttnSplit &p, int pos, int &lo, int &kept, int &total) {
    lo = p.window > 0 && pos - p.window + 1 > 0 ? pos - p.window + 1 : 0;
    kept = p.keep_first < lo ? p.keep_first : lo;
    if (p.chunk > 0) {  // the token's chunk starts no earlier than any kept first key that lies outside it
        const int first = pos / p.chunk * p.chunk;
        if (first > lo) lo = first;
        if (first > 0) kept = 0;
    }
    total = kept + pos - lo + 1;
}

// The score of a product q . k: scaled, then capped where the layer caps its scores.
__device__ __forceinline__ float score_of(const AttnSplit &p, float dot) {
    const float z = dot * p.scale;
    return p.softcap > 0.0f ? p.softcap * tanhf(z / p.softcap) : z;
}

// q (float32, 16-byte aligned, the same for every thread: a broadcast) . k (this thread's key row)
template <typename T> __device__ __forceinline__ float dot_q(const float *q, const T *k, int hd);
template <> __device__ __forceinline__ float dot_q<float>(const float *q, const float *k, int hd) {
    float acc = 0.0f;
    for (int i = 0; i < hd; i += 4) {
        const float4 v = *(const float4 *)(k + i), w = *(const float4 *)(q + i);
        acc = fmaf(w.x, v.x, acc), acc = fmaf(w.y, v.y, acc), acc = fmaf(w.z, v.z, acc), acc = fmaf(w.w, v.w, acc);
    }
    return acc;
}
template <> __device__ __forceinline__ float dot_q<__nv_bfloat16>(const float *q, const __nv_bfloat16 *k, int hd) {
    float a0 = 0.0f, a1 = 0.0f;
    for (int i = 0; i < hd; i += 8) {
        const uint4 raw = *(const uint4 *)(k + i);
        const float4 w0 = *(const float4 *)(q + i), w1 = *(const float4 *)(q + i + 4);
        const __nv_bfloat162 *h = (const __nv_bfloat162 *)&raw;
        const float2 f0 = __bfloat1622float2(h[0]), f1 = __bfloat1622float2(h[1]), f2 = __bfloat1622float2(h[2]),
                     f3 = __bfloat1622float2(h[3]);
        a0 = fmaf(w0.x, f0.x, a0), a1 = fmaf(w0.y, f0.y, a1), a0 = fmaf(w0.z, f1.x, a0), a1 = fmaf(w0.w, f1.y, a1);
        a0 = fmaf(w1.x, f2.x, a0), a1 = fmaf(w1.y, f2.y, a1), a0 = fmaf(w1.z, f3.x, a0), a1 = fmaf(w1.w, f3.y, a1);
    }
    return a0 + a1;
}

// STAGED: the part's 128 key rows come into shared memory by cp.async, all at once (padded by 16 bytes so that a thread
// reading its own row meets no bank conflict), and once the scores are made the 128 value rows into the same memory,
// under the softmax; else each thread reads global memory.
// GMAX: the group's size rounded up to 1, 2, 4, 8 or 16 (what the loops over its heads are unrolled to).
// A float32 number as three bfloat16 numbers that add up to it (its 24 bits), each pair packed for one operand register.
__device__ __forceinline__ void as_split3(float x, float y, uint32_t &hi, uint32_t &mid, uint32_t &lo) {
    const __nv_bfloat16 xh = __float2bfloat16_rn(x), yh = __float2bfloat16_rn(y);
    const float xr = x - __bfloat162float(xh), yr = y - __bfloat162float(yh);
    const __nv_bfloat16 xm = __float2bfloat16_rn(xr), ym = __float2bfloat16_rn(yr);
    const __nv_bfloat16 xl = __float2bfloat16_rn(xr - __bfloat162float(xm)), yl = __float2bfloat16_rn(yr - __bfloat162float(ym));
    hi = (uint32_t)__bfloat16_as_ushort(xh) | ((uint32_t)__bfloat16_as_ushort(yh) << 16);
    mid = (uint32_t)__bfloat16_as_ushort(xm) | ((uint32_t)__bfloat16_as_ushort(ym) << 16);
    lo = (uint32_t)__bfloat16_as_ushort(xl) | ((uint32_t)__bfloat16_as_ushort(yl) << 16);
}

template <typename T, bool STAGED, int GMAX> __global__ void __launch_bounds__(AS_THREADS) attention_split_kernel(AttnSplit p) {
    extern __shared__ __align__(16) float as_smem[];
    const int group = p.n_heads / p.n_kv_heads, hd = p.head_dim, vd = p.v_dim, kd = p.maps * hd;  // kd: a key row
    float *q_s = as_smem;                      // [group][hd]
    float *p_s = q_s + group * hd;             // [group][128]
    float *red = p_s + group * AS_THREADS;     // [4][group] maxima, then sums
    const int k_pitch = kd * (int)sizeof(T) + 16;
    uint8_t *k_s = (uint8_t *)(red + ((4 * group + 3) & ~3));  // [128][k_pitch]
    uint8_t *v_s = k_s;                                        // [128][vd], once the keys are done with
    __shared__ long long k_off[AS_THREADS], v_off[AS_THREADS];
    const int t = blockIdx.x, kvh = blockIdx.y, part = blockIdx.z, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    // the step's indices and the page table were written by kernels further back than the one just before
    const int seq = p.token_seq[t];
    const int pos = p.token_pos[t];
    int lo = 0, kept = 0, total = 0;
    if (seq >= 0) visible_keys(p, pos, lo, kept, total);
    if (part * AS_THREADS >= total) {  // (the fold knows how many parts a row has)
        pdl_wait();
        return;
    }
    const int slot = p.seq_slot[seq], n_valid = total - part * AS_THREADS < AS_THREADS ? total - part * AS_THREADS : AS_THREADS;
    const int number = part * AS_THREADS + tid;
    const bool valid = number < total;
    if (valid) {
        const int j = number < kept ? number : lo + number - kept;
        const int page = cache_page(p.cache, slot, j);
        const int ckv = kvh / p.runs, cn = p.n_kv_heads / p.runs;
        v_off[tid] = cache_offset(p.v_cache, page, ckv, cn, j, p.values_in_keys ? kd : vd);
        k_off[tid] = cache_offset(p.cache, page, ckv, cn, j, kd);
    }
    pdl_wait();
    const T *q = (const T *)p.q + (long long)t * p.q_row + (long long)kvh * group * hd;
    for (int e = tid; e < group * hd; e += AS_THREADS) q_s[e] = to_float(q[e]);
    __syncthreads();
    if (STAGED) {
        const uint32_t k_dst = (uint32_t)__cvta_generic_to_shared(k_s);
        const int k_chunks = kd * (int)sizeof(T) / 16;
        for (int e = tid; e < n_valid * k_chunks; e += AS_THREADS) {
            const int r = e / k_chunks, c = e - r * k_chunks;
            asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(k_dst + r * k_pitch + c * 16),
                         "l"((const uint8_t *)((const T *)p.k_pool + k_off[r]) + c * 16) : "memory");
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
        asm volatile("cp.async.wait_group 0;" ::: "memory");  // the keys are here
        __syncthreads();
    }
    float sc[GMAX];
    if (valid) {
        const T *k = STAGED ? (const T *)(k_s + tid * k_pitch) : (const T *)p.k_pool + k_off[tid];
#pragma unroll
        for (int g = 0; g < GMAX; g++)
            if (g < group) sc[g] = score_of(p, dot_q<T>(q_s + g * hd, k + (p.maps == 2 && (g & 1) ? hd : 0), hd));
    } else {
#pragma unroll
        for (int g = 0; g < GMAX; g++) sc[g] = -INFINITY;
    }
    // per head: the part's maximum, the weights against it, their sum
#pragma unroll
    for (int g = 0; g < GMAX; g++) {
        if (g < group) {
            const float m = warp_max(sc[g]);
            if (lane == 0) red[warp * group + g] = m;
        }
    }
    __syncthreads();
    if (STAGED && !p.values_in_keys) {  // every thread has read its key row: the values come into the same memory, under the softmax
        const uint32_t v_dst = (uint32_t)__cvta_generic_to_shared(v_s);
        const int v_chunks = vd * (int)sizeof(T) / 16;
        for (int e = tid; e < n_valid * v_chunks; e += AS_THREADS) {
            const int r = e / v_chunks, c = e - r * v_chunks;
            asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(v_dst + (r * v_chunks + c) * 16),
                         "l"((const uint8_t *)((const T *)p.v_pool + v_off[r]) + c * 16) : "memory");
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    }
    float top[GMAX];
#pragma unroll
    for (int g = 0; g < GMAX; g++) {
        if (g < group) {
            top[g] = fmaxf(fmaxf(red[g], red[group + g]), fmaxf(red[2 * group + g], red[3 * group + g]));
            sc[g] = valid ? expf(sc[g] - top[g]) : 0.0f;
            p_s[g * AS_THREADS + tid] = sc[g];
        }
    }
    __syncthreads();
#pragma unroll
    for (int g = 0; g < GMAX; g++) {
        if (g < group) {
            const float s = warp_sum(sc[g]);
            if (lane == 0) red[warp * group + g] = s;
        }
    }
    if (STAGED && !p.values_in_keys) asm volatile("cp.async.wait_group 0;" ::: "memory");  // the values are here
    __syncthreads();
    // weighted values: a thread a value column (two for values beyond 128), every head of the group per value read
    float acc0[GMAX], acc1[GMAX];
#pragma unroll
    for (int g = 0; g < GMAX; g++) acc0[g] = acc1[g] = 0.0f;
    const T *v_base = (const T *)p.v_pool;
    if (tid < vd) {
        for (int jj = 0; jj < n_valid; jj++) {
            const T *v = !STAGED ? v_base + v_off[jj]
                         : p.values_in_keys ? (const T *)(k_s + jj * k_pitch) : (const T *)v_s + (long long)jj * vd;
            const float a = to_float(v[tid]);
#pragma unroll
            for (int g = 0; g < GMAX; g++)
                if (g < group) acc0[g] = fmaf(p_s[g * AS_THREADS + jj], a, acc0[g]);
            if (tid + AS_THREADS < vd) {
                const float b = to_float(v[tid + AS_THREADS]);
#pragma unroll
                for (int g = 0; g < GMAX; g++)
                    if (g < group) acc1[g] = fmaf(p_s[g * AS_THREADS + jj], b, acc1[g]);
            }
        }
    }
#pragma unroll
    for (int g = 0; g < GMAX; g++) {
        if (g < group) {
            float *dst = p.parts + (((long long)t * p.n_heads + kvh * group + g) * p.n_parts + part) * (vd + 2);
            if (tid < vd) dst[tid] = acc0[g];
            if (tid + AS_THREADS < vd) dst[tid + AS_THREADS] = acc1[g];
            if (tid == 0) {
                dst[vd] = top[g];
                dst[vd + 1] = (red[g] + red[group + g]) + (red[2 * group + g] + red[3 * group + g]);
            }
        }
    }
}

// The same in bfloat16 with both products on the warp-level tensor cores, the group's heads as the 16 rows of a tile (key rows
// a multiple of 16 elements, values a multiple of 8 up to 256). A CTA takes PART keys; they, their values (OWN_V; else a
// value is the first elements of its key row: latent rows) and the queries come into shared memory by cp.async, zeros in
// the places of keys and heads there are none of. Where a head has two maps its query stands in its map's half of a row as
// wide as a key's, zeros in the other, so that one product makes both maps' scores. A warp makes the scores of PART / 4 keys and
// has them in registers: maxima and sums meet over the warps through shared memory. The weighted values: the float32
// weights as three bfloat16 parts that hold their 24 bits, each multiplied with the same value fragments, so that the
// weights stay float32 in effect.
template <int PART, bool OWN_V> __global__ void __launch_bounds__(AS_THREADS) attention_split_tiles_kernel(AttnSplit p) {
    extern __shared__ __align__(16) float as_smem[];
    constexpr int KEYS = PART / 4, NT = KEYS / 8, P_PITCH = PART + 8;  // a warp's keys, its tiles of 8
    const int group = p.n_heads / p.n_kv_heads, hd = p.head_dim, vd = p.v_dim, kd = p.maps * hd, pitch = kd * 2 + 16;
    const int v_pitch = OWN_V ? ((vd + 15) & ~15) * 2 + 16 : pitch;
    float *p_s = as_smem;                           // [16][P_PITCH] weights
    float *red = p_s + 16 * P_PITCH;                // [2][4][16] the warps' maxima, then their sums
    uint8_t *q_s = (uint8_t *)(red + 128);          // [16][pitch]
    uint8_t *k_s = q_s + 16 * pitch;                // [PART][pitch]
    uint8_t *v_s = OWN_V ? k_s + PART * pitch : k_s;  // [PART][v_pitch]
    __shared__ long long k_off[PART], v_off[OWN_V ? PART : 1];
    const int t = blockIdx.x, run = blockIdx.y, part = blockIdx.z, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int g = lane >> 2, c2 = (lane & 3) * 2;
    // the step's indices, the page table and the keys of earlier steps were written by kernels further back than the one just
    // before (which makes the queries and the token's own key): they are read before the wait
    const int seq = p.token_seq[t];
    const int pos = p.token_pos[t];
    int lo = 0, kept = 0, total = 0;
    if (seq >= 0) visible_keys(p, pos, lo, kept, total);
    if (part * PART >= total) {  // (the fold knows how many parts a row has)
        pdl_wait();
        return;
    }
    const int slot = p.seq_slot[seq], n_valid = min(total - part * PART, PART);
    if (tid < PART) {
        const int number = part * PART + min(tid, n_valid - 1), j = number < kept ? number : lo + number - kept;
        const int cn = p.n_kv_heads / p.runs, page = cache_page(p.cache, slot, j);
        k_off[tid] = cache_offset(p.cache, page, run / p.runs, cn, j, kd);
        if (OWN_V) v_off[OWN_V ? tid : 0] = cache_offset(p.v_cache, page, run / p.runs, cn, j, vd);
    }
    const uint32_t q_at = (uint32_t)__cvta_generic_to_shared(q_s), k_at = (uint32_t)__cvta_generic_to_shared(k_s);
    const int chunks = kd / 8, v_chunks = vd / 8;
    const uint32_t v_at = (uint32_t)__cvta_generic_to_shared(v_s);
    const __nv_bfloat16 *q = (const __nv_bfloat16 *)p.q + (long long)t * p.q_row + (long long)run * group * hd;
    // where the token's own key lies among the part's (it is the last that is seen)
    const int own = part * PART + n_valid == total ? n_valid - 1 : PART;
    __syncthreads();
    for (int e = tid; e < PART * chunks; e += AS_THREADS) {
        const int r = e / chunks, c = e - r * chunks;
        if (r == own) continue;
        asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(k_at + r * pitch + c * 16),
                     "l"((const __nv_bfloat16 *)p.k_pool + k_off[r] + c * 8), "r"(r < n_valid ? 16 : 0) : "memory");
    }
    if (OWN_V)
        for (int e = tid; e < PART * v_chunks; e += AS_THREADS) {
            const int r = e / v_chunks, c = e - r * v_chunks;
            if (r == own) continue;
            asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(v_at + r * v_pitch + c * 16),
                         "l"((const __nv_bfloat16 *)p.v_pool + v_off[OWN_V ? r : 0] + c * 8), "r"(r < n_valid ? 16 : 0) : "memory");
        }
    pdl_wait();
    if (own < PART) {
        for (int c = tid; c < chunks; c += AS_THREADS)
            asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(k_at + own * pitch + c * 16),
                         "l"((const __nv_bfloat16 *)p.k_pool + k_off[own] + c * 8) : "memory");
        if (OWN_V)
            for (int c = tid; c < v_chunks; c += AS_THREADS)
                asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(v_at + own * v_pitch + c * 16),
                             "l"((const __nv_bfloat16 *)p.v_pool + v_off[OWN_V ? own : 0] + c * 8) : "memory");
    }
    const int slice = chunks / p.maps;  // 16-byte pieces of a map
    for (int e = tid; e < 16 * chunks; e += AS_THREADS) {
        const int r = e / chunks, c = e - r * chunks, first = r % p.maps * slice;
        const bool in = r < group && c >= first && c < first + slice;
        asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(q_at + r * pitch + c * 16),
                     "l"(q + (long long)min(r, group - 1) * hd + (in ? c - first : 0) * 8), "r"(in ? 16 : 0) : "memory");
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();

    float s[NT][4];
#pragma unroll
    for (int nt = 0; nt < NT; nt++) s[nt][0] = s[nt][1] = s[nt][2] = s[nt][3] = 0.0f;
    const uint32_t qa = q_at + (lane & 15) * pitch + (lane >> 4) * 16;
    const uint32_t ka = k_at + (warp * KEYS + (lane & 7) + ((lane >> 4) << 3)) * pitch + ((lane >> 3) & 1) * 16;
#pragma unroll 4
    for (int kk = 0; kk < kd / 16; kk++) {
        uint32_t a[4];
        ldsm_x4(qa + kk * 32, a[0], a[1], a[2], a[3]);
#pragma unroll
        for (int tp = 0; tp < NT / 2; tp++) {
            uint32_t b0, b1, b2, b3;
            ldsm_x4(ka + tp * 16 * pitch + kk * 32, b0, b1, b2, b3);
            mma_bf16(s[2 * tp], a, b0, b1);
            mma_bf16(s[2 * tp + 1], a, b2, b3);
        }
    }
    // rows g and g + 8 (heads), keys warp * KEYS + 8 nt + c2 + {0, 1}
    float top[2] = {-INFINITY, -INFINITY}, sum[2] = {0.0f, 0.0f};
#pragma unroll
    for (int nt = 0; nt < NT; nt++)
#pragma unroll
        for (int e = 0; e < 4; e++) {
            s[nt][e] = warp * KEYS + nt * 8 + c2 + (e & 1) < n_valid ? score_of(p, s[nt][e]) : -INFINITY;
            top[e >> 1] = fmaxf(top[e >> 1], s[nt][e]);
        }
#pragma unroll
    for (int r = 0; r < 2; r++) {
        top[r] = quad_max(top[r]);
        if (c2 == 0) red[warp * 16 + g + 8 * r] = top[r];
    }
    __syncthreads();
#pragma unroll
    for (int r = 0; r < 2; r++) {
        const float *m = red + g + 8 * r;
        top[r] = fmaxf(fmaxf(m[0], m[16]), fmaxf(m[32], m[48]));  // (the part's first key is a real one)
    }
#pragma unroll
    for (int nt = 0; nt < NT; nt++) {
#pragma unroll
        for (int e = 0; e < 4; e++) s[nt][e] = expf(s[nt][e] - top[e >> 1]), sum[e >> 1] += s[nt][e];
        float *w = p_s + g * P_PITCH + warp * KEYS + nt * 8 + c2;
        *(float2 *)w = make_float2(s[nt][0], s[nt][1]);
        *(float2 *)(w + 8 * P_PITCH) = make_float2(s[nt][2], s[nt][3]);
    }
#pragma unroll
    for (int r = 0; r < 2; r++) {
        sum[r] = quad_sum(sum[r]);
        if (c2 == 0) red[64 + warp * 16 + g + 8 * r] = sum[r];
    }
    __syncthreads();
    // out[head][column]: a warp has every fourth pair of tiles of 8 columns; a key step's weights are split once for all of them
    float o[4][8];
#pragma unroll
    for (int i = 0; i < 4; i++)
#pragma unroll
        for (int e = 0; e < 8; e++) o[i][e] = 0.0f;
    const int n_pairs = (vd + 15) / 16;
    const uint32_t va = v_at + ((lane & 7) + ((lane >> 3) & 1) * 8) * v_pitch + (lane >> 4) * 16;
#pragma unroll
    for (int ks = 0; ks < PART / 16; ks++) {
        if (ks * 16 >= n_valid) break;
        uint32_t hi[4], mid[4], low[4];
#pragma unroll
        for (int f = 0; f < 4; f++) {  // fragment register f: rows g + 8 (f & 1), keys 16 ks + 8 (f >> 1) + c2
            const float2 w = *(const float2 *)(p_s + (g + 8 * (f & 1)) * P_PITCH + ks * 16 + 8 * (f >> 1) + c2);
            as_split3(w.x, w.y, hi[f], mid[f], low[f]);
        }
#pragma unroll
        for (int i = 0; i < 4; i++) {
            const int pair = warp + 4 * i;
            if (pair >= n_pairs) break;
            uint32_t b0, b1, b2, b3;
            ldsm_x4_t(va + ks * 16 * v_pitch + pair * 32, b0, b1, b2, b3);
            mma_bf16(o[i], hi, b0, b1), mma_bf16(o[i] + 4, hi, b2, b3);
            mma_bf16(o[i], mid, b0, b1), mma_bf16(o[i] + 4, mid, b2, b3);
            mma_bf16(o[i], low, b0, b1), mma_bf16(o[i] + 4, low, b2, b3);
        }
    }
#pragma unroll
    for (int i = 0; i < 4; i++) {
        const int pair = warp + 4 * i;
        if (pair >= n_pairs) break;
#pragma unroll
        for (int r = 0; r < 2; r++) {
            if (g + 8 * r >= group) continue;
            float *dst = p.parts + (((long long)t * p.n_heads + run * group + g + 8 * r) * p.n_parts + part) * (vd + 2) + pair * 16 + c2;
            *(float2 *)dst = make_float2(o[i][2 * r], o[i][2 * r + 1]);
            if (pair * 16 + 8 < vd) *(float2 *)(dst + 8) = make_float2(o[i][4 + 2 * r], o[i][4 + 2 * r + 1]);
        }
    }
    if (tid < group) {
        float *dst = p.parts + (((long long)t * p.n_heads + run * group + tid) * p.n_parts + part) * (vd + 2);
        const float *m = red + tid;
        dst[vd] = fmaxf(fmaxf(m[0], m[16]), fmaxf(m[32], m[48]));
        dst[vd + 1] = (m[64] + m[80]) + (m[96] + m[112]);
    }
}

// Folds a row's parts over latents and carries the heads' results out of the latent space in one kernel:
//   out[t, h, :] = W[h] (sum over the parts of their weighted latents, over the sum of their sums) (times a gate per head).
// A CTA has 32 output features of one head for up to 8 rows: its weights are asked for before the wait, a warp folds one
// row (lanes along the latent's columns, two a lane) and leaves it in shared memory in bfloat16, and the product runs on
// the warp-level tensor cores, two warps with 16 features each. rank a multiple of 8.
#define AL_ROWS 8
#define AL_THREADS (32 * AL_ROWS)
#define AL_OUTS 32
#define AL_TURN 8   // blocks of 32 columns whose weights a warp has in flight
#define AL_PARTS 4  // parts whose loads a warp has in flight
struct LatentOut {
    const __nv_bfloat16 *w;  // [heads][outs][rank]
    __nv_bfloat16 *out;      // row t, head h at out + t * ldo + h * outs
    long long ldo;
    int outs, n_rows;
};
__device__ __forceinline__ uint4 al_load16(const __nv_bfloat16 *p, bool ok) { return ok ? __ldg((const uint4 *)p) : make_uint4(0, 0, 0, 0); }

__global__ void __launch_bounds__(AL_THREADS) latent_fold_out_kernel(AttnSplit p, LatentOut l) {
    extern __shared__ __align__(16) uint8_t al_smem[];  // [AL_ROWS][pitch] bfloat16
    const int rank = p.v_dim, blocks = (rank + 31) / 32, pitch = blocks * 32 + 8;
    __nv_bfloat16 *mixed = (__nv_bfloat16 *)al_smem;
    const int tiles = (l.outs + AL_OUTS - 1) / AL_OUTS, h = blockIdx.x / tiles, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int r = lane >> 2, c = lane & 3, o0 = blockIdx.x % tiles * AL_OUTS + warp * 16, t0 = blockIdx.y * AL_ROWS;
    const __nv_bfloat16 *w_lo = l.w + ((long long)h * l.outs + o0 + r) * rank + 8 * c, *w_hi = w_lo + 8LL * rank;
    const bool multiplies = warp < AL_OUTS / 16;
    const bool has_lo = multiplies && o0 + r < l.outs, has_hi = multiplies && o0 + r + 8 < l.outs;
    uint4 a_lo[AL_TURN], a_hi[AL_TURN];
    auto load_weights = [&](int kb) {
#pragma unroll
        for (int u = 0; u < AL_TURN; u++) {
            const bool in = kb + u < blocks && (kb + u) * 32 + 8 * c < rank;
            a_lo[u] = al_load16(w_lo + (kb + u) * 32, in && has_lo), a_hi[u] = al_load16(w_hi + (kb + u) * 32, in && has_hi);
        }
    };
    load_weights(0);
    const float sink = p.sink ? p.sink[h] : -INFINITY;
    const int t = t0 + warp, seq = t < l.n_rows ? p.token_seq[t] : -1, pos = seq >= 0 ? p.token_pos[t] : 0;  // (older than the kernel just before)
    pdl_wait();
    {
        __nv_bfloat16 *dst = mixed + warp * pitch;
        int lo, kept, total;
        visible_keys(p, pos, lo, kept, total);
        const int n = seq >= 0 ? (total + p.part_keys - 1) / p.part_keys : 0;
        const float *src = p.parts + ((long long)t * p.n_heads + h) * p.n_parts * (rank + 2);
        float top = sink, sum = 0.0f;
        float2 acc[4];  // a lane's columns 2 lane + 64 u and the next (rank up to 256)
#pragma unroll
        for (int u = 0; u < 4; u++) acc[u] = make_float2(0.0f, 0.0f);
        if (n > 32) {  // (up to 32 parts a lane's own maximum is the one it has below)
            for (int k = lane; k < n; k += 32) top = fmaxf(top, src[(long long)k * (rank + 2) + rank]);
            top = warp_max(top);
        }
        for (int k0 = 0; k0 < n; k0 += 32) {
            const int left = min(32, n - k0);
            const float2 own = lane < left ? *(const float2 *)(src + (long long)(k0 + lane) * (rank + 2) + rank) : make_float2(-INFINITY, 0.0f);
            if (n <= 32) top = warp_max(fmaxf(top, own.x));
            const float w = expf(own.x - top);  // (0 in lanes without a part)
            sum = fmaf(own.y, w, sum);
            for (int k = 0; k < left; k += AL_PARTS) {
                float2 v[AL_PARTS][4];
#pragma unroll
                for (int i = 0; i < AL_PARTS; i++)
#pragma unroll
                    for (int u = 0; u < 4; u++)
                        v[i][u] = k + i < left && 2 * lane + 64 * u < rank ? *(const float2 *)(src + (long long)(k0 + k + i) * (rank + 2) + 2 * lane + 64 * u)
                                                                          : make_float2(0.0f, 0.0f);
#pragma unroll
                for (int i = 0; i < AL_PARTS; i++) {
                    const float wk = __shfl_sync(0xffffffffu, w, (k + i) & 31);
#pragma unroll
                    for (int u = 0; u < 4; u++) acc[u].x = fmaf(v[i][u].x, wk, acc[u].x), acc[u].y = fmaf(v[i][u].y, wk, acc[u].y);
                }
            }
        }
        sum = warp_sum(sum) + (p.sink ? expf(sink - top) : 0.0f);
        const float inv = n > 0 ? 1.0f / sum : 0.0f;
#pragma unroll
        for (int u = 0; u < 4; u++)
            if (2 * lane + 64 * u < blocks * 32)
                *(__nv_bfloat162 *)(dst + 2 * lane + 64 * u) = __floats2bfloat162_rn(acc[u].x * inv, acc[u].y * inv);
    }
    __syncthreads();
    if (!multiplies) return;
    float acc[4] = {0.0f, 0.0f, 0.0f, 0.0f};
    const __nv_bfloat16 *x = mixed + r * pitch + 8 * c;
    for (int kb = 0; kb < blocks; kb += AL_TURN) {
        if (kb) load_weights(kb);
#pragma unroll
        for (int u = 0; u < AL_TURN; u++) {
            if (kb + u >= blocks) break;
            const uint4 b = *(const uint4 *)(x + (kb + u) * 32);
            // (16 consecutive bytes of both operands' rows: the columns sit in the product's slots in the same way)
            const uint32_t a0[4] = {a_lo[u].x, a_hi[u].x, a_lo[u].y, a_hi[u].y}, a1[4] = {a_lo[u].z, a_hi[u].z, a_lo[u].w, a_hi[u].w};
            mma_bf16(acc, a0, b.x, b.y);
            mma_bf16(acc, a1, b.z, b.w);
        }
    }
    // accumulator: features o0 + r and o0 + r + 8, rows 2 c and 2 c + 1
#pragma unroll
    for (int e = 0; e < 4; e++) {
        const int t = t0 + 2 * c + (e & 1), o = o0 + r + 8 * (e >> 1);
        if (t >= l.n_rows || o >= l.outs) continue;
        float v = acc[e];
        if (p.gate) v *= 1.0f / (1.0f + expf(-to_float(((const __nv_bfloat16 *)p.gate)[(long long)t * p.ldg + h])));
        l.out[(long long)t * l.ldo + (long long)h * l.outs + o] = __float2bfloat16_rn(v);
    }
}

// The weighted values of a row's parts over the sum of their sums (and the sink's), all against the largest maximum: columns
// tid and tid + AS_THREADS of one head. A lane has a part's weight; all parts' loads of a round are in flight together.
#define AF_PARTS 8
__device__ __forceinline__ void fold_parts(const float *src, int n, int vd, float sink, bool has_sink, float &a, float &b) {
    const int tid = threadIdx.x, lane = tid & 31;
    float top = sink, sum = 0.0f;
    a = b = 0.0f;
    if (n > 32) {  // (up to 32 parts a lane's own maximum is the one it has below)
        for (int k = lane; k < n; k += 32) top = fmaxf(top, src[(long long)k * (vd + 2) + vd]);
        top = warp_max(top);
    }
    for (int k0 = 0; k0 < n; k0 += 32) {
        const int left = min(32, n - k0);
        const float *own = src + (long long)(k0 + lane) * (vd + 2) + vd;
        const float m = lane < left ? own[0] : -INFINITY, l = lane < left ? own[1] : 0.0f;
        if (n <= 32) top = warp_max(fmaxf(top, m));
        const float w = expf(m - top);  // (0 in lanes without a part)
        sum = fmaf(l, w, sum);
        for (int k = 0; k < left; k += AF_PARTS) {
            float x[AF_PARTS], y[AF_PARTS];
#pragma unroll
            for (int i = 0; i < AF_PARTS; i++) {
                const float *part = src + (long long)(k0 + k + i) * (vd + 2);
                x[i] = k + i < left && tid < vd ? part[tid] : 0.0f;
                y[i] = k + i < left && tid + AS_THREADS < vd ? part[tid + AS_THREADS] : 0.0f;
            }
#pragma unroll
            for (int i = 0; i < AF_PARTS; i++) {
                const float wk = __shfl_sync(0xffffffffu, w, (k + i) & 31);
                a = fmaf(x[i], wk, a), b = fmaf(y[i], wk, b);
            }
        }
    }
    sum = warp_sum(sum) + (has_sink ? expf(sink - top) : 0.0f);
    a /= sum, b /= sum;
}

// One CTA per (token, head); with two maps a head, per head: out[t, h] of the maps 2 h and 2 h + 1.
template <typename T, int MAPS> __global__ void __launch_bounds__(AS_THREADS) attention_fold_kernel(AttnSplit p) {
    __shared__ float scratch[33];
    const int t = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, vd = p.v_dim, heads = p.n_heads / MAPS;
    float sink[MAPS];
#pragma unroll
    for (int m = 0; m < MAPS; m++) sink[m] = p.sink ? p.sink[MAPS * h + m] : -INFINITY;  // weights: ahead of the wait
    const int seq = p.token_seq[t], pos = p.token_pos[t];
    pdl_wait();
    T *out = (T *)p.out + ((long long)t * heads + h) * vd;
    if (seq < 0) {
        for (int d = tid; d < vd; d += AS_THREADS) out[d] = from_float<T>(0.0f);
        return;
    }
    int lo, kept, total;
    visible_keys(p, pos, lo, kept, total);
    const int n = (total + p.part_keys - 1) / p.part_keys;
    float a[MAPS], b[MAPS];
#pragma unroll
    for (int m = 0; m < MAPS; m++)
        fold_parts(p.parts + ((long long)t * p.n_heads + MAPS * h + m) * p.n_parts * (vd + 2), n, vd, sink[m], p.sink != nullptr, a[m], b[m]);
    if (MAPS == 2) {
        a[0] = differential_value(p.diff, a[0], a[MAPS - 1]), b[0] = differential_value(p.diff, b[0], b[MAPS - 1]);  // (0 beyond vd)
        const float scale = differential_scale(p.diff, block_sum(fmaf(a[0], a[0], b[0] * b[0]), scratch), vd);
        a[0] *= scale, b[0] *= scale;
    }
    const float g = p.gate ? 1.0f / (1.0f + expf(-to_float(((const T *)p.gate)[(long long)t * p.ldg + h]))) : 1.0f;
    if (tid < vd) out[tid] = from_float<T>(a[0] * g);
    if (tid + AS_THREADS < vd) out[tid + AS_THREADS] = from_float<T>(b[0] * g);
}

// max_keys: an upper bound of the keys any row of the step sees (its position + 1, or window + keep_first);
// parts: float32 scratch of at least tokens * heads * ceil(max_keys / 64) * (v_dim + 2). to (null: none): the fold carries the
// heads' results out of the latent space.
static int attention_split(const LatentOut *to, const DifferentialHead *diff, int values_in_keys, int chunk, float softcap, const void *q, long long q_row, void *out, int dtype, int n_tokens, int n_heads,
                                   int n_kv_heads, int head_dim, int v_dim, float scale, int window, int keep_first,
                                   const float *sink, const int *token_seq, const int *token_pos, const int *seq_slot,
                                   const void *k_pool, const void *v_pool, const int *page_table, int table_width,
                                   int ring_pages, int pinned_pages, int tokens_per_page, int max_keys, float *parts,
                                   long long parts_floats, const void *gate, long long ldg, void *stream) {
    if (n_tokens <= 0) return 0;
    const int maps = diff ? 2 : 1;
    if (maps * head_dim > 2 * AS_MAX_DIM || head_dim > AS_MAX_DIM || head_dim % 8 || head_dim < 8) ABK_REFUSE("attention_split: head_dim %d is not a multiple of 8 up to %d", head_dim, AS_MAX_DIM);
    if (v_dim < 1 || v_dim > AS_MAX_DIM) ABK_REFUSE("attention_split: value size %d is not 1 to %d", v_dim, AS_MAX_DIM);
    int runs = 1;
    if (n_kv_heads >= 1 && n_heads % n_kv_heads == 0 && n_heads / n_kv_heads > AS_MAX_GROUP) {
        // more query heads to a kv head than a CTA takes: they go in runs of the largest divisor up to 16 (of whole heads,
        // where a head has two maps), each run a CTA of its own over the same cache rows
        const int group = n_heads / n_kv_heads;
        int run = AS_MAX_GROUP;
        while (run > 1 && (group % run || run % maps)) run--;
        if (run % maps == 0) runs = group / run, n_kv_heads *= runs;
    }
    if (n_kv_heads < 1 || n_heads % n_kv_heads || n_heads / n_kv_heads > AS_MAX_GROUP)
        ABK_REFUSE("attention_split: %d query heads to %d kv heads (groups of up to %d)", n_heads, n_kv_heads, AS_MAX_GROUP);
    if (maps == 2 && (n_heads / n_kv_heads % 2 || values_in_keys || gate))
        ABK_REFUSE("attention_split: the two maps of a head go with values of their own and no gate");
    if (n_heads > 65535 || n_kv_heads > 65535 || max_keys < 1) ABK_REFUSE("attention_split: %d heads, %d keys", n_heads, max_keys);
    AttnSplit p;
    p.q = q, p.q_row = q_row, p.parts = parts, p.out = out, p.n_heads = n_heads, p.n_kv_heads = n_kv_heads;
    p.head_dim = head_dim, p.v_dim = v_dim, p.scale = scale, p.window = window > 0 ? window : 0;
    p.keep_first = window > 0 && keep_first > 0 ? keep_first : 0, p.sink = sink;
    p.chunk = chunk > 0 ? chunk : 0, p.softcap = softcap > 0.0f ? softcap : 0.0f;
    p.token_seq = token_seq, p.token_pos = token_pos, p.seq_slot = seq_slot, p.k_pool = k_pool, p.v_pool = v_pool;
    p.cache.page_table = page_table, p.cache.table_width = table_width, p.cache.ring_pages = ring_pages;
    p.cache.tokens_per_page = tokens_per_page, p.cache.pinned_pages = pinned_pages;
    p.v_cache = p.cache;
    // (with values of their own and few heads to a kv head the other kernel's smaller CTAs do as well or better: 64 rows of 2,176
    // keys, groups of two, 195 us against 257)
    const bool tensor = dtype == ABK_BF16 && (values_in_keys || maps == 2 || n_heads / n_kv_heads >= 8) && maps * head_dim % 16 == 0 && v_dim % 8 == 0 && q_row % 8 == 0 &&
                        !(((uintptr_t)k_pool | (uintptr_t)v_pool | (uintptr_t)q) & 15);
    if (to && (!tensor || ((uintptr_t)to->w & 15))) ABK_REFUSE("attention_split: latents of %d in rows of %d are not what the fused fold takes", v_dim, head_dim);
    // parts of 64 keys where values have rows of their own (more CTAs to an SM: 64 rows of 2,176 keys, two maps a head, 212 us against
    // 270), and over latent rows where parts of 128 would not fill the GPU
    p.part_keys = tensor && (!values_in_keys || (long long)n_tokens * n_kv_heads * ((max_keys + 127) / 128) < 2 * abk_sm_count()) ? 64 : 128;
    p.n_parts = (max_keys + p.part_keys - 1) / p.part_keys;
    p.values_in_keys = values_in_keys, p.runs = runs, p.gate = gate, p.ldg = ldg;
    p.maps = maps, p.diff = diff ? *diff : DifferentialHead();
    if (values_in_keys && v_dim > head_dim) ABK_REFUSE("attention_split: values of %d inside keys of %d", v_dim, head_dim);
    if (p.n_parts > 65535) ABK_REFUSE("attention_split: %d keys are more than a grid takes", max_keys);
    if ((long long)n_tokens * n_heads * p.n_parts * (v_dim + 2) > parts_floats)
        ABK_REFUSE("attention_split: the scratch memory holds %lld floats, the step needs %lld", parts_floats,
                   (long long)n_tokens * n_heads * p.n_parts * (v_dim + 2));
    const int group = n_heads / n_kv_heads;
    const bool bf = dtype == ABK_BF16;
    const int esize = bf ? 2 : 4;
    const size_t small = (size_t)(group * head_dim + group * AS_THREADS + ((4 * group + 3) & ~3)) * 4;
    size_t rows = (size_t)AS_THREADS * (maps * head_dim * esize + 16);  // the keys' rows, then the values' in the same place
    if (!values_in_keys && rows < (size_t)AS_THREADS * v_dim * esize) rows = (size_t)AS_THREADS * v_dim * esize;
    const size_t staged = small + rows;
    // rows of keys and of values that are whole 16-byte pieces at 16-byte places can be staged in shared memory
    const bool stage = (head_dim * esize) % 16 == 0 && (values_in_keys || (v_dim * esize) % 16 == 0) && staged <= 100 * 1024 &&
                       !(((uintptr_t)k_pool | (uintptr_t)v_pool) & 15);
    const size_t smem = stage ? staged : small;
    cudaStream_t s = (cudaStream_t)stream;
    dim3 grid(n_tokens, n_kv_heads, p.n_parts), fold(n_tokens, n_heads / maps);
#define SPLIT_LAUNCH(T, STAGED, GMAX, ...)                                                                \
    do {                                                                                                  \
        if (smem + 4096 > 48 * 1024) { /* (the kernel's own 2 KB of static shared memory count too) */    \
            cudaError_t e = abk_allow_shared_memory((const void *)attention_split_kernel<T, STAGED, GMAX, ##__VA_ARGS__>, (int)smem); \
            if (e != cudaSuccess) return (int)e;                                                          \
        }                                                                                                 \
        abk_launch(attention_split_kernel<T, STAGED, GMAX, ##__VA_ARGS__>, grid, dim3(AS_THREADS), smem, s, p);         \
    } while (0)
#define SPLIT_BY_GROUP(T, STAGED)                   \
    do {                                            \
        if (group <= 1) SPLIT_LAUNCH(T, STAGED, 1); \
        else if (group <= 2) SPLIT_LAUNCH(T, STAGED, 2); \
        else if (group <= 4) SPLIT_LAUNCH(T, STAGED, 4); \
        else if (group <= 8) SPLIT_LAUNCH(T, STAGED, 8); \
        else SPLIT_LAUNCH(T, STAGED, 16);           \
    } while (0)
    if (tensor) {
        const int v_pitch = values_in_keys ? 0 : ((v_dim + 15) & ~15) * 2 + 16;
        const size_t bytes = (16 * (p.part_keys + 8) + 128) * 4 + (size_t)(16 + p.part_keys) * (maps * head_dim * 2 + 16) + (size_t)p.part_keys * v_pitch;
#define TILES_LAUNCH(PART, OWN_V)                                                                                             \
    do {                                                                                                                      \
        if (bytes + 4096 > 48 * 1024) {                                                                                       \
            cudaError_t e = abk_allow_shared_memory((const void *)attention_split_tiles_kernel<PART, OWN_V>, (int)bytes);     \
            if (e != cudaSuccess) return (int)e;                                                                              \
        }                                                                                                                     \
        abk_launch(attention_split_tiles_kernel<PART, OWN_V>, grid, dim3(AS_THREADS), bytes, s, p);                           \
    } while (0)
        if (!values_in_keys) TILES_LAUNCH(64, true);
        else if (p.part_keys == 64) TILES_LAUNCH(64, false);
        else TILES_LAUNCH(128, false);
#undef TILES_LAUNCH
        if (to) {
            LatentOut l = *to;
            l.n_rows = n_tokens;
            const size_t mixed = (size_t)AL_ROWS * ((v_dim + 31) / 32 * 32 + 8) * 2;
            int rc = ABK_LAUNCH_RESULT();
            if (rc) return rc;
            abk_launch(latent_fold_out_kernel, dim3(n_heads * ((l.outs + AL_OUTS - 1) / AL_OUTS), (n_tokens + AL_ROWS - 1) / AL_ROWS),
                       dim3(AL_THREADS), mixed, s, p, l);
            return ABK_LAUNCH_RESULT();
        }
    } else if (bf && stage) SPLIT_BY_GROUP(__nv_bfloat16, true);
    else if (bf) SPLIT_BY_GROUP(__nv_bfloat16, false);
    else if (stage) SPLIT_BY_GROUP(float, true);
    else SPLIT_BY_GROUP(float, false);
#undef SPLIT_BY_GROUP
#undef SPLIT_LAUNCH
    int rc = ABK_LAUNCH_RESULT();
    if (rc) return rc;
    if (maps == 2) {
        if (bf) abk_launch(attention_fold_kernel<__nv_bfloat16, 2>, fold, dim3(AS_THREADS), 0, s, p);
        else abk_launch(attention_fold_kernel<float, 2>, fold, dim3(AS_THREADS), 0, s, p);
    } else {
        if (bf) abk_launch(attention_fold_kernel<__nv_bfloat16, 1>, fold, dim3(AS_THREADS), 0, s, p);
        else abk_launch(attention_fold_kernel<float, 1>, fold, dim3(AS_THREADS), 0, s, p);
    }
    return ABK_LAUNCH_RESULT();
}

extern "C" int abk_attention_split(const void *q, long long q_row, void *out, int dtype, int n_tokens, int n_heads,
                                   int n_kv_heads, int head_dim, int v_dim, float scale, int window, int keep_first,
                                   const float *sink, const int *token_seq, const int *token_pos, const int *seq_slot,
                                   const void *k_pool, const void *v_pool, const int *page_table, int table_width,
                                   int ring_pages, int pinned_pages, int tokens_per_page, int max_keys, float *parts,
                                   long long parts_floats, int chunk, float softcap, const void *gate, long long ldg,
                                   void *stream) {
    return attention_split(nullptr, nullptr, 0, chunk, softcap, q, q_row, out, dtype, n_tokens, n_heads, n_kv_heads, head_dim, v_dim, scale, window, keep_first,
                           sink, token_seq, token_pos, seq_slot, k_pool, v_pool, page_table, table_width, ring_pages,
                           pinned_pages, tokens_per_page, max_keys, parts, parts_floats, gate, ldg, stream);
}

// The two maps of differential attention: n_heads counts every map of every head, a key row holds 2 * head_dim elements;
// out [tokens, n_heads / 2 * v_dim] = keep * o / sqrt(mean(o^2) + eps), o = a1 - lambda * a2.
extern "C" int abk_attention_split_maps(const void *q, long long q_row, void *out, int dtype, int n_tokens, int n_heads,
                                        int n_kv_heads, int head_dim, int v_dim, float scale, int window, int keep_first,
                                        const float *sink, const int *token_seq, const int *token_pos, const int *seq_slot,
                                        const void *k_pool, const void *v_pool, const int *page_table, int table_width,
                                        int ring_pages, int pinned_pages, int tokens_per_page, int max_keys, float *parts,
                                        long long parts_floats, int chunk, float softcap, float lambda, float eps, float keep,
                                        void *stream) {
    const DifferentialHead diff = {lambda, eps, keep};
    return attention_split(nullptr, &diff, 0, chunk, softcap, q, q_row, out, dtype, n_tokens, n_heads, n_kv_heads, head_dim, v_dim, scale, window,
                           keep_first, sink, token_seq, token_pos, seq_slot, k_pool, v_pool, page_table, table_width, ring_pages,
                           pinned_pages, tokens_per_page, max_keys, parts, parts_floats, nullptr, 0, stream);
}

// Keys that carry their values (a value is the first v_dim elements of its key row; one pool): attention over shared
// latent rows (csrc/latent.cu), every query head in the one group.
// w (null: none; bfloat16 [heads][outs][v_dim]): out is then [tokens][ldo], head h's `outs` results at h * outs, the weighted
// latents times w (times sigmoid(gate) with a gate per token and head); else out is [tokens][n_heads * v_dim], the weighted
// latents themselves.
extern "C" int abk_attention_split_values_in_keys(const void *q, long long q_row, void *out, int dtype, int n_tokens,
                                                  int n_heads, int n_kv_heads, int head_dim, int v_dim, float scale,
                                                  const float *sink, const int *token_seq, const int *token_pos,
                                                  const int *seq_slot, const void *k_pool, const int *page_table,
                                                  int table_width, int ring_pages, int tokens_per_page, int window, int max_keys,
                                                  float *parts, long long parts_floats, const void *w, int outs, long long ldo,
                                                  const void *gate, long long ldg, void *stream) {
    LatentOut to;
    to.w = (const __nv_bfloat16 *)w, to.out = (__nv_bfloat16 *)out, to.ldo = ldo, to.outs = outs, to.n_rows = 0;
    return attention_split(w ? &to : nullptr, nullptr, 1, 0, 0.0f, q, q_row, out, dtype, n_tokens, n_heads, n_kv_heads, head_dim, v_dim,
                           scale, window, 0, sink, token_seq, token_pos, seq_slot, k_pool, k_pool, page_table, table_width, ring_pages,
                           0, tokens_per_page, max_keys, parts, parts_floats, gate, ldg, stream);
}
