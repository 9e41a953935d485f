// Causal attention without a softmax: the weight of a key a token sees is the sigmoid of its score, each key for itself,
// and the heads' weights are mixed before they meet the values. For query head h (kv head h / (H / G)), token i, key j <= i:
//
//   z_h  = scale * (q_hi . k_j);   with a cap c: z_h <- c tanh(z_h / c);   z_h <- z_h - slope_h (i - j) + shift_h
//   a_h  = 1 / (1 + e^-z_h);       m_h = sum_g mix[h, g] a_g  (no mix: m_h = a_h);       out_hi = sum_j m_h(i, j) v_j
//
// Scores, weights (mixed or not) and sums are float32. Since nothing is normalized over the keys, what runs of keys
// contribute to a token simply adds up: there is no maximum to agree on.
//
//   general   any sizes, either type, keys and values from the paged cache: a CTA a token (and a run of output columns).
//             The float32 path, portions of prompts, and every size the other two refuse.
#define ABK_DEFINE_ERROR
#include "common.cuh"

struct AttnSigmoid {
    const void *q;       // row t, head h at q + t * q_row + h * head_dim
    long long q_row;
    void *out;           // [tokens, n_heads * v_dim]
    int n_heads, n_kv_heads, head_dim, v_dim;
    float scale, softcap;       // softcap 0: scores are not capped
    const float *slopes;        // [n_heads] or null
    const float *shift;         // [n_heads] or null
    const float *mix;           // [n_heads, n_heads] (out, in) or null
    const int *token_seq, *token_pos, *seq_slot;
    const void *k_pool, *v_pool;
    PagedCache cache;
    int vector_rows;     // key rows are whole 16-byte pieces at 16-byte places
};

// The weight of a raw score (the product q . k) at a distance, in float32 with the exact functions.
__device__ __forceinline__ float sigmoid_weight(float dot, float scale, float cap, float slope, float back, float shift) {
    float z = dot * scale;
    if (cap > 0.0f) z = cap * tanhf(z / cap);
    z = fmaf(-slope, back, z) + shift;
    return 1.0f / (1.0f + expf(-z));
}

// ---------------------------------------------------------------- general
#define SG_THREADS 256
#define SG_KEYS 32
#define SG_COLS 8  // output columns a thread sums

template <typename T> __device__ __forceinline__ float sg_dot(const float *q, const T *k, int hd, bool vec);
template <> __device__ __forceinline__ float sg_dot<float>(const float *q, const float *k, int hd, bool vec) {
    float acc = 0.0f;
    if (vec) {
        for (int i = 0; i < hd; i += 4) {
            const float4 v = *(const float4 *)(k + i);
            acc = fmaf(q[i], v.x, acc), acc = fmaf(q[i + 1], v.y, acc), acc = fmaf(q[i + 2], v.z, acc), acc = fmaf(q[i + 3], v.w, acc);
        }
    } else {
        for (int i = 0; i < hd; i++) acc = fmaf(q[i], k[i], acc);
    }
    return acc;
}
template <> __device__ __forceinline__ float sg_dot<__nv_bfloat16>(const float *q, const __nv_bfloat16 *k, int hd, bool vec) {
    float acc = 0.0f;
    if (vec) {
        for (int i = 0; i < hd; i += 8) {
            const uint4 raw = *(const uint4 *)(k + i);
            const __nv_bfloat162 *h = (const __nv_bfloat162 *)&raw;
#pragma unroll
            for (int u = 0; u < 4; u++) {
                const float2 f = __bfloat1622float2(h[u]);
                acc = fmaf(q[i + 2 * u], f.x, acc), acc = fmaf(q[i + 2 * u + 1], f.y, acc);
            }
        }
    } else {
        for (int i = 0; i < hd; i++) acc = fmaf(q[i], __bfloat162float(k[i]), acc);
    }
    return acc;
}

template <typename T> __global__ void __launch_bounds__(SG_THREADS) attention_sigmoid_kernel(AttnSigmoid p) {
    extern __shared__ __align__(16) float sg_smem[];
    const int H = p.n_heads, G = p.n_kv_heads, D = p.head_dim, VD = p.v_dim, R = H / G;
    float *q_s = sg_smem;                 // [H][D]
    float *a_s = q_s + ((H * D + 3) & ~3);  // [H][SG_KEYS]: the weights
    float *m_s = a_s + H * SG_KEYS;       // [H][SG_KEYS]: mixed
    __shared__ int page_s[SG_KEYS];
    const int t = blockIdx.x, tid = threadIdx.x;
    const int col0 = blockIdx.y * SG_THREADS * SG_COLS, cols = min(SG_THREADS * SG_COLS, H * VD - col0);
    pdl_wait();
    const int seq = p.token_seq[t];
    T *out = (T *)p.out + (long long)t * H * VD + col0;
    if (seq < 0) {  // padding
        for (int c = tid; c < cols; c += SG_THREADS) out[c] = from_float<T>(0.0f);
        return;
    }
    const int pos = p.token_pos[t], slot = p.seq_slot[seq];
    const T *q = (const T *)p.q + (long long)t * p.q_row;
    for (int e = tid; e < H * D; e += SG_THREADS) q_s[e] = to_float(q[e]);
    const int h_lo = col0 / VD, h_hi = (col0 + cols - 1) / VD;  // the heads of this CTA's columns
    float acc[SG_COLS];
    int kv[SG_COLS], hd_of[SG_COLS], at[SG_COLS];
#pragma unroll
    for (int u = 0; u < SG_COLS; u++) {
        const int c = min(tid + u * SG_THREADS, cols - 1) + col0;
        acc[u] = 0.0f, hd_of[u] = c / VD, kv[u] = hd_of[u] / R, at[u] = c % VD;
    }
    const long long v_page = (long long)p.cache.tokens_per_page * VD;
    for (int base = 0; base <= pos; base += SG_KEYS) {
        const int n = min(SG_KEYS, pos + 1 - base);
        __syncthreads();  // q is there; the tile before is done with
        if (tid < n) page_s[tid] = cache_page(p.cache, slot, base + tid);
        __syncthreads();
        for (int e = tid; e < H * SG_KEYS; e += SG_THREADS) {
            const int h = e / SG_KEYS, j = e % SG_KEYS;
            float a = 0.0f;
            if (j < n) {
                const T *k = (const T *)p.k_pool + cache_offset(p.cache, page_s[j], h / R, G, base + j, D);
                a = sigmoid_weight(sg_dot<T>(q_s + h * D, k, D, p.vector_rows), p.scale, p.softcap, p.slopes ? p.slopes[h] : 0.0f,
                                   (float)(pos - base - j), p.shift ? p.shift[h] : 0.0f);
            }
            a_s[e] = a;
        }
        __syncthreads();
        const float *w_s = a_s;
        if (p.mix) {
            for (int e = tid; e < (h_hi - h_lo + 1) * SG_KEYS; e += SG_THREADS) {
                const int h = h_lo + e / SG_KEYS, j = e % SG_KEYS;
                float m = 0.0f;
                for (int g = 0; g < H; g++) m = fmaf(p.mix[(long long)h * H + g], a_s[g * SG_KEYS + j], m);
                m_s[h * SG_KEYS + j] = m;
            }
            __syncthreads();
            w_s = m_s;
        }
        for (int j = 0; j < n; j++) {
            const T *v = (const T *)p.v_pool + (long long)page_s[j] * G * v_page + (long long)((base + j) % p.cache.tokens_per_page) * VD;
#pragma unroll
            for (int u = 0; u < SG_COLS; u++)
                if (u * SG_THREADS < cols) acc[u] = fmaf(w_s[hd_of[u] * SG_KEYS + j], to_float(v[kv[u] * v_page + at[u]]), acc[u]);
        }
    }
#pragma unroll
    for (int u = 0; u < SG_COLS; u++)
        if (tid + u * SG_THREADS < cols) out[tid + u * SG_THREADS] = from_float<T>(acc[u]);
}

static int sigmoid_params(AttnSigmoid &p, const void *q, long long q_row, void *out, int n_heads, int n_kv_heads, int head_dim,
                          int v_dim, float scale, float softcap, const float *slopes, const float *shift, const float *mix,
                          const int *token_seq, const int *token_pos, const int *seq_slot, const void *k_pool, const void *v_pool,
                          const int *page_table, int table_width, int tokens_per_page) {
    if (n_kv_heads < 1 || n_heads < 1 || n_heads % n_kv_heads)
        ABK_REFUSE("attention_sigmoid: %d query heads do not divide into %d kv heads", n_heads, n_kv_heads);
    if (head_dim < 1 || v_dim < 1 || softcap < 0.0f) ABK_REFUSE("attention_sigmoid: heads of %d, values of %d, a cap of %g", head_dim, v_dim, softcap);
    p.q = q, p.q_row = q_row, p.out = out, p.n_heads = n_heads, p.n_kv_heads = n_kv_heads, p.head_dim = head_dim, p.v_dim = v_dim;
    p.scale = scale, p.softcap = softcap, p.slopes = slopes, p.shift = shift, p.mix = mix;
    p.token_seq = token_seq, p.token_pos = token_pos, p.seq_slot = seq_slot, p.k_pool = k_pool, p.v_pool = v_pool;
    p.cache.page_table = page_table, p.cache.table_width = table_width, p.cache.ring_pages = 0;
    p.cache.tokens_per_page = tokens_per_page, p.cache.pinned_pages = 0;
    p.vector_rows = 0;
    return 0;
}

extern "C" int abk_attention_sigmoid(const void *q, long long q_row, void *out, int dtype, int n_tokens, int n_heads, int n_kv_heads,
                                     int head_dim, int v_dim, float scale, float softcap, const float *slopes, const float *shift,
                                     const float *mix, const int *token_seq, const int *token_pos, const int *seq_slot,
                                     const void *k_pool, const void *v_pool, const int *page_table, int table_width,
                                     int tokens_per_page, void *stream) {
    if (n_tokens <= 0) return 0;
    AttnSigmoid p;
    const int rc = sigmoid_params(p, q, q_row, out, n_heads, n_kv_heads, head_dim, v_dim, scale, softcap, slopes, shift, mix, token_seq,
                                  token_pos, seq_slot, k_pool, v_pool, page_table, table_width, tokens_per_page);
    if (rc) return rc;
    p.vector_rows = head_dim * (dtype == ABK_BF16 ? 2 : 4) % 16 == 0 && !((uintptr_t)k_pool & 15);
    const long long floats = ((long long)n_heads * head_dim + 3) / 4 * 4 + 2LL * n_heads * SG_KEYS;
    if (floats * 4 > 200 * 1024) ABK_REFUSE("attention_sigmoid: %d heads of %d are more than a CTA holds", n_heads, head_dim);
    const int smem = (int)floats * 4;
    const long long runs = ((long long)n_heads * v_dim + SG_THREADS * SG_COLS - 1) / (SG_THREADS * SG_COLS);
    if (runs > 65535) ABK_REFUSE("attention_sigmoid: %d heads of %d values are more than a grid takes", n_heads, v_dim);
    const void *kernel = dtype == ABK_BF16 ? (const void *)attention_sigmoid_kernel<__nv_bfloat16> : (const void *)attention_sigmoid_kernel<float>;
    if (smem > 40 * 1024) {
        cudaError_t e = abk_allow_shared_memory(kernel, smem);
        if (e != cudaSuccess) return (int)e;
    }
    const dim3 grid(n_tokens, (unsigned)runs);
    if (dtype == ABK_BF16)
        abk_launch(attention_sigmoid_kernel<__nv_bfloat16>, grid, dim3(SG_THREADS), (size_t)smem, (cudaStream_t)stream, p);
    else
        abk_launch(attention_sigmoid_kernel<float>, grid, dim3(SG_THREADS), (size_t)smem, (cudaStream_t)stream, p);
    return ABK_LAUNCH_RESULT();
}
