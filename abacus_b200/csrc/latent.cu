// Latent attention: what stands around the attention kernels when keys and values are kept as one low-rank
// latent row per token that all heads share.
//
// A token's cache row is [c | r | 0...]: c (rank elements) is the normed down-projection, r (rot elements) one
// rotated key part shared by the heads, zeros up to the row's padded size. Head h's key is [U_h c | r] and its value
// V_h c. The scores need no key of full size: (U_h c) . q = c . (U_h^T q), so a query head is carried into the
// latent space once, [U_h^T q_plain | q_rotated], and attention runs over the cache rows themselves with one kv
// head whose values are the first `rank` elements of its keys; V_h is applied to the weighted sum of latents.
//
//   latent_prep   per token: c = w * x / sqrt(mean(x^2) + eps) over the first `rank` columns of the down-projection,
//                 the rotation of the shared key part and of every query head's rotated part (pairs (2i, 2i+1) or (i, i + rot_dims / 2),
//                 angle table [position][rot_dims / 2]; elements beyond rot_dims pass unchanged), the cache write (a
//                 windowed layer's ring of pages: only what is still there after the step), the same row among the step's
//                 own where a prompt's attention reads it from there, and the query parts put where the attention
//                 kernel wants them.
//   latent_prep_product  both for a step of a few rows in bfloat16: latent_prep with the plain query parts carried into the
//                 latent space by the same launch.
//   head_product  out[t, h, :] = W[h] x[t, h, :] for every head: a product per head with a matrix of its own
//                 (U_h^T on the plain query part, V_h on the weighted latents), float32 sums in a fixed order.
//   latent_rows   the cache rows of the step's own tokens, gathered into consecutive rows (for a prompt whose keys
//                 and values are made in full size from another entry's latents).
//   spread_shared a step's shared rotated key part copied behind every head's plain key part.
#define ABK_DEFINE_ERROR
#include "common.cuh"
#include "mma_tiles.cuh"

struct LatentPrep {
    const void *proj;    // row t at proj + t * ldp: query heads [heads][dim + rot] from column 0, the down-projection
    long long ldp;       // [rank + rot] from column down_at
    int down_at;
    int n_heads, dim, rot, rank, rot_dims;
    int interleaved;     // pairs (2i, 2i+1) of the rotated dimensions; 0: pairs (i, i + rot_dims / 2)
    const float *norm_w;  // [rank]
    float eps;
    const float *cos, *sin;  // [positions][rot_dims / 2]
    void *q_dst;          // head h of row t at q_dst + t * ldq + h * q_head: its rotated part goes to + q_rot_at,
    long long ldq;        // its plain part (copy_plain) to + 0; what lies beyond q_rot_at + rot in a head is zeroed
    int q_head, q_rot_at, copy_plain;
    void *pool;           // cache rows [pages][1][tokens_per_page][row]; null: nothing is written (another entry's cache)
    int row;
    PagedCache cache;
    void *rows;           // the step's own rows [tokens][ld_rows], the same contents; null: not wanted
    long long ld_rows;
    const int *token_seq, *token_pos, *seq_slot, *seq_len_after;
};

// The latent row of token t, [c | r | zeros], to its place in the cache and among the step's rows. Whole CTAs of 128 threads.
template <typename T> __device__ __forceinline__ void latent_row(const LatentPrep &p, int t, int seq, int pos, float *scratch) {
    const int tid = threadIdx.x, half = p.rot_dims / 2;
    const T *src = (const T *)p.proj + (long long)t * p.ldp;
    const float *cs = p.cos + (long long)pos * half, *sn = p.sin + (long long)pos * half;
    const T *down = src + p.down_at;
    float ss = 0.0f;
    for (int i = tid; i < p.rank; i += 128) {
        const float v = to_float(down[i]);
        ss = fmaf(v, v, ss);
    }
    ss = block_sum(ss, scratch);
    const float inv = 1.0f / sqrtf(ss / (float)p.rank + p.eps);
    T *kept = nullptr, *own = p.rows ? (T *)p.rows + (long long)t * p.ld_rows : nullptr;
    if (p.pool && cache_keeps(p.cache, pos, p.seq_len_after[seq]))
        kept = (T *)p.pool + cache_offset(p.cache, cache_page(p.cache, p.seq_slot[seq], pos), 0, 1, pos, p.row);
    auto put = [&](int i, T v) {
        if (kept) kept[i] = v;
        if (own) own[i] = v;
    };
    for (int i = tid; i < p.rank; i += 128) put(i, from_float<T>(to_float(down[i]) * inv * p.norm_w[i]));
    for (int i = tid; i < half; i += 128) {
        const int ia = p.interleaved ? 2 * i : i, ib = p.interleaved ? 2 * i + 1 : i + half;
        const float u = to_float(down[p.rank + ia]), v = to_float(down[p.rank + ib]);
        put(p.rank + ia, from_float<T>(u * cs[i] - v * sn[i]));
        put(p.rank + ib, from_float<T>(v * cs[i] + u * sn[i]));
    }
    for (int i = p.rot_dims + tid; i < p.rot; i += 128) put(p.rank + i, down[p.rank + i]);
    for (int i = p.rank + p.rot + tid; i < p.row; i += 128) put(i, from_float<T>(0.0f));
}

template <typename T> __global__ void __launch_bounds__(128) latent_prep_kernel(LatentPrep p) {
    __shared__ float scratch[33];
    const int t = blockIdx.x, tid = threadIdx.x;
    pdl_wait();
    const int seq = p.token_seq[t];
    if (seq < 0) {
        if (p.rows)
            for (int i = tid; i < p.row; i += 128) ((T *)p.rows)[(long long)t * p.ld_rows + i] = from_float<T>(0.0f);
        return;
    }
    const int pos = p.token_pos[t], half = p.rot_dims / 2;
    const T *src = (const T *)p.proj + (long long)t * p.ldp;
    const float *cs = p.cos + (long long)pos * half, *sn = p.sin + (long long)pos * half;
    if (p.pool || p.rows) latent_row<T>(p, t, seq, pos, scratch);
    T *q_out = (T *)p.q_dst + (long long)t * p.ldq;
    const int per_head = p.dim + p.rot;
    for (int e = tid; e < p.n_heads * half; e += 128) {
        const int h = e / half, i = e - h * half;
        const T *q = src + (long long)h * per_head + p.dim;
        const int ia = p.interleaved ? 2 * i : i, ib = p.interleaved ? 2 * i + 1 : i + half;
        const float u = to_float(q[ia]), v = to_float(q[ib]);
        T *d = q_out + (long long)h * p.q_head + p.q_rot_at;
        d[ia] = from_float<T>(u * cs[i] - v * sn[i]);
        d[ib] = from_float<T>(v * cs[i] + u * sn[i]);
    }
    const int rest = p.rot - p.rot_dims, tail = p.q_head - p.q_rot_at - p.rot;
    for (int e = tid; e < p.n_heads * rest; e += 128) {
        const int h = e / rest, i = p.rot_dims + e % rest;
        q_out[(long long)h * p.q_head + p.q_rot_at + i] = src[(long long)h * per_head + p.dim + i];
    }
    for (int e = tid; e < p.n_heads * tail; e += 128) {
        const int h = e / tail, i = p.q_rot_at + p.rot + e % tail;
        q_out[(long long)h * p.q_head + i] = from_float<T>(0.0f);
    }
    if (p.copy_plain)
        for (int e = tid; e < p.n_heads * p.dim; e += 128) {
            const int h = e / p.dim, i = e - h * p.dim;
            q_out[(long long)h * p.q_head + i] = src[(long long)h * per_head + i];
        }
}

// ---------------------------------------------------------------- the same in 16-byte pieces
// bfloat16 with every size a multiple of 8 and rows 16-byte aligned; the rotation over whole pieces (in halves: of a multiple
// of 16 elements). A CTA a token.
__device__ __forceinline__ uint4 lv_pack(const float *v) {
    uint4 out;
    __nv_bfloat162 *h = (__nv_bfloat162 *)&out;
#pragma unroll
    for (int j = 0; j < 4; j++) h[j] = __floats2bfloat162_rn(v[2 * j], v[2 * j + 1]);
    return out;
}
__device__ __forceinline__ void lv_unpack(const uint4 &raw, float *v) {
    const __nv_bfloat162 *h = (const __nv_bfloat162 *)&raw;
#pragma unroll
    for (int j = 0; j < 4; j++) {
        const float2 f = __bfloat1622float2(h[j]);
        v[2 * j] = f.x, v[2 * j + 1] = f.y;
    }
}
// Elements o .. o + 7 (o a multiple of 8) of the rotated part at src, turned by the position's angles cs, sn.
__device__ __forceinline__ uint4 lv_rotated(const __nv_bfloat16 *src, int o, int rot_dims, int interleaved, const float *cs, const float *sn) {
    const uint4 raw = *(const uint4 *)(src + o);
    if (o >= rot_dims) return raw;
    float v[8], out[8];
    lv_unpack(raw, v);
    if (interleaved) {
        const float4 c = *(const float4 *)(cs + o / 2), s = *(const float4 *)(sn + o / 2);
        const float cc[4] = {c.x, c.y, c.z, c.w}, ss[4] = {s.x, s.y, s.z, s.w};
#pragma unroll
        for (int j = 0; j < 4; j++) {
            out[2 * j] = v[2 * j] * cc[j] - v[2 * j + 1] * ss[j];
            out[2 * j + 1] = v[2 * j + 1] * cc[j] + v[2 * j] * ss[j];
        }
    } else {
        const int half = rot_dims / 2;
        const bool upper = o >= half;
        const int i = upper ? o - half : o;
        float other[8];
        lv_unpack(*(const uint4 *)(src + (upper ? i : o + half)), other);
#pragma unroll
        for (int j = 0; j < 8; j++) out[j] = upper ? v[j] * cs[i + j] + other[j] * sn[i + j] : v[j] * cs[i + j] - other[j] * sn[i + j];
    }
    return lv_pack(out);
}

__global__ void __launch_bounds__(128) latent_prep_vector_kernel(LatentPrep p) {
    __shared__ float scratch[33];
    const int t = blockIdx.x, tid = threadIdx.x;
    const uint4 zero = make_uint4(0, 0, 0, 0);
    const int seq = p.token_seq[t], pos = p.token_pos[t];  // (written by kernels further back than the one just before)
    pdl_wait();
    __nv_bfloat16 *own = p.rows ? (__nv_bfloat16 *)p.rows + (long long)t * p.ld_rows : nullptr;
    if (seq < 0) {
        if (own)
            for (int i = tid * 8; i < p.row; i += 1024) *(uint4 *)(own + i) = zero;
        return;
    }
    const int half = p.rot_dims / 2, per_head = p.dim + p.rot;
    const __nv_bfloat16 *src = (const __nv_bfloat16 *)p.proj + (long long)t * p.ldp;
    const float *cs = p.cos + (long long)pos * half, *sn = p.sin + (long long)pos * half;
    if (p.pool || own) {  // a row has at most 80 pieces, a thread one
        const __nv_bfloat16 *down = src + p.down_at;
        const int o = tid * 8;
        __nv_bfloat16 *kept = nullptr;
        if (p.pool && cache_keeps(p.cache, pos, p.seq_len_after[seq]))
            kept = (__nv_bfloat16 *)p.pool + cache_offset(p.cache, cache_page(p.cache, p.seq_slot[seq], pos), 0, 1, pos, p.row);
        float v[8] = {0.0f, 0.0f, 0.0f, 0.0f, 0.0f, 0.0f, 0.0f, 0.0f}, ss = 0.0f;
        if (o < p.rank) lv_unpack(*(const uint4 *)(down + o), v);
#pragma unroll
        for (int j = 0; j < 8; j++) ss = fmaf(v[j], v[j], ss);
        ss = block_sum(ss, scratch);
        const float inv = 1.0f / sqrtf(ss / (float)p.rank + p.eps);
        uint4 out = zero;
        if (o < p.rank) {
#pragma unroll
            for (int j = 0; j < 8; j++) v[j] = v[j] * inv * p.norm_w[o + j];
            out = lv_pack(v);
        } else if (o < p.rank + p.rot) {
            out = lv_rotated(down + p.rank, o - p.rank, p.rot_dims, p.interleaved, cs, sn);
        }
        if (o < p.row) {
            if (kept) *(uint4 *)(kept + o) = out;
            if (own) *(uint4 *)(own + o) = out;
        }
    }
    __nv_bfloat16 *q_out = (__nv_bfloat16 *)p.q_dst + (long long)t * p.ldq;
    const int skip = p.copy_plain ? 0 : p.dim / 8, pieces = per_head / 8 - skip;  // a head's pieces that are written from the projection
#pragma unroll 4
    for (int e = tid; e < p.n_heads * pieces; e += 128) {
        const int h = e / pieces, o = (e - h * pieces + skip) * 8;
        const __nv_bfloat16 *q = src + (long long)h * per_head;
        __nv_bfloat16 *d = q_out + (long long)h * p.q_head;
        if (o < p.dim) *(uint4 *)(d + o) = *(const uint4 *)(q + o);
        else *(uint4 *)(d + p.q_rot_at + o - p.dim) = lv_rotated(q + p.dim, o - p.dim, p.rot_dims, p.interleaved, cs, sn);
    }
    const int tail = (p.q_head - p.q_rot_at - p.rot) / 8;
    for (int e = tid; e < p.n_heads * tail; e += 128) *(uint4 *)(q_out + (long long)(e / tail) * p.q_head + p.q_rot_at + p.rot + e % tail * 8) = zero;
}

// ---------------------------------------------------------------- the same with the queries' way into the latent space
// A step of a few rows (a decode step) in bfloat16. CTA x of row tile y (8 rows): the first heads * tiles CTAs have 64 latent
// columns of one head: q_dst[t, h, :] = w[h] q_plain[t, h], a warp 16 columns on the warp-level tensor cores (its weights, which
// nobody writes, are asked for before the wait), the head's first CTA its rotated part too; the last 8 CTAs a latent row each.
// dim a multiple of 8, every row of proj and w 16-byte aligned.
#define LP_ROWS 8
#define LP_OUTS 64
#define LP_TURN 4  // blocks of 32 columns in flight
__device__ __forceinline__ uint4 lp_load16(const __nv_bfloat16 *p, bool ok) { return ok ? *(const uint4 *)p : make_uint4(0, 0, 0, 0); }

__global__ void __launch_bounds__(128) latent_prep_product_kernel(LatentPrep p, const __nv_bfloat16 *w, int n_rows) {
    __shared__ float scratch[33];
    const int tiles = (p.rank + LP_OUTS - 1) / LP_OUTS, t0 = blockIdx.y * LP_ROWS, per_head = p.dim + p.rot, half = p.rot_dims / 2;
    if ((int)blockIdx.x >= p.n_heads * tiles) {
        const int t = t0 + blockIdx.x - p.n_heads * tiles, seq = t < n_rows ? p.token_seq[t] : -1, pos = seq >= 0 ? p.token_pos[t] : 0;
        pdl_wait();
        if (seq >= 0 && p.pool) latent_row<__nv_bfloat16>(p, t, seq, pos, scratch);
        return;
    }
    const int h = blockIdx.x / tiles, tile = blockIdx.x % tiles, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int r = lane >> 2, c = lane & 3, o0 = tile * LP_OUTS + warp * 16, blocks = (p.dim + 31) / 32;
    const __nv_bfloat16 *w_lo = w + ((long long)h * p.rank + o0 + r) * p.dim + 8 * c, *w_hi = w_lo + 8LL * p.dim;
    const bool has_lo = o0 + r < p.rank, has_hi = o0 + r + 8 < p.rank;
    uint4 a_lo[LP_TURN], a_hi[LP_TURN], b[LP_TURN];
    auto load_weights = [&](int kb) {
#pragma unroll
        for (int u = 0; u < LP_TURN; u++) {
            const bool in = (kb + u) * 32 + 8 * c < p.dim;
            a_lo[u] = lp_load16(w_lo + (kb + u) * 32, in && has_lo), a_hi[u] = lp_load16(w_hi + (kb + u) * 32, in && has_hi);
        }
    };
    load_weights(0);
    pdl_wait();
    const __nv_bfloat16 *x = (const __nv_bfloat16 *)p.proj + (long long)(t0 + r) * p.ldp + (long long)h * per_head + 8 * c;
    float acc[4] = {0.0f, 0.0f, 0.0f, 0.0f};
    for (int kb = 0; kb < blocks; kb += LP_TURN) {
        if (kb) load_weights(kb);
#pragma unroll
        for (int u = 0; u < LP_TURN; u++) b[u] = lp_load16(x + (kb + u) * 32, t0 + r < n_rows && (kb + u) * 32 + 8 * c < p.dim);
#pragma unroll
        for (int u = 0; u < LP_TURN; u++) {
            const uint32_t a0[4] = {a_lo[u].x, a_hi[u].x, a_lo[u].y, a_hi[u].y}, a1[4] = {a_lo[u].z, a_hi[u].z, a_lo[u].w, a_hi[u].w};
            mma_bf16(acc, a0, b[u].x, b[u].y);
            mma_bf16(acc, a1, b[u].z, b[u].w);
        }
    }
    __nv_bfloat16 *q = (__nv_bfloat16 *)p.q_dst + (long long)h * p.q_head;
#pragma unroll
    for (int e = 0; e < 4; e++) {
        const int t = t0 + 2 * c + (e & 1), o = o0 + r + 8 * (e >> 1);
        if (t < n_rows && o < p.rank) q[(long long)t * p.ldq + o] = __float2bfloat16_rn(acc[e]);
    }
    if (tile) return;
    // the head's rotated part and the zeros behind it
    const int tail = p.q_head - p.q_rot_at - p.rot_dims;  // (what passes unchanged, then zeros)
    for (int e = threadIdx.x; e < LP_ROWS * half; e += 128) {
        const int t = t0 + e / half, i = e % half;
        if (t >= n_rows || p.token_seq[t] < 0) continue;
        const int pos = p.token_pos[t];
        const __nv_bfloat16 *src = (const __nv_bfloat16 *)p.proj + (long long)t * p.ldp + (long long)h * per_head + p.dim;
        const int ia = p.interleaved ? 2 * i : i, ib = p.interleaved ? 2 * i + 1 : i + half;
        const float cs = p.cos[(long long)pos * half + i], sn = p.sin[(long long)pos * half + i], u = to_float(src[ia]), v = to_float(src[ib]);
        __nv_bfloat16 *d = q + (long long)t * p.ldq + p.q_rot_at;
        d[ia] = __float2bfloat16_rn(u * cs - v * sn), d[ib] = __float2bfloat16_rn(v * cs + u * sn);
    }
    for (int e = threadIdx.x; e < LP_ROWS * tail; e += 128) {
        const int t = t0 + e / tail, i = p.rot_dims + e % tail;
        if (t >= n_rows) continue;
        const __nv_bfloat16 *src = (const __nv_bfloat16 *)p.proj + (long long)t * p.ldp + (long long)h * per_head + p.dim;
        q[(long long)t * p.ldq + p.q_rot_at + i] = i < p.rot ? src[i] : __float2bfloat16_rn(0.0f);
    }
}

// w (null: none; bfloat16 [heads][rank][dim]): the plain query parts times w go to + 0 of their heads in q_dst (bfloat16; not
// with copy_plain or rows).
extern "C" int abk_latent_prep(const void *proj, long long ldp, int dtype, int n_tokens, int down_at, int n_heads, int dim,
                               int rot, int rank, int rot_dims, int interleaved, const float *norm_w, float eps, const float *cos,
                               const float *sin, void *q_dst, long long ldq, int q_head, int q_rot_at, int copy_plain,
                               void *pool, int row, const int *page_table, int table_width, int ring_pages, int tokens_per_page,
                               void *rows, long long ld_rows, const int *token_seq, const int *token_pos, const int *seq_slot,
                               const int *seq_len_after, const void *w, void *stream) {
    if (n_tokens <= 0) return 0;
    if (rot_dims < 0 || rot_dims % 2 || rot_dims > rot) ABK_REFUSE("latent_prep: %d rotated dimensions of %d", rot_dims, rot);
    if (q_head < q_rot_at + rot || ((pool || rows) && row < rank + rot) || (rows && ld_rows < row))
        ABK_REFUSE("latent_prep: a head of %d or a cache row of %d does not hold %d + %d elements", q_head, row, rank, rot);
    LatentPrep p;
    p.proj = proj, p.ldp = ldp, p.down_at = down_at, p.n_heads = n_heads, p.dim = dim, p.rot = rot, p.rank = rank;
    p.rot_dims = rot_dims, p.interleaved = interleaved, p.norm_w = norm_w, p.eps = eps, p.cos = cos, p.sin = sin, p.q_dst = q_dst, p.ldq = ldq;
    p.q_head = q_head, p.q_rot_at = q_rot_at, p.copy_plain = copy_plain, p.pool = pool, p.row = row;
    p.cache.page_table = page_table, p.cache.table_width = table_width, p.cache.ring_pages = ring_pages;
    p.cache.tokens_per_page = tokens_per_page, p.cache.pinned_pages = 0, p.rows = rows, p.ld_rows = ld_rows;
    p.token_seq = token_seq, p.token_pos = token_pos, p.seq_slot = seq_slot, p.seq_len_after = seq_len_after;
    cudaStream_t s = (cudaStream_t)stream;
    if (w) {
        if (dtype != ABK_BF16 || copy_plain || rows || dim % 8 || (dim + rot) % 8 || ldp % 8 || (((uintptr_t)w | (uintptr_t)proj) & 15) || q_rot_at < rank)
            ABK_REFUSE("latent_prep: heads of %d + %d are not what the form with the product takes", dim, rot);
        const int tiles = (rank + LP_OUTS - 1) / LP_OUTS;
        abk_launch(latent_prep_product_kernel, dim3(n_heads * tiles + LP_ROWS, (n_tokens + LP_ROWS - 1) / LP_ROWS), dim3(128), 0, s, p,
                   (const __nv_bfloat16 *)w, n_tokens);
        return ABK_LAUNCH_RESULT();
    }
    const int sizes = dim | rot | rot_dims | q_head | q_rot_at | ((pool || rows) ? rank | row | down_at : 0);
    if (dtype == ABK_BF16 && sizes % 8 == 0 && ldp % 8 == 0 && ldq % 8 == 0 && (interleaved || rot_dims % 16 == 0) && row <= 1024 &&
        (!rows || ld_rows % 8 == 0) &&
        (((uintptr_t)proj | (uintptr_t)q_dst | (uintptr_t)pool | (uintptr_t)rows | (uintptr_t)cos | (uintptr_t)sin) & 15) == 0) {
        abk_launch(latent_prep_vector_kernel, dim3(n_tokens), dim3(128), 0, s, p);
        return ABK_LAUNCH_RESULT();
    }
    if (dtype == ABK_BF16) abk_launch(latent_prep_kernel<__nv_bfloat16>, dim3(n_tokens), dim3(128), 0, s, p);
    else abk_launch(latent_prep_kernel<float>, dim3(n_tokens), dim3(128), 0, s, p);
    return ABK_LAUNCH_RESULT();
}

// ---------------------------------------------------------------- the norm of a run of columns
// dst[t, i] = w[i] * src[t, i] / sqrt(mean_i(src[t, i]^2) + eps) for i < count: a latent normed where it lies among the
// columns of a product's output (rows of any pitch; dst may be src).
template <typename T>
__global__ void __launch_bounds__(128) columns_norm_kernel(const T *src, long long lds, T *dst, long long ldd, int count,
                                                           const float *w, float eps) {
    __shared__ float scratch[33];
    const long long t = blockIdx.x;
    pdl_wait();
    const T *s = src + t * lds;
    T *d = dst + t * ldd;
    float ss = 0.0f;
    for (int i = threadIdx.x; i < count; i += 128) {
        const float v = to_float(s[i]);
        ss = fmaf(v, v, ss);
    }
    ss = block_sum(ss, scratch);
    const float inv = 1.0f / sqrtf(ss / (float)count + eps);
    for (int i = threadIdx.x; i < count; i += 128) d[i] = from_float<T>(to_float(s[i]) * inv * w[i]);
}

extern "C" int abk_columns_norm(const void *src, long long lds, void *dst, long long ldd, int dtype, int n_tokens, int count,
                                const float *w, float eps, void *stream) {
    if (n_tokens <= 0 || count <= 0) return 0;
    cudaStream_t s = (cudaStream_t)stream;
    if (dtype == ABK_BF16)
        abk_launch(columns_norm_kernel<__nv_bfloat16>, dim3(n_tokens), dim3(128), 0, s, (const __nv_bfloat16 *)src, lds,
                   (__nv_bfloat16 *)dst, ldd, count, w, eps);
    else
        abk_launch(columns_norm_kernel<float>, dim3(n_tokens), dim3(128), 0, s, (const float *)src, lds, (float *)dst, ldd, count, w, eps);
    return ABK_LAUNCH_RESULT();
}

// ---------------------------------------------------------------- a product per head
#define HP_ROWS 8      // rows of x a CTA holds in shared memory
#define HP_PER_WARP 4  // output features a warp makes, one after the other

template <typename T>
__global__ void __launch_bounds__(128) head_product_kernel(const T *__restrict__ x, long long ldx, int x_head,
                                                           const T *__restrict__ w, T *__restrict__ out, long long ldo,
                                                           int o_head, int n, int in, int outs, const T *__restrict__ gate,
                                                           long long ldg) {
    extern __shared__ __align__(16) float hp_x[];  // [HP_ROWS][in4], in4 = in rounded up to 4
    const int h = blockIdx.y, r0 = blockIdx.z * HP_ROWS, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int rows = n - r0 < HP_ROWS ? n - r0 : HP_ROWS;
    pdl_wait();
    const int in4 = (in + 3) & ~3;
    for (int e = threadIdx.x; e < HP_ROWS * in; e += 128) {
        const int r = e / in, i = e - r * in;
        hp_x[r * in4 + i] = r < rows ? to_float(x[(long long)(r0 + r) * ldx + (long long)h * x_head + i]) : 0.0f;
    }
    __syncthreads();
    const bool vec = in % (16 / (int)sizeof(T)) == 0 && ((uintptr_t)w & 15) == 0;
    for (int u = 0; u < HP_PER_WARP; u++) {
        const int o = (blockIdx.x * 4 + warp) * HP_PER_WARP + u;
        if (o >= outs) break;
        const T *wr = w + ((long long)h * outs + o) * in;
        // a row of the matrix against each of the CTA's rows of x: the lanes' shares of the sums, each in its own order
        for (int r = 0; r < rows; r++) {
            float acc = 0.0f;
            lane_dots<1>(wr, 0, hp_x + r * in4, in, lane, vec, &acc);
            acc = warp_sum(acc);
            if (lane == 0) {
                if (gate) acc *= 1.0f / (1.0f + expf(-to_float(gate[(long long)(r0 + r) * ldg + h])));  // a gate per head
                out[(long long)(r0 + r) * ldo + (long long)h * o_head + o] = from_float<T>(acc);
            }
        }
    }
}

// x element (t, h, i) at x + t * ldx + h * x_head + i; w [heads][outs][in]; out element (t, h, o) at
// out + t * ldo + h * o_head + o. x, w and out are of one type. gate (null: none): head h of row t is multiplied by
// sigmoid(gate[t * ldg + h]).
extern "C" int abk_head_product(const void *x, long long ldx, int x_head, const void *w, void *out, long long ldo,
                                int o_head, int dtype, int n, int heads, int in, int outs, const void *gate, long long ldg,
                                void *stream) {
    if (n <= 0 || heads <= 0 || outs <= 0) return 0;
    if (in < 1 || in > 4096) ABK_REFUSE("head_product: an inner size of %d is not 1 to 4096", in);
    const long long row_tiles = ((long long)n + HP_ROWS - 1) / HP_ROWS;
    if (heads > 65535 || row_tiles > 65535) ABK_REFUSE("head_product: %d heads, %d rows are more than a grid takes", heads, n);
    dim3 grid((outs + 4 * HP_PER_WARP - 1) / (4 * HP_PER_WARP), heads, (unsigned)row_tiles);
    const size_t smem = (size_t)HP_ROWS * ((in + 3) & ~3) * sizeof(float);
    cudaStream_t s = (cudaStream_t)stream;
    if (dtype == ABK_BF16) {
        if (smem > 48 * 1024) {
            cudaError_t e = abk_allow_shared_memory((const void *)head_product_kernel<__nv_bfloat16>, (int)smem);
            if (e != cudaSuccess) return (int)e;
        }
        abk_launch(head_product_kernel<__nv_bfloat16>, grid, dim3(128), smem, s, (const __nv_bfloat16 *)x, ldx, x_head,
                   (const __nv_bfloat16 *)w, (__nv_bfloat16 *)out, ldo, o_head, n, in, outs, (const __nv_bfloat16 *)gate, ldg);
    } else {
        if (smem > 48 * 1024) {
            cudaError_t e = abk_allow_shared_memory((const void *)head_product_kernel<float>, (int)smem);
            if (e != cudaSuccess) return (int)e;
        }
        abk_launch(head_product_kernel<float>, grid, dim3(128), smem, s, (const float *)x, ldx, x_head, (const float *)w,
                   (float *)out, ldo, o_head, n, in, outs, (const float *)gate, ldg);
    }
    return ABK_LAUNCH_RESULT();
}

// ---------------------------------------------------------------- a prompt's keys and values in full size
// rows[t] = the first `count` elements of the cache row of token t (its sequence's slot, its position).
template <typename T>
__global__ void __launch_bounds__(128) latent_rows_kernel(const T *pool, int row, PagedCache cache, T *rows, long long ld,
                                                          int count, const int *token_seq, const int *token_pos,
                                                          const int *seq_slot) {
    const int t = blockIdx.x;
    pdl_wait();
    const int seq = token_seq[t];
    T *dst = rows + (long long)t * ld;
    if (seq < 0) {
        for (int i = threadIdx.x; i < count; i += 128) dst[i] = from_float<T>(0.0f);
        return;
    }
    const int pos = token_pos[t];
    const T *src = pool + cache_offset(cache, cache_page(cache, seq_slot[seq], pos), 0, 1, pos, row);
    for (int i = threadIdx.x; i < count; i += 128) dst[i] = src[i];
}

extern "C" int abk_latent_rows(const void *pool, int row, const int *page_table, int table_width, int tokens_per_page,
                               void *rows, long long ld, int count, int dtype, int n_tokens, const int *token_seq,
                               const int *token_pos, const int *seq_slot, void *stream) {
    if (n_tokens <= 0) return 0;
    if (count > row || count > ld) ABK_REFUSE("latent_rows: %d elements of a cache row of %d into rows of %lld", count, row, ld);
    PagedCache c;
    c.page_table = page_table, c.table_width = table_width, c.ring_pages = 0, c.tokens_per_page = tokens_per_page;
    cudaStream_t s = (cudaStream_t)stream;
    if (dtype == ABK_BF16)
        abk_launch(latent_rows_kernel<__nv_bfloat16>, dim3(n_tokens), dim3(128), 0, s, (const __nv_bfloat16 *)pool, row, c,
                   (__nv_bfloat16 *)rows, ld, count, token_seq, token_pos, seq_slot);
    else
        abk_launch(latent_rows_kernel<float>, dim3(n_tokens), dim3(128), 0, s, (const float *)pool, row, c, (float *)rows,
                   ld, count, token_seq, token_pos, seq_slot);
    return ABK_LAUNCH_RESULT();
}

// keys[t, h, at + i] = shared[t, i] for every head h and i < count (keys: rows of ldk elements, heads of k_head).
template <typename T>
__global__ void __launch_bounds__(128) spread_shared_kernel(const T *shared, long long lds, T *keys, long long ldk, int k_head,
                                                            int at, int count, int heads) {
    const int t = blockIdx.x;
    pdl_wait();
    for (int e = threadIdx.x; e < heads * count; e += 128) {
        const int h = e / count, i = e - h * count;
        keys[(long long)t * ldk + (long long)h * k_head + at + i] = shared[(long long)t * lds + i];
    }
}

extern "C" int abk_spread_shared(const void *shared, long long lds, void *keys, long long ldk, int k_head, int at, int count,
                                 int heads, int dtype, int n_tokens, void *stream) {
    if (n_tokens <= 0 || count <= 0) return 0;
    cudaStream_t s = (cudaStream_t)stream;
    if (dtype == ABK_BF16)
        abk_launch(spread_shared_kernel<__nv_bfloat16>, dim3(n_tokens), dim3(128), 0, s, (const __nv_bfloat16 *)shared, lds,
                   (__nv_bfloat16 *)keys, ldk, k_head, at, count, heads);
    else
        abk_launch(spread_shared_kernel<float>, dim3(n_tokens), dim3(128), 0, s, (const float *)shared, lds, (float *)keys,
                   ldk, k_head, at, count, heads);
    return ABK_LAUNCH_RESULT();
}
