// A minimal gated recurrence: a running average per channel whose gate and candidate read the current token alone,
//     z = sigmoid(z' + bz),  u = u' + bu,  c = u + 1/2 where u >= 0, sigmoid(u) where u < 0,
//     S_t = (1 - z_t) S_(t-1) + z_t c_t,    out_t = S_t * silu(g_t),
// z', u', g the token's projections. Everything from the projections on is float32; the state is zero at a sequence's
// start and carried in the sequence's slot.
//
//   step   one token a sequence: a thread a channel (or a pair, or four).
//   scan   prompts: a step of the recurrence is the map S -> a S + b with a = 1 - z, b = z c, and maps compose, so a
//          sequence is cut into runs that are all walked at once. A cluster of CTAs has one sequence and 32 channels (64 as
//          pairs); each of its warps has a run of 8 tokens (the gates and candidates of which it keeps in registers)
//          and makes the run's own map; the maps meet in shared memory, a thread a channel, every CTA leaving its own map with
//          all others (distributed shared memory); then every warp walks its run again from the state it now knows, for the outputs. Longer
//          sequences go round in turns, the state carried.
#define ABK_DEFINE_ERROR
#include "common.cuh"
#include "tc_common.cuh"

struct GatedAverage {
    const void *proj;  // row t at proj + t * ld: z' at z_at + c, u' at u_at + c, g at g_at + c
    long long ld;
    int z_at, u_at, g_at, width;
    const float *bz, *bu;  // [width]
    float *state;          // [slots, width]
    void *out;             // row t at out + t * ldo
    long long ldo;
    int padded;            // columns of out from width on up to here get zeros
    const int *token_seq, *seq_start, *seq_slot;
};

// to the last bits where the model is float32; by the special-function unit (a few units in the last place of float32, in
// float32 arithmetic) where its operands are bfloat16 numbers
template <typename T> __device__ __forceinline__ float ga_exp(float v) { return expf(v); }
template <> __device__ __forceinline__ float ga_exp<__nv_bfloat16>(float v) { return __expf(v); }
template <typename T> __device__ __forceinline__ float ga_inverse(float v) { return 1.0f / v; }
template <> __device__ __forceinline__ float ga_inverse<__nv_bfloat16>(float v) { return __fdividef(1.0f, v); }

// (1 - z, z c) of a token's pre-activations. e^-z' is kept below what overflows: beyond it z is 0 in float32 either way.
template <typename T> __device__ __forceinline__ void ga_map(float zp, float u, float &a, float &b) {
    const float e = ga_exp<T>(fminf(-zp, 80.0f)), z = ga_inverse<T>(1.0f + e);
    const float c = u >= 0.0f ? u + 0.5f : ga_inverse<T>(1.0f + ga_exp<T>(fminf(-u, 80.0f)));
    a = e * z, b = z * c;
}
template <typename T> __device__ __forceinline__ float ga_silu(float g) { return g * ga_inverse<T>(1.0f + ga_exp<T>(fminf(-g, 80.0f))); }

// VEC consecutive elements as floats / stored from floats.
template <int VEC> __device__ __forceinline__ void ga_load(const float *p, float *f) {
    if constexpr (VEC == 4) { const float4 v = *(const float4 *)p; f[0] = v.x, f[1] = v.y, f[2] = v.z, f[3] = v.w; }
    else if constexpr (VEC == 2) { const float2 v = *(const float2 *)p; f[0] = v.x, f[1] = v.y; }
    else f[0] = *p;
}
template <int VEC> __device__ __forceinline__ void ga_load(const __nv_bfloat16 *p, float *f) {
    if constexpr (VEC == 1) f[0] = __bfloat162float(*p);
    else {
#pragma unroll
        for (int i = 0; i < VEC / 2; i++) {
            const float2 v = __bfloat1622float2(((const __nv_bfloat162 *)p)[i]);
            f[2 * i] = v.x, f[2 * i + 1] = v.y;
        }
    }
}
template <int VEC> __device__ __forceinline__ void ga_store(float *p, const float *f) {
    if constexpr (VEC == 4) *(float4 *)p = make_float4(f[0], f[1], f[2], f[3]);
    else if constexpr (VEC == 2) *(float2 *)p = make_float2(f[0], f[1]);
    else *p = f[0];
}
template <int VEC> __device__ __forceinline__ void ga_store(__nv_bfloat16 *p, const float *f) {
    if constexpr (VEC == 1) *p = __float2bfloat16_rn(f[0]);
    else {
#pragma unroll
        for (int i = 0; i < VEC / 2; i++) ((__nv_bfloat162 *)p)[i] = __floats2bfloat162_rn(f[2 * i], f[2 * i + 1]);
    }
}

// VEC elements as they lie in memory: loads that are asked for early keep what they bring in this form, so that nothing waits
// for them before they are needed.
template <typename T, int VEC> struct GaRaw;
template <> struct GaRaw<__nv_bfloat16, 2> { uint32_t v; };
template <> struct GaRaw<__nv_bfloat16, 1> { unsigned short v; };
template <> struct GaRaw<float, 2> { float2 v; };
template <> struct GaRaw<float, 1> { float v; };
template <typename T, int VEC> __device__ __forceinline__ GaRaw<T, VEC> ga_fetch(const T *p) { return *(const GaRaw<T, VEC> *)p; }
__device__ __forceinline__ void ga_open(const GaRaw<__nv_bfloat16, 2> &r, float *f) {
    const float2 v = __bfloat1622float2(*(const __nv_bfloat162 *)&r.v);
    f[0] = v.x, f[1] = v.y;
}
__device__ __forceinline__ void ga_open(const GaRaw<__nv_bfloat16, 1> &r, float *f) { f[0] = __bfloat162float(*(const __nv_bfloat16 *)&r.v); }
__device__ __forceinline__ void ga_open(const GaRaw<float, 2> &r, float *f) { f[0] = r.v.x, f[1] = r.v.y; }
__device__ __forceinline__ void ga_open(const GaRaw<float, 1> &r, float *f) { f[0] = r.v; }

// ---------------------------------------------------------------- one token a sequence
template <typename T, int VEC> __global__ void __launch_bounds__(128) gated_average_step_kernel(GatedAverage p) {
    const int c = (blockIdx.x * 128 + threadIdx.x) * VEC, t = blockIdx.y;
    float bz[VEC], bu[VEC];
    if (c < p.width) ga_load<VEC>(p.bz + c, bz), ga_load<VEC>(p.bu + c, bu);  // weights: ahead of the wait
    pdl_wait();
    const int seq = p.token_seq[t];
    if (seq < 0) return;
    if (c >= p.width) {
        float zero[VEC];
#pragma unroll
        for (int i = 0; i < VEC; i++) zero[i] = 0.0f;
        if (c < p.padded) ga_store<VEC>((T *)p.out + (long long)t * p.ldo + c, zero);
        return;
    }
    const T *row = (const T *)p.proj + (long long)t * p.ld + c;
    float *slot = p.state + (long long)p.seq_slot[seq] * p.width + c;
    float z[VEC], u[VEC], g[VEC], s[VEC];
    ga_load<VEC>(row + p.z_at, z), ga_load<VEC>(row + p.u_at, u), ga_load<VEC>(row + p.g_at, g), ga_load<VEC>(slot, s);
#pragma unroll
    for (int i = 0; i < VEC; i++) {
        float a, b;
        ga_map<T>(z[i] + bz[i], u[i] + bu[i], a, b);
        s[i] = fmaf(a, s[i], b);
        g[i] = s[i] * ga_silu<T>(g[i]);
    }
    ga_store<VEC>(slot, s);
    ga_store<VEC>((T *)p.out + (long long)t * p.ldo + c, g);
}

// ---------------------------------------------------------------- prompts
#define GA_WARPS 16
#define GA_RUN 8     // tokens of a warp's run

template <typename T, int VEC> __global__ void __launch_bounds__(32 * GA_WARPS) gated_average_scan_kernel(GatedAverage p) {
    constexpr int CH = 32 * VEC;
    __shared__ float2 runs[GA_WARPS][CH];    // the runs' maps (a, b); then, in x, the states before the runs
    __shared__ float2 ctas[2][8][CH];        // the CTAs' maps, by the turn's parity: every CTA leaves its own with all of them
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int ranks = (int)tc::cluster_size(), rank = (int)tc::cluster_rank();
    const int c = (blockIdx.x / ranks) * CH + lane * VEC, seq = blockIdx.y;
    const bool real = c < p.width;  // (VEC divides the width)
    float bz[VEC], bu[VEC];
#pragma unroll
    for (int i = 0; i < VEC; i++) bz[i] = bu[i] = 0.0f;
    if (real) ga_load<VEC>(p.bz + c, bz), ga_load<VEC>(p.bu + c, bu);
    pdl_wait();
    const int row0 = p.seq_start[seq], n = p.seq_start[seq + 1] - row0;
    if (n <= 0) return;  // (the whole cluster: a sequence of the step's padding)
    // the first CH threads each keep a channel's state before the turn, the same in every CTA of the cluster
    const int own = (blockIdx.x / ranks) * CH + (int)threadIdx.x;
    const bool keeper = threadIdx.x < CH, owns = keeper && own < p.width;
    float *const slot = p.state + (long long)p.seq_slot[seq] * p.width + own;
    float held = owns ? *slot : 0.0f;
    const int turn_tokens = ranks * GA_WARPS * GA_RUN;
    int parity = 0;
    // a run's rows: gates and candidates are asked for a turn ahead, the outputs' gates with the turn before's outputs
    // (loads that hang on no branch fly together: a row beyond the run repeats its last)
    GaRaw<T, VEC> rz[GA_RUN], ru[GA_RUN], rg[GA_RUN];
    const T *const all = (const T *)p.proj + (long long)row0 * p.ld + c;
    auto run_of = [&](int t0, int &first) {
        first = t0 + (rank * GA_WARPS + warp) * GA_RUN;
        return min(GA_RUN, n - first);  // (not above zero: no run)
    };
    auto fetch = [&](int t0) {
        int first;
        const int cnt = run_of(t0, first);
        if (!real || cnt <= 0) return;
#pragma unroll
        for (int k = 0; k < GA_RUN; k++) {
            const T *r = all + (long long)(first + min(k, cnt - 1)) * p.ld;
            rz[k] = ga_fetch<T, VEC>(r + p.z_at), ru[k] = ga_fetch<T, VEC>(r + p.u_at);
        }
    };
    auto fetch_gates = [&](int t0) {
        int first;
        const int cnt = run_of(t0, first);
        if (!real || cnt <= 0) return;
#pragma unroll
        for (int k = 0; k < GA_RUN; k++) rg[k] = ga_fetch<T, VEC>(all + (long long)(first + min(k, cnt - 1)) * p.ld + p.g_at);
    };
    fetch(0), fetch_gates(0);
    if (ranks > 1) tc::cluster_sync();  // every CTA has started: maps may be left with it
    for (int t0 = 0; t0 < n; t0 += turn_tokens, parity ^= 1) {
        int first;
        const int cnt = run_of(t0, first);
        float a[GA_RUN][VEC], b[GA_RUN][VEC], A[VEC], B[VEC];
#pragma unroll
        for (int i = 0; i < VEC; i++) A[i] = 1.0f, B[i] = 0.0f;
        if (real && cnt > 0) {
#pragma unroll
            for (int k = 0; k < GA_RUN; k++) {
                float z[VEC], u[VEC];
                ga_open(rz[k], z), ga_open(ru[k], u);
#pragma unroll
                for (int i = 0; i < VEC; i++) {
                    ga_map<T>(z[i] + bz[i], u[i] + bu[i], a[k][i], b[k][i]);
                    if (k < cnt) A[i] *= a[k][i], B[i] = fmaf(a[k][i], B[i], b[k][i]);
                }
            }
        }
        if (t0 + turn_tokens < n) fetch(t0 + turn_tokens);
        __syncthreads();  // the turn before has read the states before its runs
#pragma unroll
        for (int i = 0; i < VEC; i++) runs[warp][lane * VEC + i] = make_float2(A[i], B[i]);
        __syncthreads();
        float2 map[GA_WARPS];
        if (keeper) {
            float2 all = make_float2(1.0f, 0.0f);
#pragma unroll
            for (int w = 0; w < GA_WARPS; w++) {
                map[w] = runs[w][threadIdx.x];
                all = make_float2(map[w].x * all.x, fmaf(map[w].x, all.y, map[w].y));
            }
            const uint32_t at = (uint32_t)__cvta_generic_to_shared(&ctas[parity][rank][threadIdx.x]);
            if (ranks == 1) ctas[parity][0][threadIdx.x] = all;
            else for (int k = 0; k < ranks; k++)
                asm volatile("st.shared::cluster.v2.f32 [%0], {%1, %2};" ::"r"(tc::peer_smem(at, k)), "f"(all.x), "f"(all.y) : "memory");
        }
        if (ranks > 1) tc::cluster_sync();
        if (keeper) {  // through the CTAs before this one and through its runs; and on to the turn's end
            float v = held, mine = held;
            for (int k = 0; k < ranks; k++) {
                if (k == rank) mine = v;
                const float2 m = ctas[parity][k][threadIdx.x];
                v = fmaf(m.x, v, m.y);
            }
            held = v;
#pragma unroll
            for (int w = 0; w < GA_WARPS; w++) {
                runs[w][threadIdx.x].x = mine;
                mine = fmaf(map[w].x, mine, map[w].y);
            }
        }
        __syncthreads();
        float s[VEC];
#pragma unroll
        for (int i = 0; i < VEC; i++) s[i] = runs[warp][lane * VEC + i].x;
        if (!real && c < p.padded) {
            float zero[VEC];
#pragma unroll
            for (int i = 0; i < VEC; i++) zero[i] = 0.0f;
            for (int k = 0; k < cnt; k++) ga_store<VEC>((T *)p.out + (long long)(row0 + first + k) * p.ldo + c, zero);
        }
        if (real && cnt > 0) {
            T *out = (T *)p.out + (long long)(row0 + first) * p.ldo + c;
#pragma unroll
            for (int k = 0; k < GA_RUN; k++) {
                if (k >= cnt) break;
                float g[VEC];
                ga_open(rg[k], g);
#pragma unroll
                for (int i = 0; i < VEC; i++) {
                    s[i] = fmaf(a[k][i], s[i], b[k][i]);
                    g[i] = s[i] * ga_silu<T>(g[i]);
                }
                ga_store<VEC>(out + (long long)k * p.ldo, g);
            }
        }
        if (t0 + turn_tokens < n) fetch_gates(t0 + turn_tokens);
    }
    if (rank == 0 && owns) *slot = held;
    if (ranks > 1) tc::cluster_sync();  // nobody leaves while a map may still be left with it
}

// padded: columns of out from width on up to there are written with zeros (a product with padded rows reads them).
// decode: every sequence of the step brings one token (row t is sequence token_seq[t]). Else ranks (1, 2, 4 or 8) CTAs
// share a sequence.
extern "C" int abk_gated_average(const void *proj, long long ld, int dtype, int z_at, int u_at, int g_at, int width,
                                 const float *bz, const float *bu, float *state, void *out, long long ldo, int padded,
                                 int n_tokens, int n_seqs, int decode, int ranks, const int *token_seq, const int *seq_start,
                                 const int *seq_slot, void *stream) {
    if (n_tokens <= 0 || n_seqs <= 0) return 0;
    if (width < 1) ABK_REFUSE("gated_average: a width of %d", width);
    if (padded < width) padded = width;
    if (n_tokens > 65535 && decode) ABK_REFUSE("gated_average: %d sequences are more than a grid takes", n_tokens);
    if (n_seqs > 65535 || (ranks != 1 && ranks != 2 && ranks != 4 && ranks != 8))
        ABK_REFUSE("gated_average: %d sequences, clusters of %d", n_seqs, ranks);
    GatedAverage p;
    p.proj = proj, p.ld = ld, p.z_at = z_at, p.u_at = u_at, p.g_at = g_at, p.width = width, p.bz = bz, p.bu = bu;
    p.state = state, p.out = out, p.ldo = ldo, p.padded = padded, p.token_seq = token_seq, p.seq_start = seq_start, p.seq_slot = seq_slot;
    const long long places = ld | z_at | u_at | g_at | ldo | width | padded;
    const bool whole = !(((uintptr_t)proj | (uintptr_t)out | (uintptr_t)bz | (uintptr_t)bu | (uintptr_t)state) & 15);
    cudaStream_t s = (cudaStream_t)stream;
    typedef __nv_bfloat16 bf;
    if (decode) {
        const int vec = whole && places % 4 == 0 ? 4 : 1;
        const dim3 grid((padded / vec + 127) / 128, n_tokens);
        if (dtype == ABK_BF16 && vec == 4) abk_launch(gated_average_step_kernel<bf, 4>, grid, dim3(128), 0, s, p);
        else if (dtype == ABK_BF16) abk_launch(gated_average_step_kernel<bf, 1>, grid, dim3(128), 0, s, p);
        else if (vec == 4) abk_launch(gated_average_step_kernel<float, 4>, grid, dim3(128), 0, s, p);
        else abk_launch(gated_average_step_kernel<float, 1>, grid, dim3(128), 0, s, p);
        return ABK_LAUNCH_RESULT();
    }
    const int vec = whole && places % 2 == 0 ? 2 : 1;
    const dim3 grid((padded + 32 * vec - 1) / (32 * vec) * ranks, n_seqs);
    const dim3 block(32 * GA_WARPS);
    if (dtype == ABK_BF16 && vec == 2) abk_launch_clusters(gated_average_scan_kernel<bf, 2>, grid, block, 0, s, ranks, p);
    else if (dtype == ABK_BF16) abk_launch_clusters(gated_average_scan_kernel<bf, 1>, grid, block, 0, s, ranks, p);
    else if (vec == 2) abk_launch_clusters(gated_average_scan_kernel<float, 2>, grid, block, 0, s, ranks, p);
    else abk_launch_clusters(gated_average_scan_kernel<float, 1>, grid, block, 0, s, ranks, p);
    return ABK_LAUNCH_RESULT();
}
