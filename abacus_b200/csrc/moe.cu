// A feed-forward of routed experts: every token goes through `top` of `experts` small feed-forward layers, chosen by
// a router.
//
//   moe_route       per token: router logits z = R x in float32 (x as stored), the `top` largest (a tie goes to the
//                   lower index), and each chosen expert's weight: sigmoid(z) (score 0) or its softmax over the
//                   chosen (score 1), or (score 2) s = softmax(z) over all router outputs, the choice by s + correction
//                   (a learned shift per output that the weights do not see), the weight s * scale. A pair is
//                   (token, k-th choice), numbered token * top + k; pairs of padding rows carry expert -1. Router
//                   outputs from `n_real` on stand for experts without matrices that return their input: such a
//                   pair carries -2 - (output - n_real), which the products skip and moe_combine_weighted knows. With
//                   `always` >= 0 every token has one more pair, its last: that expert with weight 1 (a shared expert that
//                   lies stacked behind the routed ones). With `bias` z = R x + bias. With `shared_weight` R has one row
//                   more, and sigmoid of its product is the token's weight of a shared expert.
//   routed_product  out[pair] = act(W[expert of pair] (scale of pair * x[row of pair])): a product whose matrix is
//                   chosen per row. With a scale the input is multiplied by it and rounded to its stored type first
//                   (the weight acts on the expert's input). A CTA stages the pair's row in shared memory; a warp makes
//                   an output feature at a time, lanes along the inner dimension, so the expert's rows stream
//                   coalesced. Float32 sums in a fixed order.
//   moe_combine     out[t] (+)= sum over k of pairs[t * top + k], in the order of k.
//   moe_combine_weighted  out[t] = sum over k of weight[t, k] * (pairs[t * top + k], or x[t] for an expert that returns
//                   its input), in the order of k: the weight on the experts' outputs, in float32. The pairs' rows lie in
//                   the pairs' order, or (with `place`) sorted by expert, pair p at row place[p]. With `shared`, what a
//                   shared expert left in out joins first, times its weight for the token (1 where there is none).
//   routed_product also has the gated forms: W holds gate and up rows in turns of `block` (all gates then all ups where block
//                   is their number), out = silu(gate . x) * (up . x), or the clamped form (common.cuh: gated_mul).
//   relu_squared    x = max(x, 0)^2 in place.
#define ABK_DEFINE_ERROR
#include "common.cuh"

#define MR_THREADS 256
// ROWS router rows `stride` apart (row e0 at w) against TOKENS rows in shared memory `pitch` apart: a lane's shares of the sums.
template <int ROWS, int TOKENS>
__device__ __forceinline__ void route_dots(const float *w, long long stride, const float *xs, int pitch, int d, int lane, bool vec,
                                           float (*acc)[4]) {
    if (vec) {
        for (int i = lane * 4; i < d; i += 128) {
            float4 r[ROWS];
#pragma unroll
            for (int u = 0; u < ROWS; u++) r[u] = *(const float4 *)(w + u * stride + i);
#pragma unroll
            for (int k = 0; k < TOKENS; k++) {
                const float4 a = *(const float4 *)(xs + k * pitch + i);
#pragma unroll
                for (int u = 0; u < ROWS; u++)
                    acc[k][u] = fmaf(r[u].w, a.w, fmaf(r[u].z, a.z, fmaf(r[u].y, a.y, fmaf(r[u].x, a.x, acc[k][u]))));
            }
        }
    } else {
        for (int i = lane; i < d; i += 32)
#pragma unroll
            for (int k = 0; k < TOKENS; k++)
#pragma unroll
                for (int u = 0; u < ROWS; u++) acc[k][u] = fmaf(w[u * stride + i], xs[k * pitch + i], acc[k][u]);
    }
}

// TOKENS tokens a CTA (1 for a decode step, 4 for a prompt: the router's rows are then read once for four).
template <typename T, int TOKENS>
__global__ void __launch_bounds__(MR_THREADS) moe_route_kernel(const T *x, long long ldx, const float *router, int n_tokens, int d, int experts,
                                                        int top, int score, int always, const int *token_seq,
                                                        int *pair_expert, float *pair_weight, const float *correction,
                                                        float weight_scale, int n_real, const float *bias, float *shared_weight) {
    // a token's row (d rounded up to 4); its [experts + 1] logits, [experts] taken flags, [experts] what the choice goes by
    extern __shared__ __align__(16) float mr_smem[];
    const int pitch = (d + 3) & ~3;
    float *xs = mr_smem, *scratch = xs + TOKENS * pitch;
    const int outputs = experts + (shared_weight ? 1 : 0);  // router rows: the last may be the shared expert's
    const int softmax_chosen = score == 1;
    const int t0 = blockIdx.x * TOKENS, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int per = top + (always >= 0 ? 1 : 0);  // pairs a token has: its choices, then the expert every token uses
    constexpr int W = MR_THREADS / 32;
    for (int e = warp; e < outputs; e += W)  // weights: on their way while the kernel before is still running
        for (int i = lane * 32; i < d; i += 1024) asm volatile("prefetch.global.L2 [%0];" ::"l"(router + (long long)e * d + i));
    pdl_wait();
    for (int k = 0; k < TOKENS; k++) {
        const bool on = t0 + k < n_tokens && token_seq[t0 + k] >= 0;
        for (int i = tid; i < d; i += MR_THREADS) xs[k * pitch + i] = on ? to_float(x[(long long)(t0 + k) * ldx + i]) : 0.0f;
        int *taken = (int *)(scratch + k * (3 * experts + 1) + experts + 1);
        for (int e = tid; e < experts; e += MR_THREADS) taken[e] = 0;
    }
    __syncthreads();
    const bool vec = d % 4 == 0 && ((uintptr_t)router & 15) == 0;
    for (int e = warp; e < outputs;) {  // a warp's router rows, up to four at a time so that their loads are in flight together
        const int left = (outputs - e + W - 1) / W, rows = left < 4 ? left : 4;
        float acc[TOKENS][4];
#pragma unroll
        for (int k = 0; k < TOKENS; k++) acc[k][0] = acc[k][1] = acc[k][2] = acc[k][3] = 0.0f;
        const float *w = router + (long long)e * d;
        if (rows == 4) route_dots<4, TOKENS>(w, (long long)W * d, xs, pitch, d, lane, vec, acc);
        else if (rows == 3) route_dots<3, TOKENS>(w, (long long)W * d, xs, pitch, d, lane, vec, acc);
        else if (rows == 2) route_dots<2, TOKENS>(w, (long long)W * d, xs, pitch, d, lane, vec, acc);
        else route_dots<1, TOKENS>(w, 0, xs, pitch, d, lane, vec, acc);
#pragma unroll
        for (int k = 0; k < TOKENS; k++) {
#pragma unroll
            for (int u = 0; u < 4; u++) {
                if (u >= rows) break;
                const float sum = warp_sum(acc[k][u]);
                if (lane == 0) scratch[k * (3 * experts + 1) + e + u * W] = bias && e + u * W < experts ? sum + bias[e + u * W] : sum;
            }
        }
        e += rows * W;
    }
    __syncthreads();
    if (warp >= TOKENS || t0 + warp >= n_tokens) return;  // a warp a token from here on
    const int t = t0 + warp;
    pair_expert += (long long)t * per, pair_weight += (long long)t * per;
    if (token_seq[t] < 0) {
        for (int k = lane; k < per; k += 32) pair_expert[k] = -1, pair_weight[k] = 0.0f;
        if (shared_weight && lane == 0) shared_weight[t] = 0.0f;
        return;
    }
    if (always >= 0 && lane == 0) pair_expert[top] = always, pair_weight[top] = 1.0f;
    float *z = scratch + warp * (3 * experts + 1);
    int *taken = (int *)(z + experts + 1);
    float *key = (float *)(taken + experts);
    if (shared_weight && lane == 0) shared_weight[t] = 1.0f / (1.0f + expf(-z[experts]));
    if (score == 2) {  // z becomes softmax(z) over all outputs; the choice goes by it plus the correction
        float mx = -INFINITY, sum = 0.0f;
        for (int e = lane; e < experts; e += 32) mx = fmaxf(mx, z[e]);
        mx = warp_max(mx);
        for (int e = lane; e < experts; e += 32) sum += expf(z[e] - mx);
        sum = warp_sum(sum);
        for (int e = lane; e < experts; e += 32) {
            z[e] = expf(z[e] - mx) / sum;
            key[e] = z[e] + (correction ? correction[e] : 0.0f);
        }
    } else {
        for (int e = lane; e < experts; e += 32) key[e] = z[e];
    }
    __syncwarp();
    float chosen_max = -INFINITY, denom = 0.0f;
    for (int k = 0; k < top; k++) {
        float best = -INFINITY;
        int at = 0x7fffffff;
        for (int e = lane; e < experts; e += 32)
            if (!taken[e] && (key[e] > best || at == 0x7fffffff)) best = key[e], at = e;  // (the first of a lane's own is its lowest)
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
            const float ob = __shfl_xor_sync(0xffffffffu, best, o);
            const int oa = __shfl_xor_sync(0xffffffffu, at, o);
            if (oa != 0x7fffffff && (at == 0x7fffffff || ob > best || (ob == best && oa < at))) best = ob, at = oa;
        }
        if (k == 0) chosen_max = best;
        denom += expf(best - chosen_max);
        if (lane == 0) {
            taken[at] = 1;
            pair_expert[k] = at < n_real ? at : -2 - (at - n_real);
            pair_weight[k] = score == 2 ? z[at] * weight_scale : softmax_chosen ? best : 1.0f / (1.0f + expf(-best));
        }
        __syncwarp();
    }
    if (softmax_chosen && lane == 0)
        for (int k = 0; k < top; k++) {
            pair_weight[k] = expf(pair_weight[k] - chosen_max) / denom;
        }
}

extern "C" int abk_moe_route(const void *x, long long ldx, int dtype, const float *router, int n_tokens, int d, int experts,
                             int top, int score, int always, const int *token_seq, int *pair_expert,
                             float *pair_weight, const float *correction, float weight_scale, int n_real, const float *bias,
                             float *shared_weight, void *stream) {
    if (n_tokens <= 0) return 0;
    if (top < 1 || top > experts) ABK_REFUSE("moe_route: %d of %d experts", top, experts);
    if (score < 0 || score > 2) ABK_REFUSE("moe_route: score %d is not built", score);
    if (n_real < 0 || n_real > experts) n_real = experts;
    const size_t token = (size_t)(((d + 3) & ~3) + 3 * experts + 1) * 4;
    if (token > 200 * 1024) ABK_REFUSE("moe_route: a row of %d and %d experts do not fit shared memory", d, experts);
    const bool four = n_tokens >= 4 * abk_sm_count() && 4 * token <= 100 * 1024;
    const size_t smem = four ? 4 * token : token;
    cudaStream_t s = (cudaStream_t)stream;
#define MR_LAUNCH(T, TOKENS)                                                                                                    \
    do {                                                                                                                        \
        if (smem > 48 * 1024) {                                                                                                 \
            cudaError_t e = abk_allow_shared_memory((const void *)moe_route_kernel<T, TOKENS>, (int)smem);                      \
            if (e != cudaSuccess) return (int)e;                                                                                \
        }                                                                                                                       \
        abk_launch(moe_route_kernel<T, TOKENS>, dim3((n_tokens + TOKENS - 1) / TOKENS), dim3(MR_THREADS), smem, s, (const T *)x, ldx, \
                   router, n_tokens, d, experts, top, score, always, token_seq, pair_expert, pair_weight, correction, weight_scale, \
                   n_real, bias, shared_weight);                                                                                \
    } while (0)
    if (dtype == ABK_BF16) { if (four) MR_LAUNCH(__nv_bfloat16, 4); else MR_LAUNCH(__nv_bfloat16, 1); }
    else { if (four) MR_LAUNCH(float, 4); else MR_LAUNCH(float, 1); }
#undef MR_LAUNCH
    return ABK_LAUNCH_RESULT();
}

#define RP_PER_WARP 4
// gated: w has 2 * outs rows a matrix, gate and up rows in turns of `block`
enum { RP_NONE = 0, RP_RELU_SQUARED = 1, RP_SILU_GATED = 2, RP_CLAMPED_GATED = 3 };

template <typename T, typename TO, int ACT>
__global__ void __launch_bounds__(128) routed_product_kernel(const T *__restrict__ x, long long ldx, int pairs_per_row,
                                                             const T *__restrict__ w, const int *pair_expert,
                                                             const float *pair_scale, TO *__restrict__ out, long long ldo,
                                                             int in, int outs, int block, float limit) {
    constexpr bool GATED = ACT == RP_SILU_GATED || ACT == RP_CLAMPED_GATED;
    extern __shared__ __align__(16) float rp_x[];  // [in]
    const int pair = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    pdl_wait();
    const int e = pair_expert[pair];
    const int o0 = (blockIdx.y * 4 + warp) * RP_PER_WARP;
    if (e < 0) {  // a padding row
        if (lane < RP_PER_WARP && o0 + lane < outs) out[(long long)pair * ldo + o0 + lane] = from_float<TO>(0.0f);
        return;
    }
    const T *row = x + (long long)(pair / pairs_per_row) * ldx;
    if (pair_scale) {
        const float sc = pair_scale[pair];
        for (int i = threadIdx.x; i < in; i += 128) rp_x[i] = to_float(from_float<T>(sc * to_float(row[i])));
    } else {
        for (int i = threadIdx.x; i < in; i += 128) rp_x[i] = to_float(row[i]);
    }
    __syncthreads();
    if (o0 >= outs) return;
    // (a turn is a multiple of RP_PER_WARP rows, or all of them, so that a warp's gate rows lie together, and so its up rows)
    const T *wr = w + ((long long)e * (GATED ? 2 * outs : outs) + (GATED ? o0 / block * 2 * block + o0 % block : o0)) * in;
    const bool vec = in % (16 / (int)sizeof(T)) == 0 && ((uintptr_t)w & 15) == 0;
    float acc[RP_PER_WARP] = {0.0f, 0.0f, 0.0f, 0.0f};
    float up[RP_PER_WARP] = {0.0f, 0.0f, 0.0f, 0.0f};
    if (GATED) {
        const T *wu = wr + (long long)block * in;
        if (o0 + RP_PER_WARP <= outs) lane_dots<RP_PER_WARP>(wu, in, rp_x, in, lane, vec, up);
        else
            for (int u = 0; o0 + u < outs; u++) lane_dots<1>(wu + (long long)u * in, 0, rp_x, in, lane, vec, up + u);
    }
    if (o0 + RP_PER_WARP <= outs) lane_dots<RP_PER_WARP>(wr, in, rp_x, in, lane, vec, acc);  // four rows' loads in flight together
    else
        for (int u = 0; o0 + u < outs; u++) lane_dots<1>(wr + (long long)u * in, 0, rp_x, in, lane, vec, acc + u);
#pragma unroll
    for (int u = 0; u < RP_PER_WARP; u++) {
        float v = warp_sum(acc[u]);
        if (ACT == RP_RELU_SQUARED) v = v > 0.0f ? v * v : 0.0f;
        if (ACT == RP_SILU_GATED) {  // gate and up as stored tensors of the model's type, like the dense feed-forward's
            const float g = to_float(from_float<T>(v)), w_up = to_float(from_float<T>(warp_sum(up[u])));
            v = g / (1.0f + expf(-g)) * w_up;
        }
        if (ACT == RP_CLAMPED_GATED) {
            const float g = to_float(from_float<T>(v)), w_up = to_float(from_float<T>(warp_sum(up[u])));
            v = sizeof(T) == 2 ? gated_mul(ABK_CLAMPED, g, w_up, limit) : gated_mul_exact(ABK_CLAMPED, g, w_up, limit);
        }
        if (lane == 0 && o0 + u < outs) out[(long long)pair * ldo + o0 + u] = from_float<TO>(v);
    }
}

// x: the row of pair p is x + (p / pairs_per_row) * ldx (pairs_per_row 1: a row per pair; `top`: a row per token);
// w [experts][outs][in] of x's type (gated: [experts][2 * outs][in], gate and up rows in turns of `block`, a multiple of 4
// that divides outs, or outs itself); out [pairs][ldo] of x's type or (out_f32) float32. limit: of the clamped form.
extern "C" int abk_routed_product(const void *x, long long ldx, int pairs_per_row, int dtype, const void *w,
                                  const int *pair_expert, const float *pair_scale, void *out, long long ldo, int out_f32,
                                  int activation, int n_pairs, int in, int outs, int block, float limit, void *stream) {
    if (n_pairs <= 0 || outs <= 0) return 0;
    if (in < 1 || (size_t)in * 4 > 200 * 1024) ABK_REFUSE("routed_product: an inner size of %d does not fit shared memory", in);
    if (pairs_per_row < 1) pairs_per_row = 1;
    dim3 grid(n_pairs, (outs + 4 * RP_PER_WARP - 1) / (4 * RP_PER_WARP));
    if (grid.y > 65535) ABK_REFUSE("routed_product: %d output features are more than a grid takes", outs);
    const size_t smem = (size_t)in * 4;
    cudaStream_t s = (cudaStream_t)stream;
    typedef __nv_bfloat16 bf;
#define RP_LAUNCH(T, TO, ACT)                                                                                       \
    do {                                                                                                            \
        if (smem > 48 * 1024) {                                                                                     \
            cudaError_t e = abk_allow_shared_memory((const void *)routed_product_kernel<T, TO, ACT>, (int)smem);    \
            if (e != cudaSuccess) return (int)e;                                                                    \
        }                                                                                                           \
        abk_launch(routed_product_kernel<T, TO, ACT>, grid, dim3(128), smem, s, (const T *)x, ldx, pairs_per_row,   \
                   (const T *)w, pair_expert, pair_scale, (TO *)out, ldo, in, outs, block, limit);                                \
    } while (0)
    const bool gated = activation == RP_SILU_GATED || activation == RP_CLAMPED_GATED;
    if (activation < RP_NONE || activation > RP_CLAMPED_GATED) ABK_REFUSE("routed_product: activation %d is not built", activation);
    if (gated && (block <= 0 || outs % block || (block % RP_PER_WARP && block != outs)))
        ABK_REFUSE("routed_product: turns of %d rows do not fit %d features", block, outs);
#define RP_BY_ACT(T, TO)                                                                                             \
    do {                                                                                                            \
        if (activation == RP_CLAMPED_GATED) RP_LAUNCH(T, TO, RP_CLAMPED_GATED);                                     \
        else if (activation == RP_SILU_GATED) RP_LAUNCH(T, TO, RP_SILU_GATED);                                      \
        else if (activation == RP_RELU_SQUARED) RP_LAUNCH(T, TO, RP_RELU_SQUARED);                                  \
        else RP_LAUNCH(T, TO, RP_NONE);                                                                             \
    } while (0)
    if (dtype == ABK_BF16 && out_f32) RP_BY_ACT(bf, float);
    else if (dtype == ABK_BF16) RP_BY_ACT(bf, bf);
    else RP_BY_ACT(float, float);
#undef RP_BY_ACT
#undef RP_LAUNCH
    return ABK_LAUNCH_RESULT();
}

__global__ void __launch_bounds__(256) moe_combine_kernel(const float *pairs, float *out, long long total, int d, int top,
                                                          int add) {
    pdl_wait();
    const long long i = (long long)blockIdx.x * 256 + threadIdx.x;
    if (i >= total) return;
    const long long t = i / d, j = i - t * d;
    float acc = pairs[(t * top) * d + j];
    for (int k = 1; k < top; k++) acc += pairs[(t * top + k) * d + j];
    out[i] = add ? out[i] + acc : acc;
}

// out float32 [tokens][d]; pairs float32 [tokens * top][d]; add: out already holds what the pairs join (a shared expert).
extern "C" int abk_moe_combine(const float *pairs, float *out, int n_tokens, int d, int top, int add, void *stream) {
    const long long total = (long long)n_tokens * d;
    if (total <= 0) return 0;
    abk_launch(moe_combine_kernel, dim3((unsigned)((total + 255) / 256)), dim3(256), 0, (cudaStream_t)stream, pairs, out,
               total, d, top, add);
    return ABK_LAUNCH_RESULT();
}

// VEC: four columns a thread as one 16-byte piece (d a multiple of 4).
template <typename T, bool VEC>
__global__ void __launch_bounds__(256) moe_combine_weighted_kernel(const float *pairs, const float *weight, const int *expert,
                                                                   const T *x, long long ldx, float *out, long long total, int d,
                                                                   int top, const int *place, int shared, const float *shared_weight) {
    constexpr int W = VEC ? 4 : 1;
    pdl_wait();
    const long long i = ((long long)blockIdx.x * 256 + threadIdx.x) * W;
    if (i >= total) return;
    const long long t = i / d, j = i - t * d;
    float acc[W];
#pragma unroll
    for (int u = 0; u < W; u++) acc[u] = 0.0f;
    if (shared) {  // what a shared expert left in out
        const float sw = shared_weight ? shared_weight[t] : 1.0f;
        if (VEC) {
            const float4 r = *(const float4 *)(out + i);
            acc[0] = sw * r.x, acc[W > 1 ? 1 : 0] = sw * r.y, acc[W > 2 ? 2 : 0] = sw * r.z, acc[W > 3 ? 3 : 0] = sw * r.w;
        } else {
            acc[0] = sw * out[i];
        }
    }
    for (int k = 0; k < top; k++) {
        const int e = expert[t * top + k];
        if (e == -1) continue;  // a padding row
        const long long at = place && e >= 0 ? place[t * top + k] : t * top + k;  // rows sorted by expert: the pair's place
        const float w = weight[t * top + k];
        if (VEC && e >= 0) {
            const float4 r = *(const float4 *)(pairs + at * d + j);
            acc[0] = fmaf(w, r.x, acc[0]), acc[W > 1 ? 1 : 0] = fmaf(w, r.y, acc[W > 1 ? 1 : 0]);
            acc[W > 2 ? 2 : 0] = fmaf(w, r.z, acc[W > 2 ? 2 : 0]), acc[W > 3 ? 3 : 0] = fmaf(w, r.w, acc[W > 3 ? 3 : 0]);
        } else {
#pragma unroll
            for (int u = 0; u < W; u++) acc[u] = fmaf(w, e >= 0 ? pairs[at * d + j + u] : to_float(x[t * ldx + j + u]), acc[u]);
        }
    }
    if (VEC) *(float4 *)(out + i) = make_float4(acc[0], acc[W > 1 ? 1 : 0], acc[W > 2 ? 2 : 0], acc[W > 3 ? 3 : 0]);
    else out[i] = acc[0];
}

// out float32 [tokens][d] = sum_k weight[t, k] * (pairs[t * top + k], or x[t] where expert[t, k] <= -2). place (or null):
// pair p's row in `pairs` is place[p] (rows sorted by expert), not p. shared: out holds a shared expert's output, which
// joins the sum times shared_weight[t] (null: as it is).
extern "C" int abk_moe_combine_weighted(const float *pairs, const float *weight, const int *expert, const void *x, long long ldx,
                                        int dtype, float *out, int n_tokens, int d, int top, const int *place, int shared,
                                        const float *shared_weight, void *stream) {
    const long long total = (long long)n_tokens * d;
    if (total <= 0) return 0;
    const bool vec = d % 4 == 0 && (((uintptr_t)pairs | (uintptr_t)out) & 15) == 0;
    const unsigned blocks = (unsigned)((total / (vec ? 4 : 1) + 255) / 256);
#define MC_LAUNCH(T, VEC)                                                                                                       \
    abk_launch(moe_combine_weighted_kernel<T, VEC>, dim3(blocks), dim3(256), 0, (cudaStream_t)stream, pairs, weight, expert, \
               (const T *)x, ldx, out, total, d, top, place, shared, shared_weight)
    if (dtype == ABK_BF16) { if (vec) MC_LAUNCH(__nv_bfloat16, true); else MC_LAUNCH(__nv_bfloat16, false); }
    else { if (vec) MC_LAUNCH(float, true); else MC_LAUNCH(float, false); }
#undef MC_LAUNCH
    return ABK_LAUNCH_RESULT();
}

template <typename T> __global__ void __launch_bounds__(256) relu_squared_kernel(T *x, long long total) {
    pdl_wait();
    const long long i = (long long)blockIdx.x * 256 + threadIdx.x;
    if (i >= total) return;
    const float v = to_float(x[i]);
    x[i] = from_float<T>(v > 0.0f ? v * v : 0.0f);
}

extern "C" int abk_relu_squared(void *x, int dtype, long long total, void *stream) {
    if (total <= 0) return 0;
    const unsigned blocks = (unsigned)((total + 255) / 256);
    if (dtype == ABK_BF16) abk_launch(relu_squared_kernel<__nv_bfloat16>, dim3(blocks), dim3(256), 0, (cudaStream_t)stream, (__nv_bfloat16 *)x, total);
    else abk_launch(relu_squared_kernel<float>, dim3(blocks), dim3(256), 0, (cudaStream_t)stream, (float *)x, total);
    return ABK_LAUNCH_RESULT();
}

// ------------------------------------------------------------------ experts by a table
// A token's experts by its id: pair t * top + k is expert table[token[t]][k] with weight 1 / top. Rows of padding, tokens
// outside the table and entries that name no expert give -1 (no expert) and weight 0; the latter two set bit 0 of status.
__global__ void __launch_bounds__(256) moe_table_kernel(const int *tokens, const int *token_seq, const int *table, int vocab, int experts,
                                                        int top, int n_pairs, int *pair_expert, float *pair_weight, int *status) {
    pdl_wait();
    const int i = blockIdx.x * 256 + threadIdx.x;
    if (i >= n_pairs) return;
    const int t = i / top, k = i - t * top;
    int e = -1;
    if (token_seq[t] >= 0) {
        const int tok = tokens[t];
        if (tok >= 0 && tok < vocab) e = table[(long long)tok * top + k];
        if (e < 0 || e >= experts) {
            e = -1;
            atomicOr(status, 1);
        }
    }
    pair_expert[i] = e;
    pair_weight[i] = e >= 0 ? 1.0f / (float)top : 0.0f;
}

extern "C" int abk_moe_table(const int *tokens, const int *token_seq, const int *table, int vocab, int experts, int top,
                             int n_tokens, int *pair_expert, float *pair_weight, int *status, void *stream) {
    const long long n_pairs = (long long)n_tokens * top;
    if (n_pairs <= 0) return 0;
    if (n_pairs > 0x7fffffffLL) ABK_REFUSE("moe_table: %lld pairs are more than a grid takes", n_pairs);
    abk_launch(moe_table_kernel, dim3((unsigned)((n_pairs + 255) / 256)), dim3(256), 0, (cudaStream_t)stream, tokens, token_seq,
               table, vocab, experts, top, (int)n_pairs, pair_expert, pair_weight, status);
    return ABK_LAUNCH_RESULT();
}
