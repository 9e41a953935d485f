// What the bfloat16 kernels of attention without a softmax share (attention_sigmoid.cu has the formulas): a key's weight
// from its score, and a float32 number as three bfloat16 parts.
#pragma once
#include "common.cuh"

// The constants of a head's weights, in units of log2: with y = -log2(e) z, a = 1 / (1 + 2^y).
//   no cap:  y = plain * dot + slope * back + base
//   cap c:   c tanh(s / c) = c - 2 c / (1 + e^(2 s / c)), so  y = twice_cap / (1 + 2^(to_exp * dot)) + slope * back + base
// The exponentials and reciprocals are the special-function unit's (float32, a few units in the last place).
struct __align__(16) SigmoidHead {
    float to_exp, twice_cap, slope, base;
};
__device__ __forceinline__ SigmoidHead sigmoid_head(float scale, float cap, float slope, float shift) {
    const float l2e = 1.4426950408889634f;
    SigmoidHead c;
    const bool capped = cap > 0.0f;
    c.to_exp = capped ? 2.0f * l2e * scale / cap : -l2e * scale;
    c.twice_cap = 2.0f * l2e * cap;
    c.slope = slope * l2e;
    c.base = -shift * l2e - (capped ? l2e * cap : 0.0f);
    return c;
}
__device__ __forceinline__ float sfu_exp2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
__device__ __forceinline__ float sfu_inverse(float x) {
    float y;
    asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
// away: slope * back + base of the key, made by the caller (a multiply-add, or less where keys follow one another)
__device__ __forceinline__ float sigmoid_of(bool capped, const SigmoidHead &c, float dot, float away) {
    const float y = capped ? fmaf(c.twice_cap, sfu_inverse(1.0f + sfu_exp2(c.to_exp * dot)), away) : fmaf(c.to_exp, dot, away);
    return sfu_inverse(1.0f + sfu_exp2(y));
}

// Two float32 numbers as three bfloat16 numbers each that add up to them (their 24 bits), packed in pairs.
__device__ __forceinline__ void split3_pair(float x, float y, uint32_t *part) {
#pragma unroll
    for (int k = 0; k < 3; k++) {
        const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
        part[k] = *(const uint32_t *)&h;
        if (k < 2) x -= __low2float(h), y -= __high2float(h);
    }
}
