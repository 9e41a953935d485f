// Differential attention: a head has two maps, attentions of their own over the same values, and its output is
//   o = a1 - lambda * a2,   then   keep * o / sqrt(mean(o^2) + eps)   over the head's values, in float32.
#pragma once

struct DifferentialHead {
    float lambda;  // the second map's factor, one number a layer
    float eps;
    float keep;
};
__device__ __forceinline__ float differential_value(const DifferentialHead &d, float a1, float a2) { return fmaf(-d.lambda, a2, a1); }
// What a head's values are multiplied by, given the sum of their squares.
__device__ __forceinline__ float differential_scale(const DifferentialHead &d, float squares, int size) {
    return d.keep / sqrtf(squares / (float)size + d.eps);
}
