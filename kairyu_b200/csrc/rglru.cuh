// What the kernels of the real-gated linear recurrent unit share: the short convolution over a step's rows and a request's ring of
// kept inputs, and the step from gate sums to a decay and an input term (rglru.cu says what is computed).
#pragma once
#include "common.cuh"

#define RG_MAX_TAPS 16

__device__ __forceinline__ float sigmoid_exact(float z) { return 1.0f / (1.0f + expf(-z)); }
// the same by the special-function unit's exponential, reciprocal and square root (a few ulp): the bfloat16 mode's kernels
__device__ __forceinline__ float ex2_fast(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;\n" : "=f"(y) : "f"(x));
    return y;
}
__device__ __forceinline__ float rcp_fast(float x) {
    float y;
    asm("rcp.approx.ftz.f32 %0, %1;\n" : "=f"(y) : "f"(x));
    return y;
}
__device__ __forceinline__ float sqrt_fast(float x) {
    float y;
    asm("sqrt.approx.ftz.f32 %0, %1;\n" : "=f"(y) : "f"(x));
    return y;
}
#define RG_LOG2E 1.4426950408889634f
__device__ __forceinline__ float sigmoid_fast(float z) { return rcp_fast(1.0f + ex2_fast(-RG_LOG2E * z)); }
// gelu in its tanh form, z (1 + tanh(w)) / 2 = z sigmoid(2 w)
template <bool EXACT>
__device__ __forceinline__ float gelu_tanh_f(float z) {
    const float w = 0.7978845608028654f * (z + 0.044715f * z * z * z);
    return EXACT ? 0.5f * z * (1.0f + tanhf(w)) : z * sigmoid_fast(2.0f * w);
}

// Gate sums (biases added) and the convolved input of one channel -> the decay a and the input term.  What matters of a decay close to
// one is its distance d = 1 - a from one: a rounding of a that leans one way is one of d multiplied by 1 / d, and every token of a long
// memory adds it again.  So d comes first, without the cancellation, a is 1 - d rounded once, and 1 - a^2 = d (2 - d).
template <bool EXACT>
__device__ __forceinline__ void rglru_terms(float pre_r, float pre_i, float rate, float u, float& a, float& into) {
    if (EXACT) {
        const float la = rate * sigmoid_exact(pre_r);
        const float d = -expm1f(la);
        a = la > -0.5f ? 1.0f - d : expf(la);
        into = sqrtf(d * (2.0f - d)) * sigmoid_exact(pre_i) * u;
    } else {
        const float x = -rate * sigmoid_fast(pre_r);
        // 1 - e^(-x), by its series while it is small (the first term left out is 2e-8 of the sum)
        float p = fmaf(x, 1.0f / 120.0f, -1.0f / 24.0f);
        p = fmaf(p, x, 1.0f / 6.0f);
        p = fmaf(p, x, -0.5f);
        p = fmaf(p, x, 1.0f);
        const float far = ex2_fast(-RG_LOG2E * x);
        const bool small = x < 0.1f;
        const float d = small ? p * x : 1.0f - far;
        a = small ? 1.0f - d : far;
        into = sqrt_fast(d * (2.0f - d)) * sigmoid_fast(pre_i) * u;
    }
}

struct RglruConv {
    const float* taps;  // [n_taps, W], oldest first
    const float* bias;  // [W]
    int n_taps, W;
};

// the convolved input of channel c of token t (position pos, offset o within its row's tokens); x: the step's rows of the
// x branch; ring: the request's kept inputs
template <typename T>
__device__ __forceinline__ float rglru_conv(const T* __restrict__ x, int stride, const float* __restrict__ ring, const RglruConv& conv,
                                            int t, int o, int pos, int c) {
    float z = conv.bias[c];
    for (int back = conv.n_taps - 1; back >= 0; --back) {
        if (pos - back < 0) continue;  // zeros before the start
        const float in = o - back >= 0 ? to_float(x[(size_t)(t - back) * stride + c]) : ring[(size_t)((pos - back) % conv.n_taps) * conv.W + c];
        z = fmaf(conv.taps[(size_t)(conv.n_taps - 1 - back) * conv.W + c], in, z);
    }
    return z;
}
