// A soft cap on attention scores, s <- cap * tanh(s / cap), as the tensor-core attention kernels apply it: to the raw
// dot product q.k, together with the scale and the change to base 2, so that what comes out is what exp2 wants.
//
//   NONE   raw * scale * log2(e)
//   NEAR   raw * P(raw^2), P of degree 3: where |raw * scale / cap| is known to stay small (queries and keys of known
//          length), tanh(x) = x * p(x^2) with a polynomial that the host fits to that range in 64-bit; scale, cap and
//          log2(e) are in the coefficients.  Multiply-adds only: the special-function unit is left to the exponentials.
//   FULL   b - 2 b / (1 + 2^(a raw)), a = 2 scale log2(e) / cap, b = cap log2(e): tanh(x) = 1 - 2 / (1 + e^(2x)), any x
//          (2^(a raw) overflows to infinity where the result is b).  The cancellation near x = 0 leaves an absolute error
//          of an ulp of b.
#pragma once
#include "common.cuh"

#define KB_SOFTCAP_NONE 0
#define KB_SOFTCAP_NEAR 1
#define KB_SOFTCAP_FULL 2

// the host fills one of these in (kernels/__init__.py: SoftCap); entry points take a pointer to it, null: no cap
struct KbSoftcap {
    int mode;
    float a, b;
    float c[4];
};

static inline KbSoftcap kb_softcap_of(const void* host) {
    KbSoftcap none = {};
    return host ? *reinterpret_cast<const KbSoftcap*>(host) : none;
}

__device__ __forceinline__ float softcap_near(float raw, const KbSoftcap& cap) {
    const float z = raw * raw;
    return raw * fmaf(z, fmaf(z, fmaf(z, cap.c[3], cap.c[2]), cap.c[1]), cap.c[0]);
}

__device__ __forceinline__ float softcap_full(float raw, const KbSoftcap& cap) {
    return fmaf(-2.0f * cap.b, __fdividef(1.0f, 1.0f + exp2f(cap.a * raw)), cap.b);
}

// scale_log2: scale * log2(e), for the case without a cap
__device__ __forceinline__ float softcap_score(float raw, float scale_log2, const KbSoftcap& cap) {
    if (cap.mode == KB_SOFTCAP_NONE) return raw * scale_log2;
    return cap.mode == KB_SOFTCAP_NEAR ? softcap_near(raw, cap) : softcap_full(raw, cap);
}
