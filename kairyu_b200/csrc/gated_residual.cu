// The residual sum behind a gated sub-layer and the norm that reads the stream next, as one kernel:
//
//     y[t]   = values[t]                                                 or, for a mixture of experts before its sum,
//              sum_k mix[t, k] * values[at(t * K + k)] (+ extra[t])      in the order of k, 32-bit
//     x[t]  += mult * sigmoid(gate[t] + bias) * y[t]                     element by element (x: the fp32 residual stream)
//     out[r] = x[t] * rsqrt(mean(x[t]^2) + eps) * w                      (w null: x[t] itself, in the activation dtype)
//     out[r, H ..] = origin[t]                                           when `origin` (fp32 [T, H]) is given: the rows of a product
//                                                                        over the stream and the embedding output side by side
//
// for t = rows[r] (rows null: every row, and x is left updated; with rows x is not written: the listed rows' results are all
// that is wanted).  values null: nothing is added.  Sigmoid, sums, statistics and weights are 32-bit.  One block a row.
// The vector form handles four columns a thread a turn and keeps them in registers; which form runs depends on the width, the
// strides and the weights' alignment alone, never on the batch.
#include "common.cuh"

#define GR_THREADS 256
#define GR_CHUNKS 4  // four-column groups a thread of the vector form keeps at most: rows of up to 4 * 4 * 256 columns

__device__ __forceinline__ float4 load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 load4(const __nv_bfloat16* p) {
    const uint2 raw = *reinterpret_cast<const uint2*>(p);
    const float2 lo = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
    const float2 hi = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
    return make_float4(lo.x, lo.y, hi.x, hi.y);
}
__device__ __forceinline__ void store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void store4(__nv_bfloat16* p, float4 v) {
    const __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
    uint2 raw;
    raw.x = *reinterpret_cast<const unsigned*>(&lo);
    raw.y = *reinterpret_cast<const unsigned*>(&hi);
    *reinterpret_cast<uint2*>(p) = raw;
}
// a weight vector of either type
__device__ __forceinline__ float weight1(const void* p, int bf16, int i) {
    return bf16 ? to_float(((const __nv_bfloat16*)p)[i]) : ((const float*)p)[i];
}
__device__ __forceinline__ float4 weight4(const void* p, int bf16, int i) { return bf16 ? load4((const __nv_bfloat16*)p + i) : load4((const float*)p + i); }
__device__ __forceinline__ float gate_of(float g, float b) { return 1.0f / (1.0f + expf(-(g + b))); }

struct GatedSum {
    float* x;
    const void* values;       // TY
    const float* mix;         // null: plain rows
    const int* at;
    int K;
    const void* extra;        // TA
    const void* gate;         // TA
    int gate_stride;
    const void* bias;
    int bias_bf16;
    float mult;
    const void* w;
    int w_bf16;
    float eps;
    const float* origin;
    void* out;                // TA
    int out_stride;
    const int* rows;
    int H;
};

// TY: the values' dtype, TA: the activations' (gate, extra, out)
template <typename TY, typename TA>
__global__ void __launch_bounds__(GR_THREADS) gated_residual_norm_kernel(const GatedSum p) {
    extern __shared__ float row[];
    __shared__ float scratch[32];
    pdl_trigger();
    const int r = blockIdx.x;
    const int t = p.rows ? p.rows[r] : r;
    pdl_wait();
    const TY* values = (const TY*)p.values;
    const TA* gate = (const TA*)p.gate;
    const TA* extra = (const TA*)p.extra;
    const void* bias = p.bias;
    TA* out = (TA*)p.out + (size_t)r * p.out_stride;
    float* xr = p.x + (size_t)t * p.H;
    float ss = 0.0f;
    for (int i = threadIdx.x; i < p.H; i += GR_THREADS) {
        float v = xr[i];
        if (values) {
            float y;
            if (p.mix) {
                y = 0.0f;
                for (int k = 0; k < p.K; ++k) {
                    const size_t pair = (size_t)t * p.K + k;
                    y += p.mix[pair] * to_float(values[(p.at ? (size_t)p.at[pair] : pair) * p.H + i]);
                }
                if (extra) y += to_float(extra[(size_t)t * p.H + i]);
            } else {
                y = to_float(values[(size_t)t * p.H + i]);
            }
            v += p.mult * gate_of(to_float(gate[(size_t)t * p.gate_stride + i]), bias ? weight1(bias, p.bias_bf16, i) : 0.0f) * y;
            if (!p.rows) xr[i] = v;
        }
        row[i] = v;
        ss += v * v;
    }
    const void* w = p.w;
    const float inv = w ? rsqrtf(block_sum(ss, scratch) / (float)p.H + p.eps) : 1.0f;
    for (int i = threadIdx.x; i < p.H; i += GR_THREADS) {
        out[i] = from_float<TA>(w ? row[i] * inv * weight1(w, p.w_bf16, i) : row[i]);
        if (p.origin) out[p.H + i] = from_float<TA>(p.origin[(size_t)t * p.H + i]);
    }
}

// CHUNKS: four-column groups a thread keeps
template <typename TY, typename TA, int CHUNKS>
__global__ void __launch_bounds__(GR_THREADS) gated_residual_norm_vec_kernel(const GatedSum p) {
    __shared__ float scratch[32];
    pdl_trigger();
    const int r = blockIdx.x;
    const int t = p.rows ? p.rows[r] : r;
    const int H = p.H;
    const void* bias = p.bias;
    const void* w = p.w;
    pdl_wait();
    const TY* values = (const TY*)p.values;
    TA* out = (TA*)p.out + (size_t)r * p.out_stride;
    float* xr = p.x + (size_t)t * H;
    // every load of the row goes out before the first store, so that they are all in flight together
    float4 kept[CHUNKS], y[CHUNKS], g[CHUNKS];
#pragma unroll
    for (int c = 0; c < CHUNKS; ++c) {
        const int i = (c * GR_THREADS + threadIdx.x) * 4;
        if (i >= H) continue;
        kept[c] = load4(xr + i);
        if (values) {
            g[c] = load4((const TA*)p.gate + (size_t)t * p.gate_stride + i);
            if (!p.mix) y[c] = load4(values + (size_t)t * H + i);
        }
    }
    if (p.mix) {
#pragma unroll
        for (int c = 0; c < CHUNKS; ++c) y[c] = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
        for (int k0 = 0; k0 < p.K; k0 += 2) {  // two of the token's rows at a time, in the order of k
            const size_t pair = (size_t)t * p.K + k0;
            const bool second = k0 + 1 < p.K;
            const float m0 = p.mix[pair], m1 = second ? p.mix[pair + 1] : 0.0f;
            const TY* row0 = values + (p.at ? (size_t)p.at[pair] : pair) * H;
            const TY* row1 = second ? values + (p.at ? (size_t)p.at[pair + 1] : pair + 1) * H : row0;
#pragma unroll
            for (int c = 0; c < CHUNKS; ++c) {
                const int i = (c * GR_THREADS + threadIdx.x) * 4;
                if (i >= H) continue;
                const float4 a = load4(row0 + i), b = load4(row1 + i);
                y[c].x += m0 * a.x; y[c].y += m0 * a.y; y[c].z += m0 * a.z; y[c].w += m0 * a.w;
                if (second) { y[c].x += m1 * b.x; y[c].y += m1 * b.y; y[c].z += m1 * b.z; y[c].w += m1 * b.w; }
            }
        }
        if (p.extra) {
#pragma unroll
            for (int c = 0; c < CHUNKS; ++c) {
                const int i = (c * GR_THREADS + threadIdx.x) * 4;
                if (i >= H) continue;
                const float4 e = load4((const TA*)p.extra + (size_t)t * H + i);
                y[c].x += e.x; y[c].y += e.y; y[c].z += e.z; y[c].w += e.w;
            }
        }
    }
    float ss = 0.0f;
#pragma unroll
    for (int c = 0; c < CHUNKS; ++c) {
        const int i = (c * GR_THREADS + threadIdx.x) * 4;
        if (i >= H) continue;
        float4 v = kept[c];
        if (values) {
            const float4 b = bias ? weight4(bias, p.bias_bf16, i) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
            v.x += p.mult * gate_of(g[c].x, b.x) * y[c].x;
            v.y += p.mult * gate_of(g[c].y, b.y) * y[c].y;
            v.z += p.mult * gate_of(g[c].z, b.z) * y[c].z;
            v.w += p.mult * gate_of(g[c].w, b.w) * y[c].w;
            if (!p.rows) store4(xr + i, v);
        }
        kept[c] = v;
        ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
    }
    const float inv = w ? rsqrtf(block_sum(ss, scratch) / (float)H + p.eps) : 1.0f;
#pragma unroll
    for (int c = 0; c < CHUNKS; ++c) {
        const int i = (c * GR_THREADS + threadIdx.x) * 4;
        if (i >= H) continue;
        float4 v = kept[c];
        if (w) {
            const float4 n = weight4(w, p.w_bf16, i);
            v = make_float4(v.x * inv * n.x, v.y * inv * n.y, v.z * inv * n.z, v.w * inv * n.w);
        }
        store4(out + i, v);
        if (p.origin) store4(out + H + i, load4(p.origin + (size_t)t * H + i));
    }
}

template <typename TY, typename TA>
static int launch_gated(const GatedSum& p, int R, bool vec, cudaStream_t stream) {
    const int chunks = (p.H + 4 * GR_THREADS - 1) / (4 * GR_THREADS);
    if (!vec) kb_launch(gated_residual_norm_kernel<TY, TA>, dim3(R), dim3(GR_THREADS), (size_t)p.H * sizeof(float), stream, p);
    else if (chunks == 1) kb_launch(gated_residual_norm_vec_kernel<TY, TA, 1>, dim3(R), dim3(GR_THREADS), 0, stream, p);
    else if (chunks == 2) kb_launch(gated_residual_norm_vec_kernel<TY, TA, 2>, dim3(R), dim3(GR_THREADS), 0, stream, p);
    else kb_launch(gated_residual_norm_vec_kernel<TY, TA, GR_CHUNKS>, dim3(R), dim3(GR_THREADS), 0, stream, p);
    return kb_launch_result();
}

KB_EXPORT int kb_gated_residual_norm(float* x, const void* values, int values_bf16, const float* mix, const int* at, int K, const void* extra,
                                     const void* gate, int gate_stride, const void* bias, int bias_bf16, float mult, const void* w, int w_bf16,
                                     float eps, const float* origin, void* out, int out_stride, int act_bf16, const int* rows, int R, int H,
                                     cudaStream_t stream) {
    if (R == 0) return 0;
    if (!x || !out || (values && !gate)) return KB_ERR_NULL;
    if (H < 1 || H > 12000 || K < 1) return KB_ERR_UNSUPPORTED_SIZE;  // the scalar form keeps the row in 48 KB of shared memory
    if (out_stride < (origin ? 2 * H : H)) return KB_ERR_BAD_ARG;
    const GatedSum p = {x, values, mix, at, K, extra, gate, gate_stride, bias, bias_bf16, mult, w, w_bf16, eps, origin, out, out_stride, rows, H};
    const uintptr_t all = (uintptr_t)x | (uintptr_t)values | (uintptr_t)extra | (uintptr_t)gate | (uintptr_t)bias | (uintptr_t)w | (uintptr_t)origin | (uintptr_t)out;
    const bool vec = H % 4 == 0 && H <= 4 * GR_CHUNKS * GR_THREADS && gate_stride % 4 == 0 && out_stride % 4 == 0 && all % 16 == 0;
    if (act_bf16) {
        if (values_bf16) return launch_gated<__nv_bfloat16, __nv_bfloat16>(p, R, vec, stream);
        return launch_gated<float, __nv_bfloat16>(p, R, vec, stream);
    }
    if (values_bf16) return KB_ERR_BAD_ARG;
    return launch_gated<float, float>(p, R, vec, stream);
}
