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

#define GR_THREADS 256      // of the scalar form
#define GR_VEC_THREADS 512  // of the vector form, at most: a row's loads are then all in flight at once up to 2,048 columns
#define GR_CHUNKS 4         // four-column groups a thread of the vector form keeps

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
    const void* bias;         // TB
    float mult;
    const void* w;            // TW
    float eps;
    const float* origin;
    void* out;                // TA
    int out_stride;
    const int* rows;
    int H;
};

// TY: the values' dtype, TA: the activations' (gate, extra, out), TB: gate bias, TW: norm weight
template <typename TY, typename TA, typename TB, typename TW>
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
    const TB* bias = (const TB*)p.bias;
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
            v += p.mult * gate_of(to_float(gate[(size_t)t * p.gate_stride + i]), bias ? to_float(bias[i]) : 0.0f) * y;
            if (!p.rows) xr[i] = v;
        }
        row[i] = v;
        ss += v * v;
    }
    const TW* w = (const TW*)p.w;
    const float inv = w ? rsqrtf(block_sum(ss, scratch) / (float)p.H + p.eps) : 1.0f;
    for (int i = threadIdx.x; i < p.H; i += GR_THREADS) {
        out[i] = from_float<TA>(w ? row[i] * inv * to_float(w[i]) : row[i]);
        if (p.origin) out[p.H + i] = from_float<TA>(p.origin[(size_t)t * p.H + i]);
    }
}

template <typename TY, typename TA, typename TB, typename TW>
__global__ void __launch_bounds__(GR_VEC_THREADS) gated_residual_norm_vec_kernel(const GatedSum p) {
    __shared__ float scratch[32];
    pdl_trigger();
    const int r = blockIdx.x;
    const int t = p.rows ? p.rows[r] : r;
    const int H = p.H;
    const TB* bias = (const TB*)p.bias;
    const TW* w = (const TW*)p.w;
    pdl_wait();
    const TY* values = (const TY*)p.values;
    TA* out = (TA*)p.out + (size_t)r * p.out_stride;
    float* xr = p.x + (size_t)t * H;
    float4 kept[GR_CHUNKS];
    float ss = 0.0f;
#pragma unroll
    for (int c = 0; c < GR_CHUNKS; ++c) {
        const int i = (c * (int)blockDim.x + threadIdx.x) * 4;
        if (i >= H) break;
        float4 v = load4(xr + i);
        if (values) {
            float4 y;
            if (p.mix) {
                y = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
#pragma unroll 4
                for (int k = 0; k < p.K; ++k) {
                    const size_t pair = (size_t)t * p.K + k;
                    const float m = p.mix[pair];
                    const float4 part = load4(values + (p.at ? (size_t)p.at[pair] : pair) * H + i);
                    y.x += m * part.x; y.y += m * part.y; y.z += m * part.z; y.w += m * part.w;
                }
                if (p.extra) {
                    const float4 e = load4((const TA*)p.extra + (size_t)t * H + i);
                    y.x += e.x; y.y += e.y; y.z += e.z; y.w += e.w;
                }
            } else {
                y = load4(values + (size_t)t * H + i);
            }
            const float4 g = load4((const TA*)p.gate + (size_t)t * p.gate_stride + i);
            const float4 b = bias ? load4(bias + i) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
            v.x += p.mult * gate_of(g.x, b.x) * y.x;
            v.y += p.mult * gate_of(g.y, b.y) * y.y;
            v.z += p.mult * gate_of(g.z, b.z) * y.z;
            v.w += p.mult * gate_of(g.w, b.w) * y.w;
            if (!p.rows) store4(xr + i, v);
        }
        kept[c] = v;
        ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
    }
    const float inv = w ? rsqrtf(block_sum(ss, scratch) / (float)H + p.eps) : 1.0f;
#pragma unroll
    for (int c = 0; c < GR_CHUNKS; ++c) {
        const int i = (c * (int)blockDim.x + threadIdx.x) * 4;
        if (i >= H) break;
        float4 v = kept[c];
        if (w) {
            const float4 n = load4(w + i);
            v = make_float4(v.x * inv * n.x, v.y * inv * n.y, v.z * inv * n.z, v.w * inv * n.w);
        }
        store4(out + i, v);
        if (p.origin) store4(out + H + i, load4(p.origin + (size_t)t * H + i));
    }
}

template <typename TY, typename TA>
static int launch_gated(const GatedSum& p, int R, int bias_bf16, int w_bf16, bool vec, cudaStream_t stream) {
    const size_t smem = vec ? 0 : (size_t)p.H * sizeof(float);
    const int wanted = (p.H / 4 + 31) / 32 * 32;
    const int threads = wanted > GR_VEC_THREADS ? GR_VEC_THREADS : wanted;
#define LAUNCH(TB, TW)                                                                                                          \
    do {                                                                                                                        \
        if (vec) kb_launch(gated_residual_norm_vec_kernel<TY, TA, TB, TW>, dim3(R), dim3(threads), smem, stream, p);              \
        else kb_launch(gated_residual_norm_kernel<TY, TA, TB, TW>, dim3(R), dim3(GR_THREADS), smem, stream, p);                   \
    } while (0)
    if (bias_bf16) {
        if (w_bf16) LAUNCH(__nv_bfloat16, __nv_bfloat16); else LAUNCH(__nv_bfloat16, float);
    } else {
        if (w_bf16) LAUNCH(float, __nv_bfloat16); else LAUNCH(float, float);
    }
#undef LAUNCH
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
    const GatedSum p = {x, values, mix, at, K, extra, gate, gate_stride, bias, mult, w, eps, origin, out, out_stride, rows, H};
    const uintptr_t all = (uintptr_t)x | (uintptr_t)values | (uintptr_t)extra | (uintptr_t)gate | (uintptr_t)bias | (uintptr_t)w | (uintptr_t)origin | (uintptr_t)out;
    const bool vec = H % 4 == 0 && H <= 4 * GR_CHUNKS * GR_VEC_THREADS && gate_stride % 4 == 0 && out_stride % 4 == 0 && all % 16 == 0;
    if (act_bf16) {
        if (values_bf16) return launch_gated<__nv_bfloat16, __nv_bfloat16>(p, R, bias_bf16, w_bf16, vec, stream);
        return launch_gated<float, __nv_bfloat16>(p, R, bias_bf16, w_bf16, vec, stream);
    }
    if (values_bf16) return KB_ERR_BAD_ARG;
    return launch_gated<float, float>(p, R, bias_bf16, w_bf16, vec, stream);
}
