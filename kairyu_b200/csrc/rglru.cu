// The real-gated linear recurrent unit: per channel c of W and request one number S, kept in 32-bit and rewritten by
// every token,
//
//     u   = conv(x)                           a short causal convolution over time per channel, with a bias
//     r   = sigmoid(Wr_b u_b + br)            u in `parts` equal parts of n channels, one [n, n] matrix a part
//     i   = sigmoid(Wi_b u_b + bi)
//     la  = rate_c r                          rate_c = -8 softplus(lam_c), formed once at loading; log a = la
//     S   <- e^la S + sqrt(1 - e^(2 la)) i u
//     out = S gelu(y)                         y: the other branch of the packed projection [y | x]
//
// Everything between the projections and `out` is 32-bit.  What a request keeps: S [W], and the convolution's last inputs as
// a ring [taps, W]: the input of position p stands in row p % taps, so that a step of single tokens writes a row that
// none of its reads touches.
//
// Kernels:
//   rglru_gates       any size, FMA: convolution, both gates, -> a and the input term, for every token of the step
//   rglru_scan        the walk over each request's tokens, the gelu branch, S and the ring left updated.  A request's tokens may
//                     be cut into segments that warps walk side by side: each first finds what its segment does to S (a factor
//                     and an offset), the warps before it say what S it starts from, and it walks again.
//   rglru_step        a step of single tokens in one kernel, on tensor cores (bfloat16)
#include "common.cuh"
#include "linear_recurrence.cuh"

#define RG_MAX_TAPS 16

__device__ __forceinline__ float sigmoid_exact(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float gelu_tanh_f(float z) { return 0.5f * z * (1.0f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z))); }

// 1 - e^(-y) for y >= 0: the series of the exponential where the difference would cancel
__device__ __forceinline__ float one_minus_exp_neg(float y) {
    float p = -1.0f / 40320.0f;
    p = fmaf(p, y, 1.0f / 5040.0f);
    p = fmaf(p, y, -1.0f / 720.0f);
    p = fmaf(p, y, 1.0f / 120.0f);
    p = fmaf(p, y, -1.0f / 24.0f);
    p = fmaf(p, y, 1.0f / 6.0f);
    p = fmaf(p, y, -0.5f);
    p = fmaf(p, y, 1.0f);
    return y < 0.35f ? p * y : 1.0f - expf(-y);
}

// gate sums (biases added) and the convolved input of one channel -> the decay a and the input term
__device__ __forceinline__ void rglru_terms(float pre_r, float pre_i, float rate, float u, float& a, float& into) {
    const float la = rate * sigmoid_exact(pre_r);
    a = expf(la);
    into = sqrtf(one_minus_exp_neg(-2.0f * la)) * sigmoid_exact(pre_i) * u;
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

// ------------------------------------------------------------------ gates, any size
// grid (token tiles of RG_TOKENS, parts, column tiles of RG_COLS); w_t: [2, parts, n, n] as [gate][part][in][out], T's dtype
#define RG_TOKENS 16
#define RG_COLS 64

template <typename T>
__global__ void __launch_bounds__(256)
rglru_gates_kernel(const T* __restrict__ x, int stride, const RglruConv conv, const float* __restrict__ rings, const int* __restrict__ row_ids,
                   const int* __restrict__ qo_indptr, const int* __restrict__ positions, const int* __restrict__ state_slots,
                   const T* __restrict__ w_t, const float* __restrict__ gate_bias, const float* __restrict__ rate, int parts, int n,
                   float* __restrict__ a_out, float* __restrict__ into_out, int num_rows, int num_tokens, int* flag) {
    extern __shared__ float u[];  // [RG_TOKENS][n]
    const int W = parts * n;
    const int first = blockIdx.x * RG_TOKENS, part = blockIdx.y;
    pdl_wait();
    for (int idx = threadIdx.x; idx < RG_TOKENS * n; idx += blockDim.x) {
        const int t = first + idx / n, c = part * n + idx % n;
        float v = 0.0f;
        if (t < num_tokens) {
            const int row = row_ids[t];
            if (row < 0 || row >= num_rows) {
                if (flag) atomicOr(flag, KB_FLAG_BAD_ROW);
            } else {
                const float* ring = rings ? rings + (size_t)state_slots[row] * conv.n_taps * W : nullptr;
                v = rglru_conv(x, stride, ring, conv, t, t - qo_indptr[row], positions[t], c);
            }
        }
        u[idx] = v;
    }
    __syncthreads();
    const int col = blockIdx.z * RG_COLS + threadIdx.x % RG_COLS;  // column of the part
    const int group = threadIdx.x / RG_COLS;                       // its tokens: group, group + 4, ...
    if (col >= n) return;
    float acc_r[RG_TOKENS / 4], acc_i[RG_TOKENS / 4];
#pragma unroll
    for (int j = 0; j < RG_TOKENS / 4; ++j) acc_r[j] = acc_i[j] = 0.0f;
    const T* wr = w_t + (size_t)part * n * n + col;
    const T* wi = wr + (size_t)parts * n * n;
    for (int k = 0; k < n; ++k) {
        const float r = to_float(wr[(size_t)k * n]), i = to_float(wi[(size_t)k * n]);
#pragma unroll
        for (int j = 0; j < RG_TOKENS / 4; ++j) {
            const float v = u[(group + 4 * j) * n + k];
            acc_r[j] = fmaf(r, v, acc_r[j]);
            acc_i[j] = fmaf(i, v, acc_i[j]);
        }
    }
    const int c = part * n + col;
#pragma unroll
    for (int j = 0; j < RG_TOKENS / 4; ++j) {
        const int t = first + group + 4 * j;
        if (t >= num_tokens) break;
        float a, into;
        rglru_terms(acc_r[j] + gate_bias[c], acc_i[j] + gate_bias[W + c], rate[c], u[(group + 4 * j) * n + col], a, into);
        a_out[(size_t)t * W + c] = a;
        into_out[(size_t)t * W + c] = into;
    }
}

// ------------------------------------------------------------------ the walk
// grid (channel groups of 32, rows), a warp a segment of the row's tokens; one warp: no segments, the plain walk
#define RG_MAX_SEGMENTS 32
#define RG_AHEAD 8  // tokens fetched ahead of their turn

template <typename T>
__global__ void rglru_scan_kernel(const float* __restrict__ a_in, const float* __restrict__ into_in, const T* __restrict__ x, const T* __restrict__ y,
                                  int stride, int W, int n_taps, float* __restrict__ states, float* __restrict__ rings,
                                  const int* __restrict__ qo_indptr, const int* __restrict__ positions, const int* __restrict__ state_slots,
                                  T* __restrict__ out) {
    __shared__ float seg_a[RG_MAX_SEGMENTS][32], seg_b[RG_MAX_SEGMENTS][32];
    const int row = blockIdx.y;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, segments = blockDim.x >> 5;
    const int c = blockIdx.x * 32 + lane;
    const bool live = c < W;
    const int t0 = qo_indptr[row], t1 = qo_indptr[row + 1];
    const int slot = state_slots[row];
    pdl_wait();
    if (t0 >= t1) return;  // (the whole block)
    const int per = (t1 - t0 + segments - 1) / segments;
    const int s0 = min(t0 + warp * per, t1), s1 = min(s0 + per, t1);
    float S = live ? states[(size_t)slot * W + c] : 0.0f;
    if (segments > 1) {
        float A = 1.0f, B = 0.0f;
        if (live && s1 < t1) {  // what the last segment does to S nobody asks
            for (int t = s0; t < s1; t += RG_AHEAD) {
                float av[RG_AHEAD], bv[RG_AHEAD];
#pragma unroll
                for (int j = 0; j < RG_AHEAD; ++j) {
                    const bool in = t + j < s1;
                    av[j] = in ? a_in[(size_t)(t + j) * W + c] : 1.0f;
                    bv[j] = in ? into_in[(size_t)(t + j) * W + c] : 0.0f;
                }
#pragma unroll
                for (int j = 0; j < RG_AHEAD; ++j) {
                    B = fmaf(av[j], B, bv[j]);
                    A *= av[j];
                }
            }
        }
        seg_a[warp][lane] = A;
        seg_b[warp][lane] = B;
        __syncthreads();  // (every warp has read the state by now)
        for (int w = 0; w < warp; ++w) S = fmaf(seg_a[w][lane], S, seg_b[w][lane]);
    }
    if (!live) return;
    for (int t = s0; t < s1; t += RG_AHEAD) {
        float av[RG_AHEAD], bv[RG_AHEAD], yv[RG_AHEAD];
#pragma unroll
        for (int j = 0; j < RG_AHEAD; ++j) {
            const bool in = t + j < s1;
            av[j] = in ? a_in[(size_t)(t + j) * W + c] : 1.0f;
            bv[j] = in ? into_in[(size_t)(t + j) * W + c] : 0.0f;
            yv[j] = in ? to_float(y[(size_t)(t + j) * stride + c]) : 0.0f;
        }
#pragma unroll
        for (int j = 0; j < RG_AHEAD; ++j) {
            S = fmaf(av[j], S, bv[j]);
            if (t + j < s1) out[(size_t)(t + j) * W + c] = from_float<T>(S * gelu_tanh_f(yv[j]));
        }
    }
    if (s0 < s1 && s1 == t1) {  // the segment that ends the row
        states[(size_t)slot * W + c] = S;
        if (rings) {
            float* ring = rings + (size_t)slot * n_taps * W;
            for (int t = max(t1 - n_taps, t0); t < t1; ++t) ring[(size_t)(positions[t] % n_taps) * W + c] = to_float(x[(size_t)t * stride + c]);
        }
    }
}

// packed: [tokens, stride], columns [y | x] of W each.  rings: [slots, n_taps, W] (null with one tap); states: [slots, W].
// w_t: [2, parts, n, n] (gate, part, in, out); gate_bias: [2, W]; rate: [W]; a, into: scratch [tokens, W].
KB_EXPORT int kb_rglru_gates(const void* x, int stride, int is_bf16, const float* taps, const float* conv_bias, int n_taps, const float* rings,
                             const int* row_ids, const int* qo_indptr, const int* positions, const int* state_slots, const void* w_t,
                             const float* gate_bias, const float* rate, int parts, int n, float* a, float* into, int num_rows, int T, int* flag,
                             cudaStream_t stream) {
    if (T == 0) return 0;
    if (!x || !taps || !conv_bias || !row_ids || !qo_indptr || !positions || !state_slots || !w_t || !gate_bias || !rate || !a || !into) return KB_ERR_NULL;
    if (n_taps < 1 || n_taps > RG_MAX_TAPS || parts < 1 || parts > 65535 || n < 1) return KB_ERR_UNSUPPORTED_SIZE;
    if (n_taps > 1 && !rings) return KB_ERR_NULL;
    const size_t smem = (size_t)RG_TOKENS * n * sizeof(float);
    if (smem > 200 * 1024) return KB_ERR_UNSUPPORTED_SIZE;
    const RglruConv conv = {taps, conv_bias, n_taps, parts * n};
    const dim3 grid((T + RG_TOKENS - 1) / RG_TOKENS, parts, (n + RG_COLS - 1) / RG_COLS);
#define LAUNCH(TT)                                                                                                                     \
    do {                                                                                                                               \
        const cudaError_t e = cudaFuncSetAttribute(rglru_gates_kernel<TT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);     \
        if (e != cudaSuccess) return (int)e;                                                                                           \
        kb_launch(rglru_gates_kernel<TT>, grid, dim3(256), smem, stream, (const TT*)x, stride, conv, rings, row_ids, qo_indptr, positions, \
                  state_slots, (const TT*)w_t, gate_bias, rate, parts, n, a, into, num_rows, T, flag);                                  \
    } while (0)
    if (is_bf16) LAUNCH(__nv_bfloat16); else LAUNCH(float);
#undef LAUNCH
    return kb_launch_result();
}

// segments: 1 (the plain walk: a sum's order does not depend on where a prompt was cut) to 32
KB_EXPORT int kb_rglru_scan(const float* a, const float* into, const void* x, const void* y, int stride, int is_bf16, int W, int n_taps,
                            float* states, float* rings, const int* qo_indptr, const int* positions, const int* state_slots, void* out, int num_rows,
                            int segments, cudaStream_t stream) {
    if (num_rows == 0) return 0;
    if (!a || !into || !x || !y || !states || !qo_indptr || !positions || !state_slots || !out) return KB_ERR_NULL;
    if (W < 1 || n_taps < 1 || n_taps > RG_MAX_TAPS || segments < 1 || segments > RG_MAX_SEGMENTS || num_rows > 65535) return KB_ERR_BAD_ARG;
    if (n_taps > 1 && !rings) return KB_ERR_NULL;
    const dim3 grid((W + 31) / 32, num_rows), block(32 * segments);
    if (is_bf16)
        kb_launch(rglru_scan_kernel<__nv_bfloat16>, grid, block, 0, stream, a, into, (const __nv_bfloat16*)x, (const __nv_bfloat16*)y, stride, W,
                  n_taps, states, rings, qo_indptr, positions, state_slots, (__nv_bfloat16*)out);
    else
        kb_launch(rglru_scan_kernel<float>, grid, block, 0, stream, a, into, (const float*)x, (const float*)y, stride, W, n_taps, states, rings,
                  qo_indptr, positions, state_slots, (float*)out);
    return kb_launch_result();
}
