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
//   rglru_gates_tc5   (rglru_tc5.cu) the same on the 5th-generation tensor cores (bfloat16)
//   rglru_scan        the walk over each request's tokens, the gelu branch, S and the ring left updated.  A request's tokens may
//                     be cut into segments that warps walk side by side: each first finds what its segment does to S (a factor
//                     and an offset), the warps before it say what S it starts from, and it walks again.
//   rglru_step        a step of single tokens in one kernel, on tensor cores (bfloat16)
//
// On tensor cores u enters the gates' products as two bfloat16 numbers, its rounding and the rounding of what is left (sixteen
// bits of u and more), against weights that are bfloat16 as stored, with 32-bit sums.
#include "rglru.cuh"

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
        rglru_terms<true>(acc_r[j] + gate_bias[c], acc_i[j] + gate_bias[W + c], rate[c], u[(group + 4 * j) * n + col], a, into);
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

// ------------------------------------------------------------------ a step of single tokens
// A block owns 16 channels of one part, both gates: warps 0-3 the rows of r, 4-7 those of i, the four of a gate cut the sum over
// the part's n inputs in turns of 64.  The weight rows are the 16-row operand of mma.sync m16n8k16 and eight tokens its columns; a lane
// holds 16 consecutive inputs of a row and of a token, which feed four products (a sum's order of k is free as long as both
// agree).  The partial sums meet in shared memory in warp order, and 128 threads, one a (token, channel), finish: gates, S, gelu.
// w: [2, parts, np, np] (gate, part, out, in), zeros beyond n; np is n rounded up to 16.
struct RgReg8 {
    uint32_t r[8];
};
__device__ __forceinline__ RgReg8 rg_load32(const void* p) {
    RgReg8 v;
    asm volatile("ld.global.nc.v8.u32 {%0,%1,%2,%3,%4,%5,%6,%7}, [%8];\n"
                 : "=r"(v.r[0]), "=r"(v.r[1]), "=r"(v.r[2]), "=r"(v.r[3]), "=r"(v.r[4]), "=r"(v.r[5]), "=r"(v.r[6]), "=r"(v.r[7])
                 : "l"(p));
    return v;
}
__device__ __forceinline__ void rg_mma(float (&d)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
    asm volatile(
        "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
        : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
        : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}

#define RG_STEP_THREADS 256
#define RG_STEP_K 64

__global__ void __launch_bounds__(RG_STEP_THREADS)
rglru_step_kernel(const __nv_bfloat16* __restrict__ x, const __nv_bfloat16* __restrict__ y, int stride, const RglruConv conv, float* __restrict__ states,
                  float* __restrict__ rings, const int* __restrict__ row_ids, const int* __restrict__ positions, const int* __restrict__ state_slots,
                  const __nv_bfloat16* __restrict__ w, const float* __restrict__ gate_bias, const float* __restrict__ rate, int parts, int n, int np,
                  __nv_bfloat16* __restrict__ out, int num_rows, int num_tokens, int* flag) {
    extern __shared__ __align__(16) unsigned char rg_smem[];
    const int pitch = np + 8;  // elements between tokens: 16-byte aligned, off a multiple of the banks
    __nv_bfloat16* hi = reinterpret_cast<__nv_bfloat16*>(rg_smem);  // [8][pitch]
    __nv_bfloat16* lo = hi + 8 * pitch;
    __shared__ float partial[8][16][9];
    __shared__ float own[8][16];  // u of the block's channels
    __shared__ int s_slot[8], s_pos[8];
    const int tiles = (np + 15) / 16;
    const int part = blockIdx.x / tiles, col0 = (blockIdx.x % tiles) * 16;
    const int W = parts * n;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int g = lane >> 2, tq = lane & 3;
    const int gate = warp >> 2, kwarp = warp & 3;
    const int steps = (np + RG_STEP_K - 1) / RG_STEP_K;
    RgReg8 zero;
#pragma unroll
    for (int i = 0; i < 8; ++i) zero.r[i] = 0u;
    const __nv_bfloat16* w_lo = w + ((size_t)(gate * parts + part) * np + col0 + g) * np;  // np is a multiple of 16: all 16 rows exist
    const __nv_bfloat16* w_hi = w_lo + (size_t)8 * np;
    auto load_weights = [&](int step, RgReg8& a, RgReg8& b) {
        const int k = step * RG_STEP_K + tq * 16;
        const bool in = k < np;
        a = in ? rg_load32(w_lo + k) : zero;
        b = in ? rg_load32(w_hi + k) : zero;
    };
    // the weights of this warp's first turn do not depend on the kernel before; with no more turns than warps they are all it needs
    RgReg8 first_lo, first_hi;
    load_weights(kwarp, first_lo, first_hi);
    pdl_wait();
    for (int t0 = blockIdx.y * 8; t0 < num_tokens; t0 += gridDim.y * 8) {
        if (threadIdx.x < 8) {
            const int t = t0 + threadIdx.x;
            int slot = -1, pos = 0;
            if (t < num_tokens) {
                const int row = row_ids[t];
                if (row < 0 || row >= num_rows) {
                    if (flag) atomicOr(flag, KB_FLAG_BAD_ROW);
                } else {
                    slot = state_slots[row];
                    pos = positions[t];
                }
            }
            s_slot[threadIdx.x] = slot;
            s_pos[threadIdx.x] = pos;
        }
        __syncthreads();  // (also: the tile before is done with the shared tiles)
        for (int idx = threadIdx.x; idx < 8 * np; idx += RG_STEP_THREADS) {
            const int m = idx / np, k = idx - m * np;
            float u = 0.0f;
            if (k < n && s_slot[m] >= 0) {
                const float* ring = rings ? rings + (size_t)s_slot[m] * conv.n_taps * W : nullptr;
                u = rglru_conv(x, stride, ring, conv, t0 + m, 0, s_pos[m], part * n + k);
            }
            const __nv_bfloat16 rounded = __float2bfloat16_rn(u);
            hi[m * pitch + k] = rounded;
            lo[m * pitch + k] = __float2bfloat16_rn(u - __bfloat162float(rounded));
            if (k >= col0 && k < col0 + 16) own[m][k - col0] = u;
        }
        __syncthreads();
        float acc[4] = {0.0f, 0.0f, 0.0f, 0.0f};
        for (int step = kwarp; step < steps; step += 4) {
            RgReg8 a = first_lo, b = first_hi;
            if (step != kwarp) load_weights(step, a, b);
            const int k = step * RG_STEP_K + tq * 16;
            uint32_t h[8], l[8];
            if (k < np) {
                *reinterpret_cast<uint4*>(h) = *reinterpret_cast<const uint4*>(hi + g * pitch + k);
                *reinterpret_cast<uint4*>(h + 4) = *reinterpret_cast<const uint4*>(hi + g * pitch + k + 8);
                *reinterpret_cast<uint4*>(l) = *reinterpret_cast<const uint4*>(lo + g * pitch + k);
                *reinterpret_cast<uint4*>(l + 4) = *reinterpret_cast<const uint4*>(lo + g * pitch + k + 8);
            } else {
#pragma unroll
                for (int i = 0; i < 8; ++i) h[i] = l[i] = 0u;
            }
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                rg_mma(acc, a.r[2 * j], b.r[2 * j], a.r[2 * j + 1], b.r[2 * j + 1], h[2 * j], h[2 * j + 1]);
                rg_mma(acc, a.r[2 * j], b.r[2 * j], a.r[2 * j + 1], b.r[2 * j + 1], l[2 * j], l[2 * j + 1]);
            }
        }
        partial[warp][g][2 * tq] = acc[0];
        partial[warp][g][2 * tq + 1] = acc[1];
        partial[warp][g + 8][2 * tq] = acc[2];
        partial[warp][g + 8][2 * tq + 1] = acc[3];
        __syncthreads();
        if (threadIdx.x < 128) {
            const int m = threadIdx.x >> 4, col = threadIdx.x & 15;
            const int t = t0 + m, c = part * n + col0 + col;
            if (s_slot[m] >= 0 && col0 + col < n) {
                float pre_r = gate_bias[c], pre_i = gate_bias[W + c];
#pragma unroll
                for (int k = 0; k < 4; ++k) {
                    pre_r += partial[k][col][m];
                    pre_i += partial[4 + k][col][m];
                }
                float a, into;
                rglru_terms<false>(pre_r, pre_i, rate[c], own[m][col], a, into);
                float* state = states + (size_t)s_slot[m] * W + c;
                const float S = fmaf(a, *state, into);
                *state = S;
                if (rings) rings[((size_t)s_slot[m] * conv.n_taps + s_pos[m] % conv.n_taps) * W + c] = __bfloat162float(x[(size_t)t * stride + c]);
                out[(size_t)t * W + c] = __float2bfloat16_rn(S * gelu_tanh_f(__bfloat162float(y[(size_t)t * stride + c])));
            }
        }
        __syncthreads();  // the next tile's slots and positions overwrite this one's
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

// A step whose rows carry one token each, bfloat16.  w: [2, parts, np, np] (gate, part, out, in), np a multiple of 16, 32-byte aligned.
KB_EXPORT int kb_rglru_step(const void* x, const void* y, int stride, const float* taps, const float* conv_bias, int n_taps, float* states, float* rings,
                            const int* row_ids, const int* positions, const int* state_slots, const void* w, const float* gate_bias, const float* rate,
                            int parts, int n, int np, void* out, int num_rows, int T, int* flag, cudaStream_t stream) {
    if (T == 0) return 0;
    if (!x || !y || !taps || !conv_bias || !states || !row_ids || !positions || !state_slots || !w || !gate_bias || !rate || !out) return KB_ERR_NULL;
    if (n_taps < 1 || n_taps > RG_MAX_TAPS || parts < 1 || n < 1 || np < n || np % 16 != 0 || np > 4096 || (uintptr_t)w % 32 != 0) return KB_ERR_UNSUPPORTED_SIZE;
    if (n_taps > 1 && !rings) return KB_ERR_NULL;
    const size_t smem = (size_t)2 * 8 * (np + 8) * sizeof(__nv_bfloat16);
    if (smem > 48 * 1024) {
        const cudaError_t e = cudaFuncSetAttribute(rglru_step_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return (int)e;
    }
    // blocks a token group: a few an SM in all, each walking its share of the token tiles
    const int blocks = parts * (np / 16), tiles = (T + 7) / 8;
    int groups = (4 * 148 + blocks - 1) / blocks;
    if (groups > tiles) groups = tiles;
    const RglruConv conv = {taps, conv_bias, n_taps, parts * n};
    kb_launch(rglru_step_kernel, dim3(blocks, groups), dim3(RG_STEP_THREADS), smem, stream, (const __nv_bfloat16*)x, (const __nv_bfloat16*)y, stride, conv,
              states, rings, row_ids, positions, state_slots, (const __nv_bfloat16*)w, gate_bias, rate, parts, n, np, (__nv_bfloat16*)out, num_rows, T, flag);
    return kb_launch_result();
}
