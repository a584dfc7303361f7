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
// Kernels, 32-bit mode:
//   rglru_gates       convolution and both gates on FMAs -> a and the input term, for every token of the step
//   rglru_scan        the walk over each request's tokens, the gelu branch, S and the ring left updated
// bfloat16 mode:
//   rglru_convolve    u of every token, as two bfloat16 planes: its rounding, and the rounding of what that leaves (sixteen bits of u and
//                     more); the gates' products take both planes against weights that are bfloat16 as stored, with 32-bit sums
//   rglru_gates_tc5   (rglru_tc5.cu) the gates of a step with prompt portions, on the 5th-generation tensor cores -> a and the input term
//   rglru_scan        as above; a request's tokens are cut into segments that warps walk side by side: each first finds what its segment
//                     does to S (a factor and an offset), those before it say what S it starts from, and it walks again
//   rglru_step        the gates and the recurrence of a step of single tokens in one kernel (mma.sync)
#include <cooperative_groups.h>

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
// grid (channel groups of 32 x the cluster's blocks, rows): a row's tokens are cut into (blocks of the cluster x warps of a block) segments,
// a warp a segment, a lane a channel.  One warp in one block: no segments, the plain walk.
#define RG_MAX_WARPS 16
#define RG_MAX_CLUSTER 8
#define RG_AHEAD 8  // tokens fetched ahead of their turn

template <typename T, bool EXACT>
__global__ void __launch_bounds__(32 * RG_MAX_WARPS)
rglru_scan_kernel(const float* __restrict__ a_in, const float* __restrict__ into_in, const T* __restrict__ x, const T* __restrict__ y, int stride, int W,
                  int n_taps, float* __restrict__ states, float* __restrict__ rings, const int* __restrict__ qo_indptr,
                  const int* __restrict__ positions, const int* __restrict__ state_slots, T* __restrict__ out) {
    namespace cg = cooperative_groups;
    __shared__ float seg_a[RG_MAX_WARPS][32], seg_b[RG_MAX_WARPS][32];
    __shared__ float block_a[32], block_b[32];  // what the block's segments together do to S
    cg::cluster_group cluster = cg::this_cluster();
    const int rank = (int)cluster.block_rank(), blocks = (int)cluster.num_blocks();
    const int row = blockIdx.y;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5;
    const int c = (blockIdx.x / blocks) * 32 + lane;
    const bool live = c < W;
    const int t0 = qo_indptr[row], t1 = qo_indptr[row + 1];
    const int slot = state_slots[row];
    pdl_wait();
    if (t0 >= t1) return;  // (the whole cluster)
    const int segments = warps * blocks;
    const int per = (t1 - t0 + segments - 1) / segments;
    const int s0 = min(t0 + (rank * warps + warp) * per, t1), s1 = min(s0 + per, t1);
    float S = live ? states[(size_t)slot * W + c] : 0.0f;
    if (segments > 1) {
        float A = 1.0f, B = 0.0f;
        if (live && s1 < t1) {  // what the last segment does to S nobody asks
            const float* ap = a_in + (size_t)s0 * W + c;
            const float* bp = into_in + (size_t)s0 * W + c;
            int left = s1 - s0;
            for (; left >= RG_AHEAD; left -= RG_AHEAD) {
                float av[RG_AHEAD], bv[RG_AHEAD];
#pragma unroll
                for (int j = 0; j < RG_AHEAD; ++j) {
                    av[j] = ap[(size_t)j * W];
                    bv[j] = bp[(size_t)j * W];
                }
                ap += (size_t)RG_AHEAD * W;
                bp += (size_t)RG_AHEAD * W;
#pragma unroll
                for (int j = 0; j < RG_AHEAD; ++j) {
                    B = fmaf(av[j], B, bv[j]);
                    A *= av[j];
                }
            }
            for (; left > 0; --left, ap += W, bp += W) {
                B = fmaf(*ap, B, *bp);
                A *= *ap;
            }
        }
        seg_a[warp][lane] = A;
        seg_b[warp][lane] = B;
        __syncthreads();
        if (blocks > 1) {
            if (warp == 0) {
                float a = 1.0f, b = 0.0f;
                for (int w = 0; w < warps; ++w) {
                    b = fmaf(seg_a[w][lane], b, seg_b[w][lane]);
                    a *= seg_a[w][lane];
                }
                block_a[lane] = a;
                block_b[lane] = b;
            }
            cluster.sync();  // (also: every block has read the state by now)
            for (int r = 0; r < rank; ++r) S = fmaf(cluster.map_shared_rank(block_a, r)[lane], S, cluster.map_shared_rank(block_b, r)[lane]);
        }
        for (int w = 0; w < warp; ++w) S = fmaf(seg_a[w][lane], S, seg_b[w][lane]);
    }
    if (live) {
        const float* ap = a_in + (size_t)s0 * W + c;
        const float* bp = into_in + (size_t)s0 * W + c;
        const T* yp = y + (size_t)s0 * stride + c;
        T* op = out + (size_t)s0 * W + c;
        int left = s1 - s0;
        for (; left >= RG_AHEAD; left -= RG_AHEAD) {
            float av[RG_AHEAD], bv[RG_AHEAD], yv[RG_AHEAD];
#pragma unroll
            for (int j = 0; j < RG_AHEAD; ++j) {
                av[j] = ap[(size_t)j * W];
                bv[j] = bp[(size_t)j * W];
                yv[j] = to_float(yp[(size_t)j * stride]);
            }
            ap += (size_t)RG_AHEAD * W;
            bp += (size_t)RG_AHEAD * W;
            yp += (size_t)RG_AHEAD * stride;
#pragma unroll
            for (int j = 0; j < RG_AHEAD; ++j) {
                S = fmaf(av[j], S, bv[j]);
                op[(size_t)j * W] = from_float<T>(S * gelu_tanh_f<EXACT>(yv[j]));
            }
            op += (size_t)RG_AHEAD * W;
        }
        for (; left > 0; --left, ap += W, bp += W, yp += stride, op += W) {
            S = fmaf(*ap, S, *bp);
            *op = from_float<T>(S * gelu_tanh_f<EXACT>(to_float(*yp)));
        }
        if (s0 < s1 && s1 == t1) {  // the segment that ends the row
            states[(size_t)slot * W + c] = S;
            if (rings) {
                float* ring = rings + (size_t)slot * n_taps * W;
                for (int t = max(t1 - n_taps, t0); t < t1; ++t) ring[(size_t)(positions[t] % n_taps) * W + c] = to_float(x[(size_t)t * stride + c]);
            }
        }
    }
    if (blocks > 1) cluster.sync();  // no block leaves while another may read its shared memory
}

// ------------------------------------------------------------------ the convolution alone (bfloat16)
// hi, lo: [tokens, parts * np], a part's n columns and zeros behind them (np: n rounded up to 16): u = hi + lo to sixteen bits and more.
// VEC: a thread takes eight channels of RG_CONV_TOKENS consecutive tokens; else one channel of one token.  `single`: every row
// carries one token; the kernel then also writes the token's input to its ring (a row none of its reads touches).
#define RG_CONV_TOKENS 2

__device__ __forceinline__ void rg_split(float u, __nv_bfloat16& hi, __nv_bfloat16& lo) {
    hi = __float2bfloat16_rn(u);
    lo = __float2bfloat16_rn(u - __bfloat162float(hi));
}

__device__ __forceinline__ void rg_floats8(const float* at, float (&v)[8]) {
    *reinterpret_cast<float4*>(v) = *reinterpret_cast<const float4*>(at);
    *reinterpret_cast<float4*>(v + 4) = *reinterpret_cast<const float4*>(at + 4);
}
__device__ __forceinline__ void rg_unpack8(const uint4& raw, float (&v)[8]) {
    const __nv_bfloat162* two = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
    for (int e = 0; e < 4; ++e) {
        const float2 f = __bfloat1622float2(two[e]);
        v[2 * e] = f.x;
        v[2 * e + 1] = f.y;
    }
}

// KT: the number of taps, or 0: any
template <bool VEC, int KT>
__global__ void __launch_bounds__(256)
rglru_convolve_kernel(const __nv_bfloat16* __restrict__ x, int stride, const RglruConv conv, float* rings, const int* __restrict__ row_ids,
                      const int* __restrict__ qo_indptr, const int* __restrict__ positions, const int* __restrict__ state_slots, int parts, int n, int np,
                      __nv_bfloat16* __restrict__ hi, __nv_bfloat16* __restrict__ lo, int single, int num_rows, int num_tokens, int* flag) {
    if (single) pdl_trigger();  // (few blocks; a portion's would make room for the next kernel's too early)
    constexpr int TOKENS = VEC ? RG_CONV_TOKENS : 1, CHANNELS = VEC ? 8 : 1;
    const int wide = parts * np, groups = wide / CHANNELS;
    const int taps = KT > 0 ? KT : conv.n_taps;
    const long long idx = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    const int at = (int)(idx % groups) * CHANNELS, first = (int)(idx / groups) * TOKENS;
    if (first >= num_tokens) return;
    const int part = at / np, k = at - part * np;
    const int c = part * n + k;
    int off[TOKENS], pos[TOKENS], slot[TOKENS];  // a token's place among its request's tokens of this step, its position, its request's slot
#pragma unroll
    for (int i = 0; i < TOKENS; ++i) {
        const int t = first + i;
        off[i] = pos[i] = 0;
        slot[i] = -1;
        if (t < num_tokens) {
            const int row = row_ids[t];
            if (row < 0 || row >= num_rows) {
                if (flag && at == 0) atomicOr(flag, KB_FLAG_BAD_ROW);
            } else {
                off[i] = t - qo_indptr[row];
                pos[i] = positions[t];
                slot[i] = state_slots[row];
            }
        }
    }
    pdl_wait();
    if constexpr (!VEC) {
        float u = 0.0f;
        if (k < n && slot[0] >= 0) {
            float* ring = rings ? rings + (size_t)slot[0] * taps * conv.W : nullptr;
            u = rglru_conv(x, stride, ring, conv, first, off[0], pos[0], c);
            if (single && ring) ring[(size_t)(pos[0] % taps) * conv.W + c] = __bfloat162float(x[(size_t)first * stride + c]);
        }
        rg_split(u, hi[(size_t)first * wide + at], lo[(size_t)first * wide + at]);
    } else {
        float u[TOKENS][8];
        if (k < n) {
            float b[8];
            rg_floats8(conv.bias + c, b);
#pragma unroll
            for (int i = 0; i < TOKENS; ++i)
#pragma unroll
                for (int e = 0; e < 8; ++e) u[i][e] = b[e];
            // the step's rows these tokens and their taps reach, fetched once (KT > 0); a row before the tokens may be another request's, and
            // is then not used
            constexpr int SPAN = KT > 0 ? KT + TOKENS - 1 : 1;
            uint4 window[SPAN];
            if constexpr (KT > 0) {
#pragma unroll
                for (int i = 0; i < SPAN; ++i) {
                    const int t = first + i - (KT - 1);
                    window[i] = t >= 0 && t < num_tokens ? *reinterpret_cast<const uint4*>(x + (size_t)t * stride + c) : make_uint4(0, 0, 0, 0);
                }
            }
#pragma unroll
            for (int j = 0; j < (KT > 0 ? KT : RG_MAX_TAPS); ++j) {  // oldest input first: the order of the taps
                if (j >= taps) break;
                const int back = taps - 1 - j;
                float w[8];
                rg_floats8(conv.taps + (size_t)j * conv.W + c, w);
#pragma unroll
                for (int i = 0; i < TOKENS; ++i) {
                    if (slot[i] < 0) continue;
                    float in[8];
                    if (off[i] >= back) {
                        rg_unpack8(KT > 0 ? window[KT > 0 ? i + j : 0] : *reinterpret_cast<const uint4*>(x + (size_t)(first + i - back) * stride + c), in);
                    } else if (pos[i] >= back) {
                        rg_floats8(rings + ((size_t)slot[i] * taps + (pos[i] - back) % taps) * conv.W + c, in);
                    } else {
                        continue;  // before the sequence's start
                    }
#pragma unroll
                    for (int e = 0; e < 8; ++e) u[i][e] = fmaf(w[e], in[e], u[i][e]);
                }
            }
            if (single && rings) {
#pragma unroll
                for (int i = 0; i < TOKENS; ++i) {
                    if (slot[i] < 0) continue;
                    float in[8];
                    rg_unpack8(*reinterpret_cast<const uint4*>(x + (size_t)(first + i) * stride + c), in);
                    float* ring = rings + ((size_t)slot[i] * taps + pos[i] % taps) * conv.W + c;
                    *reinterpret_cast<float4*>(ring) = make_float4(in[0], in[1], in[2], in[3]);
                    *reinterpret_cast<float4*>(ring + 4) = make_float4(in[4], in[5], in[6], in[7]);
                }
            }
        }
#pragma unroll
        for (int i = 0; i < TOKENS; ++i) {
            if (first + i >= num_tokens) break;
            __align__(16) __nv_bfloat16 h[8], l[8];
#pragma unroll
            for (int e = 0; e < 8; ++e) rg_split(k < n && slot[i] >= 0 ? u[i][e] : 0.0f, h[e], l[e]);
            *reinterpret_cast<uint4*>(hi + (size_t)(first + i) * wide + at) = *reinterpret_cast<const uint4*>(h);
            *reinterpret_cast<uint4*>(lo + (size_t)(first + i) * wide + at) = *reinterpret_cast<const uint4*>(l);
        }
    }
}

// ------------------------------------------------------------------ gates and recurrence of a step of single tokens
// A block owns 16 channels of one part, both gates: warps 0-3 the rows of r, 4-7 those of i, the four of a gate cut the sum over
// the part's inputs in turns of 64.  The weight rows are the 16-row operand of mma.sync m16n8k16 and eight tokens its columns; a lane
// holds 16 consecutive inputs of a row and of a token, which feed four products (a sum's order of k is free as long as both
// agree).  The partial sums meet in shared memory in warp order, and a thread a (token, channel) finishes: gates, S, gelu.
// w: [2, parts, np, np] (gate, part, out, in), zeros beyond n; hi, lo: [tokens, parts * np].
struct RgReg8 {
    uint32_t r[8];
};
__device__ __forceinline__ RgReg8 rg_load32(const void* p) {
    RgReg8 v;
    asm volatile("ld.global.v8.u32 {%0,%1,%2,%3,%4,%5,%6,%7}, [%8];\n"
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

// NT: tiles of eight tokens a turn
template <int NT>
__global__ void __launch_bounds__(RG_STEP_THREADS)
rglru_step_kernel(const __nv_bfloat16* __restrict__ hi, const __nv_bfloat16* __restrict__ lo, const __nv_bfloat16* __restrict__ y, int stride,
                  float* __restrict__ states, const int* __restrict__ row_ids, const int* __restrict__ state_slots, const __nv_bfloat16* __restrict__ w,
                  const float* __restrict__ gate_bias, const float* __restrict__ rate, int parts, int n, int np, __nv_bfloat16* __restrict__ out,
                  int num_rows, int num_tokens, int* flag) {
    __shared__ float partial[8][NT * 8][17];  // [warp][token][channel]
    const int tiles = np / 16;
    const int part = blockIdx.x / tiles, col0 = (blockIdx.x % tiles) * 16;
    const int W = parts * n, wide = parts * np;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int g = lane >> 2, tq = lane & 3;
    const int gate = warp >> 2, kwarp = warp & 3;
    const int steps = (np + RG_STEP_K - 1) / RG_STEP_K;
    RgReg8 zero;
#pragma unroll
    for (int i = 0; i < 8; ++i) zero.r[i] = 0u;
    const __nv_bfloat16* w_lo = w + ((size_t)(gate * parts + part) * np + col0 + g) * np;  // np is a multiple of 16: all 16 rows exist
    const __nv_bfloat16* w_hi = w_lo + (size_t)8 * np;
    // the weights of this warp's first turn do not depend on the kernel before; with no more turns than warps they are all it needs
    const bool any = kwarp * RG_STEP_K + tq * 16 < np;
    const RgReg8 first_lo = any ? rg_load32(w_lo + kwarp * RG_STEP_K + tq * 16) : zero;
    const RgReg8 first_hi = any ? rg_load32(w_hi + kwarp * RG_STEP_K + tq * 16) : zero;
    pdl_wait();
    for (int t0 = blockIdx.y * NT * 8; t0 < num_tokens; t0 += gridDim.y * NT * 8) {
        // what the finishing threads need, asked for ahead of the products
        constexpr int FINISH = (NT * 8 * 16 + RG_STEP_THREADS - 1) / RG_STEP_THREADS;
        float held_state[FINISH], held_y[FINISH], held_u[FINISH];
        float* where[FINISH];
#pragma unroll
        for (int f = 0; f < FINISH; ++f) {
            const int idx = f * RG_STEP_THREADS + threadIdx.x, m = idx >> 4, col = idx & 15, t = t0 + m, c = part * n + col0 + col;
            where[f] = nullptr;
            held_state[f] = held_y[f] = held_u[f] = 0.0f;
            if (m < NT * 8 && t < num_tokens && col0 + col < n) {
                const int row = row_ids[t];
                if (row < 0 || row >= num_rows) {
                    if (flag) atomicOr(flag, KB_FLAG_BAD_ROW);
                } else {
                    where[f] = states + (size_t)state_slots[row] * W + c;
                    held_state[f] = *where[f];
                    held_y[f] = __bfloat162float(y[(size_t)t * stride + c]);
                    const size_t at = (size_t)t * wide + part * np + col0 + col;
                    held_u[f] = __bfloat162float(hi[at]) + __bfloat162float(lo[at]);
                }
            }
        }
        float acc[NT][4];
#pragma unroll
        for (int tile = 0; tile < NT; ++tile) acc[tile][0] = acc[tile][1] = acc[tile][2] = acc[tile][3] = 0.0f;
        for (int step = kwarp; step < steps; step += 4) {
            const int k = step * RG_STEP_K + tq * 16;
            const bool in = k < np;
            RgReg8 a = first_lo, b = first_hi;
            if (step != kwarp) {
                a = in ? rg_load32(w_lo + k) : zero;
                b = in ? rg_load32(w_hi + k) : zero;
            }
            RgReg8 h[NT], l[NT];
#pragma unroll
            for (int tile = 0; tile < NT; ++tile) {
                const int t = t0 + tile * 8 + g;
                const bool both = in && t < num_tokens;
                const size_t at = (size_t)t * wide + part * np + k;
                h[tile] = both ? rg_load32(hi + at) : zero;
                l[tile] = both ? rg_load32(lo + at) : zero;
            }
#pragma unroll
            for (int j = 0; j < 4; ++j)
#pragma unroll
                for (int tile = 0; tile < NT; ++tile) {
                    rg_mma(acc[tile], a.r[2 * j], b.r[2 * j], a.r[2 * j + 1], b.r[2 * j + 1], h[tile].r[2 * j], h[tile].r[2 * j + 1]);
                    rg_mma(acc[tile], a.r[2 * j], b.r[2 * j], a.r[2 * j + 1], b.r[2 * j + 1], l[tile].r[2 * j], l[tile].r[2 * j + 1]);
                }
        }
        if (t0 != (int)blockIdx.y * NT * 8) __syncthreads();  // the turn before has been read
#pragma unroll
        for (int tile = 0; tile < NT; ++tile) {
            partial[warp][tile * 8 + 2 * tq][g] = acc[tile][0];
            partial[warp][tile * 8 + 2 * tq + 1][g] = acc[tile][1];
            partial[warp][tile * 8 + 2 * tq][g + 8] = acc[tile][2];
            partial[warp][tile * 8 + 2 * tq + 1][g + 8] = acc[tile][3];
        }
        __syncthreads();
#pragma unroll
        for (int f = 0; f < FINISH; ++f) {
            if (where[f] == nullptr) continue;
            const int idx = f * RG_STEP_THREADS + threadIdx.x, m = idx >> 4, col = idx & 15, t = t0 + m, c = part * n + col0 + col;
            float pre_r = gate_bias[c], pre_i = gate_bias[W + c];
#pragma unroll
            for (int k = 0; k < 4; ++k) {
                pre_r += partial[k][m][col];
                pre_i += partial[4 + k][m][col];
            }
            float a, into;
            rglru_terms<false>(pre_r, pre_i, rate[c], held_u[f], a, into);
            const float S = fmaf(a, held_state[f], into);
            *where[f] = S;
            out[(size_t)t * W + c] = __float2bfloat16_rn(S * gelu_tanh_f<false>(held_y[f]));
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

// warps (1 to 16) of each of `cluster` (1, 2, 4 or 8) blocks share a row's tokens; 1 and 1: the plain walk, in which a sum's order does not
// depend on where a prompt was cut.  Both 0: chosen from the width and the number of tokens.
KB_EXPORT int kb_rglru_scan(const float* a, const float* into, const void* x, const void* y, int stride, int is_bf16, int W, int n_taps,
                            float* states, float* rings, const int* qo_indptr, const int* positions, const int* state_slots, void* out, int num_rows,
                            int T, int warps, int cluster, cudaStream_t stream) {
    if (num_rows == 0) return 0;
    if (!a || !into || !x || !y || !states || !qo_indptr || !positions || !state_slots || !out) return KB_ERR_NULL;
    if (W < 1 || n_taps < 1 || n_taps > RG_MAX_TAPS || num_rows > 65535) return KB_ERR_BAD_ARG;
    if (n_taps > 1 && !rings) return KB_ERR_NULL;
    if (warps == 0 && cluster == 0) {
        // segments of sixteen tokens and more of an average row; blocks until there are two for most SMs (2,048 tokens: width 2,048 takes 27 us with
        // clusters of four, 33 of eight, 53 of one; width 4,096 45 with clusters of two, 49 of four, 61 of one)
        const int groups = (W + 31) / 32;
        long long segments = ((long long)T / num_rows + 15) / 16;
        warps = segments < 1 ? 1 : segments > RG_MAX_WARPS ? RG_MAX_WARPS : (int)segments;
        cluster = 1;
        while (cluster < RG_MAX_CLUSTER && segments >= 2 * cluster * warps && (long long)groups * num_rows * cluster * 2 <= 2 * 148) cluster *= 2;
    }
    if (warps < 1 || warps > RG_MAX_WARPS || cluster < 1 || cluster > RG_MAX_CLUSTER || (cluster & (cluster - 1)) != 0) return KB_ERR_BAD_ARG;
    cudaLaunchConfig_t config = {};
    config.gridDim = dim3(((W + 31) / 32) * cluster, num_rows);
    config.blockDim = dim3(32 * warps);
    config.stream = stream;
    cudaLaunchAttribute attributes[2];
    attributes[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attributes[0].val.programmaticStreamSerializationAllowed = 1;
    attributes[1].id = cudaLaunchAttributeClusterDimension;
    attributes[1].val.clusterDim.x = cluster;
    attributes[1].val.clusterDim.y = attributes[1].val.clusterDim.z = 1;
    config.attrs = attributes;
    config.numAttrs = 2;
    if (is_bf16)
        cudaLaunchKernelEx(&config, rglru_scan_kernel<__nv_bfloat16, false>, a, into, (const __nv_bfloat16*)x, (const __nv_bfloat16*)y, stride, W, n_taps, states,
                           rings, qo_indptr, positions, state_slots, (__nv_bfloat16*)out);
    else
        cudaLaunchKernelEx(&config, rglru_scan_kernel<float, true>, a, into, (const float*)x, (const float*)y, stride, W, n_taps, states, rings, qo_indptr,
                           positions, state_slots, (float*)out);
    return kb_launch_result();
}

// hi, lo: [T, parts * np] bfloat16; single: every row carries one token, and the rings are left updated
KB_EXPORT int kb_rglru_convolve(const void* x, int stride, const float* taps, const float* conv_bias, int n_taps, float* rings, const int* row_ids,
                                const int* qo_indptr, const int* positions, const int* state_slots, int parts, int n, int np, void* hi, void* lo, int single,
                                int num_rows, int T, int* flag, cudaStream_t stream) {
    if (T == 0) return 0;
    if (!x || !taps || !conv_bias || !row_ids || !qo_indptr || !positions || !state_slots || !hi || !lo) return KB_ERR_NULL;
    if (n_taps < 1 || n_taps > RG_MAX_TAPS || parts < 1 || n < 1 || np < n || np % 16 != 0) return KB_ERR_UNSUPPORTED_SIZE;
    if (n_taps > 1 && !rings) return KB_ERR_NULL;
    const RglruConv conv = {taps, conv_bias, n_taps, parts * n};
    const bool vec = n % 8 == 0 && stride % 8 == 0 &&
                     ((uintptr_t)x | (uintptr_t)taps | (uintptr_t)conv_bias | (uintptr_t)rings | (uintptr_t)hi | (uintptr_t)lo) % 16 == 0;
    const long long wide = (long long)parts * np;
    const long long items = vec ? (wide / 8) * ((T + RG_CONV_TOKENS - 1) / RG_CONV_TOKENS) : wide * T;
    const long long blocks = (items + 255) / 256;
    if (blocks > 0x7fffffffll) return KB_ERR_UNSUPPORTED_SIZE;
#define LAUNCH(VEC, KT)                                                                                                                       \
    kb_launch(rglru_convolve_kernel<VEC, KT>, dim3((unsigned)blocks), dim3(256), 0, stream, (const __nv_bfloat16*)x, stride, conv, rings, row_ids, qo_indptr, \
              positions, state_slots, parts, n, np, (__nv_bfloat16*)hi, (__nv_bfloat16*)lo, single, num_rows, T, flag)
    if (!vec) LAUNCH(false, 0); else if (n_taps == 4) LAUNCH(true, 4); else LAUNCH(true, 0);
#undef LAUNCH
    return kb_launch_result();
}

// The gates and the recurrence of a step whose rows carry one token each, bfloat16.  hi, lo: what kb_rglru_convolve left; w: [2, parts, np, np] (gate,
// part, out, in); np a multiple of 16, all three 32-byte aligned.
KB_EXPORT int kb_rglru_step(const void* hi, const void* lo, const void* y, int stride, float* states, const int* row_ids, const int* state_slots, const void* w,
                            const float* gate_bias, const float* rate, int parts, int n, int np, void* out, int num_rows, int T, int* flag,
                            cudaStream_t stream) {
    if (T == 0) return 0;
    if (!hi || !lo || !y || !states || !row_ids || !state_slots || !w || !gate_bias || !rate || !out) return KB_ERR_NULL;
    if (parts < 1 || n < 1 || np < n || np % 16 != 0 || ((uintptr_t)w | (uintptr_t)hi | (uintptr_t)lo) % 32 != 0) return KB_ERR_UNSUPPORTED_SIZE;
    // blocks a token group: a few an SM in all, each walking its share of the token tiles
    const int blocks = parts * (np / 16);
    const int turn = T <= 8 ? 8 : 32, turns = (T + turn - 1) / turn;
    int groups = (4 * 148 + blocks - 1) / blocks;
    if (groups > turns) groups = turns;
#define LAUNCH(NT)                                                                                                                             \
    kb_launch(rglru_step_kernel<NT>, dim3(blocks, groups), dim3(RG_STEP_THREADS), 0, stream, (const __nv_bfloat16*)hi, (const __nv_bfloat16*)lo,   \
              (const __nv_bfloat16*)y, stride, states, row_ids, state_slots, (const __nv_bfloat16*)w, gate_bias, rate, parts, n, np, (__nv_bfloat16*)out, \
              num_rows, T, flag)
    if (T <= 8) LAUNCH(1); else LAUNCH(4);
#undef LAUNCH
    return kb_launch_result();
}
