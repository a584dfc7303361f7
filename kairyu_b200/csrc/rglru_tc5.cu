// The gates of the real-gated linear recurrent unit for prompt portions, on the 5th-generation tensor cores (bfloat16 mode; rglru.cu
// says what is computed).
//
// A block owns 128 tokens of the step (whatever requests they belong to) and 64 channels of one part, both gates: the product is
// [128 tokens] x [64 rows of Wr | 64 rows of Wi], summed over the part's n inputs, one accumulator of 128 columns in tensor memory.
// The A operand is made here: per band of 64 inputs the 256 threads convolve (four tokens of eight channels each), split u into
// its rounding to bfloat16 and the rounding of the rest, and store both in the operand's swizzled layout; the weights' band comes by
// TMA.  Two stages: while the tensor cores work on one band, the threads make the next.  Behind the last band the sums go through
// shared memory to threads that have the channel's u again (the convolution once more) and form the decay and the input term.
//
// Every wait is bounded (umma.cuh); a block whose wait runs out raises its flag, waits for its copies in flight and frees its tensor memory.
#include "rglru.cuh"
#include "umma.cuh"

#define RT_THREADS 256
#define RT_TOKENS 128
#define RT_COLS 64  // channels a block
#define RT_BAND 64  // inputs a band

struct RtCfg {
    static constexpr int A_BYTES = RT_TOKENS * 128;      // one of u's two parts: 128 rows of 64 bfloat16
    static constexpr int B_BYTES = 2 * RT_COLS * 128;    // the rows of Wr, then those of Wi
    static constexpr int STAGE = 2 * A_BYTES + B_BYTES;
    static constexpr int PITCH = 68;                     // floats a row of the sums' staging
    static constexpr int OFF_BAR = 2 * STAGE;
    static constexpr int NUM_BARS = 5;                   // full[2], empty[2], done
    static constexpr size_t SMEM = 1024 + OFF_BAR + NUM_BARS * 8 + 16 + 3 * RT_TOKENS * 4;
    static constexpr int TMEM_COLUMNS = 128;
    static_assert(2 * RT_TOKENS * PITCH * 4 <= 2 * STAGE, "the sums' staging fits the stages");
};

// u of four consecutive tokens (rows r0 .. r0 + 3 of the block's tile) and eight channels from c on; KT: the taps, or 0 (any number)
template <int KT>
__device__ __forceinline__ void rt_convolve(const __nv_bfloat16* __restrict__ x, int stride, const float* __restrict__ rings, const RglruConv& conv,
                                            int tile0, int r0, const int* s_off, const int* s_pos, const int* s_slot, int c, float (&u)[4][8]) {
    const int taps = KT > 0 ? KT : conv.n_taps;
    {
        float b[8];
        *reinterpret_cast<float4*>(b) = *reinterpret_cast<const float4*>(conv.bias + c);
        *reinterpret_cast<float4*>(b + 4) = *reinterpret_cast<const float4*>(conv.bias + c + 4);
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
            for (int e = 0; e < 8; ++e) u[i][e] = b[e];
    }
    auto row8 = [&](int t) -> uint4 { return *reinterpret_cast<const uint4*>(x + (size_t)t * stride + c); };
    // the step's rows that these tokens and their taps may reach, fetched once (KT > 0)
    constexpr int SPAN = KT > 0 ? KT + 3 : 1;
    uint4 window[SPAN];
    if constexpr (KT > 0) {
#pragma unroll
        for (int i = 0; i < SPAN; ++i) {
            const int r = r0 + i - (KT - 1);
            const int t = tile0 + r;
            const bool in = t >= 0 && (r < RT_TOKENS ? (r < 0 || s_slot[r] >= 0) : false);
            window[i] = in ? row8(t) : make_uint4(0, 0, 0, 0);
        }
    }
#pragma unroll
    for (int k = 0; k < (KT > 0 ? KT : RG_MAX_TAPS); ++k) {  // oldest input first: the order of the taps
        if (k >= taps) break;
        const int back = taps - 1 - k;
        float w[8];
        *reinterpret_cast<float4*>(w) = *reinterpret_cast<const float4*>(conv.taps + (size_t)k * conv.W + c);
        *reinterpret_cast<float4*>(w + 4) = *reinterpret_cast<const float4*>(conv.taps + (size_t)k * conv.W + c + 4);
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const int r = r0 + i;
            const int slot = s_slot[r];
            if (slot < 0) continue;
            float in[8];
            if (s_off[r] >= back) {
                const uint4 raw = KT > 0 ? window[KT > 0 ? i + k : 0] : row8(tile0 + r - back);
                const __nv_bfloat162* two = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const float2 f = __bfloat1622float2(two[e]);
                    in[2 * e] = f.x;
                    in[2 * e + 1] = f.y;
                }
            } else if (s_pos[r] >= back) {
                const float* ring = rings + ((size_t)slot * conv.n_taps + (s_pos[r] - back) % conv.n_taps) * conv.W + c;
                *reinterpret_cast<float4*>(in) = *reinterpret_cast<const float4*>(ring);
                *reinterpret_cast<float4*>(in + 4) = *reinterpret_cast<const float4*>(ring + 4);
            } else {
                continue;  // before the sequence's start
            }
#pragma unroll
            for (int e = 0; e < 8; ++e) u[i][e] = fmaf(w[e], in[e], u[i][e]);
        }
    }
}

template <int KT>
__global__ void __launch_bounds__(RT_THREADS, 2)
rglru_gates_tc5_kernel(const __grid_constant__ CUtensorMap map_w, const __nv_bfloat16* __restrict__ x, int stride, const RglruConv conv,
                       const float* __restrict__ rings, const int* __restrict__ row_ids, const int* __restrict__ qo_indptr,
                       const int* __restrict__ positions, const int* __restrict__ state_slots, const float* __restrict__ gate_bias,
                       const float* __restrict__ rate, int parts, int n, int np, float* __restrict__ a_out, float* __restrict__ into_out,
                       int num_rows, int num_tokens, int* flag) {
    using Cfg = RtCfg;
    extern __shared__ unsigned char rt_smem[];
    unsigned char* base = reinterpret_cast<unsigned char*>(((uintptr_t)rt_smem + 1023) & ~(uintptr_t)1023);
    uint64_t* full = reinterpret_cast<uint64_t*>(base + Cfg::OFF_BAR);
    uint64_t* empty = full + 2;
    uint64_t* done = full + 4;
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(full + Cfg::NUM_BARS);
    volatile int* abort_word = reinterpret_cast<volatile int*>(tmem_slot + 1);
    int* s_off = reinterpret_cast<int*>(tmem_slot + 4);  // a token's place within its request's tokens of this step
    int* s_pos = s_off + RT_TOKENS;
    int* s_slot = s_pos + RT_TOKENS;                     // -1: no token

    const int W = parts * n;
    const int tiles = (n + RT_COLS - 1) / RT_COLS;
    const int part = blockIdx.x / tiles, col0 = (blockIdx.x % tiles) * RT_COLS;
    const int tile0 = blockIdx.y * RT_TOKENS;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int bands = (n + RT_BAND - 1) / RT_BAND;

    if (threadIdx.x == 0) {
        prefetch_tensormap(&map_w);
        mbar_init(full, 1);
        mbar_init(full + 1, 1);
        mbar_init(empty, 1);
        mbar_init(empty + 1, 1);
        mbar_init(done, 1);
        *abort_word = 0;
        asm volatile("fence.mbarrier_init.release.cluster;\n" ::: "memory");
    }
    if (warp == 1) tmem_alloc(tmem_slot, Cfg::TMEM_COLUMNS);
    if (threadIdx.x < RT_TOKENS) {
        const int t = tile0 + threadIdx.x;
        int off = 0, pos = 0, slot = -1;
        if (t < num_tokens) {
            const int row = row_ids[t];
            if (row < 0 || row >= num_rows) {
                if (flag) atomicOr(flag, KB_FLAG_BAD_ROW);
            } else {
                off = t - qo_indptr[row];
                pos = positions[t];
                slot = state_slots[row];
            }
        }
        s_off[threadIdx.x] = off;
        s_pos[threadIdx.x] = pos;
        s_slot[threadIdx.x] = slot;
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem_base = *tmem_slot;
    auto fetch_weights = [&](int band) {  // one thread
        unsigned char* b = base + (band & 1) * Cfg::STAGE + 2 * Cfg::A_BYTES;
        mbar_arrive_expect_tx(full + (band & 1), Cfg::B_BYTES);
        tma_load_2d_plain(b, &map_w, band * RT_BAND, part * np + col0, full + (band & 1));
        tma_load_2d_plain(b + RT_COLS * 128, &map_w, band * RT_BAND, (parts + part) * np + col0, full + (band & 1));
    };
    if (threadIdx.x == 0) {  // weights do not depend on the kernel before this one
        fetch_weights(0);
        if (bands > 1) fetch_weights(1);
    }
    pdl_wait();

    const int cg = threadIdx.x & 7, r0 = (threadIdx.x >> 3) * 4;  // this thread's eight channels and four tokens
    constexpr uint32_t idesc = umma_idesc(2 * RT_COLS);
    bool ok = true;
    for (int band = 0; band < bands; ++band) {
        const int s = band & 1;
        unsigned char* stage = base + s * Cfg::STAGE;
        if (band >= 2) {  // the products of the band before last have read this stage
            ok = mbar_wait(empty + s, ((band >> 1) - 1) & 1, abort_word);
            if (ok && threadIdx.x == 0) fetch_weights(band);
        }
        if (ok) {
            const int k = band * RT_BAND + cg * 8;
            float u[4][8];
            if (k < n) {
                rt_convolve<KT>(x, stride, rings, conv, tile0, r0, s_off, s_pos, s_slot, part * n + k, u);
            }
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const int r = r0 + i;
                uint32_t hi[4], lo[4];
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const bool in = k < n && s_slot[r] >= 0;
                    const float v0 = in ? u[i][2 * e] : 0.0f, v1 = in ? u[i][2 * e + 1] : 0.0f;
                    const __nv_bfloat162 h = __floats2bfloat162_rn(v0, v1);
                    const float2 back = __bfloat1622float2(h);
                    const __nv_bfloat162 l = __floats2bfloat162_rn(v0 - back.x, v1 - back.y);
                    hi[e] = *reinterpret_cast<const uint32_t*>(&h);
                    lo[e] = *reinterpret_cast<const uint32_t*>(&l);
                }
                const int at = r * 128 + ((cg ^ (r & 7)) << 4);
                *reinterpret_cast<uint4*>(stage + at) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
                *reinterpret_cast<uint4*>(stage + Cfg::A_BYTES + at) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
            }
            fence_proxy_async_smem();
        }
        if (__syncthreads_or(!ok)) {
            ok = false;
            break;
        }
        if (threadIdx.x == 0) {
            if (mbar_wait(full + s, (band >> 1) & 1, abort_word)) {
                tc_fence_after();
                const uint32_t a = smem_addr(stage), b = a + 2 * Cfg::A_BYTES;
#pragma unroll
                for (int kk = 0; kk < RT_BAND / 16; ++kk) {
                    const uint64_t b_desc = umma_desc_sw128(b + kk * 32);
                    umma_bf16(tmem_base, umma_desc_sw128(a + kk * 32), b_desc, idesc, (band > 0 || kk > 0) ? 1u : 0u);
                    umma_bf16(tmem_base, umma_desc_sw128(a + Cfg::A_BYTES + kk * 32), b_desc, idesc, 1u);
                }
                umma_commit(empty + s);
                if (band == bands - 1) umma_commit(done);
            } else {
                *abort_word = 1;  // the others leave at their next wait
            }
        }
    }
    if (ok) ok = mbar_wait(done, 0, abort_word);
    ok = !__syncthreads_or(!ok);
    if (ok) {
        tc_fence_after();
        // sums -> shared memory, a row a token: r's 64 columns, then i's (the stages are free: every product has read its operands)
        float* sums_r = reinterpret_cast<float*>(base);
        float* sums_i = sums_r + RT_TOKENS * Cfg::PITCH;
        {
            const int quarter = warp & 3, half = warp >> 2;
            const int row = quarter * 32 + lane;
            const uint32_t at = tmem_base + ((uint32_t)(quarter * 32) << 16) + half * 32;
            uint32_t v[32];
#pragma unroll
            for (int g = 0; g < 2; ++g) {
                tmem_load32_nowait(at + g * RT_COLS, v);
                tmem_wait_ld();
                float* dst = (g ? sums_i : sums_r) + row * Cfg::PITCH + half * 32;
#pragma unroll
                for (int e = 0; e < 8; ++e) *reinterpret_cast<uint4*>(dst + 4 * e) = make_uint4(v[4 * e], v[4 * e + 1], v[4 * e + 2], v[4 * e + 3]);
            }
        }
        tc_fence_before();
        __syncthreads();
        const int col = col0 + cg * 8;
        if (col < n) {
            const int c = part * n + col;
            float u[4][8];
            rt_convolve<KT>(x, stride, rings, conv, tile0, r0, s_off, s_pos, s_slot, c, u);
            float br[8], bi[8], rt[8];
#pragma unroll
            for (int e = 0; e < 8; e += 4) {
                *reinterpret_cast<float4*>(br + e) = *reinterpret_cast<const float4*>(gate_bias + c + e);
                *reinterpret_cast<float4*>(bi + e) = *reinterpret_cast<const float4*>(gate_bias + W + c + e);
                *reinterpret_cast<float4*>(rt + e) = *reinterpret_cast<const float4*>(rate + c + e);
            }
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const int r = r0 + i;
                if (s_slot[r] < 0) continue;
                float a[8], into[8];
#pragma unroll
                for (int e = 0; e < 8; e += 4) {
                    const float4 pr = *reinterpret_cast<const float4*>(sums_r + r * Cfg::PITCH + cg * 8 + e);
                    const float4 pi = *reinterpret_cast<const float4*>(sums_i + r * Cfg::PITCH + cg * 8 + e);
                    rglru_terms<false>(pr.x + br[e], pi.x + bi[e], rt[e], u[i][e], a[e], into[e]);
                    rglru_terms<false>(pr.y + br[e + 1], pi.y + bi[e + 1], rt[e + 1], u[i][e + 1], a[e + 1], into[e + 1]);
                    rglru_terms<false>(pr.z + br[e + 2], pi.z + bi[e + 2], rt[e + 2], u[i][e + 2], a[e + 2], into[e + 2]);
                    rglru_terms<false>(pr.w + br[e + 3], pi.w + bi[e + 3], rt[e + 3], u[i][e + 3], a[e + 3], into[e + 3]);
                }
                const size_t at = (size_t)(tile0 + r) * W + c;
#pragma unroll
                for (int e = 0; e < 8; e += 4) {
                    *reinterpret_cast<float4*>(a_out + at + e) = make_float4(a[e], a[e + 1], a[e + 2], a[e + 3]);
                    *reinterpret_cast<float4*>(into_out + at + e) = make_float4(into[e], into[e + 1], into[e + 2], into[e + 3]);
                }
            }
        }
    } else if (threadIdx.x == 0) {
        if (flag) atomicOr(flag, KB_FLAG_TIMEOUT);
        volatile int ignore = 0;  // copies in flight target this block's shared memory: one more short wait each
        for (int s = 0; s < 2; ++s) {
            mbar_wait(full + s, 0, &ignore, 1024);
            mbar_wait(full + s, 1, &ignore, 1024);
        }
    }
    tc_fence_before();
    __syncthreads();
    if (warp == 1) {
        tc_fence_after();
        tmem_dealloc(tmem_base, Cfg::TMEM_COLUMNS);
    }
}

// map_w: host pointer to a tensor map (gemm_tc5.cu: kb_tc5_encode_map) of the gates' matrices [2 * parts * np, np] (gate, part, out; in) with boxes of
// 64 rows; np: n rounded up to 16.  n and the packed rows in steps of eight columns, 16-byte aligned.
KB_EXPORT int kb_rglru_gates_tc5(const void* map_w, const void* x, int stride, const float* taps, const float* conv_bias, int n_taps, const float* rings,
                                 const int* row_ids, const int* qo_indptr, const int* positions, const int* state_slots, const float* gate_bias,
                                 const float* rate, int parts, int n, int np, float* a, float* into, int num_rows, int T, int* flag, cudaStream_t stream) {
    if (T == 0) return 0;
    if (!map_w || !x || !taps || !conv_bias || !row_ids || !qo_indptr || !positions || !state_slots || !gate_bias || !rate || !a || !into) return KB_ERR_NULL;
    if (n_taps < 1 || n_taps > RG_MAX_TAPS || parts < 1 || n < 8 || n % 8 != 0 || np < n || np % 16 != 0 || stride % 8 != 0) return KB_ERR_UNSUPPORTED_SIZE;
    if (n_taps > 1 && !rings) return KB_ERR_NULL;
    if (((uintptr_t)x | (uintptr_t)taps | (uintptr_t)conv_bias | (uintptr_t)rings | (uintptr_t)gate_bias | (uintptr_t)rate | (uintptr_t)a | (uintptr_t)into) % 16 != 0)
        return KB_ERR_BAD_ARG;
    const int token_tiles = (T + RT_TOKENS - 1) / RT_TOKENS;
    if (token_tiles > 65535) return KB_ERR_UNSUPPORTED_SIZE;
    const RglruConv conv = {taps, conv_bias, n_taps, parts * n};
    const dim3 grid(parts * ((n + RT_COLS - 1) / RT_COLS), token_tiles);
#define LAUNCH(KT)                                                                                                                          \
    do {                                                                                                                                    \
        const cudaError_t e = cudaFuncSetAttribute(rglru_gates_tc5_kernel<KT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)RtCfg::SMEM); \
        if (e != cudaSuccess) return (int)e;                                                                                                \
        kb_launch(rglru_gates_tc5_kernel<KT>, grid, dim3(RT_THREADS), RtCfg::SMEM, stream, *(const CUtensorMap*)map_w,                        \
                  (const __nv_bfloat16*)x, stride, conv, rings, row_ids, qo_indptr, positions, state_slots, gate_bias, rate, parts, n, np, a, into, \
                  num_rows, T, flag);                                                                                                        \
    } while (0)
    if (n_taps == 4) LAUNCH(4); else LAUNCH(0);
#undef LAUNCH
    return kb_launch_result();
}
