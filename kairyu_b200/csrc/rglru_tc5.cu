// The gates of the real-gated linear recurrent unit for prompt portions, on the 5th-generation tensor cores (bfloat16 mode; rglru.cu
// says what is computed).
//
// A block owns 128 tokens of the step (whatever requests they belong to) and 64 channels of one part, both gates: the product is
// [128 tokens] x [64 rows of Wr | 64 rows of Wi], summed over the part's inputs, one accumulator of 128 columns in tensor memory.  The
// convolved inputs are two bfloat16 planes, u = hi + lo, and both are multiplied with the same weights into that accumulator.  One
// thread brings bands of 64 inputs (both planes' and the weights') by TMA through two stages, one issues the products, and then all
// 256 threads finish: the sums go through shared memory to threads that own four tokens of eight channels each and form the decay
// and the input term from them.  Columns of u beyond a part's width are the next part's: they meet weights that are zero.
//
// Every wait is bounded (umma.cuh); a block whose wait runs out raises its flag, waits for its copies in flight and frees its tensor memory.
#include "rglru.cuh"
#include "umma.cuh"

#define RT_THREADS 256
#define RT_TOKENS 128
#define RT_COLS 64  // channels a block
#define RT_BAND 64  // inputs a band

struct RtCfg {
    static constexpr int A_BYTES = RT_TOKENS * 128;      // one of u's two planes: 128 rows of 64 bfloat16
    static constexpr int B_BYTES = 2 * RT_COLS * 128;    // the rows of Wr, then those of Wi
    static constexpr int STAGE = 2 * A_BYTES + B_BYTES;
    static constexpr int PITCH = 68;                     // floats a row of the sums' staging
    static constexpr int OFF_BAR = 2 * STAGE;
    static constexpr int NUM_BARS = 5;                   // full[2], empty[2], done
    static constexpr size_t SMEM = 1024 + OFF_BAR + NUM_BARS * 8 + 16;
    static constexpr int TMEM_COLUMNS = 128;
    static_assert(2 * RT_TOKENS * PITCH * 4 <= 2 * STAGE, "the sums' staging fits the stages");
};

// VEC: a part's width is a multiple of eight, and so are a thread's channels all in or all out, in 16-byte groups
template <bool VEC>
__global__ void __launch_bounds__(RT_THREADS, 2)
rglru_gates_tc5_kernel(const __grid_constant__ CUtensorMap map_w, const __grid_constant__ CUtensorMap map_hi, const __grid_constant__ CUtensorMap map_lo,
                       const __nv_bfloat16* __restrict__ hi, const __nv_bfloat16* __restrict__ lo, const float* __restrict__ gate_bias,
                       const float* __restrict__ rate, int parts, int n, int np, float* __restrict__ a_out, float* __restrict__ into_out, int num_tokens,
                       int* flag) {
    using Cfg = RtCfg;
    extern __shared__ unsigned char rt_smem[];
    unsigned char* base = reinterpret_cast<unsigned char*>(((uintptr_t)rt_smem + 1023) & ~(uintptr_t)1023);
    uint64_t* full = reinterpret_cast<uint64_t*>(base + Cfg::OFF_BAR);
    uint64_t* empty = full + 2;
    uint64_t* done = full + 4;
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(full + Cfg::NUM_BARS);
    volatile int* abort_word = reinterpret_cast<volatile int*>(tmem_slot + 1);

    const int W = parts * n, wide = parts * np;
    const int tiles = (n + RT_COLS - 1) / RT_COLS;
    const int part = blockIdx.x / tiles, col0 = (blockIdx.x % tiles) * RT_COLS;
    const int tile0 = blockIdx.y * RT_TOKENS;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int bands = (np + RT_BAND - 1) / RT_BAND;

    if (threadIdx.x == 0) {
        prefetch_tensormap(&map_w);
        prefetch_tensormap(&map_hi);
        prefetch_tensormap(&map_lo);
        for (int i = 0; i < Cfg::NUM_BARS; ++i) mbar_init(full + i, 1);
        *abort_word = 0;
        asm volatile("fence.mbarrier_init.release.cluster;\n" ::: "memory");
    }
    if (warp == 1) tmem_alloc(tmem_slot, Cfg::TMEM_COLUMNS);
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem_base = *tmem_slot;
    if (warp == 0 && lane == 0) {
        // ---------------- copies
        auto weights = [&](int band) {
            unsigned char* b = base + (band & 1) * Cfg::STAGE + 2 * Cfg::A_BYTES;
            mbar_arrive_expect_tx(full + (band & 1), Cfg::STAGE);
            tma_load_2d_plain(b, &map_w, band * RT_BAND, part * np + col0, full + (band & 1));
            tma_load_2d_plain(b + RT_COLS * 128, &map_w, band * RT_BAND, (parts + part) * np + col0, full + (band & 1));
        };
        auto inputs = [&](int band) {
            unsigned char* a = base + (band & 1) * Cfg::STAGE;
            tma_load_2d_plain(a, &map_hi, part * np + band * RT_BAND, tile0, full + (band & 1));
            tma_load_2d_plain(a + Cfg::A_BYTES, &map_lo, part * np + band * RT_BAND, tile0, full + (band & 1));
        };
        weights(0);  // weights do not depend on the kernel before this one
        if (bands > 1) weights(1);
        pdl_wait();
        inputs(0);
        if (bands > 1) inputs(1);
        for (int band = 2; band < bands; ++band) {
            if (!mbar_wait(empty + (band & 1), ((band >> 1) - 1) & 1, abort_word)) {  // the products of the band before last have read the stage
                *abort_word = 1;
                break;
            }
            weights(band);
            inputs(band);
        }
    } else if (warp == 1 && lane == 0) {
        // ---------------- products
        constexpr uint32_t idesc = umma_idesc(2 * RT_COLS);
        bool ok = true;
        for (int band = 0; band < bands && ok; ++band) {
            const int s = band & 1;
            ok = mbar_wait(full + s, (band >> 1) & 1, abort_word);
            if (!ok) {
                *abort_word = 1;
                break;
            }
            tc_fence_after();
            const uint32_t a = smem_addr(base + s * Cfg::STAGE), b = a + 2 * Cfg::A_BYTES;
#pragma unroll
            for (int k = 0; k < RT_BAND / 16; ++k) {
                const uint64_t b_desc = umma_desc_sw128(b + k * 32);
                umma_bf16(tmem_base, umma_desc_sw128(a + k * 32), b_desc, idesc, (band > 0 || k > 0) ? 1u : 0u);
                umma_bf16(tmem_base, umma_desc_sw128(a + Cfg::A_BYTES + k * 32), b_desc, idesc, 1u);
            }
            umma_commit(empty + s);
        }
        if (ok) umma_commit(done);
    }
    __syncwarp();
    pdl_wait();
    const int cg = threadIdx.x & 7, r0 = (threadIdx.x >> 3) * 4;  // this thread's eight channels and four tokens
    const int col = col0 + cg * 8, c = part * n + col;
    // u of its channels, asked for while the products run
    uint4 uh[4], ul[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const bool in = col < n && tile0 + r0 + i < num_tokens;
        const size_t at = (size_t)(tile0 + r0 + i) * wide + part * np + col;
        uh[i] = in ? *reinterpret_cast<const uint4*>(hi + at) : make_uint4(0, 0, 0, 0);
        ul[i] = in ? *reinterpret_cast<const uint4*>(lo + at) : make_uint4(0, 0, 0, 0);
    }
    bool ok = mbar_wait(done, 0, abort_word);
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
        if (col < n) {
            float br[8], bi[8], rt[8];
#pragma unroll
            for (int e = 0; e < 8; ++e) {
                const bool in = VEC || col + e < n;
                br[e] = in ? gate_bias[c + e] : 0.0f;
                bi[e] = in ? gate_bias[W + c + e] : 0.0f;
                rt[e] = in ? rate[c + e] : 0.0f;
            }
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const int r = r0 + i;
                if (tile0 + r >= num_tokens) break;
                const __nv_bfloat162* h2 = reinterpret_cast<const __nv_bfloat162*>(&uh[i]);
                const __nv_bfloat162* l2 = reinterpret_cast<const __nv_bfloat162*>(&ul[i]);
                float a[8], into[8];
#pragma unroll
                for (int e = 0; e < 8; e += 2) {
                    const float2 h = __bfloat1622float2(h2[e / 2]), l = __bfloat1622float2(l2[e / 2]);
                    const float2 pr = *reinterpret_cast<const float2*>(sums_r + r * Cfg::PITCH + cg * 8 + e);
                    const float2 pi = *reinterpret_cast<const float2*>(sums_i + r * Cfg::PITCH + cg * 8 + e);
                    rglru_terms<false>(pr.x + br[e], pi.x + bi[e], rt[e], h.x + l.x, a[e], into[e]);
                    rglru_terms<false>(pr.y + br[e + 1], pi.y + bi[e + 1], rt[e + 1], h.y + l.y, a[e + 1], into[e + 1]);
                }
                const size_t at = (size_t)(tile0 + r) * W + c;
                if constexpr (VEC) {
#pragma unroll
                    for (int e = 0; e < 8; e += 4) {
                        *reinterpret_cast<float4*>(a_out + at + e) = make_float4(a[e], a[e + 1], a[e + 2], a[e + 3]);
                        *reinterpret_cast<float4*>(into_out + at + e) = make_float4(into[e], into[e + 1], into[e + 2], into[e + 3]);
                    }
                } else {
#pragma unroll
                    for (int e = 0; e < 8; ++e) {
                        if (col + e >= n) break;
                        a_out[at + e] = a[e];
                        into_out[at + e] = into[e];
                    }
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

// Host pointers to tensor maps (gemm_tc5.cu: kb_tc5_encode_map): map_w of the gates' matrices [2 * parts * np, np] (gate, part, out; in) with boxes of 64
// rows, map_hi and map_lo of the planes [T, parts * np] with boxes of 128 rows; hi and lo: the planes; np: n rounded up to 16.
KB_EXPORT int kb_rglru_gates_tc5(const void* map_w, const void* map_hi, const void* map_lo, const void* hi, const void* lo, const float* gate_bias,
                                 const float* rate, int parts, int n, int np, float* a, float* into, int T, int* flag, cudaStream_t stream) {
    if (T == 0) return 0;
    if (!map_w || !map_hi || !map_lo || !hi || !lo || !gate_bias || !rate || !a || !into) return KB_ERR_NULL;
    if (parts < 1 || n < 1 || np < n || np % 16 != 0 || ((uintptr_t)hi | (uintptr_t)lo) % 16 != 0) return KB_ERR_UNSUPPORTED_SIZE;
    const int token_tiles = (T + RT_TOKENS - 1) / RT_TOKENS;
    if (token_tiles > 65535) return KB_ERR_UNSUPPORTED_SIZE;
    const dim3 grid(parts * ((n + RT_COLS - 1) / RT_COLS), token_tiles);
#define LAUNCH(VEC)                                                                                                                            \
    do {                                                                                                                                       \
        const cudaError_t e = cudaFuncSetAttribute(rglru_gates_tc5_kernel<VEC>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)RtCfg::SMEM); \
        if (e != cudaSuccess) return (int)e;                                                                                                   \
        kb_launch(rglru_gates_tc5_kernel<VEC>, grid, dim3(RT_THREADS), RtCfg::SMEM, stream, *(const CUtensorMap*)map_w, *(const CUtensorMap*)map_hi, \
                  *(const CUtensorMap*)map_lo, (const __nv_bfloat16*)hi, (const __nv_bfloat16*)lo, gate_bias, rate, parts, n, np, a, into, T, flag); \
    } while (0)
    if (n % 8 == 0 && ((uintptr_t)a | (uintptr_t)into) % 16 == 0) LAUNCH(true); else LAUNCH(false);
#undef LAUNCH
    return kb_launch_result();
}
