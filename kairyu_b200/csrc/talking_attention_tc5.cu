// Flash attention for prompt portions where all query heads of a position share ONE wide key row and take their values from
// their own key/value head, on the 5th-generation tensor cores: attention whose heads' scores are mixed before the softmax,
// the mix folded into the queries (talking_attention.cu):
//
//     S = Q K^T * scale      Q [tokens, H, G * D] mixed queries, K: the G key/value heads' keys of a position side by side
//     P = softmax rows online over the keys a query sees: itself and the window - 1 before it (window 0: all), and the
//         sequence's first keep_first tokens
//     O_h = P_h V_c(h)
//
// A block takes 128 / (H / G) queries of one key/value head: row r of its tile is query r / (H / G), head r % (H / G) of that
// key/value head's query heads, so the 128 rows of every product share one pass over keys and values.  Keys go in tiles of
// 64 at absolute multiples of 64: first the tiles of the kept first tokens, then those of the window.  The queries live in
// tensor memory (two bf16 columns a 32-bit one: 256 of its 512 columns for key rows of 512), which leaves the whole shared
// memory to the keys and values on their way.  Roles (288 threads):
//   warps 0-3  softmax: thread r owns row r; moves its queries from shared memory (where they lie in the keys' buffers before
//              the first keys do) into tensor memory, then reads its row of S from there, writes P as bf16 pairs over it, and
//              rescales O in tensor memory only when the row maximum has grown by more than 2^8 since the reference it scales by;
//   warps 4-7  producer: cp.async of a tile's keys or values into its buffer, each 16-byte group put where the 128-byte swizzle
//              of the tensor cores' operand wants it.  (A TMA copy brings a page's run of rows of one 64-column band: with pages
//              of 16 positions and wide keys that is 32 copies a tile beside those of the values, more than an SM can issue
//              beside the products; a thread's cp.async takes any page size, and pads columns up to 64 and rows beyond the
//              last key with zeros.)
//   warp 8     one thread issues tcgen05.mma: S (128 x 64, two buffers), O += P V.  Q K^T runs two tiles ahead of P V.
// A buffer holds a whole tile: with a barrier for every band of a tile the issuing thread spent 540 cycles a band of four
// products on waiting and committing, three times what the products take.
// The items are produced in the order the products consume them, K0 K1 V0 K2 V1 ..., and a producer warp that has to wait
// for a free buffer first reports everything it has issued, so no wait can be circular.
//
// Every wait on an mbarrier is bounded: a role that gives up raises KB_FLAG_TIMEOUT, the other roles leave through a shared
// abort word, and the block frees its tensor memory and returns.
// Sizes: D a multiple of 8 up to 128, G * D up to 512, H / G up to 128, any page size.
#include "umma.cuh"

#define TA_THREADS 288
#define TA_PRODUCERS 128
#define TA_BM 128
#define TA_BN 64
#define TA_BAND (TA_BN * 128)  // bytes of one 64-column band of 64 rows
#define TA_PASSES (TA_BN * 8 / TA_PRODUCERS)  // rows of a band a producer thread copies 16 bytes of
#define TA_MAX_BANDS 8
#define TA_K_STAGES 3          // the queries lie in the last two of them before the second tile's keys do
#define TA_V_STAGES 2
#define TA_LOG2E 1.4426950408889634f
#define TA_RESCALE_STEP 8.0f
#define TA_TMEM_COLUMNS 512
#define KB_FLAG_MISALIGNED 32

__device__ __forceinline__ float ta_ex2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;\n" : "=f"(y) : "f"(x));
    return y;
}
__device__ __forceinline__ bool ta_ready(uint64_t* bar, uint32_t parity) {
    uint32_t done;
    asm volatile("{\n .reg .pred p;\n mbarrier.test_wait.parity.shared::cta.b64 p, [%1], %2;\n selp.u32 %0, 1, 0, p;\n}\n"
                 : "=r"(done)
                 : "r"(smem_addr(bar)), "r"(parity)
                 : "memory");
    return done != 0;
}
__device__ __forceinline__ void ta_copy16(uint32_t dst, const void* src, bool valid) {
    const int bytes = valid ? 16 : 0;  // 0: the 16 bytes are filled with zeros and nothing is read
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"(dst), "l"(src), "r"(bytes) : "memory");
}
__device__ __forceinline__ void ta_commit() { asm volatile("cp.async.commit_group;\n" ::: "memory"); }
template <int N>
__device__ __forceinline__ void ta_wait() { asm volatile("cp.async.wait_group %0;\n" ::"n"(N) : "memory"); }

template <int VB>  // 64-column bands of a value row
__global__ void __launch_bounds__(TA_THREADS, 1)
talking_attention_tc5_kernel(const __nv_bfloat16* __restrict__ q, int q_stride, __nv_bfloat16* __restrict__ out, int out_stride,
                             const __nv_bfloat16* __restrict__ k_cache, const __nv_bfloat16* __restrict__ v_cache,
                             const int* __restrict__ qo_indptr, const int* __restrict__ seq_lens, const int* __restrict__ block_table,
                             int max_pages, const int* __restrict__ tile_rows, const int* __restrict__ tile_starts, int H, int G, int D,
                             int key_bands, int page_size, int page_shift, int num_pages, float scale, int window,
                             int keep_first, int* flag) {
    extern __shared__ __align__(1024) unsigned char smem[];
    const uint32_t k_bytes = key_bands * TA_BAND, v_bytes = VB * TA_BAND;
    unsigned char* sV = smem + TA_K_STAGES * k_bytes;
    uint64_t* bars = reinterpret_cast<uint64_t*>(sV + TA_V_STAGES * v_bytes);
    uint64_t* k_full = bars;
    uint64_t* k_empty = k_full + TA_K_STAGES;
    uint64_t* v_full = k_empty + TA_K_STAGES;
    uint64_t* v_empty = v_full + TA_V_STAGES;
    uint64_t* q_loaded = v_empty + TA_V_STAGES;  // the queries lie in shared memory
    uint64_t* q_stored = q_loaded + 1;           // ... and in tensor memory
    uint64_t* s_full = q_stored + 1;             // one per S buffer
    // two each, used in turn: the softmax may be a tile ahead of the products, and a barrier whose phase is told by its
    // parity cannot be two phases ahead of who waits on it
    uint64_t* p_full = s_full + 2;
    uint64_t* pv_done = p_full + 2;
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(pv_done + 2);
    volatile int* abort_word = reinterpret_cast<volatile int*>(tmem_slot + 1);
    // tensor memory: two S buffers of 64 columns (P, bf16 pairs, overwrites the first half of its S), O, the queries
    constexpr int S_COL = 0, O_COL = 2 * TA_BN, Q_COL = O_COL + VB * 64;

    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    if (threadIdx.x == 0) {
        for (int s = 0; s < TA_K_STAGES; ++s) {
            mbar_init(k_full + s, TA_PRODUCERS / 32);
            mbar_init(k_empty + s, 1);
        }
        for (int s = 0; s < TA_V_STAGES; ++s) {
            mbar_init(v_full + s, TA_PRODUCERS / 32);
            mbar_init(v_empty + s, 1);
        }
        mbar_init(q_loaded, TA_PRODUCERS / 32);
        mbar_init(q_stored, 4);
        for (int i = 0; i < 2; ++i) {
            mbar_init(s_full + i, 1);
            mbar_init(p_full + i, 4);
            mbar_init(pv_done + i, 1);
        }
        *abort_word = 0;
        if ((smem_addr(smem) & 1023u) != 0) {  // the swizzled layouts below assume it
            if (flag) atomicOr(flag, KB_FLAG_MISALIGNED);
            *abort_word = 1;
        }
        asm volatile("fence.mbarrier_init.release.cluster;\n" ::: "memory");
        fence_proxy_async_smem();
    }
    if (warp == 8) tmem_alloc(tmem_slot, TA_TMEM_COLUMNS);
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem_base = *tmem_slot;
    pdl_wait();

    // the tile: later tiles of a portion see more keys and go first
    const int group = H / G, kvh = blockIdx.x;
    const int per_tile = TA_BM / group;  // queries
    const int tile = (int)gridDim.y - 1 - (int)blockIdx.y;
    const int row = tile_rows[tile];
    const int q0 = tile_starts[tile];
    const int tok0 = qo_indptr[row];
    const int portion = qo_indptr[row + 1] - tok0;
    const int queries = min(per_tile, portion - q0);
    const int first_pos = seq_lens[row] - portion + q0;
    const int last_pos = first_pos + queries - 1;
    const int key_end = last_pos + 1;
    const int key_lo = (window > 0 && first_pos + 1 > window) ? first_pos + 1 - window : 0;
    const int first_kt = key_lo / TA_BN;
    const int kept_kt = min((min(keep_first, key_lo) + TA_BN - 1) / TA_BN, first_kt);  // tiles of kept tokens the window has passed
    const int num_kt = queries > 0 ? kept_kt + last_pos / TA_BN - first_kt + 1 : 0;
    auto key_of = [&](int n) { return (n < kept_kt ? n : first_kt + n - kept_kt) * TA_BN; };

    if (*abort_word || num_kt == 0) {
        // fall through to the common exit
    } else if (warp >= 4 && warp < 8) {
        // ---------------- producer: 8 lanes a row, 16 rows a pass
        const int tid = threadIdx.x - 128;
        const int chunk = tid & 7, row0 = tid >> 3;
        const int key_width = G * D;
        const uint32_t row_at = smem_addr(smem) + row0 * 128 + (uint32_t)((chunk ^ (row0 & 7)) * 16);  // a thread's rows are 16 apart: one swizzle
        const uint32_t v_at = row_at + TA_K_STAGES * k_bytes;
        const int* table = block_table + (size_t)row * max_pages;
        bool ok = true;
        uint64_t* older = nullptr;  // the barriers of the last two items issued, not reported yet
        uint64_t* newer = nullptr;
        auto report = [&](uint64_t* bar) {  // one arrival a warp
            __syncwarp();
            if (lane == 0 && bar) mbar_arrive(bar);
        };
        auto flush = [&]() {
            ta_wait<0>();
            fence_proxy_async_smem();
            report(older);
            report(newer);
            older = newer = nullptr;
        };
        auto wait_free = [&](uint64_t* bar, uint32_t parity) {
            if (__all_sync(0xffffffffu, ta_ready(bar, parity))) return true;
            flush();
            ok = __all_sync(0xffffffffu, mbar_wait(bar, parity, abort_word));
            if (!ok) {
                if (lane == 0 && !*abort_word && flag) atomicOr(flag, KB_FLAG_TIMEOUT);
                *abort_word = 1;
            }
            return ok;
        };
        auto end_item = [&](uint64_t* bar) {  // the copies issued since the last call belong to `bar`
            ta_commit();
            if (older) {
                ta_wait<2>();
                fence_proxy_async_smem();
                report(older);
            }
            older = newer;
            newer = bar;
        };
        // the queries: row r at r * bands * 128 bytes behind the first keys' buffer, a band's 16-byte groups turned by the row
        for (int r = row0; r < TA_BM; r += 16) {
            const int qi = r / group;
            const bool in_tile = qi < queries && r < per_tile * group;
            const __nv_bfloat16* src = q + (size_t)(tok0 + q0 + (in_tile ? qi : 0)) * q_stride + (size_t)(kvh * group + (in_tile ? r - qi * group : 0)) * key_width;
            const uint32_t dst = smem_addr(smem) + k_bytes + r * key_bands * 128 + (uint32_t)((chunk ^ (r & 7)) * 16);
            for (int b = 0; b < key_bands; ++b) {
                const int col = b * 64 + chunk * 8;
                const bool valid = in_tile && col < key_width;
                ta_copy16(dst + b * 128, src + (valid ? col : 0), valid);
            }
        }
        end_item(q_loaded);
        int place[TA_PASSES], place_before[TA_PASSES];
#pragma unroll
        for (int i = 0; i < TA_PASSES; ++i) place[i] = -1;
        int k_slot = 0, k_use = 0;
        for (int n = 0; n <= num_kt && ok; ++n) {
#pragma unroll
            for (int i = 0; i < TA_PASSES; ++i) place_before[i] = place[i];
            if (n < num_kt) {
                const int key0 = key_of(n);
#pragma unroll
                for (int i = 0; i < TA_PASSES; ++i) {
                    const int key = key0 + row0 + i * 16;
                    int at = -1;
                    if (key < key_end) {
                        const int page_index = page_shift >= 0 ? key >> page_shift : key / page_size;
                        const int page = page_index < max_pages ? table[page_index] : -1;  // -1: a page the window has given back
                        if (page >= 0 && page < num_pages) at = page * page_size + (key - page_index * page_size);
                    }
                    place[i] = at;
                }
                if (n == 1 && !wait_free(q_stored, 0)) break;  // the queries have left the buffers of the tiles after the first
                if (k_use > 0 && !wait_free(k_empty + k_slot, (k_use - 1) & 1)) break;
                for (int b = 0; b < key_bands; ++b) {
                    const int col = b * 64 + chunk * 8;
#pragma unroll
                    for (int i = 0; i < TA_PASSES; ++i) {
                        const bool valid = place[i] >= 0 && col < key_width;
                        ta_copy16(row_at + k_slot * k_bytes + b * TA_BAND + i * 2048, k_cache + (valid ? (size_t)place[i] * key_width + col : 0), valid);
                    }
                }
                end_item(k_full + k_slot);
                if (++k_slot == TA_K_STAGES) {
                    k_slot = 0;
                    ++k_use;
                }
            }
            if (n > 0) {  // the values of the tile before
                const int m = n - 1, v_slot = m % TA_V_STAGES;
                if (m >= TA_V_STAGES && !wait_free(v_empty + v_slot, (m / TA_V_STAGES - 1) & 1)) break;
#pragma unroll
                for (int b = 0; b < VB; ++b) {
                    const int col = b * 64 + chunk * 8;
#pragma unroll
                    for (int i = 0; i < TA_PASSES; ++i) {
                        const bool valid = place_before[i] >= 0 && col < D;
                        ta_copy16(v_at + v_slot * v_bytes + b * TA_BAND + i * 2048, v_cache + (valid ? (size_t)place_before[i] * key_width + kvh * D + col : 0), valid);
                    }
                }
                end_item(v_full + v_slot);
            }
        }
        flush();
    } else if (warp == 8) {
        // ---------------- products (one thread)
        if (lane == 0) {
            constexpr uint32_t idesc_qk = umma_idesc(TA_BN);
            constexpr uint32_t idesc_pv = umma_idesc_b_mn(VB * 64);
            const uint64_t k_desc = umma_desc_sw128(smem_addr(smem));
            const uint64_t v_desc = umma_desc_mn_sw128(smem_addr(sV), TA_BAND, 1024);
            bool ok = true;
            int k_slot = 0, k_use = 0;
            auto give_up = [&]() {
                if (!*abort_word && flag) atomicOr(flag, KB_FLAG_TIMEOUT);
                *abort_word = 1;
                ok = false;
            };
            auto issue_qk = [&](int n) {
                if (!mbar_wait(k_full + k_slot, k_use & 1, abort_word)) {
                    give_up();
                    return;
                }
                tc_fence_after();
                const uint64_t kb = k_desc + (uint64_t)((k_slot * k_bytes) >> 4);
                const uint32_t s_at = tmem_base + S_COL + (n & 1) * TA_BN, q_at = tmem_base + Q_COL;
#pragma unroll
                for (int b = 0; b < TA_MAX_BANDS; ++b)
                    if (b < key_bands) {
#pragma unroll
                        for (int k = 0; k < 4; ++k)  // 16 columns: 8 columns of the queries in tensor memory, 32 bytes along the keys' swizzled row
                            umma_bf16_a_tmem(s_at, q_at + b * 32 + k * 8, kb + (uint64_t)((b * TA_BAND + k * 32) >> 4), idesc_qk, (b > 0 || k > 0) ? 1u : 0u);
                    }
                umma_commit(k_empty + k_slot);
                umma_commit(s_full + (n & 1));
                if (++k_slot == TA_K_STAGES) {
                    k_slot = 0;
                    ++k_use;
                }
            };
            if (!mbar_wait(q_stored, 0, abort_word)) give_up();
            tc_fence_after();
            if (ok) issue_qk(0);
            if (ok && num_kt > 1) issue_qk(1);
            for (int n = 0; n < num_kt && ok; ++n) {
                const int v_slot = n % TA_V_STAGES;
                if (!mbar_wait(p_full + (n & 1), (n >> 1) & 1, abort_word) || !mbar_wait(v_full + v_slot, (n / TA_V_STAGES) & 1, abort_word)) {
                    give_up();
                    break;
                }
                tc_fence_after();
                const uint64_t vb = v_desc + (uint64_t)((v_slot * v_bytes) >> 4);
#pragma unroll
                for (int ks = 0; ks < TA_BN / 16; ++ks)  // 16 keys: 8 columns of P in tensor memory, 16 rows (2 KB) of V
                    umma_bf16_a_tmem(tmem_base + O_COL, tmem_base + S_COL + (n & 1) * TA_BN + ks * 8, vb + (uint64_t)(ks * 128), idesc_pv,
                                     (n > 0 || ks > 0) ? 1u : 0u);
                umma_commit(v_empty + v_slot);
                umma_commit(pv_done + (n & 1));
                // the softmax holds S_n in registers (it has written P_n), and the pipe keeps the order of products: S_n's
                // buffer takes tile n + 2
                if (n + 2 < num_kt) issue_qk(n + 2);
            }
        }
    } else if (warp < 4) {
        // ---------------- softmax and epilogue: thread r owns row r
        const int r = threadIdx.x;
        const uint32_t lane_base = tmem_base + ((uint32_t)(warp * 32) << 16);
        const float sl2 = scale * TA_LOG2E;
        const int qi = r / group;
        const bool valid = qi < queries && r < per_tile * group;
        const int pos = valid ? first_pos + qi : last_pos;
        const int lo = (window > 0 && pos + 1 > window) ? pos + 1 - window : 0;
        const int lo_last = (window > 0 && last_pos + 1 > window) ? last_pos + 1 - window : 0;
        float m_ref = -INFINITY;  // the maximum the row's P and O are scaled by
        float l = 0.0f;
        bool ok = true;
        // the row's queries, a band of 64 columns (32 of tensor memory) at a time
        if (!mbar_wait(q_loaded, 0, abort_word)) ok = false;
        if (ok) {
            for (int b = 0; b < key_bands; ++b) {
                const unsigned char* src = smem + k_bytes + (r * key_bands + b) * 128;
                uint32_t band[32];
#pragma unroll
                for (int i = 0; i < 8; ++i) {
                    const uint4 v = *reinterpret_cast<const uint4*>(src + ((i ^ (r & 7)) * 16));
                    band[4 * i] = v.x;
                    band[4 * i + 1] = v.y;
                    band[4 * i + 2] = v.z;
                    band[4 * i + 3] = v.w;
                }
                tmem_store32(lane_base + Q_COL + b * 32, band);
            }
            tmem_wait_st();
            tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(q_stored);
        }
        for (int n = 0; n < num_kt && ok; ++n) {
            const int key0 = key_of(n);
            if (!mbar_wait(s_full + (n & 1), (n >> 1) & 1, abort_word)) { ok = false; break; }
            tc_fence_after();
            const uint32_t s_at = lane_base + S_COL + (n & 1) * TA_BN;
            uint32_t raw[2][32];
#pragma unroll
            for (int c = 0; c < 2; ++c) tmem_load32_nowait(s_at + c * 32, raw[c]);
            tmem_wait_ld();
            // on the raw scores for a positive scale: the maximum is taken before the scale, which then enters the exponent's
            // argument with the reference as one fused multiply-add; a scale of another sign is applied first
            const bool all_seen = key0 + TA_BN - 1 <= first_pos && (key0 >= lo_last || key0 + TA_BN <= keep_first);
            if (!all_seen) {
#pragma unroll
                for (int c = 0; c < TA_BN; ++c) {
                    const int key = key0 + c;
                    if (!(key <= pos && (key >= lo || key < keep_first))) raw[c >> 5][c & 31] = __float_as_uint(sl2 >= 0.0f ? -INFINITY : INFINITY);
                }
            }
            float mx4[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
            if (sl2 >= 0.0f) {
#pragma unroll
                for (int c = 0; c < TA_BN; ++c) mx4[c & 3] = fmaxf(mx4[c & 3], __uint_as_float(raw[c >> 5][c & 31]));
            } else {
#pragma unroll
                for (int c = 0; c < TA_BN; ++c) mx4[c & 3] = fmaxf(mx4[c & 3], -__uint_as_float(raw[c >> 5][c & 31]));
            }
            const float top = fmaxf(fmaxf(mx4[0], mx4[1]), fmaxf(mx4[2], mx4[3]));
            const float mx = top == -INFINITY ? -INFINITY : top * fabsf(sl2);
            float alpha = 1.0f;
            if (m_ref == -INFINITY) {
                m_ref = mx;  // nothing accumulated for this row yet
            } else if (mx > m_ref + TA_RESCALE_STEP) {
                alpha = exp2f(m_ref - mx);
                m_ref = mx;
            }
            // only a rescale of O needs the P V before complete; every phase of the two pv_done barriers is observed all the
            // same, in order and two tiles late
            if (n > 1 && !mbar_wait(pv_done + (n & 1), ((n - 2) >> 1) & 1, abort_word)) { ok = false; break; }
            if (__any_sync(0xffffffffu, alpha != 1.0f)) {
                if (n > 0 && !mbar_wait(pv_done + ((n - 1) & 1), ((n - 1) >> 1) & 1, abort_word)) { ok = false; break; }
                tc_fence_after();
#pragma unroll
                for (int c = 0; c < VB * 2; ++c) {
                    uint32_t o[32];
                    tmem_load32_nowait(lane_base + O_COL + c * 32, o);
                    tmem_wait_ld();
#pragma unroll
                    for (int i = 0; i < 32; ++i) o[i] = __float_as_uint(__uint_as_float(o[i]) * alpha);
                    tmem_store32(lane_base + O_COL + c * 32, o);
                }
                tmem_wait_st();
                l *= alpha;
            }
            const float base = m_ref == -INFINITY ? 0.0f : -m_ref;
            float sum4[4] = {0.0f, 0.0f, 0.0f, 0.0f};
            uint32_t packed[32];
#pragma unroll
            for (int c = 0; c < TA_BN; c += 2) {
                const float s0 = __uint_as_float(raw[c >> 5][c & 31]), s1 = __uint_as_float(raw[c >> 5][(c & 31) + 1]);
                const float p0 = ta_ex2(fmaf(s0, sl2, base)), p1 = ta_ex2(fmaf(s1, sl2, base));
                sum4[c & 2] += p0;
                sum4[(c & 2) + 1] += p1;
                __nv_bfloat162 pair = __floats2bfloat162_rn(p0, p1);
                packed[c >> 1] = *reinterpret_cast<uint32_t*>(&pair);
            }
            tmem_store32(s_at, packed);
            l += (sum4[0] + sum4[1]) + (sum4[2] + sum4[3]);
            tmem_wait_st();
            tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(p_full + (n & 1));
        }
        if (ok && num_kt > 1 && !mbar_wait(pv_done + ((num_kt - 2) & 1), ((num_kt - 2) >> 1) & 1, abort_word)) ok = false;
        if (ok && !mbar_wait(pv_done + ((num_kt - 1) & 1), ((num_kt - 1) >> 1) & 1, abort_word)) ok = false;
        if (ok) {
            tc_fence_after();
            const float inv = l > 0.0f ? 1.0f / l : 0.0f;
            __nv_bfloat16* dst = out + (size_t)(tok0 + q0 + (valid ? qi : 0)) * out_stride + (size_t)(kvh * group + (valid ? r - qi * group : 0)) * D;
#pragma unroll
            for (int c = 0; c < VB * 2; ++c) {
                uint32_t o[32];
                tmem_load32_nowait(lane_base + O_COL + c * 32, o);
                tmem_wait_ld();
                if (valid) {
#pragma unroll
                    for (int i = 0; i < 4; ++i) {
                        if (c * 32 + i * 8 >= D) continue;
                        uint32_t w[4];
#pragma unroll
                        for (int e = 0; e < 4; ++e) {
                            __nv_bfloat162 pair = __floats2bfloat162_rn(__uint_as_float(o[8 * i + 2 * e]) * inv, __uint_as_float(o[8 * i + 2 * e + 1]) * inv);
                            w[e] = *reinterpret_cast<uint32_t*>(&pair);
                        }
                        *reinterpret_cast<uint4*>(dst + c * 32 + i * 8) = make_uint4(w[0], w[1], w[2], w[3]);
                    }
                }
            }
            tc_fence_before();
        } else {
            if (lane == 0 && !*abort_word && flag) atomicOr(flag, KB_FLAG_TIMEOUT);
            *abort_word = 1;
        }
    }
    tc_fence_before();
    __syncthreads();
    if (warp == 8) {
        tc_fence_after();
        tmem_dealloc(tmem_base, TA_TMEM_COLUMNS);
    }
}

#define TA_SMEM_MAX ((TA_K_STAGES * TA_MAX_BANDS + TA_V_STAGES * 2) * TA_BAND + (2 * TA_K_STAGES + 2 * TA_V_STAGES + 8) * 8 + 16)

static int ta_key_bands(int G, int D) { return (G * D + 63) / 64; }
static int ta_value_bands(int D) { return (D + 63) / 64; }

KB_EXPORT int kb_talking_attention_tc5_supported(int H, int G, int D) {
    return G >= 1 && H >= 1 && H % G == 0 && H / G <= TA_BM && D >= 8 && D <= 128 && D % 8 == 0
           && ta_key_bands(G, D) <= TA_MAX_BANDS;
}

// list_rows / list_starts: the request row and the first query of each tile of 128 / (H / G) queries of the step's portions.
KB_EXPORT int kb_talking_attention_tc5(const void* q, int q_stride, void* out, int out_stride, const void* k_cache, const void* v_cache,
                                       const int* qo_indptr, const int* seq_lens, const int* block_table, int max_pages,
                                       const int* list_rows, const int* list_starts, int count, int H, int G, int D, int page_size,
                                       int num_pages, float scale, int window, int keep_first, int* flag, cudaStream_t stream) {
    if (count == 0) return 0;
    if (!q || !out || !k_cache || !v_cache || !qo_indptr || !seq_lens || !block_table || !list_rows || !list_starts) return KB_ERR_NULL;
    if (!kb_talking_attention_tc5_supported(H, G, D)) return KB_ERR_UNSUPPORTED_SIZE;
    if (count > 65535 || page_size < 1 || keep_first < 0 || q_stride % 8 || out_stride % 8
        || (((uintptr_t)q | (uintptr_t)out | (uintptr_t)k_cache | (uintptr_t)v_cache) % 16)) return KB_ERR_BAD_ARG;
    if ((long long)num_pages * page_size > 0x7fffffffLL) return KB_ERR_UNSUPPORTED_SIZE;
    const int bands = ta_key_bands(G, D), vb = ta_value_bands(D);
    const size_t smem = TA_SMEM_MAX - (size_t)((TA_MAX_BANDS - bands) * TA_K_STAGES + (2 - vb) * TA_V_STAGES) * TA_BAND;
    int shift = -1;
    if ((page_size & (page_size - 1)) == 0) {
        shift = 0;
        while ((1 << shift) < page_size) ++shift;
    }
#define LAUNCH(VB)                                                                                                                          \
    do {                                                                                                                                    \
        static bool configured = false;                                                                                                     \
        if (!configured) {                                                                                                                  \
            cudaFuncSetAttribute(talking_attention_tc5_kernel<VB>, cudaFuncAttributeMaxDynamicSharedMemorySize, TA_SMEM_MAX);               \
            configured = true;                                                                                                              \
        }                                                                                                                                   \
        kb_launch(talking_attention_tc5_kernel<VB>, dim3(G, count), dim3(TA_THREADS), smem, stream, (const __nv_bfloat16*)q, q_stride,       \
                  (__nv_bfloat16*)out, out_stride, (const __nv_bfloat16*)k_cache, (const __nv_bfloat16*)v_cache, qo_indptr, seq_lens,        \
                  block_table, max_pages, list_rows, list_starts, H, G, D, bands, page_size, shift, num_pages, scale, window,        \
                  keep_first, flag);                                                                                                        \
    } while (0)
    if (vb == 1) LAUNCH(1); else LAUNCH(2);
#undef LAUNCH
    return kb_launch_result();
}
