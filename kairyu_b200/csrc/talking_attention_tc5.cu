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
// 128 at absolute multiples of 128: first the tiles of the kept first tokens, then those of the window.  Roles (256 threads; eight warps, so
// that a thread may hold its 128 scores in registers):
//   warps 0-3  softmax: thread r owns row r; reads its row of S from tensor memory, writes P as bf16 pairs over it, rescales O
//              in tensor memory only when the row maximum has grown by more than 2^8 since the reference it scales by;
//   warps 4-5  producer: cp.async of the queries (once), of the keys, one 64-column band of a tile at a time through a ring of
//              buffers, and of the values (one buffer), each 16-byte group put where the 128-byte swizzle of the tensor cores'
//              operand wants it.  (A TMA copy brings a page's run of rows of one band: with pages of 16 positions and wide
//              keys that is 8 copies for every 256 cycles of products, more than an SM can issue; a thread's cp.async takes
//              any page size, and pads columns up to 64 and rows beyond the last key with zeros.)
//   warp 6     one thread issues tcgen05.mma: S (128 x 128, two buffers) band by band, O += P V.  Q K^T runs two tiles
//              ahead of P V.
// The items (bands of keys, tiles of values) are produced in the order the products consume them, K0 K1 V0 K2 V1 ..., and a
// producer thread that has to wait for a free buffer first reports everything it has issued, so no wait can be circular.
//
// Every wait on an mbarrier is bounded: a role that gives up raises KB_FLAG_TIMEOUT, the other roles leave through a shared
// abort word, and the block frees its tensor memory and returns.
// Sizes: D a multiple of 8 up to 128, G * D up to 640, H / G up to 128, any page size.
#include "umma.cuh"

#define TA_THREADS 256
#define TA_PRODUCERS 64
#define TA_PASSES (TA_BN * 8 / TA_PRODUCERS)  // rows of a band a producer thread copies 16 bytes of
#define TA_BM 128
#define TA_BN 128
#define TA_BAND (TA_BN * 128)  // bytes of one 64-column band of 128 rows
#define TA_MAX_STAGES 8
#define TA_LOG2E 1.4426950408889634f
#define TA_RESCALE_STEP 8.0f
#define TA_S_COL 0      // two S buffers of 128 columns; P (bf16 pairs) overwrites the first half of its S
#define TA_O_COL 256
#define TA_TMEM_COLUMNS 512
#define KB_FLAG_MISALIGNED 32

__device__ __forceinline__ float ta_ex2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;\n" : "=f"(y) : "f"(x));
    return y;
}
__device__ __forceinline__ bool ta_ready(uint64_t* bar, uint32_t parity) {
    uint32_t done;
    asm volatile("{\n .reg .pred p;\n mbarrier.try_wait.parity.shared::cta.b64 p, [%1], %2;\n selp.u32 %0, 1, 0, p;\n}\n"
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

// A producer thread's items in flight: reported (fence, then one arrival) in the order they were issued.
struct TaInFlight {
    uint64_t* older = nullptr;
    uint64_t* newer = nullptr;
    __device__ __forceinline__ void flush() {
        if (!newer) return;
        ta_wait<0>();
        fence_proxy_async_smem();
        if (older) mbar_arrive(older);
        mbar_arrive(newer);
        older = newer = nullptr;
    }
    __device__ __forceinline__ void push(uint64_t* bar) {  // the copies issued since the last push belong to `bar`
        ta_commit();
        if (older) {  // two items stay in flight behind this one
            ta_wait<2>();
            fence_proxy_async_smem();
            mbar_arrive(older);
        }
        older = newer;
        newer = bar;
    }
};

template <int VB>  // 64-column bands of a value row
__global__ void __launch_bounds__(TA_THREADS, 1)
talking_attention_tc5_kernel(const __nv_bfloat16* __restrict__ q, int q_stride, __nv_bfloat16* __restrict__ out, int out_stride,
                             const __nv_bfloat16* __restrict__ k_cache, const __nv_bfloat16* __restrict__ v_cache,
                             const int* __restrict__ qo_indptr, const int* __restrict__ seq_lens, const int* __restrict__ block_table,
                             int max_pages, const int* __restrict__ tile_rows, const int* __restrict__ tile_starts, int H, int G, int D,
                             int key_bands, int stages, int page_size, int page_shift, int num_pages, float scale, int window,
                             int keep_first, int* flag) {
    extern __shared__ __align__(1024) unsigned char smem[];
    unsigned char* sQ = smem;
    unsigned char* sK = sQ + (size_t)key_bands * TA_BAND;
    unsigned char* sV = sK + (size_t)stages * TA_BAND;
    uint64_t* bars = reinterpret_cast<uint64_t*>(sV + VB * TA_BAND);
    uint64_t* q_full = bars;
    uint64_t* k_full = bars + 1;
    uint64_t* k_empty = k_full + TA_MAX_STAGES;
    uint64_t* v_full = k_empty + TA_MAX_STAGES;
    uint64_t* v_empty = v_full + 1;
    uint64_t* s_full = v_empty + 1;   // one per S buffer
    // two each, used in turn: the softmax may be a tile ahead of the products, and a barrier whose phase is told by its
    // parity cannot be two phases ahead of who waits on it
    uint64_t* p_full = s_full + 2;
    uint64_t* pv_done = p_full + 2;
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(pv_done + 2);
    volatile int* abort_word = reinterpret_cast<volatile int*>(tmem_slot + 1);

    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    if (threadIdx.x == 0) {
        mbar_init(q_full, TA_PRODUCERS);
        for (int s = 0; s < stages; ++s) {
            mbar_init(k_full + s, TA_PRODUCERS);
            mbar_init(k_empty + s, 1);
        }
        mbar_init(v_full, TA_PRODUCERS);
        mbar_init(v_empty, 1);
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
    if (warp == 6) tmem_alloc(tmem_slot, TA_TMEM_COLUMNS);
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
    } else if (warp == 4 || warp == 5) {
        // ---------------- producer: 8 lanes a row, 8 rows a pass
        const int tid = threadIdx.x - 128;
        const int chunk = tid & 7, row0 = tid >> 3;
        const int key_width = G * D;
        const uint32_t swizzled = (uint32_t)((chunk ^ (row0 & 7)) * 16);  // rows of a thread differ by 8: one swizzle for all
        const int* table = block_table + (size_t)row * max_pages;
        TaInFlight flight;
        bool ok = true;
        auto wait_free = [&](uint64_t* bar, uint32_t parity) {
            if (ta_ready(bar, parity)) return true;
            flight.flush();
            if (mbar_wait(bar, parity, abort_word)) return true;
            if (!*abort_word && flag) atomicOr(flag, KB_FLAG_TIMEOUT);
            *abort_word = 1;
            return false;
        };
        for (int b = 0; b < key_bands; ++b) {
            const int col = b * 64 + chunk * 8;
#pragma unroll
            for (int i = 0; i < TA_PASSES; ++i) {
                const int r = row0 + i * 8;
                const int qi = r / group;
                const bool valid = qi < queries && col < key_width;
                const __nv_bfloat16* src = q + (size_t)(tok0 + q0 + (valid ? qi : 0)) * q_stride + (size_t)(kvh * group + (valid ? r - qi * group : 0)) * key_width + (valid ? col : 0);
                ta_copy16(smem_addr(sQ) + b * TA_BAND + r * 128 + swizzled, src, valid);
            }
        }
        flight.push(q_full);
        int place[TA_PASSES], place_before[TA_PASSES];
        uint32_t slot = 0, use = 0;  // of the key ring
        for (int n = 0; n <= num_kt && ok; ++n) {
            if (n < num_kt) {
                const int key0 = key_of(n);
#pragma unroll
                for (int i = 0; i < TA_PASSES; ++i) {
                    const int key = key0 + row0 + i * 8;
                    int at = -1;
                    if (key < key_end) {
                        const int page_index = page_shift >= 0 ? key >> page_shift : key / page_size;
                        const int page = page_index < max_pages ? table[page_index] : -1;  // -1: a page the window has given back
                        if (page >= 0 && page < num_pages) at = page * page_size + (key - page_index * page_size);
                    }
                    place[i] = at;
                }
                for (int b = 0; b < key_bands; ++b) {
                    if (use > 0 && !wait_free(k_empty + slot, (use - 1) & 1)) {
                        ok = false;
                        break;
                    }
                    const int col = b * 64 + chunk * 8;
                    const uint32_t dst = smem_addr(sK) + slot * TA_BAND + row0 * 128 + swizzled;
#pragma unroll
                    for (int i = 0; i < TA_PASSES; ++i) {
                        const bool valid = place[i] >= 0 && col < key_width;
                        ta_copy16(dst + i * 1024, k_cache + (valid ? (size_t)place[i] * key_width + col : 0), valid);
                    }
                    flight.push(k_full + slot);
                    if (++slot == (uint32_t)stages) {
                        slot = 0;
                        ++use;
                    }
                }
            }
            if (n > 0 && ok) {  // the values of the tile before
                if (n > 1 && !wait_free(v_empty, (n - 2) & 1)) {
                    ok = false;
                    break;
                }
#pragma unroll
                for (int b = 0; b < VB; ++b) {
                    const int col = b * 64 + chunk * 8;
                    const uint32_t dst = smem_addr(sV) + b * TA_BAND + row0 * 128 + swizzled;
#pragma unroll
                    for (int i = 0; i < TA_PASSES; ++i) {
                        const bool valid = place_before[i] >= 0 && col < D;
                        ta_copy16(dst + i * 1024, v_cache + (valid ? (size_t)place_before[i] * key_width + kvh * D + col : 0), valid);
                    }
                }
                flight.push(v_full);
            }
#pragma unroll
            for (int i = 0; i < TA_PASSES; ++i) place_before[i] = place[i];
        }
        flight.flush();
        ta_wait<0>();
    } else if (warp == 6) {
        // ---------------- products (one thread)
        if (lane == 0) {
            constexpr uint32_t idesc_qk = umma_idesc(TA_BN);
            constexpr uint32_t idesc_pv = umma_idesc_b_mn(VB * 64);
            const uint64_t q_desc = umma_desc_sw128(smem_addr(sQ));
            const uint64_t k_desc = umma_desc_sw128(smem_addr(sK));
            const uint64_t v_desc = umma_desc_mn_sw128(smem_addr(sV), TA_BAND, 1024);
            bool ok = true;
            uint32_t slot = 0, use = 0;
            auto give_up = [&]() {
                if (!*abort_word && flag) atomicOr(flag, KB_FLAG_TIMEOUT);
                *abort_word = 1;
                ok = false;
            };
            auto issue_qk = [&](int n) {
                for (int b = 0; b < key_bands; ++b) {
                    if (!mbar_wait(k_full + slot, use & 1, abort_word)) {
                        give_up();
                        return;
                    }
                    tc_fence_after();
                    const uint64_t qb = q_desc + (uint64_t)((b * TA_BAND) >> 4);
                    const uint64_t kb = k_desc + (uint64_t)((slot * TA_BAND) >> 4);
#pragma unroll
                    for (int k = 0; k < 4; ++k)  // 16 columns = 32 bytes along the swizzled row
                        umma_bf16(tmem_base + TA_S_COL + (n & 1) * TA_BN, qb + (uint64_t)(k * 2), kb + (uint64_t)(k * 2), idesc_qk, (b > 0 || k > 0) ? 1u : 0u);
                    umma_commit(k_empty + slot);
                    if (++slot == (uint32_t)stages) {
                        slot = 0;
                        ++use;
                    }
                }
                umma_commit(s_full + (n & 1));
            };
            if (!mbar_wait(q_full, 0, abort_word)) give_up();
            if (ok) issue_qk(0);
            if (ok && num_kt > 1) issue_qk(1);
            for (int n = 0; n < num_kt && ok; ++n) {
                if (!mbar_wait(p_full + (n & 1), (n >> 1) & 1, abort_word) || !mbar_wait(v_full, n & 1, abort_word)) {
                    give_up();
                    break;
                }
                tc_fence_after();
#pragma unroll
                for (int ks = 0; ks < TA_BN / 16; ++ks)  // 16 keys: 8 columns of P in tensor memory, 16 rows (2 KB) of V
                    umma_bf16_a_tmem(tmem_base + TA_O_COL, tmem_base + TA_S_COL + (n & 1) * TA_BN + ks * 8, v_desc + (uint64_t)(ks * 128), idesc_pv,
                                     (n > 0 || ks > 0) ? 1u : 0u);
                umma_commit(v_empty);
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
        for (int n = 0; n < num_kt; ++n) {
            const int key0 = key_of(n);
            if (!mbar_wait(s_full + (n & 1), (n >> 1) & 1, abort_word)) { ok = false; break; }
            tc_fence_after();
            const uint32_t s_at = lane_base + TA_S_COL + (n & 1) * TA_BN;
            uint32_t raw[4][32];
#pragma unroll
            for (int c = 0; c < 4; ++c) tmem_load32_nowait(s_at + c * 32, raw[c]);
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
                    tmem_load32_nowait(lane_base + TA_O_COL + c * 32, o);
                    tmem_wait_ld();
#pragma unroll
                    for (int i = 0; i < 32; ++i) o[i] = __float_as_uint(__uint_as_float(o[i]) * alpha);
                    tmem_store32(lane_base + TA_O_COL + c * 32, o);
                }
                tmem_wait_st();
                l *= alpha;
            }
            const float base = m_ref == -INFINITY ? 0.0f : -m_ref;
            float sum4[4] = {0.0f, 0.0f, 0.0f, 0.0f};
#pragma unroll
            for (int half = 0; half < 2; ++half) {
                uint32_t packed[32];
#pragma unroll
                for (int c = 0; c < 64; c += 2) {
                    const int at = half * 64 + c;
                    const float s0 = __uint_as_float(raw[at >> 5][at & 31]), s1 = __uint_as_float(raw[at >> 5][(at & 31) + 1]);
                    const float p0 = ta_ex2(fmaf(s0, sl2, base)), p1 = ta_ex2(fmaf(s1, sl2, base));
                    sum4[c & 2] += p0;
                    sum4[(c & 2) + 1] += p1;
                    __nv_bfloat162 pair = __floats2bfloat162_rn(p0, p1);
                    packed[c >> 1] = *reinterpret_cast<uint32_t*>(&pair);
                }
                tmem_store32(s_at + half * 32, packed);
            }
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
                tmem_load32_nowait(lane_base + TA_O_COL + c * 32, o);
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
    if (warp == 6) {
        tc_fence_after();
        tmem_dealloc(tmem_base, TA_TMEM_COLUMNS);
    }
}

#define TA_SMEM_LIMIT (227 * 1024)
#define TA_BAR_BYTES ((1 + 2 * TA_MAX_STAGES + 8) * 8 + 16)

static int ta_key_bands(int G, int D) { return (G * D + 63) / 64; }
static int ta_value_bands(int D) { return (D + 63) / 64; }
static int ta_stages(int G, int D) {
    const int room = TA_SMEM_LIMIT - TA_BAR_BYTES - (ta_key_bands(G, D) + ta_value_bands(D)) * TA_BAND;
    const int stages = room / TA_BAND;
    return stages > TA_MAX_STAGES ? TA_MAX_STAGES : stages;
}

KB_EXPORT int kb_talking_attention_tc5_supported(int H, int G, int D) {
    return G >= 1 && H >= 1 && H % G == 0 && H / G <= TA_BM && D >= 8 && D <= 128 && D % 8 == 0 && ta_stages(G, D) >= 2;
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
    const int bands = ta_key_bands(G, D), vb = ta_value_bands(D), stages = ta_stages(G, D);
    const size_t smem = (size_t)(bands + stages + vb) * TA_BAND + TA_BAR_BYTES;
    int shift = -1;
    if ((page_size & (page_size - 1)) == 0) {
        shift = 0;
        while ((1 << shift) < page_size) ++shift;
    }
#define LAUNCH(VB)                                                                                                                          \
    do {                                                                                                                                    \
        static bool configured = false;                                                                                                     \
        if (!configured) {                                                                                                                  \
            cudaFuncSetAttribute(talking_attention_tc5_kernel<VB>, cudaFuncAttributeMaxDynamicSharedMemorySize, TA_SMEM_LIMIT);               \
            configured = true;                                                                                                              \
        }                                                                                                                                   \
        kb_launch(talking_attention_tc5_kernel<VB>, dim3(G, count), dim3(TA_THREADS), smem, stream, (const __nv_bfloat16*)q, q_stride,       \
                  (__nv_bfloat16*)out, out_stride, (const __nv_bfloat16*)k_cache, (const __nv_bfloat16*)v_cache, qo_indptr, seq_lens,        \
                  block_table, max_pages, list_rows, list_starts, H, G, D, bands, stages, page_size, shift, num_pages, scale, window,        \
                  keep_first, flag);                                                                                                        \
    } while (0)
    if (vb == 1) LAUNCH(1); else LAUNCH(2);
#undef LAUNCH
    return kb_launch_result();
}
