// Flash attention of single tokens where all query heads of a position share ONE wide key row and take their values from their
// own key/value head (the mixed queries of talking_attention.cu), on mma.sync m16n8k16 with 32-bit scores, softmax and sums:
//
//     S = Q K^T * scale      Q [tokens, H, G * D], K: the G key/value heads' keys of a position side by side
//     P = softmax over the keys the token sees: itself and the window - 1 before it (window 0: all), and the sequence's first
//         keep_first tokens;   O_h = P_h V_c(h)
//
// The H heads are the rows of the products (sixteen a product, as many as a product has anyway), so the wide key row costs no
// more than G separate heads' keys would, and a request's keys and values are read once for all heads.
// A block walks a share of one request's keys in tiles of 32 at absolute multiples of 32, first the tiles of the kept first
// tokens, then the window's.  The tiles' keys and values go into a ring of buffers, in the order they are used: K0 K1 V0 K2 V1 ...
// (by TMA, one copy a run of a page's positions with all its columns, where key rows are whole 64-column bands and pages a power
// of two of 8 positions or more; else four warps copy 16 bytes a lane: cp.async keeps about 30 KB an SM on their way whatever it
// is asked for, half of what the memory wants).  Sixteen warps work on them, a turn at a time, in two phases:
//   products  S of tile n + 1 (warp w: 16 of its keys, an eighth of the key columns, whose part of the queries the warp holds in
//             registers) and O += P V of tile n (warp w: its 16-column units of the value row; a unit lies in one key/value
//             head and takes that head's rows of P);
//   softmax   of tile n + 1, a warp a row, a lane a key: the eighths' scores are added up, the row's maximum moves on, P goes
//             to shared memory.  A lane keeps its share of the row's sum to itself until the end.
// With the keys split over blocks the unnormalised results are combined by a second kernel in split order, so a result
// depends on the token's position and the number of splits.
// Waits on the ring's barriers are bounded by time: who gives up raises KB_FLAG_TIMEOUT and the block's abort word, later waits end
// at once, and the block runs to its end over whatever the buffers hold.
#include "attention_mma.cuh"

#include <cuda.h>
#include <cudaTypedefs.h>

#define TD_WARPS 16      // that work on the tiles
#define TD_COPY_WARPS 4  // that fetch them without TMA (with it: one)
#define TD_WORKERS (TD_WARPS * 32)
#define TD_THREADS(tma) ((TD_WARPS + ((tma) ? 1 : TD_COPY_WARPS)) * 32)
#define TD_PARTS (TD_WARPS / 2)  // shares of the key columns
#define TD_MAX_RING 8
#define TD_IN_FLIGHT 3   // items a copying thread leaves unreported behind the one it has just issued
#define TD_KEYS 32
#define TD_P_STRIDE (TD_KEYS + 8)
#define TD_S_STRIDE (TD_KEYS + 4)
#define TD_SMEM_LIMIT (226 * 1024)

__device__ __forceinline__ void td_arrive(uint64_t* bar) {
    asm volatile("mbarrier.arrive.shared::cta.b64 _, [%0];\n" ::"r"(smem_u32(bar)) : "memory");
}
__device__ __forceinline__ bool td_wait(uint64_t* bar, uint32_t parity, volatile int* abort_word) {
    return !*abort_word && mbar_wait(bar, parity);
}

__device__ __forceinline__ void td_tma(void* dst, const CUtensorMap* map, int within, int page, uint64_t* bar) {
    asm volatile("cp.async.bulk.tensor.4d.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%3, %4, %5, %6}], [%2];\n" ::"r"(
                     smem_u32(dst)),
                 "l"(map), "r"(smem_u32(bar)), "r"(0), "r"(within), "r"(0), "r"(page)
                 : "memory");
}

struct TdShape {
    int H, G, D, width;  // width = G * D
    int row_tiles;       // sixteens of query heads: 1 or 2
    int ring;            // buffers of a tile's keys or values
    int tma;
};

__host__ __device__ static inline size_t td_smem(const TdShape& s) {
    const size_t stride = s.width + (s.tma ? 0 : 8), rows = 16 * s.row_tiles;
    return ((size_t)s.ring * TD_KEYS * stride + rows * TD_P_STRIDE) * sizeof(__nv_bfloat16)
           + (TD_PARTS * rows * TD_S_STRIDE + 3 * rows) * sizeof(float) + 2 * TD_MAX_RING * 8 + 16;
}

// MT: sixteens of heads; STEPS: 16-column steps of the key row a warp's share has at most (of the value row's 16-column units
// a warp owns half as many, or one)
template <int MT, int STEPS, bool TMA>
__global__ void __launch_bounds__(TD_THREADS(TMA))
talking_decode_kernel(const __grid_constant__ CUtensorMap map_k, const __grid_constant__ CUtensorMap map_v, const __nv_bfloat16* __restrict__ q, int q_stride, __nv_bfloat16* __restrict__ out, int out_stride,
                      const __nv_bfloat16* __restrict__ k_cache, const __nv_bfloat16* __restrict__ v_cache, const int* __restrict__ seq_lens,
                      const int* __restrict__ block_table, int max_pages, const int* __restrict__ list_rows,
                      const int* __restrict__ list_tokens, const TdShape shape, int page_size, int page_shift, int num_pages, float scale,
                      int window, int keep_first, int splits, float* __restrict__ part_o, float* __restrict__ part_ml, int* flag) {
    extern __shared__ __align__(1024) unsigned char td_shared[];
    constexpr int UNITS = STEPS > 1 ? STEPS / 2 : 1, ROWS = 16 * MT, ROW_TURNS = ROWS / TD_WARPS;
    const int H = shape.H, D = shape.D, width = shape.width, stride = width + (TMA ? 0 : 8), ring = shape.ring;
    const size_t tile_size = (size_t)TD_KEYS * stride;
    __nv_bfloat16* sRing = reinterpret_cast<__nv_bfloat16*>(td_shared);
    __nv_bfloat16* sP = sRing + ring * tile_size;
    float* sS = reinterpret_cast<float*>(sP + ROWS * TD_P_STRIDE);  // [share of the columns][row][key]
    float* sAlpha = sS + TD_PARTS * ROWS * TD_S_STRIDE;
    float* sM = sAlpha + ROWS;
    float* sL = sM + ROWS;
    uint64_t* full = reinterpret_cast<uint64_t*>(sL + ROWS);
    uint64_t* empty = full + TD_MAX_RING;
    volatile int* abort_word = reinterpret_cast<volatile int*>(empty + TD_MAX_RING);
    // Where 16 bytes (columns 8 c .. 8 c + 7 of row r) of a tile lie, in elements.  Brought by TMA: runs of positions, in a run
    // the 64-column bands one after the other, a band's rows 128 bytes apart with their 16-byte groups turned by the row.
    const int run_shift = page_shift < 5 ? page_shift : 5, run_rows = 1 << run_shift;  // TMA: pages of a power of two
    static_assert(TD_KEYS == 32, "runs of up to 2^5 rows");
    auto at16 = [&](int r, int c) {
        if constexpr (TMA) return ((r >> run_shift) << run_shift) * width + ((c >> 3) << (run_shift + 6)) + ((r & (run_rows - 1)) << 6) + (((c & 7) ^ (r & 7)) << 3);
        else return r * stride + c * 8;
    };

    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int g = lane >> 2, tq = lane & 3, mm = lane >> 3;
    const int split = blockIdx.x, index = blockIdx.y;
    const int row = list_rows[index], token = list_tokens[index];
    const int pos = seq_lens[row] - 1;
    const int* table = block_table + (size_t)row * max_pages;
    const int group = H / shape.G;
    const int key_lo = (window > 0 && pos + 1 > window) ? pos + 1 - window : 0;
    const int first_kt = key_lo / TD_KEYS;
    const int kept_kt = min((min(keep_first, key_lo) + TD_KEYS - 1) / TD_KEYS, first_kt);
    const int all_kt = kept_kt + pos / TD_KEYS - first_kt + 1;
    const int per = (all_kt + splits - 1) / splits;
    const int begin = split * per, num_kt = min(per, all_kt - begin);
    auto key_of = [&](int n) { return (begin + n < kept_kt ? begin + n : first_kt + begin + n - kept_kt) * TD_KEYS; };
    if (num_kt <= 0) {  // a short row leaves the last splits without keys (splits > 1: split 0 always has some)
        pdl_wait();
        for (int h = threadIdx.x; h < H; h += TD_THREADS(TMA)) {
            float* ml = part_ml + (((size_t)split * gridDim.y + index) * H + h) * 2;
            ml[0] = -INFINITY;
            ml[1] = 0.0f;
        }
        return;
    }
    if (threadIdx.x == 0) {
        for (int i = 0; i < ring; ++i) {
            mbar_init(full + i, TMA ? 1 : TD_COPY_WARPS);
            mbar_init(empty + i, TD_WARPS);
        }
        *abort_word = 0;
        fence_barrier_init();
    }
    __syncthreads();
    auto give_up = [&]() {
        if (lane == 0 && !*abort_word && flag) atomicOr(flag, KB_FLAG_TIMEOUT);
        *abort_word = 1;
    };

    if (TMA && warp >= TD_WARPS) {
        // ---------------- copies by TMA: a lane a run of positions
        const int runs = TD_KEYS >> run_shift;
        int slot = 0, use = 0;
        bool waited = false;
        auto fetch = [&](const CUtensorMap* map, int n) {
            // what the kernel before writes is the newest position: older tiles may be fetched ahead of it
            if (!waited && (use > 0 || key_of(n) + TD_KEYS > pos)) {
                pdl_wait();
                waited = true;
            }
            if (use > 0 && !__all_sync(0xffffffffu, td_wait(empty + slot, (use - 1) & 1, abort_word))) {
                give_up();
                return false;
            }
            if (lane == 0) mbar_arrive_expect_tx(full + slot, (uint32_t)(TD_KEYS * width * sizeof(__nv_bfloat16)));
            __syncwarp();
            if (lane < runs) {
                const int key = key_of(n) + lane * run_rows;
                const int page_index = key >> page_shift;
                int page = 0, within = 0;  // the reserved page stands in for rows nobody may see
                if (key <= pos && page_index < max_pages) {
                    const int p = table[page_index];
                    if (p >= 0 && p < num_pages) {
                        page = p;
                        within = key - (page_index << page_shift);
                    }
                }
                td_tma(sRing + slot * tile_size + (size_t)lane * run_rows * width, map, within, page, full + slot);
            }
            if (++slot == ring) {
                slot = 0;
                ++use;
            }
            return true;
        };
        bool ok = true;
        for (int n = 0; n <= num_kt && ok; ++n) {
            if (n < num_kt) ok = fetch(&map_k, n);
            if (n > 0 && ok) ok = fetch(&map_v, n - 1);
        }
        if (!waited) pdl_wait();
        return;  // the workers wait for every copy before they leave
    }
    if (!TMA && warp >= TD_WARPS) {
        // ---------------- copies: a warp takes every fourth row of a tile
        const int copier = warp - TD_WARPS;
        constexpr int ROWS_HERE = TD_KEYS / TD_COPY_WARPS;
        const int chunks = width / 8;
        int place[ROWS_HERE], place_before[ROWS_HERE];  // where the warp's key rows of a tile lie (in positions of the pool), -1: nowhere
#pragma unroll
        for (int i = 0; i < ROWS_HERE; ++i) place[i] = -1;
        int slot = 0, use = 0, reported = 0, pending = 0;
        bool ok = true;
        auto report = [&](int left) {
            __syncwarp();
            for (; pending > left; --pending) {
                if (lane == 0) td_arrive(full + reported);
                if (++reported == ring) reported = 0;
            }
        };
        auto fetch = [&](const __nv_bfloat16* cache, const int (&at)[ROWS_HERE]) {
            if (use > 0) {
                if (!__all_sync(0xffffffffu, mbar_wait(empty + slot, (use - 1) & 1, 1))) {  // report everything issued before waiting: no wait can be circular
                    cp_async_wait<0>();
                    report(0);
                    ok = __all_sync(0xffffffffu, td_wait(empty + slot, (use - 1) & 1, abort_word));
                    if (!ok) {
                        give_up();
                        return;
                    }
                }
            }
            __nv_bfloat16* tile = sRing + slot * tile_size;
#pragma unroll
            for (int i = 0; i < ROWS_HERE; ++i) {
                const bool valid = at[i] >= 0;
                const __nv_bfloat16* src = cache + (size_t)(valid ? at[i] : 0) * width;
                __nv_bfloat16* dst = tile + (size_t)(copier + i * TD_COPY_WARPS) * stride;
#pragma unroll 2
                for (int c = lane; c < chunks; c += 32) cp_async16(dst + c * 8, src + c * 8, valid);
            }
            cp_async_commit();
            ++pending;
            if (++slot == ring) {
                slot = 0;
                ++use;
            }
            if (pending > TD_IN_FLIGHT) {
                cp_async_wait<TD_IN_FLIGHT>();
                report(TD_IN_FLIGHT);
            }
        };
        for (int n = 0; n <= num_kt && ok; ++n) {
#pragma unroll
            for (int i = 0; i < ROWS_HERE; ++i) place_before[i] = place[i];
            if (n < num_kt) {
                const int key0 = key_of(n);
#pragma unroll
                for (int i = 0; i < ROWS_HERE; ++i) {
                    const int key = key0 + copier + i * TD_COPY_WARPS;
                    const int page_index = page_shift >= 0 ? key >> page_shift : key / page_size;
                    const int page = key <= pos && page_index < max_pages ? table[page_index] : -1;  // -1: a page the window has given back
                    place[i] = page >= 0 && page < num_pages ? page * page_size + (key - page_index * page_size) : -1;
                }
                if (n == 0) pdl_wait();  // the pages' numbers do not depend on the kernel before, the newest position's keys do
                fetch(k_cache, place);
            }
            if (n > 0 && ok) fetch(v_cache, place_before);
        }
        cp_async_wait<0>();
        report(0);
        return;
    }
    pdl_wait();

    // ---------------- work
    auto workers_sync = [&]() { asm volatile("bar.sync 1, %0;\n" ::"n"(TD_WORKERS) : "memory"); };
    const int steps = width / 16, per_part = (steps + TD_PARTS - 1) / TD_PARTS;
    const int key_half = warp & 1, part = warp >> 1;
    const int step0 = part * per_part, my_steps = max(0, min(per_part, steps - step0));
    // the warp's part of the queries, straight into the products' register layout (rows beyond the heads: zeros)
    uint32_t qa[MT][STEPS][4];
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
        for (int s = 0; s < STEPS; ++s) {
            const int r0 = mt * 16 + g, col = (step0 + s) * 16 + tq * 2;
            const __nv_bfloat16* src = q + (size_t)token * q_stride + col;
            const bool on = s < my_steps;
            qa[mt][s][0] = on && r0 < H ? *reinterpret_cast<const uint32_t*>(src + (size_t)r0 * width) : 0u;
            qa[mt][s][1] = on && r0 + 8 < H ? *reinterpret_cast<const uint32_t*>(src + (size_t)(r0 + 8) * width) : 0u;
            qa[mt][s][2] = on && r0 < H ? *reinterpret_cast<const uint32_t*>(src + (size_t)r0 * width + 8) : 0u;
            qa[mt][s][3] = on && r0 + 8 < H ? *reinterpret_cast<const uint32_t*>(src + (size_t)(r0 + 8) * width + 8) : 0u;
        }
    float o[UNITS][2][4];
#pragma unroll
    for (int u = 0; u < UNITS; ++u)
#pragma unroll
        for (int t = 0; t < 2; ++t) o[u][t][0] = o[u][t][1] = o[u][t][2] = o[u][t][3] = 0.0f;
    float m_row[ROW_TURNS], l_lane[ROW_TURNS];  // of the rows this warp's softmax takes: warp, warp + 8, ...
#pragma unroll
    for (int i = 0; i < ROW_TURNS; ++i) {
        m_row[i] = -INFINITY;
        l_lane[i] = 0.0f;
    }
    const float scale2 = scale * LOG2E;

    int head_of_unit[UNITS];  // the first query head of the unit's key/value head
#pragma unroll
    for (int u = 0; u < UNITS; ++u) head_of_unit[u] = ((warp + u * TD_WARPS) * 16 / D) * group;

    int slot = 0, use = 0;  // of the next item
    auto item_ready = [&]() {
        if (!td_wait(full + slot, use & 1, abort_word)) give_up();
        __syncwarp();
        return sRing + slot * tile_size;
    };
    auto item_done = [&]() {
        __syncwarp();
        if (lane == 0) td_arrive(empty + slot);
        if (++slot == ring) {
            slot = 0;
            ++use;
        }
    };
    for (int t = 0; t <= num_kt; ++t) {
        if (t < num_kt) {
            const __nv_bfloat16* tK = item_ready();
            const int k_row = key_half * 16 + (mm >> 1) * 8 + (lane & 7);
            float s[MT][2][4];
#pragma unroll
            for (int mt = 0; mt < MT; ++mt)
#pragma unroll
                for (int x = 0; x < 2; ++x) s[mt][x][0] = s[mt][x][1] = s[mt][x][2] = s[mt][x][3] = 0.0f;
#pragma unroll
            for (int ks = 0; ks < STEPS; ++ks) {
                if (ks >= my_steps) break;
                uint32_t b[4];
                ldmatrix_x4(b, tK + at16(k_row, (step0 + ks) * 2 + (mm & 1)));
#pragma unroll
                for (int mt = 0; mt < MT; ++mt) {
                    mma_16816(s[mt][0], qa[mt][ks], b[0], b[1]);
                    mma_16816(s[mt][1], qa[mt][ks], b[2], b[3]);
                }
            }
#pragma unroll
            for (int mt = 0; mt < MT; ++mt) {
                float* dst = sS + (size_t)(part * ROWS + mt * 16 + g) * TD_S_STRIDE + key_half * 16 + tq * 2;
#pragma unroll
                for (int x = 0; x < 2; ++x) {
                    *reinterpret_cast<float2*>(dst + x * 8) = make_float2(s[mt][x][0], s[mt][x][1]);
                    *reinterpret_cast<float2*>(dst + 8 * TD_S_STRIDE + x * 8) = make_float2(s[mt][x][2], s[mt][x][3]);
                }
            }
            item_done();
        }
        if (t > 0) {
            __nv_bfloat16* tV = item_ready();
            if constexpr (TMA) {
                // Rows nobody may see get probability 0, but 0 * NaN is NaN and what lies there may be anything: clear them, a
                // warp its own columns
                const int key0 = key_of(t - 1), key = key0 + lane;
                if (key0 + TD_KEYS - 1 > pos || (key0 < key_lo && key0 + TD_KEYS > keep_first)) {
                    if (!(key <= pos && (key >= key_lo || key < keep_first))) {
#pragma unroll
                        for (int u = 0; u < UNITS; ++u) {
                            const int unit = warp + u * TD_WARPS;
                            if (unit >= steps) break;
                            *reinterpret_cast<uint4*>(tV + at16(lane, unit * 2)) = make_uint4(0u, 0u, 0u, 0u);
                            *reinterpret_cast<uint4*>(tV + at16(lane, unit * 2 + 1)) = make_uint4(0u, 0u, 0u, 0u);
                        }
                    }
                    fence_proxy_async();  // these writes stay ordered before the copy that refills the buffer
                    __syncwarp();
                }
            }
#pragma unroll
            for (int u = 0; u < UNITS; ++u) {
                const int unit = warp + u * TD_WARPS;
                if (unit >= steps) break;
                const int head0 = head_of_unit[u];
                const float alpha0 = sAlpha[min(head0 + g, H - 1)], alpha1 = sAlpha[min(head0 + g + 8, H - 1)];
#pragma unroll
                for (int x = 0; x < 2; ++x) {
                    o[u][x][0] *= alpha0;
                    o[u][x][1] *= alpha0;
                    o[u][x][2] *= alpha1;
                    o[u][x][3] *= alpha1;
                }
                // rows beyond the group hold other heads' weights: their results are dropped
                const __nv_bfloat16* p_at = sP + (size_t)min(head0 + (mm & 1) * 8 + (lane & 7), H - 1) * TD_P_STRIDE + (mm >> 1) * 8;
#pragma unroll
                for (int kk = 0; kk < TD_KEYS / 16; ++kk) {
                    uint32_t a[4], b[4];
                    ldmatrix_x4(a, p_at + kk * 16);
                    ldmatrix_x4_trans(b, tV + at16(kk * 16 + (mm & 1) * 8 + (lane & 7), unit * 2 + (mm >> 1)));
                    mma_16816(o[u][0], a, b[0], b[1]);
                    mma_16816(o[u][1], a, b[2], b[3]);
                }
            }
            item_done();
        }
        workers_sync();
        if (t < num_kt) {
            const int key = key_of(t) + lane;
            const bool seen = key <= pos && (key >= key_lo || key < keep_first);
            float value[ROW_TURNS], top[ROW_TURNS];
#pragma unroll
            for (int i = 0; i < ROW_TURNS; ++i) {
                const float* src = sS + (size_t)(warp + i * TD_WARPS) * TD_S_STRIDE + lane;
                float raw = 0.0f;
#pragma unroll
                for (int x = 0; x < TD_PARTS; ++x) raw += src[x * ROWS * TD_S_STRIDE];
                value[i] = seen ? raw * scale2 : -INFINITY;
                top[i] = value[i];
            }
#pragma unroll
            for (int offset = 16; offset > 0; offset >>= 1)
#pragma unroll
                for (int i = 0; i < ROW_TURNS; ++i) top[i] = fmaxf(top[i], __shfl_xor_sync(0xffffffffu, top[i], offset));
#pragma unroll
            for (int i = 0; i < ROW_TURNS; ++i) {
                const int r = warp + i * TD_WARPS;
                const float m_new = fmaxf(m_row[i], top[i]);
                const float base = m_new == -INFINITY ? 0.0f : m_new;
                const float p = exp2f(value[i] - base);
                const float alpha = exp2f(m_row[i] - base);
                l_lane[i] = l_lane[i] * alpha + p;
                m_row[i] = m_new;
                sP[r * TD_P_STRIDE + lane] = __float2bfloat16_rn(p);
                if (lane == 0) sAlpha[r] = alpha;
            }
        }
        workers_sync();
    }
#pragma unroll
    for (int i = 0; i < ROW_TURNS; ++i) {
        const float sum = warp_sum(l_lane[i]);
        if (lane == 0) {
            sM[warp + i * TD_WARPS] = m_row[i];
            sL[warp + i * TD_WARPS] = sum;
        }
    }
    workers_sync();
#pragma unroll
    for (int u = 0; u < UNITS; ++u) {
        const int unit = warp + u * TD_WARPS;
        if (unit >= steps) break;
        const int c = unit * 16 / D, col = unit * 16 - c * D + tq * 2;
#pragma unroll
        for (int half = 0; half < 2; ++half) {
            const int in_group = g + half * 8;
            if (in_group >= group) continue;
            const int h = c * group + in_group;
            if (splits > 1) {
                float* dst = part_o + (((size_t)split * gridDim.y + index) * H + h) * D + col;
#pragma unroll
                for (int x = 0; x < 2; ++x) *reinterpret_cast<float2*>(dst + x * 8) = make_float2(o[u][x][half * 2], o[u][x][half * 2 + 1]);
            } else {
                const float inv = sL[h] > 0.0f ? 1.0f / sL[h] : 0.0f;
                __nv_bfloat16* dst = out + (size_t)token * out_stride + (size_t)h * D + col;
#pragma unroll
                for (int x = 0; x < 2; ++x)
                    *reinterpret_cast<__nv_bfloat162*>(dst + x * 8) = __floats2bfloat162_rn(o[u][x][half * 2] * inv, o[u][x][half * 2 + 1] * inv);
            }
        }
    }
    if (TMA && *abort_word && threadIdx.x == 0) {
        // copies that are still in flight target this block's shared memory: one more short wait on the barriers they complete
        for (int i = 0; i < ring; ++i) {
            mbar_wait(full + i, 0, 1024);
            mbar_wait(full + i, 1, 1024);
        }
    }
    if (splits > 1)
        for (int h = threadIdx.x; h < H; h += TD_WORKERS) {
            float* ml = part_ml + (((size_t)split * gridDim.y + index) * H + h) * 2;
            ml[0] = sM[h];
            ml[1] = sL[h];
        }
}

// The splits' results of a token and head, in split order.
__global__ void __launch_bounds__(128)
talking_decode_merge_kernel(const float* __restrict__ part_o, const float* __restrict__ part_ml, __nv_bfloat16* __restrict__ out,
                            int out_stride, const int* __restrict__ list_tokens, int H, int D, int splits, int count) {
    pdl_trigger();
    const int index = blockIdx.x, h = blockIdx.y;
    const int token = list_tokens[index];
    pdl_wait();
    float top = -INFINITY;
    for (int s = 0; s < splits; ++s) top = fmaxf(top, part_ml[(((size_t)s * count + index) * H + h) * 2]);
    for (int d = threadIdx.x; d < D; d += 128) {
        float value = 0.0f, denom = 0.0f;
#pragma unroll 4
        for (int s = 0; s < splits; ++s) {
            const size_t at = ((size_t)s * count + index) * H + h;
            const float m = part_ml[at * 2];
            if (m == -INFINITY) continue;
            const float weight = exp2f(m - top);
            denom += part_ml[at * 2 + 1] * weight;
            value += part_o[at * D + d] * weight;
        }
        out[(size_t)token * out_stride + (size_t)h * D + d] = __float2bfloat16_rn(denom > 0.0f ? value / denom : 0.0f);
    }
}

static bool td_shape(int H, int G, int D, int page_size, TdShape* shape) {
    if (G < 1 || H < 1 || H % G != 0 || H / G > 16 || H > 32 || D < 16 || D % 16 != 0 || G * D > 512) return false;
    TdShape s = {H, G, D, G * D, (H + 15) / 16, TD_MAX_RING, 0};
    s.tma = s.width % 64 == 0 && page_size >= 8 && (page_size & (page_size - 1)) == 0;
    while (td_smem(s) > TD_SMEM_LIMIT) --s.ring;  // five at the widest row and 32 heads
    *shape = s;
    return true;
}

KB_EXPORT int kb_talking_decode_supported(int H, int G, int D) {
    TdShape shape;
    return td_shape(H, G, D, 16, &shape) ? 1 : 0;
}

// Whether the kernel wants the caches' tensor maps (kb_talking_decode_encode_map) for these sizes.
KB_EXPORT int kb_talking_decode_uses_tma(int H, int G, int D, int page_size) {
    TdShape shape;
    return td_shape(H, G, D, page_size, &shape) && shape.tma ? 1 : 0;
}

// Writes a 128-byte tensor map (host memory, 64-byte aligned) over a bf16 cache [num_pages, page_size, width]: four dimensions
// (64 columns, positions, bands of columns, pages), boxes of min(page_size, 32) positions with every band.  128-byte swizzle.
KB_EXPORT int kb_talking_decode_encode_map(void* map_out, const void* base, long long num_pages, int page_size, int width) {
    if (!map_out || !base) return KB_ERR_NULL;
    if (((uintptr_t)map_out % 64) != 0 || ((uintptr_t)base % 16) != 0) return KB_ERR_BAD_ARG;
    if (width % 64 != 0 || width > 512 || page_size < 8 || (page_size & (page_size - 1)) != 0 || num_pages < 1) return KB_ERR_UNSUPPORTED_SIZE;
    static PFN_cuTensorMapEncodeTiled encode = nullptr;
    if (!encode) {
        void* fn = nullptr;
        cudaDriverEntryPointQueryResult status;
        const cudaError_t e = cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &fn, cudaEnableDefault, &status);
        if (e != cudaSuccess) return (int)e;
        if (!fn) return KB_ERR_NULL;
        encode = (PFN_cuTensorMapEncodeTiled)fn;
    }
    const cuuint64_t dims[4] = {64, (cuuint64_t)page_size, (cuuint64_t)(width / 64), (cuuint64_t)num_pages};
    const cuuint64_t strides[3] = {(cuuint64_t)width * 2, 128, (cuuint64_t)page_size * width * 2};
    const cuuint32_t box[4] = {64, (cuuint32_t)(page_size < TD_KEYS ? page_size : TD_KEYS), (cuuint32_t)(width / 64), 1};
    const cuuint32_t elem[4] = {1, 1, 1, 1};
    const CUresult r = encode((CUtensorMap*)map_out, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 4, const_cast<void*>(base), dims, strides, box, elem,
                              CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                              CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
    return r == CUDA_SUCCESS ? 0 : 1000 + (int)r;
}

// How many blocks share a token's keys: enough to fill the device once, each with at least two tiles.
KB_EXPORT int kb_talking_decode_splits(int count, int keys, int H, int G, int D, int page_size) {
    TdShape shape;
    static int sms = 0;
    if (sms == 0) {
        int device = 0;
        cudaGetDevice(&device);
        cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, device);
    }
    if (count < 1 || !td_shape(H, G, D, page_size, &shape)) return 1;
    const int resident = (int)((227 * 1024) / (td_smem(shape) + 1024));
    const int places = sms * (resident < 1 ? 1 : resident > 2 ? 2 : resident);
    const int tiles = (keys + TD_KEYS - 1) / TD_KEYS;
    int splits = places / count;
    if (splits > tiles / 2) splits = tiles / 2;
    return splits < 1 ? 1 : splits > 64 ? 64 : splits;
}

template <int MT, int STEPS, bool TMA>
static void launch_decode(size_t smem, cudaStream_t stream, const CUtensorMap& map_k, const CUtensorMap& map_v, const void* q, int q_stride, void* out, int out_stride, const void* k_cache,
                          const void* v_cache, const int* seq_lens, const int* block_table, int max_pages, const int* list_rows,
                          const int* list_tokens, const TdShape& shape, int count, int page_size, int shift, int num_pages, float scale,
                          int window, int keep_first, int splits, float* part_o, float* part_ml, int* flag) {
    static bool configured = false;
    if (!configured) {
        cudaFuncSetAttribute(talking_decode_kernel<MT, STEPS, TMA>, cudaFuncAttributeMaxDynamicSharedMemorySize, TD_SMEM_LIMIT);
        configured = true;
    }
    kb_launch(talking_decode_kernel<MT, STEPS, TMA>, dim3(splits, count), dim3(TD_THREADS(TMA)), smem, stream, map_k, map_v, (const __nv_bfloat16*)q, q_stride,
              (__nv_bfloat16*)out, out_stride, (const __nv_bfloat16*)k_cache, (const __nv_bfloat16*)v_cache, seq_lens, block_table, max_pages,
              list_rows, list_tokens, shape, page_size, shift, num_pages, scale, window, keep_first, splits, part_o, part_ml, flag);
}

// map_k, map_v: host pointers to the caches' tensor maps where kb_talking_decode_uses_tma asks for them.
KB_EXPORT int kb_talking_decode(const void* map_k, const void* map_v, const void* q, int q_stride, void* out, int out_stride, const void* k_cache, const void* v_cache,
                                const int* seq_lens, const int* block_table, int max_pages, const int* list_rows, const int* list_tokens,
                                int count, int H, int G, int D, int page_size, int num_pages, float scale, int window, int keep_first,
                                int splits, float* part_o, float* part_ml, int* flag, cudaStream_t stream) {
    if (count == 0) return 0;
    if (!q || !out || !k_cache || !v_cache || !seq_lens || !block_table || !list_rows || !list_tokens || (splits > 1 && (!part_o || !part_ml))) return KB_ERR_NULL;
    TdShape shape;
    if (!td_shape(H, G, D, page_size, &shape)) return KB_ERR_UNSUPPORTED_SIZE;
    if (shape.tma && (!map_k || !map_v)) return KB_ERR_NULL;
    if (count > 65535 || splits < 1 || page_size < 1 || keep_first < 0 || q_stride % 8 || out_stride % 2
        || (((uintptr_t)q | (uintptr_t)k_cache | (uintptr_t)v_cache) % 16) || ((uintptr_t)out % 4)) return KB_ERR_BAD_ARG;
    if ((long long)num_pages * page_size > 0x7fffffffLL) return KB_ERR_UNSUPPORTED_SIZE;
    const size_t smem = td_smem(shape);
    int shift = -1;
    if ((page_size & (page_size - 1)) == 0) {
        shift = 0;
        while ((1 << shift) < page_size) ++shift;
    }
    const CUtensorMap none = {};
    const CUtensorMap& mk = shape.tma ? *reinterpret_cast<const CUtensorMap*>(map_k) : none;
    const CUtensorMap& mv = shape.tma ? *reinterpret_cast<const CUtensorMap*>(map_v) : none;
#define LAUNCH_AS(MT, STEPS, TMA)                                                                                                              \
    launch_decode<MT, STEPS, TMA>(smem, stream, mk, mv, q, q_stride, out, out_stride, k_cache, v_cache, seq_lens, block_table, max_pages,      \
                                  list_rows, list_tokens, shape, count, page_size, shift, num_pages, scale, window, keep_first, splits, part_o, \
                                  part_ml, flag)
#define LAUNCH(MT, STEPS)                         \
    do {                                          \
        if (shape.tma) LAUNCH_AS(MT, STEPS, true); \
        else LAUNCH_AS(MT, STEPS, false);          \
    } while (0)
    if (shape.row_tiles == 1) {
        if (shape.width <= 128) LAUNCH(1, 1);
        else if (shape.width <= 256) LAUNCH(1, 2);
        else LAUNCH(1, 4);
    } else {
        if (shape.width <= 128) LAUNCH(2, 1);
        else if (shape.width <= 256) LAUNCH(2, 2);
        else LAUNCH(2, 4);
    }
#undef LAUNCH
#undef LAUNCH_AS
    if (splits > 1)
        kb_launch(talking_decode_merge_kernel, dim3(count, H), dim3(128), 0, stream, (const float*)part_o, (const float*)part_ml, (__nv_bfloat16*)out,
                  out_stride, list_tokens, H, D, splits, count);
    return kb_launch_result();
}
