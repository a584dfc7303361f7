// Flash attention of single tokens where all query heads of a position share ONE wide key row and take their values from their
// own key/value head (the mixed queries of talking_attention.cu), on mma.sync m16n8k16 with 32-bit scores, softmax and sums:
//
//     S = Q K^T * scale      Q [tokens, H, G * D], K: the G key/value heads' keys of a position side by side
//     P = softmax over the keys the token sees: itself and the window - 1 before it (window 0: all), and the sequence's first
//         keep_first tokens;   O_h = P_h V_c(h)
//
// The H heads are the rows of the products (sixteen a product, as many as a product has anyway), so the wide key row costs no
// more than G separate heads' keys would, and a request's keys and values are read once for all heads.
// A block (8 warps) walks a share of one request's keys in tiles of 32 at absolute multiples of 32, first the tiles of the kept
// first tokens, then the window's, through a ring of cp.async buffers.  Per tile: S, each warp 8 keys and half of the key
// columns; softmax, a warp a row at a time with a lane a key; P V, each warp its 16-column units of the value row (a unit
// lies in one key/value head and takes that head's rows of P).  With the keys split over blocks the unnormalised results
// are combined by a second kernel in split order, so a result depends on the token's position and the number of splits.
#include "attention_mma.cuh"

#define TD_THREADS 256
#define TD_WARPS 8
#define TD_KEYS 32
#define TD_P_STRIDE (TD_KEYS + 8)
#define TD_S_STRIDE (TD_KEYS + 2)
#define TD_SMEM_LIMIT (220 * 1024)

struct TdShape {
    int H, G, D, width;  // width = G * D
    int row_tiles;       // sixteens of query heads
    int stages;
};

__host__ __device__ static inline size_t td_smem(const TdShape& s) {
    const size_t stride = s.width + 8, rows = 16 * s.row_tiles;
    return (rows * stride + (size_t)s.stages * 2 * TD_KEYS * stride + rows * TD_P_STRIDE) * sizeof(__nv_bfloat16)
           + (2 * rows * TD_S_STRIDE + 3 * rows) * sizeof(float);
}

template <int UNITS>  // 16-column units of the value row a warp owns at most
__global__ void __launch_bounds__(TD_THREADS)
talking_decode_kernel(const __nv_bfloat16* __restrict__ q, int q_stride, __nv_bfloat16* __restrict__ out, int out_stride,
                      const __nv_bfloat16* __restrict__ k_cache, const __nv_bfloat16* __restrict__ v_cache, const int* __restrict__ seq_lens,
                      const int* __restrict__ block_table, int max_pages, const int* __restrict__ list_rows,
                      const int* __restrict__ list_tokens, const TdShape shape, int page_size, int page_shift, int num_pages, float scale,
                      int window, int keep_first, int splits, float* __restrict__ part_o, float* __restrict__ part_ml) {
    extern __shared__ __align__(16) unsigned char smem_raw[];
    const int H = shape.H, D = shape.D, width = shape.width, stride = width + 8, rows = 16 * shape.row_tiles, stages = shape.stages;
    __nv_bfloat16* sQ = reinterpret_cast<__nv_bfloat16*>(smem_raw);
    __nv_bfloat16* sKV = sQ + (size_t)rows * stride;  // per stage: 32 key rows, then 32 value rows
    const size_t stage_size = (size_t)2 * TD_KEYS * stride;
    __nv_bfloat16* sP = sKV + stages * stage_size;
    float* sS = reinterpret_cast<float*>(sP + (size_t)rows * TD_P_STRIDE);  // [column half][row][key]
    float* sAlpha = sS + 2 * rows * TD_S_STRIDE;
    float* sM = sAlpha + rows;
    float* sL = sM + rows;

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
        for (int h = threadIdx.x; h < H; h += TD_THREADS) {
            float* ml = part_ml + (((size_t)split * gridDim.y + index) * H + h) * 2;
            ml[0] = -INFINITY;
            ml[1] = 0.0f;
        }
        return;
    }
    const int chunks = width / 8;
    auto load_tile = [&](int n, int stage) {
        __nv_bfloat16* tK = sKV + stage * stage_size;
        __nv_bfloat16* tV = tK + (size_t)TD_KEYS * stride;
        const int key0 = key_of(n);
#pragma unroll
        for (int i = 0; i < TD_KEYS / TD_WARPS; ++i) {
            const int r = warp + i * TD_WARPS;
            const int key = key0 + r;
            bool valid = key <= pos;
            size_t place = 0;
            if (valid) {
                const int page_index = page_shift >= 0 ? key >> page_shift : key / page_size;
                const int page = page_index < max_pages ? table[page_index] : -1;  // -1: a page the window has given back
                valid = page >= 0 && page < num_pages;
                if (valid) place = ((size_t)page * page_size + (key - page_index * page_size)) * width;
            }
            for (int c = lane; c < chunks; c += 32) {
                cp_async16(tK + (size_t)r * stride + c * 8, k_cache + place + (valid ? c * 8 : 0), valid);
                cp_async16(tV + (size_t)r * stride + c * 8, v_cache + place + (valid ? c * 8 : 0), valid);
            }
        }
    };
    pdl_wait();
    for (int r = warp; r < rows; r += TD_WARPS)
        for (int c = lane; c < chunks; c += 32)
            cp_async16(sQ + (size_t)r * stride + c * 8, q + (size_t)token * q_stride + (r < H ? (size_t)r * width + c * 8 : 0), r < H);
    // one copy group a tile, also where there is no tile left, so that "all but the last groups" always names the tile at hand
    for (int ahead = 0; ahead < stages - 1; ++ahead) {
        if (ahead < num_kt) load_tile(ahead, ahead);
        cp_async_commit();
    }
    for (int r = threadIdx.x; r < rows; r += TD_THREADS) {
        sM[r] = -INFINITY;
        sL[r] = 0.0f;
    }

    float o[UNITS][2][4];
#pragma unroll
    for (int u = 0; u < UNITS; ++u)
#pragma unroll
        for (int t = 0; t < 2; ++t) o[u][t][0] = o[u][t][1] = o[u][t][2] = o[u][t][3] = 0.0f;
    const int units = width / 16;
    const int ksteps = width / 16, half_steps = (ksteps + 1) / 2;
    const int key_group = warp & 3, part = warp >> 2;
    const int k_begin = part ? half_steps : 0, k_end = part ? ksteps : half_steps;
    const float scale2 = scale * LOG2E;

    int stage = 0;
    for (int n = 0; n < num_kt; ++n) {
        if (n + stages - 1 < num_kt) load_tile(n + stages - 1, (stage + stages - 1) % stages);  // the buffer of the tile before
        cp_async_commit();
        if (stages == 3) cp_async_wait<2>(); else cp_async_wait<1>();
        __syncthreads();
        const __nv_bfloat16* tK = sKV + stage * stage_size;
        const __nv_bfloat16* tV = tK + (size_t)TD_KEYS * stride;
        // S: this warp's 8 keys, its half of the key columns, sixteen heads at a time
        for (int mt = 0; mt < shape.row_tiles; ++mt) {
            float s[4] = {0.0f, 0.0f, 0.0f, 0.0f};
            const __nv_bfloat16* q_at = sQ + (size_t)(mt * 16 + (mm & 1) * 8 + (lane & 7)) * stride + (mm >> 1) * 8;
            const __nv_bfloat16* k_at = tK + (size_t)(key_group * 8 + (lane & 7)) * stride + mm * 8;
#pragma unroll 4
            for (int ks = k_begin; ks < k_end; ks += 2) {
                uint32_t a[4], b[4];
                ldmatrix_x4(b, k_at + ks * 16);  // the keys' columns of two steps
                ldmatrix_x4(a, q_at + ks * 16);
                mma_16816(s, a, b[0], b[1]);
                if (ks + 1 < k_end) {
                    ldmatrix_x4(a, q_at + ks * 16 + 16);
                    mma_16816(s, a, b[2], b[3]);
                }
            }
            float* dst = sS + ((size_t)part * rows + mt * 16 + g) * TD_S_STRIDE + key_group * 8 + tq * 2;
            *reinterpret_cast<float2*>(dst) = make_float2(s[0], s[1]);
            *reinterpret_cast<float2*>(dst + 8 * TD_S_STRIDE) = make_float2(s[2], s[3]);
        }
        __syncthreads();
        // softmax: a warp a row, a lane a key
        {
            const int key = key_of(n) + lane;
            const bool seen = key <= pos && (key >= key_lo || key < keep_first);
            for (int r = warp; r < H; r += TD_WARPS) {
                const float raw = (sS[(size_t)r * TD_S_STRIDE + lane] + sS[((size_t)rows + r) * TD_S_STRIDE + lane]) * scale2;
                const float value = seen ? raw : -INFINITY;
                const float before = sM[r];
                const float top = fmaxf(before, warp_max(value));
                const float base = top == -INFINITY ? 0.0f : top;
                const float p = exp2f(value - base);
                const float alpha = exp2f(before - base);
                const float sum = warp_sum(p);
                sP[(size_t)r * TD_P_STRIDE + lane] = __float2bfloat16_rn(p);
                __syncwarp();
                if (lane == 0) {
                    sM[r] = top;
                    sL[r] = sL[r] * alpha + sum;
                    sAlpha[r] = alpha;
                }
            }
        }
        __syncthreads();
        // O: this warp's units of the value row
#pragma unroll
        for (int u = 0; u < UNITS; ++u) {
            const int unit = warp + u * TD_WARPS;
            if (unit >= units) break;
            const int head0 = (unit * 16 / D) * group;  // the first query head of the unit's key/value head
            const float alpha0 = sAlpha[min(head0 + g, H - 1)], alpha1 = sAlpha[min(head0 + g + 8, H - 1)];
#pragma unroll
            for (int t = 0; t < 2; ++t) {
                o[u][t][0] *= alpha0;
                o[u][t][1] *= alpha0;
                o[u][t][2] *= alpha1;
                o[u][t][3] *= alpha1;
            }
            // rows beyond the group hold other heads' weights: their results are dropped
            const __nv_bfloat16* p_at = sP + (size_t)min(head0 + (mm & 1) * 8 + (lane & 7), H - 1) * TD_P_STRIDE + (mm >> 1) * 8;
#pragma unroll
            for (int kk = 0; kk < TD_KEYS / 16; ++kk) {
                uint32_t a[4], b[4];
                ldmatrix_x4(a, p_at + kk * 16);
                ldmatrix_x4_trans(b, tV + (size_t)(kk * 16 + (mm & 1) * 8 + (lane & 7)) * stride + unit * 16 + (mm >> 1) * 8);
                mma_16816(o[u][0], a, b[0], b[1]);
                mma_16816(o[u][1], a, b[2], b[3]);
            }
        }
        __syncthreads();  // the buffer is refilled by the next turn's request
        stage = (stage + 1) % stages;
    }
    cp_async_wait<0>();
#pragma unroll
    for (int u = 0; u < UNITS; ++u) {
        const int unit = warp + u * TD_WARPS;
        if (unit >= units) break;
        const int c = unit * 16 / D, col = unit * 16 - c * D + tq * 2;
#pragma unroll
        for (int half = 0; half < 2; ++half) {
            const int in_group = g + half * 8;
            if (in_group >= group) continue;
            const int h = c * group + in_group;
            if (splits > 1) {
                float* dst = part_o + (((size_t)split * gridDim.y + index) * H + h) * D + col;
#pragma unroll
                for (int t = 0; t < 2; ++t) *reinterpret_cast<float2*>(dst + t * 8) = make_float2(o[u][t][half * 2], o[u][t][half * 2 + 1]);
            } else {
                const float inv = sL[h] > 0.0f ? 1.0f / sL[h] : 0.0f;
                __nv_bfloat16* dst = out + (size_t)token * out_stride + (size_t)h * D + col;
#pragma unroll
                for (int t = 0; t < 2; ++t)
                    *reinterpret_cast<__nv_bfloat162*>(dst + t * 8) = __floats2bfloat162_rn(o[u][t][half * 2] * inv, o[u][t][half * 2 + 1] * inv);
            }
        }
    }
    if (splits > 1)
        for (int h = threadIdx.x; h < H; h += TD_THREADS) {
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

static bool td_shape(int H, int G, int D, TdShape* shape) {
    if (G < 1 || H < 1 || H % G != 0 || H / G > 16 || H > 64 || D < 16 || D % 16 != 0 || G * D > 16 * TD_WARPS * 8) return false;
    TdShape s = {H, G, D, G * D, (H + 15) / 16, 3};
    if (td_smem(s) > TD_SMEM_LIMIT) s.stages = 2;
    if (td_smem(s) > TD_SMEM_LIMIT) return false;
    *shape = s;
    return true;
}

KB_EXPORT int kb_talking_decode_supported(int H, int G, int D) {
    TdShape shape;
    return td_shape(H, G, D, &shape) ? 1 : 0;
}

// How many blocks share a token's keys: enough to fill the device once, each with at least two tiles.
KB_EXPORT int kb_talking_decode_splits(int count, int keys, int H, int G, int D) {
    TdShape shape;
    static int sms = 0;
    if (sms == 0) {
        int device = 0;
        cudaGetDevice(&device);
        cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, device);
    }
    if (count < 1 || !td_shape(H, G, D, &shape)) return 1;
    const int resident = (int)((227 * 1024) / (td_smem(shape) + 1024));
    const int places = sms * (resident < 1 ? 1 : resident > 4 ? 4 : resident);
    const int tiles = (keys + TD_KEYS - 1) / TD_KEYS;
    int splits = places / count;
    if (splits > tiles / 2) splits = tiles / 2;
    return splits < 1 ? 1 : splits > 64 ? 64 : splits;
}

KB_EXPORT int kb_talking_decode(const void* q, int q_stride, void* out, int out_stride, const void* k_cache, const void* v_cache,
                                const int* seq_lens, const int* block_table, int max_pages, const int* list_rows, const int* list_tokens,
                                int count, int H, int G, int D, int page_size, int num_pages, float scale, int window, int keep_first,
                                int splits, float* part_o, float* part_ml, cudaStream_t stream) {
    if (count == 0) return 0;
    if (!q || !out || !k_cache || !v_cache || !seq_lens || !block_table || !list_rows || !list_tokens || (splits > 1 && (!part_o || !part_ml))) return KB_ERR_NULL;
    TdShape shape;
    if (!td_shape(H, G, D, &shape)) return KB_ERR_UNSUPPORTED_SIZE;
    if (count > 65535 || splits < 1 || page_size < 1 || keep_first < 0 || q_stride % 8 || out_stride % 2
        || (((uintptr_t)q | (uintptr_t)k_cache | (uintptr_t)v_cache) % 16) || ((uintptr_t)out % 4)) return KB_ERR_BAD_ARG;
    const size_t smem = td_smem(shape);
    int shift = -1;
    if ((page_size & (page_size - 1)) == 0) {
        shift = 0;
        while ((1 << shift) < page_size) ++shift;
    }
#define LAUNCH(U)                                                                                                                             \
    do {                                                                                                                                      \
        static bool configured = false;                                                                                                       \
        if (!configured) {                                                                                                                    \
            cudaFuncSetAttribute(talking_decode_kernel<U>, cudaFuncAttributeMaxDynamicSharedMemorySize, TD_SMEM_LIMIT);                         \
            configured = true;                                                                                                                \
        }                                                                                                                                     \
        kb_launch(talking_decode_kernel<U>, dim3(splits, count), dim3(TD_THREADS), smem, stream, (const __nv_bfloat16*)q, q_stride,            \
                  (__nv_bfloat16*)out, out_stride, (const __nv_bfloat16*)k_cache, (const __nv_bfloat16*)v_cache, seq_lens, block_table,         \
                  max_pages, list_rows, list_tokens, shape, page_size, shift, num_pages, scale, window, keep_first, splits,       \
                  part_o, part_ml);                                                                                                           \
    } while (0)
    const int per_warp = (shape.width / 16 + TD_WARPS - 1) / TD_WARPS;
    if (per_warp <= 2) LAUNCH(2);
    else if (per_warp <= 4) LAUNCH(4);
    else LAUNCH(8);
#undef LAUNCH
    if (splits > 1)
        kb_launch(talking_decode_merge_kernel, dim3(count, H), dim3(128), 0, stream, (const float*)part_o, (const float*)part_ml, (__nv_bfloat16*)out,
                  out_stride, list_tokens, H, D, splits, count);
    return kb_launch_result();
}
