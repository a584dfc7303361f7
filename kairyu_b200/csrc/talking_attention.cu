// What goes before attention whose heads' scores are mixed before the softmax ("talking heads"):
//
//     score_h(i, j) = sum_g T[h, g] * (q_g(i) . k_c(g)(j)) * scale          c(g): the key/value head of query head g
//
// The mix is linear in the queries, so it needs no pass over the scores: with the key/value heads' keys of a position side
// by side as ONE row of G * D columns, and the mixed query
//
//     Q_h(i) = [ sum_{g of head 0} T[h, g] q_g(i) | sum_{g of head 1} T[h, g] q_g(i) | ... ]      G * D columns
//
// score_h(i, j) = Q_h(i) . [k_0(j) | k_1(j) | ...] * scale, and attention is that of query heads which all share one key
// row and take their values from their own key/value head.  The mixed queries are formed here in 32-bit from the rotated
// 32-bit queries and rounded once.
//
// One block a token, on the packed rows [q | k | (v) | ...]:
//   q (32-bit) turns by the token's position (the first 2 * rot_half columns of a head, pairs (i, i + rot_half)), is mixed,
//   and goes to `mixed` [tokens, H * G * D]; k turns and goes to its page; the value row (the columns from v_offset on: with
//   v_offset = k_offset a value is the key as projected, before its turn) goes to its page.
#include "common.cuh"

#define TP_THREADS 256

template <typename T, int VEC>
struct Columns {
    float v[VEC];
};

template <typename T, int VEC>
__device__ __forceinline__ Columns<T, VEC> load_columns(const T* p) {
    Columns<T, VEC> c;
    if constexpr (VEC == 8 && sizeof(T) == 2) {
        const uint4 raw = *reinterpret_cast<const uint4*>(p);
        const uint32_t words[4] = {raw.x, raw.y, raw.z, raw.w};
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const float2 f = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&words[i]));
            c.v[2 * i] = f.x;
            c.v[2 * i + 1] = f.y;
        }
    } else {
#pragma unroll
        for (int i = 0; i < VEC; ++i) c.v[i] = to_float(p[i]);
    }
    return c;
}

template <typename T, int VEC>
__device__ __forceinline__ void store_columns(T* p, const float (&v)[VEC]) {
    if constexpr (VEC == 8 && sizeof(T) == 2) {
        uint32_t words[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const __nv_bfloat162 pair = __floats2bfloat162_rn(v[2 * i], v[2 * i + 1]);
            words[i] = *reinterpret_cast<const uint32_t*>(&pair);
        }
        *reinterpret_cast<uint4*>(p) = make_uint4(words[0], words[1], words[2], words[3]);
    } else {
#pragma unroll
        for (int i = 0; i < VEC; ++i) p[i] = from_float<T>(v[i]);
    }
}

// VEC columns from `d` on of a head's row, turned (VEC divides rot_half and D, or is 1)
template <typename T, int VEC>
__device__ __forceinline__ Columns<T, VEC> turned(const T* head, int d, int half, const float* cos_row, const float* sin_row) {
    Columns<T, VEC> own = load_columns<T, VEC>(head + d);
    if (d >= 2 * half) return own;
    const bool first = d < half;
    const Columns<T, VEC> other = load_columns<T, VEC>(head + (first ? d + half : d - half));
    const int a = first ? d : d - half;
    float cs[VEC], sn[VEC];
    if constexpr (VEC == 8) {
#pragma unroll
        for (int i = 0; i < 8; i += 4) {  // rows of the tables start on 16 bytes: half is a multiple of 8
            const float4 c4 = *reinterpret_cast<const float4*>(cos_row + a + i), s4 = *reinterpret_cast<const float4*>(sin_row + a + i);
            cs[i] = c4.x; cs[i + 1] = c4.y; cs[i + 2] = c4.z; cs[i + 3] = c4.w;
            sn[i] = s4.x; sn[i + 1] = s4.y; sn[i + 2] = s4.z; sn[i + 3] = s4.w;
        }
    } else {
#pragma unroll
        for (int i = 0; i < VEC; ++i) {
            cs[i] = cos_row[a + i];
            sn[i] = sin_row[a + i];
        }
    }
#pragma unroll
    for (int i = 0; i < VEC; ++i) {
        const float c = cs[i], s = sn[i];
        own.v[i] = first ? own.v[i] * c - other.v[i] * s : own.v[i] * c + other.v[i] * s;
    }
    return own;
}

// GROUP: query heads a key/value head that the mixing loop keeps in registers (0: it reads them from shared memory)
template <typename T, int VEC, int GROUP>
__global__ void __launch_bounds__(TP_THREADS)
talking_prepare_kernel(const T* __restrict__ packed, int stride, int k_offset, int v_offset, int H, int G, int D, const float* __restrict__ talk,
                       const float* __restrict__ cos, const float* __restrict__ sin, int half, int max_pos, const int* __restrict__ positions,
                       const int* __restrict__ row_ids, const int* __restrict__ block_table, int max_pages, int num_rows,
                       const int* __restrict__ write_from, T* __restrict__ k_cache, T* __restrict__ v_cache, int page_size, int num_pages,
                       T* __restrict__ mixed, int mixed_stride, int* flag) {
    extern __shared__ __align__(16) float shared[];
    float* qs = shared;                  // [H * D] turned queries
    float* ts = shared + (size_t)H * D;  // [H * H]
    const int t = blockIdx.x;
    const int pos = positions[t];
    const int row = row_ids[t];
    for (int i = threadIdx.x; i < H * H; i += TP_THREADS) ts[i] = talk[i];
    int page = -1;
    bool write = k_cache != nullptr;
    if (write && (row < 0 || row >= num_rows)) {
        if (threadIdx.x == 0 && flag) atomicOr(flag, KB_FLAG_BAD_ROW);
        write = false;
    }
    if (write && write_from && pos < write_from[row]) write = false;
    if (write) {
        const int page_index = pos / page_size;
        page = (pos >= 0 && page_index < max_pages) ? block_table[(size_t)row * max_pages + page_index] : -1;
        if (page < 0 || page >= num_pages) {
            if (threadIdx.x == 0 && flag) atomicOr(flag, KB_FLAG_BAD_PAGE);
            write = false;
        }
    }
    int turn = half;
    if (turn > 0 && (pos < 0 || pos >= max_pos)) {
        if (threadIdx.x == 0 && flag) atomicOr(flag, KB_FLAG_BAD_POS);
        turn = 0;
    }
    const float* cos_row = cos + (size_t)(turn > 0 ? pos : 0) * half;
    const float* sin_row = sin + (size_t)(turn > 0 ? pos : 0) * half;
    pdl_wait();
    const T* src = packed + (size_t)t * stride;
    for (int e = threadIdx.x * VEC; e < H * D; e += TP_THREADS * VEC) {
        const int head = e / D, d = e - head * D;
        const Columns<T, VEC> c = turned<T, VEC>(src + head * D, d, turn, cos_row, sin_row);
        if constexpr (VEC == 8) {
            *reinterpret_cast<float4*>(qs + e) = make_float4(c.v[0], c.v[1], c.v[2], c.v[3]);
            *reinterpret_cast<float4*>(qs + e + 4) = make_float4(c.v[4], c.v[5], c.v[6], c.v[7]);
        } else {
#pragma unroll
            for (int i = 0; i < VEC; ++i) qs[e + i] = c.v[i];
        }
    }
    if (write) {
        const size_t place = ((size_t)page * page_size + (pos - (pos / page_size) * page_size)) * G * D;
        for (int e = threadIdx.x * VEC; e < G * D; e += TP_THREADS * VEC) {
            const int head = e / D, d = e - head * D;
            const Columns<T, VEC> c = turned<T, VEC>(src + k_offset + head * D, d, turn, cos_row, sin_row);
            store_columns<T, VEC>(k_cache + place + e, c.v);
            const Columns<T, VEC> raw = load_columns<T, VEC>(src + v_offset + e);
            store_columns<T, VEC>(v_cache + place + e, raw.v);
        }
    }
    __syncthreads();
    const int group = H / G, row_width = G * D;
    T* dst = mixed + (size_t)t * mixed_stride;
    if constexpr (GROUP > 0) {
        // a thread holds its eight columns of the group's queries in registers and walks the heads
        const int columns = row_width / 8;
        const int lanes = columns < TP_THREADS ? columns : TP_THREADS;
        const int walkers = TP_THREADS / lanes;  // threads that share the heads of a column group
        const int walker = threadIdx.x / lanes;
        for (int e = threadIdx.x - walker * lanes; e < columns && walker < walkers; e += lanes) {
            const int c = e * 8 / D, d = e * 8 - c * D;
            float4 lo[GROUP], hi[GROUP];
#pragma unroll
            for (int g = 0; g < GROUP; ++g)
                if (g < group) {
                    lo[g] = *reinterpret_cast<const float4*>(qs + (size_t)(c * group + g) * D + d);
                    hi[g] = *reinterpret_cast<const float4*>(qs + (size_t)(c * group + g) * D + d + 4);
                }
            for (int h = walker; h < H; h += walkers) {
                float acc[8] = {0.0f, 0.0f, 0.0f, 0.0f, 0.0f, 0.0f, 0.0f, 0.0f};
                const float* weight = ts + h * H + c * group;
#pragma unroll
                for (int g = 0; g < GROUP; ++g)
                    if (g < group) {
                        const float w = weight[g];
                        acc[0] = fmaf(w, lo[g].x, acc[0]); acc[1] = fmaf(w, lo[g].y, acc[1]); acc[2] = fmaf(w, lo[g].z, acc[2]); acc[3] = fmaf(w, lo[g].w, acc[3]);
                        acc[4] = fmaf(w, hi[g].x, acc[4]); acc[5] = fmaf(w, hi[g].y, acc[5]); acc[6] = fmaf(w, hi[g].z, acc[6]); acc[7] = fmaf(w, hi[g].w, acc[7]);
                    }
                store_columns<T, 8>(dst + (size_t)h * row_width + e * 8, acc);
            }
        }
    } else {
        for (int e = threadIdx.x * VEC; e < H * row_width; e += TP_THREADS * VEC) {
            const int h = e / row_width, rest = e - h * row_width;
            const int c = rest / D, d = rest - c * D;
            float acc[VEC];
#pragma unroll
            for (int i = 0; i < VEC; ++i) acc[i] = 0.0f;
            const float* weight = ts + h * H + c * group;
            const float* q = qs + (size_t)c * group * D + d;
            for (int g = 0; g < group; ++g) {
                const float w = weight[g];
                if constexpr (VEC == 8) {
                    const float4 lo = *reinterpret_cast<const float4*>(q + (size_t)g * D), hi = *reinterpret_cast<const float4*>(q + (size_t)g * D + 4);
                    acc[0] = fmaf(w, lo.x, acc[0]); acc[1] = fmaf(w, lo.y, acc[1]); acc[2] = fmaf(w, lo.z, acc[2]); acc[3] = fmaf(w, lo.w, acc[3]);
                    acc[4] = fmaf(w, hi.x, acc[4]); acc[5] = fmaf(w, hi.y, acc[5]); acc[6] = fmaf(w, hi.z, acc[6]); acc[7] = fmaf(w, hi.w, acc[7]);
                } else {
#pragma unroll
                    for (int i = 0; i < VEC; ++i) acc[i] = fmaf(w, q[(size_t)g * D + i], acc[i]);
                }
            }
            store_columns<T, VEC>(dst + e, acc);
        }
    }
}

template <typename T, int VEC, int GROUP>
static int launch_prepare(const void* packed, int stride, int tokens, int k_offset, int v_offset, int H, int G, int D, const float* talk,
                          const float* cos, const float* sin, int half, int max_pos, const int* positions, const int* row_ids,
                          const int* block_table, int max_pages, int num_rows, const int* write_from, void* k_cache, void* v_cache,
                          int page_size, int num_pages, void* mixed, int mixed_stride, int* flag, cudaStream_t stream) {
    const size_t smem = ((size_t)H * D + (size_t)H * H) * sizeof(float);
    if (smem > 200 * 1024) return KB_ERR_UNSUPPORTED_SIZE;
    if (smem > 48 * 1024) cudaFuncSetAttribute(talking_prepare_kernel<T, VEC, GROUP>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    kb_launch(talking_prepare_kernel<T, VEC, GROUP>, dim3(tokens), dim3(TP_THREADS), smem, stream, (const T*)packed, stride, k_offset, v_offset, H, G, D,
              talk, cos, sin, half, max_pos, positions, row_ids, block_table, max_pages, num_rows, write_from, (T*)k_cache, (T*)v_cache, page_size,
              num_pages, (T*)mixed, mixed_stride, flag);
    return kb_launch_result();
}

KB_EXPORT int kb_talking_prepare(const void* packed, int stride, int is_bf16, int tokens, int k_offset, int v_offset, int H, int G, int D,
                                 const float* talk, const float* cos, const float* sin, int half, int max_pos, const int* positions,
                                 const int* row_ids, const int* block_table, int max_pages, int num_rows, const int* write_from, void* k_cache,
                                 void* v_cache, int page_size, int num_pages, void* mixed, int mixed_stride, int* flag, cudaStream_t stream) {
    if (tokens == 0) return 0;
    if (!packed || !talk || !positions || !row_ids || !mixed || (half > 0 && (!cos || !sin)) || (k_cache && (!v_cache || !block_table))) return KB_ERR_NULL;
    if (G < 1 || H < 1 || H % G != 0 || D < 1 || half < 0 || 2 * half > D || (k_cache && page_size < 1)) return KB_ERR_BAD_ARG;
#define ARGS packed, stride, tokens, k_offset, v_offset, H, G, D, talk, cos, sin, half, max_pos, positions, row_ids, block_table, max_pages, num_rows, \
             write_from, k_cache, v_cache, page_size, num_pages, mixed, mixed_stride, flag, stream
    if (!is_bf16) return launch_prepare<float, 1, 0>(ARGS);
    const bool vec = D % 8 == 0 && half % 8 == 0 && stride % 8 == 0 && k_offset % 8 == 0 && v_offset % 8 == 0 && mixed_stride % 8 == 0
                     && (((uintptr_t)packed | (uintptr_t)k_cache | (uintptr_t)v_cache | (uintptr_t)mixed | (uintptr_t)cos | (uintptr_t)sin) % 16) == 0;
    if (!vec) return launch_prepare<__nv_bfloat16, 1, 0>(ARGS);
    const int group = H / G;
    if (group == 1) return launch_prepare<__nv_bfloat16, 8, 1>(ARGS);
    if (group == 2) return launch_prepare<__nv_bfloat16, 8, 2>(ARGS);
    if (group <= 4) return launch_prepare<__nv_bfloat16, 8, 4>(ARGS);
    if (group <= 8) return launch_prepare<__nv_bfloat16, 8, 8>(ARGS);
    return launch_prepare<__nv_bfloat16, 8, 0>(ARGS);
#undef ARGS
}
