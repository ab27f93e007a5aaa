// Attention with two softmax maps per head that share one value and are subtracted: what comes before and behind the
// attention kernels.
//
// A head h has two queries and a key/value head g two keys of `dim` numbers each and one value of `vdim` numbers.  A cached
// key is [k1 | k2] and a cached value [v], both in heads of `slot` >= max(2 dim, vdim) numbers; the queries become two of
// `slot` numbers, [q1 | 0] and [0 | q2], so that the attention kernels see 2 H query heads on G key/value heads, query head
// 2h + m on key head h / (H / G), and a map's score is its own product alone.
//
// diff_prepare: a token's projected row  q [H][2][dim] | k [G][2][dim] | v [G][vdim]  (offsets in elements) becomes queries
// and pages.  q and k: x / sqrt(mean(x^2) + eps) * gain per head and map (dim numbers, one gain for all queries and one for
// all keys); queries are then multiplied by 1 + temp_coef * ln(floor((p + 1) / temp_every) + 1) of their position p
// (temp_every 0: not).  has_kv 0: queries only (keys and values lie in another layer's pages).
//
// diff_combine: from the attention's rows [2 H][slot], per head
//     o = a1 - share * a2,     out = o / sqrt(mean(o^2) + eps) * scale * sigmoid(gate_h)
// with `gate` one number per head behind the projections (null: no gate).
//
// Statistics, factors and sums are float32.  V numbers an access (16 bytes), `lanes` lanes per unit of work.
#include "common.cuh"

namespace ps {

constexpr int DIFF_WARPS = 4;

template <typename T, int V> struct DiffPack;
template <> struct DiffPack<float, 4> { using type = float4; };
template <> struct DiffPack<__nv_bfloat16, 8> { using type = uint4; };
template <> struct DiffPack<float, 1> { using type = float; };
template <> struct DiffPack<__nv_bfloat16, 1> { using type = __nv_bfloat16; };

__device__ __forceinline__ void diff_unpack(const float4& p, float (&x)[4]) { x[0] = p.x; x[1] = p.y; x[2] = p.z; x[3] = p.w; }
__device__ __forceinline__ void diff_unpack(const uint4& p, float (&x)[8]) {
    const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&p);
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const float2 f = __bfloat1622float2(h[i]);
        x[2 * i] = f.x;
        x[2 * i + 1] = f.y;
    }
}
__device__ __forceinline__ void diff_unpack(const float& p, float (&x)[1]) { x[0] = p; }
__device__ __forceinline__ void diff_unpack(const __nv_bfloat16& p, float (&x)[1]) { x[0] = __bfloat162float(p); }
__device__ __forceinline__ void diff_pack(const float (&x)[4], float4& p) { p = make_float4(x[0], x[1], x[2], x[3]); }
__device__ __forceinline__ void diff_pack(const float (&x)[8], uint4& p) {
    __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&p);
#pragma unroll
    for (int i = 0; i < 4; ++i) h[i] = __floats2bfloat162_rn(x[2 * i], x[2 * i + 1]);
}
__device__ __forceinline__ void diff_pack(const float (&x)[1], float& p) { p = x[0]; }
__device__ __forceinline__ void diff_pack(const float (&x)[1], __nv_bfloat16& p) { p = __float2bfloat16_rn(x[0]); }

// A unit of work is one (head, map) of the queries, one of the keys, or one value head; `lanes` (a power of two) lanes of a
// warp share it.  A lane's numbers are V * (lane + lanes * i).
template <typename T, int V>
__global__ void __launch_bounds__(DIFF_WARPS * 32)
diff_prepare_kernel(const T* __restrict__ row, long long row_stride, int k_offset, int v_offset,
                    const float* __restrict__ q_gain, const float* __restrict__ k_gain, float eps, float temp_coef,
                    int temp_every, const int* __restrict__ token_row, const int* __restrict__ positions,
                    const int* __restrict__ block_table, int bt_stride, T* __restrict__ k_pool, T* __restrict__ v_pool,
                    long long page_stride, int page_size, T* __restrict__ q_out, long long q_stride, int n_heads,
                    int n_kv_heads, int dim, int vdim, int slot, int has_kv, int lanes) {
    using P = typename DiffPack<T, V>::type;
    const int t = blockIdx.x;
    // positions, rows and the block table are static for the step: read before the wait
    const int p = positions[t];
    const float heat = temp_every > 0 ? 1.0f + temp_coef * logf((float)((p + 1) / temp_every) + 1.0f) : 1.0f;
    long long page_base = -1;
    if (has_kv) {
        const int page = block_table[(size_t)token_row[t] * bt_stride + p / page_size];
        if (page >= 0) page_base = (long long)page * page_stride + (long long)(p % page_size) * slot;
    }
    pdl_prologue();
    row = pdl_fresh(row);
    const T* mine = row + (size_t)t * row_stride;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int per_warp = 32 / lanes, group = lane / lanes, gl = lane - group * lanes;
    const int queries = 2 * n_heads, keys = has_kv ? 2 * n_kv_heads : 0, total = queries + keys + (has_kv ? n_kv_heads : 0);
    for (int base = (blockIdx.y * DIFF_WARPS + warp) * per_warp; base < total; base += gridDim.y * DIFF_WARPS * per_warp) {
        const int unit = base + group;
        const bool here = unit < total, is_query = unit < queries, is_value = unit >= queries + keys;
        const int index = is_query ? unit : is_value ? unit - queries - keys : unit - queries;
        if (here && is_value) {                              // (the lanes of a unit branch together; others wait at the sum)
            const T* src = mine + v_offset + (size_t)index * vdim;
            T* dst = page_base >= 0 ? v_pool + page_base + (long long)index * page_size * slot : nullptr;
            if (dst) {
                for (int d = V * gl; d < slot; d += V * lanes) {
                    float x[V];
#pragma unroll
                    for (int e = 0; e < V; ++e) x[e] = 0.f;
                    if (d < vdim) diff_unpack(*reinterpret_cast<const P*>(src + d), x);
                    P packed;
                    diff_pack(x, packed);
                    *reinterpret_cast<P*>(dst + d) = packed;
                }
            }
        }
        const T* src = mine + (is_query ? 0 : k_offset) + (size_t)index * dim;
        const bool normed = here && !is_value;
        float sq = 0.f;
        if (normed) {
            for (int d = V * gl; d < dim; d += V * lanes) {
                float x[V];
                diff_unpack(*reinterpret_cast<const P*>(src + d), x);
#pragma unroll
                for (int e = 0; e < V; ++e) sq = fmaf(x[e], x[e], sq);
            }
        }
        for (int o = lanes >> 1; o > 0; o >>= 1) sq += __shfl_xor_sync(0xffffffffu, sq, o);
        if (!normed) continue;
        const float inverse = 1.0f / sqrtf(sq / (float)dim + eps);
        const float factor = is_query ? heat : 1.0f;
        const float* gain = is_query ? q_gain : k_gain;
        const int map = index & 1, first = map * dim;
        // a query's row of `slot` numbers is its map's and zeros; of a key's row the first map's unit writes its own numbers,
        // the second the rest
        T* dst;
        int from, to;
        if (is_query) {
            dst = q_out + (size_t)t * q_stride + (size_t)unit * slot;
            from = 0, to = slot;
        } else {
            if (page_base < 0) continue;
            dst = k_pool + page_base + (long long)(index >> 1) * page_size * slot;
            from = first, to = map ? slot : dim;
        }
        for (int d = from + V * gl; d < to; d += V * lanes) {
            float x[V];
#pragma unroll
            for (int e = 0; e < V; ++e) x[e] = 0.f;
            if (d >= first && d < first + dim) {
                diff_unpack(*reinterpret_cast<const P*>(src + d - first), x);
#pragma unroll
                for (int e = 0; e < V; ++e) x[e] = x[e] * inverse * gain[d - first + e] * factor;
            }
            P packed;
            diff_pack(x, packed);
            *reinterpret_cast<P*>(dst + d) = packed;
        }
    }
}

// V neighbouring numbers of a map's result: of the output's type, or float32
template <typename T, int V>
__device__ __forceinline__ void diff_fetch(const T* p, float (&x)[V]) {
    if constexpr (V == 8 && sizeof(T) == 4) {
        const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
        x[0] = a.x; x[1] = a.y; x[2] = a.z; x[3] = a.w; x[4] = b.x; x[5] = b.y; x[6] = b.z; x[7] = b.w;
    } else {
        diff_unpack(*reinterpret_cast<const typename DiffPack<T, V>::type*>(p), x);
    }
}

template <typename TM, typename T, int V>
__global__ void __launch_bounds__(DIFF_WARPS * 32)
diff_combine_kernel(const TM* __restrict__ maps, long long maps_stride, const T* __restrict__ gate, long long gate_stride,
                    T* __restrict__ out, long long out_stride, float share, float eps, float scale, int rows, int n_heads,
                    int vdim, int slot, int lanes) {
    using P = typename DiffPack<T, V>::type;
    pdl_prologue();
    maps = pdl_fresh(maps);
    gate = pdl_fresh(gate);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int per_warp = 32 / lanes, group = lane / lanes, gl = lane - group * lanes;
    const long long total = (long long)rows * n_heads;
    const float inv = 1.0f / (float)vdim;
    for (long long base = ((long long)blockIdx.x * DIFF_WARPS + warp) * per_warp; base < total;
         base += (long long)gridDim.x * DIFF_WARPS * per_warp) {
        const long long unit = base + group;
        const bool here = unit < total;
        const int t = here ? (int)(unit / n_heads) : 0, h = here ? (int)(unit - (long long)t * n_heads) : 0;
        const TM* a1 = maps + (size_t)t * maps_stride + (size_t)(2 * h) * slot;
        const TM* a2 = a1 + slot;
        float sq = 0.f, held[V];                             // the first V numbers of a lane stay in registers
        if (here) {
            for (int d = V * gl; d < vdim; d += V * lanes) {
                float x[V], y[V];
                diff_fetch(a1 + d, x);
                diff_fetch(a2 + d, y);
#pragma unroll
                for (int e = 0; e < V; ++e) {
                    x[e] = fmaf(-share, y[e], x[e]);
                    sq = fmaf(x[e], x[e], sq);
                    if (d == V * gl) held[e] = x[e];
                }
            }
        }
        for (int o = lanes >> 1; o > 0; o >>= 1) sq += __shfl_xor_sync(0xffffffffu, sq, o);
        if (!here) continue;
        float factor = scale / sqrtf(sq * inv + eps);
        if (gate) factor /= 1.0f + expf(-to_float(gate[(size_t)t * gate_stride + h]));
        T* dst = out + (size_t)t * out_stride + (size_t)h * vdim;
        for (int d = V * gl; d < vdim; d += V * lanes) {
            float x[V];
            if (d == V * gl) {
#pragma unroll
                for (int e = 0; e < V; ++e) x[e] = held[e];
            } else {
                float y[V];
                diff_fetch(a1 + d, x);
                diff_fetch(a2 + d, y);
#pragma unroll
                for (int e = 0; e < V; ++e) x[e] = fmaf(-share, y[e], x[e]);
            }
#pragma unroll
            for (int e = 0; e < V; ++e) x[e] *= factor;
            P packed;
            diff_pack(x, packed);
            *reinterpret_cast<P*>(dst + d) = packed;
        }
    }
}

inline int diff_lanes(int numbers, int V) {
    int lanes = 1;
    while (lanes < 32 && lanes * V < numbers) lanes <<= 1;
    return lanes;
}

template <typename T, int V>
int launch_diff_prepare(const void* row, long long row_stride, int k_offset, int v_offset, const float* q_gain,
                        const float* k_gain, float eps, float temp_coef, int temp_every, const int* token_row,
                        const int* positions, const int* block_table, int bt_stride, void* k_pool, void* v_pool,
                        long long page_stride, int page_size, void* q_out, long long q_stride, int T_, int n_heads,
                        int n_kv_heads, int dim, int vdim, int slot, int has_kv, cudaStream_t s) {
    const int lanes = diff_lanes(slot, V), units = 2 * n_heads + (has_kv ? 3 * n_kv_heads : 0);
    const int per_cta = DIFF_WARPS * (32 / lanes);
    int split = (units + per_cta - 1) / per_cta;
    if (T_ >= 1024 && split > 4) split = 4;                  // many tokens: a CTA walks several units
    return launch_pdl(diff_prepare_kernel<T, V>, dim3(T_, split), dim3(DIFF_WARPS * 32), 0, s, (const T*)row, row_stride,
                      k_offset, v_offset, q_gain, k_gain, eps, temp_coef, temp_every, token_row, positions, block_table,
                      bt_stride, (T*)k_pool, (T*)v_pool, page_stride, page_size, (T*)q_out, q_stride, n_heads, n_kv_heads, dim,
                      vdim, slot, has_kv, lanes);
}

template <typename TM, typename T, int V>
int launch_diff_combine(const void* maps, long long maps_stride, const void* gate, long long gate_stride, void* out,
                        long long out_stride, float share, float eps, float scale, int rows, int n_heads, int vdim, int slot,
                        cudaStream_t s) {
    const int lanes = diff_lanes(vdim, V), per_cta = DIFF_WARPS * (32 / lanes);
    const long long ctas = ((long long)rows * n_heads + per_cta - 1) / per_cta;
    return launch_pdl(diff_combine_kernel<TM, T, V>, dim3((unsigned)(ctas < 148 * 16 ? ctas : 148 * 16)), dim3(DIFF_WARPS * 32), 0, s,
                      (const TM*)maps, maps_stride, (const T*)gate, gate_stride, (T*)out, out_stride, share, eps, scale, rows,
                      n_heads, vdim, slot, lanes);
}

}  // namespace ps

// row [T] rows of `dtype`, row_stride apart: queries at 0, keys at k_offset, values at v_offset (see the top of the file);
// gains float32 [dim]; q_out [T][2 * n_heads * slot]; pools: pages of [n_kv_heads][page_size][slot].  has_kv 0: no keys and
// values in the row, nothing is written to pages.
PS_EXPORT int ps_diff_prepare(const void* row, long long row_stride, int k_offset, int v_offset, const float* q_gain,
                              const float* k_gain, float eps, float temp_coef, int temp_every, const int* token_row,
                              const int* positions, const int* block_table, int bt_stride, void* k_pool, void* v_pool,
                              long long page_stride, int page_size, void* q_out, long long q_stride, int T, int n_heads,
                              int n_kv_heads, int dim, int vdim, int slot, int has_kv, int dtype, void* stream) {
    if (T <= 0) return PS_OK;
    if (!row || !q_gain || !positions || !q_out || n_heads <= 0 || n_kv_heads <= 0 || n_heads % n_kv_heads || dim <= 0 ||
        vdim <= 0 || slot < 2 * dim || slot < vdim || temp_every < 0)
        return PS_ERR_BAD_ARGUMENT;
    if (has_kv && (!k_gain || !k_pool || !v_pool || !token_row || !block_table || page_size <= 0)) return PS_ERR_BAD_ARGUMENT;
    cudaStream_t s = (cudaStream_t)stream;
    const int V = dtype == PS_F32 ? 4 : 8;
    const bool wide = dim % V == 0 && vdim % V == 0 && slot % V == 0 && row_stride % V == 0 && q_stride % V == 0 &&
                      page_stride % V == 0 && k_offset % V == 0 && v_offset % V == 0 &&
                      !(((uintptr_t)row | (uintptr_t)q_out | (uintptr_t)k_pool | (uintptr_t)v_pool) & 15);
#define PS_DIFF_PREPARE(TYPE, V)                                                                                        \
    return ps::launch_diff_prepare<TYPE, V>(row, row_stride, k_offset, v_offset, q_gain, k_gain, eps, temp_coef, temp_every, \
                                            token_row, positions, block_table, bt_stride, k_pool, v_pool, page_stride,   \
                                            page_size, q_out, q_stride, T, n_heads, n_kv_heads, dim, vdim, slot, has_kv, s)
    if (dtype == PS_F32) {
        if (wide) PS_DIFF_PREPARE(float, 4);
        PS_DIFF_PREPARE(float, 1);
    }
    if (dtype == PS_BF16) {
        if (wide) PS_DIFF_PREPARE(__nv_bfloat16, 8);
        PS_DIFF_PREPARE(__nv_bfloat16, 1);
    }
#undef PS_DIFF_PREPARE
    return PS_ERR_UNSUPPORTED;
}

// maps [T][2 * n_heads * slot] of maps_dtype (`dtype` or float32), gate [T][n_heads] or null, out [T][n_heads * vdim] of `dtype`
PS_EXPORT int ps_diff_combine(const void* maps, long long maps_stride, const void* gate, long long gate_stride, void* out,
                              long long out_stride, float share, float eps, float scale, int T, int n_heads, int vdim,
                              int slot, int maps_dtype, int dtype, void* stream) {
    if (T <= 0) return PS_OK;
    if (!maps || !out || n_heads <= 0 || vdim <= 0 || slot < vdim) return PS_ERR_BAD_ARGUMENT;
    cudaStream_t s = (cudaStream_t)stream;
    const int V = dtype == PS_F32 ? 4 : 8;
    const bool wide = vdim % V == 0 && slot % V == 0 && maps_stride % V == 0 && out_stride % V == 0 &&
                      !(((uintptr_t)maps | (uintptr_t)out) & 15);
#define PS_DIFF_COMBINE(MAPS, TYPE, V)                                                                                  \
    return ps::launch_diff_combine<MAPS, TYPE, V>(maps, maps_stride, gate, gate_stride, out, out_stride, share, eps, scale, T, \
                                                  n_heads, vdim, slot, s)
    using bf = __nv_bfloat16;
    if (dtype == PS_F32 && maps_dtype == PS_F32) {
        if (wide) PS_DIFF_COMBINE(float, float, 4);
        PS_DIFF_COMBINE(float, float, 1);
    }
    if (dtype == PS_BF16 && maps_dtype == PS_F32) {
        if (wide) PS_DIFF_COMBINE(float, bf, 8);
        PS_DIFF_COMBINE(float, bf, 1);
    }
    if (dtype == PS_BF16 && maps_dtype == PS_BF16) {
        if (wide) PS_DIFF_COMBINE(bf, bf, 8);
        PS_DIFF_COMBINE(bf, bf, 1);
    }
#undef PS_DIFF_COMBINE
    return PS_ERR_UNSUPPORTED;
}
