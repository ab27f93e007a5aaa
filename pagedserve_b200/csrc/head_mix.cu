// Mixing of the heads of an attention layer, behind the products with the values.
//
// A layer whose heads' weights are mixed before they meet the values,
//     w'_h(i, j) = sum_g M[h][g] w_g(i, j),   result_h = sum_j w'_h(i, j) v_G(h)(j),   G(h) = h / (heads / kv_heads),
// is linear in the weights: with all[g][e] = sum_j w_g(i, j) v_e(j), what attention leaves when every query head meets the
// values of every key/value head,
//     result_h = sum_g M[h][g] all[g][G(h)].
// all: [T][heads][kv_heads][dim] (compute type), M: float32 [heads][heads], out: [T][heads * dim] (compute type); sums in
// float32, g rising.
#include "common.cuh"

namespace ps {

constexpr int HEAD_MIX_THREADS = 128;
constexpr int HEAD_MIX_BLOCK = 8;               // result heads a thread sums at once

// V neighbouring numbers of a head per thread
template <typename T, int V>
struct HeadMixPack;
template <> struct HeadMixPack<float, 1> { using type = float; };
template <> struct HeadMixPack<__nv_bfloat16, 1> { using type = __nv_bfloat16; };
template <> struct HeadMixPack<float, 2> { using type = float2; };
template <> struct HeadMixPack<__nv_bfloat16, 2> { using type = __nv_bfloat162; };
__device__ __forceinline__ void head_mix_unpack(float p, float (&x)[1]) { x[0] = p; }
__device__ __forceinline__ void head_mix_unpack(__nv_bfloat16 p, float (&x)[1]) { x[0] = __bfloat162float(p); }
__device__ __forceinline__ void head_mix_unpack(float2 p, float (&x)[2]) { x[0] = p.x; x[1] = p.y; }
__device__ __forceinline__ void head_mix_unpack(__nv_bfloat162 p, float (&x)[2]) {
    const float2 f = __bfloat1622float2(p);
    x[0] = f.x; x[1] = f.y;
}
__device__ __forceinline__ void head_mix_pack(const float (&x)[1], float& p) { p = x[0]; }
__device__ __forceinline__ void head_mix_pack(const float (&x)[1], __nv_bfloat16& p) { p = __float2bfloat16_rn(x[0]); }
__device__ __forceinline__ void head_mix_pack(const float (&x)[2], float2& p) { p = make_float2(x[0], x[1]); }
__device__ __forceinline__ void head_mix_pack(const float (&x)[2], __nv_bfloat162& p) { p = __floats2bfloat162_rn(x[0], x[1]); }

template <typename T, int V>
__global__ void __launch_bounds__(HEAD_MIX_THREADS)
head_mix_kernel(const T* __restrict__ all, long long all_stride, const float* __restrict__ mix, T* __restrict__ out,
                long long out_stride, int heads, int kv_heads, int dim) {
    using P = typename HeadMixPack<T, V>::type;
    pdl_prologue();
    all = pdl_fresh(all);
    const int unit = blockIdx.y * HEAD_MIX_THREADS + threadIdx.x, units = kv_heads * (dim / V);
    if (unit >= units) return;
    const int group = unit / (dim / V), d = (unit - group * (dim / V)) * V;
    const int per = heads / kv_heads;
    const T* source = all + (size_t)blockIdx.x * all_stride + group * dim + d;
    T* target = out + (size_t)blockIdx.x * out_stride + d;
    for (int h0 = group * per; h0 < (group + 1) * per; h0 += HEAD_MIX_BLOCK) {
        const int n = min(HEAD_MIX_BLOCK, (group + 1) * per - h0);
        float sum[HEAD_MIX_BLOCK][V];
#pragma unroll
        for (int b = 0; b < HEAD_MIX_BLOCK; ++b)
#pragma unroll
            for (int e = 0; e < V; ++e) sum[b][e] = 0.f;
#pragma unroll 4
        for (int g = 0; g < heads; ++g) {
            float x[V];
            head_mix_unpack(*reinterpret_cast<const P*>(source + (size_t)g * kv_heads * dim), x);
#pragma unroll
            for (int b = 0; b < HEAD_MIX_BLOCK; ++b) {
                const float m = b < n ? mix[(size_t)(h0 + b) * heads + g] : 0.f;
#pragma unroll
                for (int e = 0; e < V; ++e) sum[b][e] = fmaf(m, x[e], sum[b][e]);
            }
        }
#pragma unroll
        for (int b = 0; b < HEAD_MIX_BLOCK; ++b) {
            if (b < n) {
                P packed;
                head_mix_pack(sum[b], packed);
                *reinterpret_cast<P*>(target + (size_t)(h0 + b) * dim) = packed;
            }
        }
    }
}

// The same by pieces of 16 bytes, for sizes, strides and addresses that allow it: a thread owns a piece of one head slot of
// one token for all of its group's result heads.  M lies in shared memory by columns, every group's heads padded to
// blocks of HEAD_MIX_BLOCK with zeros, so that a block's weights are two accesses for all threads of the group.
template <typename T> struct HeadMixPiece;
template <> struct HeadMixPiece<float> { static constexpr int V = 4; };
template <> struct HeadMixPiece<__nv_bfloat16> { static constexpr int V = 8; };
__device__ __forceinline__ void head_mix_unpack(const uint4& p, float (&x)[4]) {
    x[0] = __uint_as_float(p.x); x[1] = __uint_as_float(p.y); x[2] = __uint_as_float(p.z); x[3] = __uint_as_float(p.w);
}
__device__ __forceinline__ void head_mix_unpack(const uint4& p, float (&x)[8]) {
    const __nv_bfloat162* pair = reinterpret_cast<const __nv_bfloat162*>(&p);
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const float2 f = __bfloat1622float2(pair[i]);
        x[2 * i] = f.x;
        x[2 * i + 1] = f.y;
    }
}
__device__ __forceinline__ uint4 head_mix_piece(const float (&x)[4]) {
    return make_uint4(__float_as_uint(x[0]), __float_as_uint(x[1]), __float_as_uint(x[2]), __float_as_uint(x[3]));
}
__device__ __forceinline__ uint4 head_mix_piece(const float (&x)[8]) {
    uint4 p;
    uint32_t* word = reinterpret_cast<uint32_t*>(&p);
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const __nv_bfloat162 pair = __floats2bfloat162_rn(x[2 * i], x[2 * i + 1]);
        word[i] = *reinterpret_cast<const uint32_t*>(&pair);
    }
    return p;
}

template <typename T>
__global__ void __launch_bounds__(HEAD_MIX_THREADS)
head_mix_pieces_kernel(const T* __restrict__ all, long long all_stride, const float* __restrict__ mix, T* __restrict__ out,
                       long long out_stride, int tokens, int heads, int kv_heads, int dim) {
    constexpr int V = HeadMixPiece<T>::V, AHEAD = 4;
    extern __shared__ __align__(16) float head_mix_smem[];          // [g][group][padded heads of the group]
    const int per = heads / kv_heads, padded = (per + HEAD_MIX_BLOCK - 1) / HEAD_MIX_BLOCK * HEAD_MIX_BLOCK;
    for (int e = threadIdx.x; e < heads * kv_heads * padded; e += HEAD_MIX_THREADS) {
        const int g = e / (kv_heads * padded), rest = e - g * kv_heads * padded, group = rest / padded, b = rest - group * padded;
        head_mix_smem[e] = b < per ? mix[(size_t)(group * per + b) * heads + g] : 0.f;
    }
    const int pieces = dim / V, units = kv_heads * pieces;
    const long long index = (long long)blockIdx.x * HEAD_MIX_THREADS + threadIdx.x;
    const int t = (int)(index / units), unit = (int)(index - (long long)t * units);
    const int group = unit / pieces, d = (unit - group * pieces) * V;
    pdl_prologue();
    all = pdl_fresh(all);
    __syncthreads();
    if (t >= tokens) return;
    const T* source = all + (size_t)t * all_stride + group * dim + d;
    T* target = out + (size_t)t * out_stride + (size_t)group * per * dim + d;
    const size_t step = (size_t)kv_heads * dim;
    for (int h0 = 0; h0 < padded; h0 += HEAD_MIX_BLOCK) {
        float sum[HEAD_MIX_BLOCK][V];
#pragma unroll
        for (int b = 0; b < HEAD_MIX_BLOCK; ++b)
#pragma unroll
            for (int e = 0; e < V; ++e) sum[b][e] = 0.f;
        const float* weights = head_mix_smem + group * padded + h0;
        for (int g0 = 0; g0 < heads; g0 += AHEAD) {
            uint4 raw[AHEAD];
#pragma unroll
            for (int a = 0; a < AHEAD; ++a)
                if (g0 + a < heads) raw[a] = *reinterpret_cast<const uint4*>(source + (g0 + a) * step);
#pragma unroll
            for (int a = 0; a < AHEAD; ++a) {
                if (g0 + a < heads) {
                    float x[V];
                    head_mix_unpack(raw[a], x);
                    const float* w = weights + (size_t)(g0 + a) * kv_heads * padded;
                    const float4 lo = *reinterpret_cast<const float4*>(w), hi = *reinterpret_cast<const float4*>(w + 4);
                    const float m[HEAD_MIX_BLOCK] = {lo.x, lo.y, lo.z, lo.w, hi.x, hi.y, hi.z, hi.w};
#pragma unroll
                    for (int b = 0; b < HEAD_MIX_BLOCK; ++b)
#pragma unroll
                        for (int e = 0; e < V; ++e) sum[b][e] = fmaf(m[b], x[e], sum[b][e]);
                }
            }
        }
#pragma unroll
        for (int b = 0; b < HEAD_MIX_BLOCK; ++b)
            if (h0 + b < per) *reinterpret_cast<uint4*>(target + (size_t)(h0 + b) * dim) = head_mix_piece(sum[b]);
    }
}

template <typename T>
inline int launch_head_mix_pieces(const void* all, long long all_stride, const float* mix, void* out, long long out_stride,
                                  int T_tokens, int heads, int kv_heads, int dim, size_t smem, cudaStream_t s) {
    auto kernel = head_mix_pieces_kernel<T>;
    static size_t raised[MAX_DEVICES] = {0};
    if (!ensure_dynamic_smem((const void*)kernel, smem, raised)) return PS_ERR_LAUNCH;
    const long long threads = (long long)T_tokens * kv_heads * (dim / HeadMixPiece<T>::V);
    return launch_pdl(kernel, dim3((unsigned)((threads + HEAD_MIX_THREADS - 1) / HEAD_MIX_THREADS)), dim3(HEAD_MIX_THREADS),
                      smem, s, (const T*)all, all_stride, mix, (T*)out, out_stride, T_tokens, heads, kv_heads, dim);
}

}  // namespace ps

PS_EXPORT int ps_head_mix(const void* all, long long all_stride, const float* mix, void* out, long long out_stride, int T,
                          int heads, int kv_heads, int dim, int dtype, void* stream) {
    if (T <= 0) return PS_OK;
    if (!all || !mix || !out || heads <= 0 || kv_heads <= 0 || heads % kv_heads || dim <= 0) return PS_ERR_BAD_ARGUMENT;
    cudaStream_t s = (cudaStream_t)stream;
    const int elem = dtype == PS_F32 ? 4 : 2;
    const int per = heads / kv_heads, padded = (per + ps::HEAD_MIX_BLOCK - 1) / ps::HEAD_MIX_BLOCK * ps::HEAD_MIX_BLOCK;
    const size_t smem = (size_t)heads * kv_heads * padded * sizeof(float);
    const int piece = 16 / elem;
    if (dim % piece == 0 && all_stride % piece == 0 && out_stride % piece == 0 && !(((uintptr_t)all | (uintptr_t)out) & 15) &&
        smem <= 48 * 1024) {
        if (dtype == PS_F32)
            return ps::launch_head_mix_pieces<float>(all, all_stride, mix, out, out_stride, T, heads, kv_heads, dim, smem, s);
        if (dtype == PS_BF16)
            return ps::launch_head_mix_pieces<__nv_bfloat16>(all, all_stride, mix, out, out_stride, T, heads, kv_heads, dim,
                                                             smem, s);
    }
    const bool pairs = dim % 2 == 0 && all_stride % 2 == 0 && out_stride % 2 == 0 &&
                       !(((uintptr_t)all | (uintptr_t)out) & (uintptr_t)(2 * elem - 1));
    const int units = kv_heads * (pairs ? dim / 2 : dim);
    const dim3 grid(T, (units + ps::HEAD_MIX_THREADS - 1) / ps::HEAD_MIX_THREADS), block(ps::HEAD_MIX_THREADS);
#define PS_HEAD_MIX(TYPE, V)                                                                                         \
    return ps::launch_pdl(ps::head_mix_kernel<TYPE, V>, grid, block, 0, s, (const TYPE*)all, all_stride, mix, (TYPE*)out, \
                          out_stride, heads, kv_heads, dim)
    if (dtype == PS_F32) {
        if (pairs) PS_HEAD_MIX(float, 2);
        PS_HEAD_MIX(float, 1);
    }
    if (dtype == PS_BF16) {
        if (pairs) PS_HEAD_MIX(__nv_bfloat16, 2);
        PS_HEAD_MIX(__nv_bfloat16, 1);
    }
#undef PS_HEAD_MIX
    return PS_ERR_UNSUPPORTED;
}
