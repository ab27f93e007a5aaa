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

}  // namespace ps

PS_EXPORT int ps_head_mix(const void* all, long long all_stride, const float* mix, void* out, long long out_stride, int T,
                          int heads, int kv_heads, int dim, int dtype, void* stream) {
    if (T <= 0) return PS_OK;
    if (!all || !mix || !out || heads <= 0 || kv_heads <= 0 || heads % kv_heads || dim <= 0) return PS_ERR_BAD_ARGUMENT;
    cudaStream_t s = (cudaStream_t)stream;
    const int elem = dtype == PS_F32 ? 4 : 2;
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
