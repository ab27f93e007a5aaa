// RMS norm in groups, and the residual sums of a layer that norms what a sublayer returns.
//
// group_rms_norm, one CTA per row:  the row of H numbers is cut into `groups` equal consecutive runs; each run is
// divided by its own sqrt(mean(run^2) + eps); the whole is multiplied by `gain` (float32 [H]).  groups = 1 is the
// plain RMS norm.  The row is read in its own type (float32, or the compute type: a product's output), held in
// shared memory as float32, and written in the output's type; `rows` gathers (out[r] = norm(x[rows[r]])).  A row
// may be normed in place.
//
// post_norm_add, one CTA per token, all float32:  a sublayer has added its result into the zeroed row y; then
//     x <- x + group_rms_norm(y) * gain;   y <- 0 (ready for the next sublayer)
// and, where the layer ends with an average over depth (`history` given: [n][tokens][H], entries 0 .. n - 2 the
// embedding output and the results of the layers before, as they left this kernel):
//     history[n - 1] <- x;   x <- sum_j weight[j] * history[j]   (j rising)
// x is also left in the compute type (`x_cast`, null where that is float32 itself) for the next product.
//
// depth_begin: history[0] <- x (if given), x_cast <- x, y <- 0.
//
// sandwich_close, one CTA per token, all float32: between two sublayers of a layer that norms what a sublayer reads and
// what it returns.  A sublayer has left its result, up to a common factor y_scale, in the zeroed row y;
//     x <- x + gain * norm(y_scale * y);   y <- 0          (norm(a) = a / sqrt(mean(a^2) + eps); gain null: only y <- 0)
//     inverse = 1 / sqrt(mean(x^2) + eps)
// and what the next sublayer wants of the new row: out <- x * inverse * next_gain (compute type), or the factor alone
// (row_scale[t] <- inverse) where the next kernel reads x itself.
#include "common.cuh"

namespace ps {

constexpr int GROUP_NORM_THREADS = 256;
constexpr int GROUP_NORM_MAX_GROUPS = 64;

// sums of squares of the runs of the staged row -> 1 / sqrt(mean + eps) per run
__device__ __forceinline__ void group_inverse_rms(const float* staged, int H, int groups, float eps, float* inverse) {
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5;
    const int run = H / groups;
    for (int g = warp; g < groups; g += warps) {
        const float* part = staged + (size_t)g * run;
        float sq = 0.f;
        for (int j = lane; j < run; j += 32) sq = fmaf(part[j], part[j], sq);
        sq = warp_sum(sq);
        if (lane == 0) inverse[g] = 1.0f / sqrtf(sq / (float)run + eps);
    }
}

template <typename TIn, typename TOut>
__global__ void __launch_bounds__(GROUP_NORM_THREADS)
group_rms_norm_kernel(const TIn* x, long long x_stride, const int* __restrict__ rows, int H, int groups,
                      const float* __restrict__ gain, float eps, TOut* out, long long out_stride) {
    extern __shared__ float staged[];
    __shared__ float inverse[GROUP_NORM_MAX_GROUPS];
    pdl_prologue();
    x = pdl_fresh(x);
    const int r = blockIdx.x;
    const TIn* source = x + (size_t)(rows ? rows[r] : r) * x_stride;
    for (int j = threadIdx.x; j < H; j += blockDim.x) staged[j] = to_float(source[j]);
    __syncthreads();
    group_inverse_rms(staged, H, groups, eps, inverse);
    __syncthreads();
    const int run = H / groups;
    TOut* target = out + (size_t)r * out_stride;
    for (int j = threadIdx.x; j < H; j += blockDim.x) target[j] = from_float<TOut>(staged[j] * inverse[j / run] * gain[j]);
}

// The same for rows in 16-byte pieces (V numbers of the input's type) and one group, or groups that are whole warps' passes
// (run a multiple of 32 V): a row stays in registers, PASSES pieces a thread; the gains are fetched before the wait.
template <typename T, int V> __device__ __forceinline__ void norm_piece(const T* p, float (&x)[V]) {
    const uint4 raw = *reinterpret_cast<const uint4*>(p);
    if constexpr (V == 4) {
        x[0] = __uint_as_float(raw.x); x[1] = __uint_as_float(raw.y); x[2] = __uint_as_float(raw.z); x[3] = __uint_as_float(raw.w);
    } else {
        const __nv_bfloat162* pair = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const float2 f = __bfloat1622float2(pair[i]);
            x[2 * i] = f.x;
            x[2 * i + 1] = f.y;
        }
    }
}
template <int V> __device__ __forceinline__ void norm_store(float* p, const float (&x)[V]) {
#pragma unroll
    for (int i = 0; i < V; i += 4) *reinterpret_cast<float4*>(p + i) = make_float4(x[i], x[i + 1], x[i + 2], x[i + 3]);
}
template <int V> __device__ __forceinline__ void norm_store(__nv_bfloat16* p, const float (&x)[V]) {
#pragma unroll
    for (int i = 0; i < V; i += 4) {
        const __nv_bfloat162 lo = __floats2bfloat162_rn(x[i], x[i + 1]), hi = __floats2bfloat162_rn(x[i + 2], x[i + 3]);
        *reinterpret_cast<uint2*>(p + i) = make_uint2(*reinterpret_cast<const uint32_t*>(&lo), *reinterpret_cast<const uint32_t*>(&hi));
    }
}

template <typename TIn, typename TOut, int PASSES>
__global__ void __launch_bounds__(GROUP_NORM_THREADS)
group_rms_norm_pieces_kernel(const TIn* x, long long x_stride, const int* __restrict__ rows, int H, int groups,
                             const float* __restrict__ gain, float eps, TOut* out, long long out_stride) {
    constexpr int V = 16 / (int)sizeof(TIn);
    __shared__ float partial[PASSES * GROUP_NORM_THREADS / 32];
    __shared__ float inverse[GROUP_NORM_MAX_GROUPS];
    const int warps = blockDim.x >> 5, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, run = H / groups;
    float g[PASSES][V];
#pragma unroll
    for (int p = 0; p < PASSES; ++p) {
        const int j = V * (threadIdx.x + p * blockDim.x);
#pragma unroll
        for (int i = 0; i < V; i += 4) {
            const float4 f = j < H ? *reinterpret_cast<const float4*>(gain + j + i) : make_float4(0.f, 0.f, 0.f, 0.f);
            g[p][i] = f.x; g[p][i + 1] = f.y; g[p][i + 2] = f.z; g[p][i + 3] = f.w;
        }
    }
    pdl_prologue();
    x = pdl_fresh(x);
    const int r = blockIdx.x;
    const TIn* source = x + (size_t)(rows ? rows[r] : r) * x_stride;
    float v[PASSES][V];
#pragma unroll
    for (int p = 0; p < PASSES; ++p) {
        const int j = V * (threadIdx.x + p * blockDim.x);
#pragma unroll
        for (int i = 0; i < V; ++i) v[p][i] = 0.f;
        if (j < H) norm_piece<TIn, V>(source + j, v[p]);
    }
#pragma unroll
    for (int p = 0; p < PASSES; ++p) {
        float sq = 0.f;
#pragma unroll
        for (int i = 0; i < V; ++i) sq = fmaf(v[p][i], v[p][i], sq);
        sq = warp_sum(sq);
        if (lane == 0) partial[p * warps + warp] = sq;                   // the pieces p * warps + warp, in the row's order
    }
    __syncthreads();
    float whole = 0.f;
    if (groups == 1) {                                                   // at most 32 partial sums: every warp adds them itself
        whole = 1.0f / sqrtf(warp_sum(lane < PASSES * warps ? partial[lane] : 0.f) / (float)run + eps);
    } else {
        const int each = run / (32 * V);                                 // partial sums of a group
        for (int k = threadIdx.x; k < groups; k += blockDim.x) {
            float total = 0.f;
            for (int i = 0; i < each; ++i) total += partial[k * each + i];
            inverse[k] = 1.0f / sqrtf(total / (float)run + eps);
        }
        __syncthreads();
    }
    TOut* target = out + (size_t)r * out_stride;
#pragma unroll
    for (int p = 0; p < PASSES; ++p) {
        const int j = V * (threadIdx.x + p * blockDim.x);
        if (j >= H) continue;
        const float scale = groups == 1 ? whole : inverse[j / run];
#pragma unroll
        for (int i = 0; i < V; ++i) v[p][i] = v[p][i] * scale * g[p][i];
        norm_store<V>(target + j, v[p]);
    }
}

// V numbers per access (4 where the width allows it).  The older entries of the history do not depend on the
// sublayer's row: their weighted sum and the residual row are fetched in the first pass, beside the row itself, so
// that their latency lies behind the row's statistics instead of behind them.
template <int V> struct PackOf;
template <> struct PackOf<1> { float v[1]; };
template <> struct __align__(16) PackOf<4> { float v[4]; };

template <int V> __device__ __forceinline__ void store_cast(float* p, const PackOf<V>& a) { *reinterpret_cast<PackOf<V>*>(p) = a; }
template <int V> __device__ __forceinline__ void store_cast(__nv_bfloat16* p, const PackOf<V>& a) {
    if constexpr (V == 4) {
        const __nv_bfloat162 lo = __floats2bfloat162_rn(a.v[0], a.v[1]), hi = __floats2bfloat162_rn(a.v[2], a.v[3]);
        uint2 packed;
        packed.x = *reinterpret_cast<const uint32_t*>(&lo);
        packed.y = *reinterpret_cast<const uint32_t*>(&hi);
        *reinterpret_cast<uint2*>(p) = packed;
    } else {
        p[0] = __float2bfloat16_rn(a.v[0]);
    }
}

template <typename TC, int V>
__global__ void __launch_bounds__(GROUP_NORM_THREADS)
post_norm_add_kernel(float* __restrict__ y, float* __restrict__ x, int H, int groups, const float* __restrict__ gain,
                     float eps, TC* __restrict__ x_cast, float* history, long long history_stride,
                     int n_history, const float* __restrict__ weight) {
    using Pack = PackOf<V>;
    extern __shared__ __align__(16) float staged[];          // the sublayer's row, the residual row, the older entries' sum
    __shared__ float inverse[GROUP_NORM_MAX_GROUPS];
    float* row = staged;
    float* kept = staged + H;
    float* older = staged + 2 * H;
    pdl_prologue();
    y = pdl_fresh(y);
    x = pdl_fresh(x);
    history = pdl_fresh(history);
    const size_t base = (size_t)blockIdx.x * H;
    for (int j = V * threadIdx.x; j < H; j += V * blockDim.x) {
        const Pack a = *reinterpret_cast<const Pack*>(y + base + j);
        const Pack b = *reinterpret_cast<const Pack*>(x + base + j);
        Pack sum;
#pragma unroll
        for (int i = 0; i < V; ++i) sum.v[i] = 0.f;
        if (history) {
            for (int d = 0; d < n_history - 1; ++d) {
                const Pack h = *reinterpret_cast<const Pack*>(history + (size_t)d * history_stride + base + j);
                const float w = weight[d];
#pragma unroll
                for (int i = 0; i < V; ++i) sum.v[i] = fmaf(w, h.v[i], sum.v[i]);
            }
        }
        Pack zero;
#pragma unroll
        for (int i = 0; i < V; ++i) zero.v[i] = 0.f;
        *reinterpret_cast<Pack*>(y + base + j) = zero;
        *reinterpret_cast<Pack*>(row + j) = a;
        *reinterpret_cast<Pack*>(kept + j) = b;
        *reinterpret_cast<Pack*>(older + j) = sum;
    }
    __syncthreads();
    group_inverse_rms(row, H, groups, eps, inverse);
    __syncthreads();
    const int run = H / groups;
    const float newest = history ? weight[n_history - 1] : 1.f;
    for (int j = V * threadIdx.x; j < H; j += V * blockDim.x) {
        const Pack g = *reinterpret_cast<const Pack*>(gain + j);
        Pack v, out;
#pragma unroll
        for (int i = 0; i < V; ++i) {
            v.v[i] = kept[j + i] + row[j + i] * inverse[(j + i) / run] * g.v[i];
            out.v[i] = history ? fmaf(newest, v.v[i], older[j + i]) : v.v[i];
        }
        if (history) *reinterpret_cast<Pack*>(history + (size_t)(n_history - 1) * history_stride + base + j) = v;
        *reinterpret_cast<Pack*>(x + base + j) = out;
        if (x_cast) store_cast<V>(x_cast + base + j, out);
    }
}

template <typename TC>
__global__ void __launch_bounds__(256)
depth_begin_kernel(const float* __restrict__ x, float* __restrict__ first, TC* __restrict__ x_cast, float* __restrict__ y,
                   long long count) {
    pdl_prologue();
    x = pdl_fresh(x);
    for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < count; i += (long long)gridDim.x * blockDim.x) {
        const float v = x[i];
        if (first) first[i] = v;
        if (x_cast) x_cast[i] = from_float<TC>(v);
        y[i] = 0.f;
    }
}

// the sum over the CTA's threads, in every thread, in a fixed order (`slots`: one float per warp)
__device__ __forceinline__ float cta_sum(float v, float* slots) {
    v = warp_sum(v);
    if ((threadIdx.x & 31) == 0) slots[threadIdx.x >> 5] = v;
    __syncthreads();
    float total = 0.f;
#pragma unroll
    for (int w = 0; w < GROUP_NORM_THREADS / 32; ++w) total += slots[w];
    return total;
}

template <typename TC, int V>
__global__ void __launch_bounds__(GROUP_NORM_THREADS)
sandwich_close_kernel(float* __restrict__ y, float* __restrict__ x, int H, const float* __restrict__ gain, float y_scale,
                      float eps, const float* __restrict__ next_gain, TC* __restrict__ out, float* __restrict__ row_scale) {
    using Pack = PackOf<V>;
    extern __shared__ __align__(16) float staged[];          // the sublayer's row, the residual row
    __shared__ float slots[2][GROUP_NORM_THREADS / 32];
    float* row = staged;
    float* kept = staged + H;
    pdl_prologue();
    y = pdl_fresh(y);
    x = pdl_fresh(x);
    const size_t base = (size_t)blockIdx.x * H;
    Pack zero;
#pragma unroll
    for (int i = 0; i < V; ++i) zero.v[i] = 0.f;
    float sq = 0.f, sq_x = 0.f;
    for (int j = V * threadIdx.x; j < H; j += V * GROUP_NORM_THREADS) {
        const Pack b = *reinterpret_cast<const Pack*>(x + base + j);
        *reinterpret_cast<Pack*>(kept + j) = b;
        if (gain) {
            Pack a = *reinterpret_cast<const Pack*>(y + base + j);
#pragma unroll
            for (int i = 0; i < V; ++i) {
                a.v[i] *= y_scale;
                sq = fmaf(a.v[i], a.v[i], sq);
            }
            *reinterpret_cast<Pack*>(row + j) = a;
        } else {
#pragma unroll
            for (int i = 0; i < V; ++i) sq_x = fmaf(b.v[i], b.v[i], sq_x);
        }
        *reinterpret_cast<Pack*>(y + base + j) = zero;
    }
    // (a thread reads back only what it has written itself: the two rows need no barrier of their own)
    if (gain) {
        const float inverse = 1.0f / sqrtf(cta_sum(sq, slots[0]) / (float)H + eps);
        for (int j = V * threadIdx.x; j < H; j += V * GROUP_NORM_THREADS) {
            const Pack g = *reinterpret_cast<const Pack*>(gain + j);
            const Pack a = *reinterpret_cast<const Pack*>(row + j);
            Pack b = *reinterpret_cast<const Pack*>(kept + j);
#pragma unroll
            for (int i = 0; i < V; ++i) {
                b.v[i] = fmaf(a.v[i] * inverse, g.v[i], b.v[i]);
                sq_x = fmaf(b.v[i], b.v[i], sq_x);
            }
            *reinterpret_cast<Pack*>(kept + j) = b;
            *reinterpret_cast<Pack*>(x + base + j) = b;
        }
    }
    if (!out && !row_scale) return;
    const float inverse = 1.0f / sqrtf(cta_sum(sq_x, slots[1]) / (float)H + eps);
    if (row_scale && threadIdx.x == 0) row_scale[blockIdx.x] = inverse;
    if (!out) return;
    for (int j = V * threadIdx.x; j < H; j += V * GROUP_NORM_THREADS) {
        const Pack g = *reinterpret_cast<const Pack*>(next_gain + j);
        Pack b = *reinterpret_cast<const Pack*>(kept + j);
#pragma unroll
        for (int i = 0; i < V; ++i) b.v[i] = b.v[i] * inverse * g.v[i];
        store_cast<V>(out + base + j, b);
    }
}

// The same with a row in registers, QUADS quads a thread whose loads are all in flight together: for widths that are
// multiples of four on aligned rows.  With many rows a CTA has as few threads as the row allows, so that many rows are
// resident; with few rows a thread has one quad.
// TAPS > 0 (steps in which every entry brings one token, token t being entry t): what comes next is a short causal
// convolution over time on the rows x / rms(x) (csrc/short_conv.cu), and an entry's one row meets its slot's kept rows here:
// out <- sum_(j < TAPS - 1) taps[c][j] kept[j][c] + taps[c][TAPS - 1] x[c] / rms(x), and the kept rows move up by one.
constexpr int CLOSE_QUADS = 4, CLOSE_MAX_THREADS = 1024;

__device__ __forceinline__ float few_warps_sum(float v, float* slots) {
    v = warp_sum(v);
    const int warps = blockDim.x >> 5;
    if (warps == 1) return v;
    if ((threadIdx.x & 31) == 0) slots[threadIdx.x >> 5] = v;
    __syncthreads();
    float total = 0.f;
    for (int w = 0; w < warps; ++w) total += slots[w];
    return total;
}

template <typename TC, int QUADS, int TAPS>
__global__ void __launch_bounds__(QUADS == 1 ? CLOSE_MAX_THREADS : CLOSE_MAX_THREADS / 2)
sandwich_close_rows_kernel(float* __restrict__ y, float* __restrict__ x, int H, const float* __restrict__ gain, float y_scale,
                           float eps, const float* __restrict__ next_gain, TC* __restrict__ out,
                           float* __restrict__ row_scale, const float* __restrict__ taps, float* kept, long long kept_stride,
                           const int* __restrict__ item_slot) {
    using Pack = PackOf<4>;
    __shared__ float slots[2][CLOSE_MAX_THREADS / 32];
    const size_t base = (size_t)blockIdx.x * H;
    Pack g[QUADS], a[QUADS], b[QUADS], zero;
#pragma unroll
    for (int i = 0; i < 4; ++i) zero.v[i] = 0.f;
    // before the wait: the gain, the taps, and the kept rows, which only this layer's kernels of an earlier step wrote
    if (gain) {
#pragma unroll
        for (int k = 0; k < QUADS; ++k) {
            const int j = 4 * (threadIdx.x + k * blockDim.x);
            g[k] = j < H ? *reinterpret_cast<const Pack*>(gain + j) : zero;
        }
    }
    constexpr int OLD = TAPS > 1 ? TAPS - 1 : 1;
    Pack old[OLD];
    float w[TAPS > 0 ? 4 * TAPS : 1];
    float* slot = nullptr;
    if constexpr (TAPS > 0) {
        static_assert(QUADS == 1, "the convolution is for one quad a thread");
        const int j = 4 * threadIdx.x;
        if (j < H) {
#pragma unroll
            for (int p = 0; p < TAPS; ++p) {
                const Pack v = *reinterpret_cast<const Pack*>(taps + (size_t)j * TAPS + 4 * p);
#pragma unroll
                for (int i = 0; i < 4; ++i) w[4 * p + i] = v.v[i];
            }
            if constexpr (TAPS > 1) {
                slot = kept + (size_t)item_slot[blockIdx.x] * kept_stride + j;
#pragma unroll
                for (int k = 0; k < TAPS - 1; ++k) old[k] = *reinterpret_cast<const Pack*>(slot + (size_t)k * H);
            }
        }
    }
    pdl_prologue();
    y = pdl_fresh(y);
    x = pdl_fresh(x);
#pragma unroll
    for (int k = 0; k < QUADS; ++k) {
        const int j = 4 * (threadIdx.x + k * blockDim.x);
        const bool here = j < H;
        b[k] = here ? *reinterpret_cast<const Pack*>(x + base + j) : zero;
        if (gain) a[k] = here ? *reinterpret_cast<const Pack*>(y + base + j) : zero;
    }
    float sq = 0.f, sq_x = 0.f;
    if (gain) {
#pragma unroll
        for (int k = 0; k < QUADS; ++k)
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                a[k].v[i] *= y_scale;
                sq = fmaf(a[k].v[i], a[k].v[i], sq);
            }
        const float inverse = 1.0f / sqrtf(few_warps_sum(sq, slots[0]) / (float)H + eps);
#pragma unroll
        for (int k = 0; k < QUADS; ++k)
#pragma unroll
            for (int i = 0; i < 4; ++i) b[k].v[i] = fmaf(a[k].v[i] * inverse, g[k].v[i], b[k].v[i]);
    }
#pragma unroll
    for (int k = 0; k < QUADS; ++k) {
        const int j = 4 * (threadIdx.x + k * blockDim.x);
#pragma unroll
        for (int i = 0; i < 4; ++i) sq_x = fmaf(b[k].v[i], b[k].v[i], sq_x);
        if (j < H) {
            if (gain) *reinterpret_cast<Pack*>(x + base + j) = b[k];
            *reinterpret_cast<Pack*>(y + base + j) = zero;
        }
    }
    if (!out && !row_scale) return;
    const float inverse = 1.0f / sqrtf(few_warps_sum(sq_x, slots[1]) / (float)H + eps);
    if (row_scale && threadIdx.x == 0) row_scale[blockIdx.x] = inverse;
    if (!out) return;
#pragma unroll
    for (int k = 0; k < QUADS; ++k) {
        const int j = 4 * (threadIdx.x + k * blockDim.x);
        if (j >= H) continue;
        if constexpr (TAPS > 0) {
            Pack unit, sum = zero;
#pragma unroll
            for (int i = 0; i < 4; ++i) unit.v[i] = b[k].v[i] * inverse;
            if constexpr (TAPS > 1) {
#pragma unroll
                for (int p = 0; p < TAPS - 1; ++p) {
#pragma unroll
                    for (int i = 0; i < 4; ++i) sum.v[i] = fmaf(w[i * TAPS + p], old[p].v[i], sum.v[i]);
                    *reinterpret_cast<Pack*>(slot + (size_t)p * H) = p + 1 < TAPS - 1 ? old[p + 1 < OLD ? p + 1 : p] : unit;
                }
            }
#pragma unroll
            for (int i = 0; i < 4; ++i) sum.v[i] = fmaf(w[i * TAPS + TAPS - 1], unit.v[i], sum.v[i]);
            store_cast<4>(out + base + j, sum);
        } else {
            const Pack n = *reinterpret_cast<const Pack*>(next_gain + j);
#pragma unroll
            for (int i = 0; i < 4; ++i) b[k].v[i] = b[k].v[i] * inverse * n.v[i];
            store_cast<4>(out + base + j, b[k]);
        }
    }
}

template <typename TC>
int launch_sandwich_rows(float* y, float* x, int T, int H, const float* gain, float y_scale, float eps, const float* next_gain,
                         void* out, float* row_scale, int n_taps, const float* taps, float* kept, long long kept_stride,
                         const int* item_slot, cudaStream_t s) {
    const bool few = n_taps > 0 || (T < 592 && H <= 4 * CLOSE_MAX_THREADS);
    const int per_thread = few ? 4 : 4 * CLOSE_QUADS;
    const dim3 block(((H + per_thread - 1) / per_thread + 31) / 32 * 32);
#define PS_CLOSE_ROWS(QUADS, TAPS)                                                                                     \
    return launch_pdl(sandwich_close_rows_kernel<TC, QUADS, TAPS>, dim3(T), block, 0, s, y, x, H, gain, y_scale, eps,    \
                      next_gain, (TC*)out, row_scale, taps, kept, kept_stride, item_slot)
    switch (n_taps) {
        case 1: PS_CLOSE_ROWS(1, 1);
        case 2: PS_CLOSE_ROWS(1, 2);
        case 3: PS_CLOSE_ROWS(1, 3);
        case 4: PS_CLOSE_ROWS(1, 4);
    }
    if (few) PS_CLOSE_ROWS(1, 0);
    PS_CLOSE_ROWS(CLOSE_QUADS, 0);
#undef PS_CLOSE_ROWS
}

template <typename TIn, typename TOut>
inline int launch_group_norm(const void* x, long long x_stride, const int* rows, int n_rows, int H, int groups,
                             const float* gain, float eps, void* out, long long out_stride, cudaStream_t s) {
    constexpr int V = 16 / (int)sizeof(TIn), OUT = (int)sizeof(TOut);
    if (H % V == 0 && x_stride % V == 0 && out_stride % (16 / OUT) == 0 && (groups == 1 || H / groups % (32 * V) == 0) &&
        !(((uintptr_t)x | (uintptr_t)gain | (uintptr_t)out) & 15) && H / V <= 4 * GROUP_NORM_THREADS) {
        const int pieces = H / V, threads = pieces < GROUP_NORM_THREADS ? (pieces + 31) / 32 * 32 : GROUP_NORM_THREADS;
        const int passes = (pieces + threads - 1) / threads;
        auto kernel = passes == 1 ? group_rms_norm_pieces_kernel<TIn, TOut, 1>
                                  : passes == 2 ? group_rms_norm_pieces_kernel<TIn, TOut, 2> : group_rms_norm_pieces_kernel<TIn, TOut, 4>;
        return launch_pdl(kernel, dim3(n_rows), dim3(threads), 0, s, (const TIn*)x, x_stride, rows, H, groups, gain, eps,
                          (TOut*)out, out_stride);
    }
    static size_t raised[MAX_DEVICES] = {0};
    if (!ensure_dynamic_smem((const void*)group_rms_norm_kernel<TIn, TOut>, (size_t)H * sizeof(float), raised)) return PS_ERR_LAUNCH;
    return launch_pdl(group_rms_norm_kernel<TIn, TOut>, dim3(n_rows), dim3(GROUP_NORM_THREADS), (size_t)H * sizeof(float),
                      s, (const TIn*)x, x_stride, rows, H, groups, gain, eps, (TOut*)out, out_stride);
}

}  // namespace ps

// x [*, H] rows of `in_dtype` with x_stride elements between rows; rows (may be null): int32 [n_rows] row indices;
// gain float32 [H]; out [n_rows, H] rows of `out_dtype`.  H must be a multiple of groups.
PS_EXPORT int ps_group_rms_norm(const void* x, long long x_stride, int in_dtype, const int* rows, int n_rows, int H,
                                int groups, const float* gain, float eps, void* out, long long out_stride,
                                int out_dtype, void* stream) {
    if (n_rows <= 0) return PS_OK;
    if (!x || !gain || !out || H <= 0 || groups <= 0 || H % groups) return PS_ERR_BAD_ARGUMENT;
    if (groups > ps::GROUP_NORM_MAX_GROUPS || (size_t)H * sizeof(float) > 200 * 1024) return PS_ERR_UNSUPPORTED;
    cudaStream_t s = (cudaStream_t)stream;
#define PS_GROUP_NORM(TIN, TOUT) \
    return ps::launch_group_norm<TIN, TOUT>(x, x_stride, rows, n_rows, H, groups, gain, eps, out, out_stride, s)
    if (in_dtype == PS_F32 && out_dtype == PS_F32) PS_GROUP_NORM(float, float);
    if (in_dtype == PS_F32 && out_dtype == PS_BF16) PS_GROUP_NORM(float, __nv_bfloat16);
    if (in_dtype == PS_BF16 && out_dtype == PS_BF16) PS_GROUP_NORM(__nv_bfloat16, __nv_bfloat16);
    if (in_dtype == PS_BF16 && out_dtype == PS_F32) PS_GROUP_NORM(__nv_bfloat16, float);
#undef PS_GROUP_NORM
    return PS_ERR_UNSUPPORTED;
}

// y, x float32 [T, H] contiguous; gain float32 [H]; x_cast [T, H] of `cast_dtype` or null; history float32
// [n_history][T][H] with history_stride elements between entries, or null; weight float32 [n_history].
PS_EXPORT int ps_post_norm_add(float* y, float* x, int T, int H, int groups, const float* gain, float eps, void* x_cast,
                               int cast_dtype, float* history, long long history_stride, int n_history,
                               const float* weight, void* stream) {
    if (T <= 0) return PS_OK;
    if (!y || !x || !gain || H <= 0 || groups <= 0 || H % groups) return PS_ERR_BAD_ARGUMENT;
    if (history && (!weight || n_history < 1)) return PS_ERR_BAD_ARGUMENT;
    const size_t smem = (size_t)3 * H * sizeof(float);
    if (groups > ps::GROUP_NORM_MAX_GROUPS || smem > 200 * 1024) return PS_ERR_UNSUPPORTED;
    if (x_cast && cast_dtype != PS_F32 && cast_dtype != PS_BF16) return PS_ERR_UNSUPPORTED;
    cudaStream_t s = (cudaStream_t)stream;
    const bool bf16 = x_cast && cast_dtype == PS_BF16;
    const bool by4 = H % 4 == 0 && history_stride % 4 == 0 &&
                     !(((uintptr_t)y | (uintptr_t)x | (uintptr_t)gain | (uintptr_t)history) & 15) &&
                     !((uintptr_t)x_cast & (bf16 ? 7 : 15));
#define PS_POST_NORM(TYPE, V)                                                                                        \
    do {                                                                                                             \
        static size_t raised[ps::MAX_DEVICES] = {0};                                                                 \
        auto kernel = ps::post_norm_add_kernel<TYPE, V>;                                                             \
        if (!ps::ensure_dynamic_smem((const void*)kernel, smem, raised)) return PS_ERR_LAUNCH;                       \
        return ps::launch_pdl(kernel, dim3(T), dim3(ps::GROUP_NORM_THREADS), smem, s, y, x, H, groups, gain, eps,    \
                              (TYPE*)x_cast, history, history_stride, n_history, weight);                            \
    } while (0)
    if (bf16) {
        if (by4) PS_POST_NORM(__nv_bfloat16, 4);
        PS_POST_NORM(__nv_bfloat16, 1);
    }
    if (by4) PS_POST_NORM(float, 4);
    PS_POST_NORM(float, 1);
#undef PS_POST_NORM
}

// x float32 [count]; first (may be null), y float32 [count]; x_cast [count] of `cast_dtype` or null.
PS_EXPORT int ps_depth_begin(const float* x, float* first, void* x_cast, int cast_dtype, float* y, long long count,
                             void* stream) {
    if (count <= 0) return PS_OK;
    if (!x || !y) return PS_ERR_BAD_ARGUMENT;
    cudaStream_t s = (cudaStream_t)stream;
    const long long blocks = (count + 255) / 256;
    const dim3 grid((unsigned)(blocks < 2368 ? blocks : 2368));
    if (!x_cast || cast_dtype == PS_F32)
        return ps::launch_pdl(ps::depth_begin_kernel<float>, grid, dim3(256), 0, s, x, first, (float*)x_cast, y, count);
    if (cast_dtype == PS_BF16)
        return ps::launch_pdl(ps::depth_begin_kernel<__nv_bfloat16>, grid, dim3(256), 0, s, x, first, (__nv_bfloat16*)x_cast,
                              y, count);
    return PS_ERR_UNSUPPORTED;
}

// y, x float32 [T, H] contiguous; gain, next_gain float32 [H] (gain null: nothing is added); out [T, H] of `out_dtype` or
// null (then next_gain may be null); row_scale float32 [T] or null.
PS_EXPORT int ps_sandwich_close(float* y, float* x, int T, int H, const float* gain, float y_scale, float eps,
                                const float* next_gain, void* out, int out_dtype, float* row_scale, void* stream) {
    if (T <= 0) return PS_OK;
    if (!y || !x || H <= 0 || (out && !next_gain)) return PS_ERR_BAD_ARGUMENT;
    const size_t smem = (size_t)2 * H * sizeof(float);
    if (smem > 200 * 1024 || (out && out_dtype != PS_F32 && out_dtype != PS_BF16)) return PS_ERR_UNSUPPORTED;
    cudaStream_t s = (cudaStream_t)stream;
    const bool bf16 = out && out_dtype == PS_BF16;
    const bool by4 = H % 4 == 0 && !(((uintptr_t)y | (uintptr_t)x | (uintptr_t)gain | (uintptr_t)next_gain) & 15) &&
                     !((uintptr_t)out & (bf16 ? 7 : 15));
    if (by4 && H <= 2 * ps::CLOSE_QUADS * ps::CLOSE_MAX_THREADS) {
        if (bf16)
            return ps::launch_sandwich_rows<__nv_bfloat16>(y, x, T, H, gain, y_scale, eps, next_gain, out, row_scale, 0, nullptr,
                                                           nullptr, 0, nullptr, s);
        return ps::launch_sandwich_rows<float>(y, x, T, H, gain, y_scale, eps, next_gain, out, row_scale, 0, nullptr, nullptr, 0,
                                               nullptr, s);
    }
#define PS_SANDWICH(TYPE, V)                                                                                         \
    do {                                                                                                             \
        static size_t raised[ps::MAX_DEVICES] = {0};                                                                 \
        auto kernel = ps::sandwich_close_kernel<TYPE, V>;                                                            \
        if (!ps::ensure_dynamic_smem((const void*)kernel, smem, raised)) return PS_ERR_LAUNCH;                       \
        return ps::launch_pdl(kernel, dim3(T), dim3(ps::GROUP_NORM_THREADS), smem, s, y, x, H, gain, y_scale, eps,   \
                              next_gain, (TYPE*)out, row_scale);                                                     \
    } while (0)
    if (bf16) {
        if (by4) PS_SANDWICH(__nv_bfloat16, 4);
        PS_SANDWICH(__nv_bfloat16, 1);
    }
    if (by4) PS_SANDWICH(float, 4);
    PS_SANDWICH(float, 1);
#undef PS_SANDWICH
}

// The close of a sublayer and, for entries of one token each, the convolution in front of the next mixer: taps float32
// [H, n_taps] (n_taps 1 to 4), kept float32 rows of kept_stride whose first (n_taps - 1) * H numbers are a slot's kept rows,
// item_slot int32 [T].  H a multiple of 4 up to 4096, everything on 16-byte boundaries (out in the compute type: 8).
PS_EXPORT int ps_sandwich_close_conv(float* y, float* x, int T, int H, const float* gain, float y_scale, float eps,
                                     const float* taps, int n_taps, float* kept, long long kept_stride, const int* item_slot,
                                     void* out, int out_dtype, void* stream) {
    if (T <= 0) return PS_OK;
    if (!y || !x || !out || !taps || H <= 0 || n_taps < 1 || (n_taps > 1 && (!kept || !item_slot))) return PS_ERR_BAD_ARGUMENT;
    if (n_taps > 4 || H % 4 != 0 || H > 4 * ps::CLOSE_MAX_THREADS || kept_stride % 4 != 0 ||
        (((uintptr_t)y | (uintptr_t)x | (uintptr_t)gain | (uintptr_t)taps | (uintptr_t)kept) & 15) ||
        ((uintptr_t)out & (out_dtype == PS_BF16 ? 7 : 15)))
        return PS_ERR_UNSUPPORTED;
    cudaStream_t s = (cudaStream_t)stream;
    if (out_dtype == PS_BF16)
        return ps::launch_sandwich_rows<__nv_bfloat16>(y, x, T, H, gain, y_scale, eps, nullptr, out, nullptr, n_taps, taps, kept,
                                                       kept_stride, item_slot, s);
    if (out_dtype == PS_F32)
        return ps::launch_sandwich_rows<float>(y, x, T, H, gain, y_scale, eps, nullptr, out, nullptr, n_taps, taps, kept,
                                               kept_stride, item_slot, s);
    return PS_ERR_UNSUPPORTED;
}
