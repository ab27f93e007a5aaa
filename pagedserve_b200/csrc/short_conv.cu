// A short causal convolution over time on every channel of a projection, with the tail of each sequence kept as state.
//
//     y_t[c] = sum_{j < taps} w[c][j] * u_(t - taps + 1 + j)[c],      u = 0 before the sequence's first token
//
// u is the projection's float32 output for the step's tokens; what lies before an entry's first token of this step
// comes from the request's slot, which holds its last taps - 1 projected rows (oldest first; zeros when the request
// is admitted).  Channels from `conv_channels` on have no convolution and are passed through (a gate's columns that
// ride in the same product).  The result is written in the compute type.
//
// Blending of values (optional), on the channels [mix_lo, mix_lo + mix_heads * head_slot): they are heads of
// `head_slot` numbers of which the first `head_values` count.  mode 1: the convolved values are also stored, float32,
// in `shared_values` [T, mix_heads * head_values]; mode 2: y <- (1 - m) y + m * shared_values[t], m = *mix.
//
// bias and act (optional): y <- act(y + bias[c]) before the result is rounded (act: one of the activation codes); kept rows
// are the projection's own.  u may be rows of the compute type too.
//
// row_scale (may be null): one float per token that multiplies its row of u wherever it is read (a row to be divided by
// its root mean square, say, whose factor an earlier kernel has formed); kept rows are stored already multiplied.
//
// The slot then receives the last taps - 1 rows of the sequence (rows of this step, and older kept rows moved up where the
// entry brought fewer than taps - 1 tokens).  The old rows are read by the entry's first taps - 1 tokens only, and one
// thread per channel works on all of those: it has read what it needs when it replaces them.
#include "common.cuh"

namespace ps {

constexpr int SHORT_CONV_MAX_TAPS = 16;

template <typename TI, typename TC>
__global__ void __launch_bounds__(256)
short_conv_kernel(const TI* __restrict__ u, long long u_stride, const float* __restrict__ weight, int taps,
                  int conv_channels, int channels, const float* __restrict__ row_scale, float* kept, long long kept_stride,
                  const int* __restrict__ token_item, const int* __restrict__ q_start, const int* __restrict__ item_slot,
                  TC* __restrict__ out, long long out_stride, int mode, int mix_lo, int mix_heads, int head_slot,
                  int head_values, float* __restrict__ shared_values, const float* __restrict__ mix,
                  const float* __restrict__ bias, int act, int tokens) {
    pdl_prologue();
    u = pdl_fresh(u);
    row_scale = pdl_fresh(row_scale);
    shared_values = pdl_fresh(shared_values);
    const long long total = (long long)tokens * channels;
    const float blend = mode == 2 ? *mix : 0.f;
    for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < total;
         i += (long long)gridDim.x * blockDim.x) {
        const int t = (int)(i / channels), c = (int)(i - (long long)t * channels);
        if (c >= conv_channels) {
            out[(size_t)t * out_stride + c] = from_float<TC>(to_float(u[(size_t)t * u_stride + c]) * (row_scale ? row_scale[t] : 1.f));
            continue;
        }
        const int item = token_item[t];
        const int first = q_start[item], end = q_start[item + 1];
        if (t != first && t - first < taps - 1) continue;             // (the thread of the first token does these)
        float* old = kept + (size_t)item_slot[item] * kept_stride;
        auto row = [&](int source) { return to_float(u[(size_t)source * u_stride + c]) * (row_scale ? row_scale[source] : 1.f); };
        const int last = t == first ? min(first + max(taps - 1, 1), end) : t + 1;
        for (int now = t; now < last; ++now) {
            float y = 0.f;
            for (int j = 0; j < taps; ++j) {
                const int source = now - (taps - 1) + j;
                // kept row k holds the projection of the token (taps - 1 - k) places before the entry's first
                const float v = source >= first ? row(source)
                                                : old[(size_t)(taps - 1 - (first - source)) * conv_channels + c];
                y = fmaf(weight[(size_t)c * taps + j], v, y);
            }
            if (bias) y += bias[c];
            y = apply_act(y, act);
            if (mode) {
                const int local = c - mix_lo;
                if (local >= 0 && local < mix_heads * head_slot) {
                    const int head = local / head_slot, place = local - head * head_slot;
                    if (place < head_values) {
                        float* common = shared_values + (size_t)now * mix_heads * head_values + head * head_values + place;
                        if (mode == 1) *common = y;
                        else y = (1.0f - blend) * y + blend * *common;
                    }
                }
            }
            out[(size_t)now * out_stride + c] = from_float<TC>(y);
        }
        if (t == first) {
            // new row k is the token at place count - (taps - 1) + k of the entry; before the entry's first token that
            // is the old row k + count, which lies above every row written so far
            const int count = end - first;
            for (int k = 0; k < taps - 1; ++k) {
                const int place = count - (taps - 1) + k;
                old[(size_t)k * conv_channels + c] = place >= 0 ? row(first + place) : old[(size_t)(k + count) * conv_channels + c];
            }
        }
    }
}

// The same for widths, strides and addresses that are multiples of four numbers and a convolution of TAPS taps known
// when the kernel is built: a thread owns four neighbouring channels and walks a run of consecutive tokens, holding the
// last TAPS - 1 projected rows of its channels in registers, so every number of u is fetched once (and TAPS - 1
// rows again where a run begins); the taps of its channels stay in registers for the whole run.  Where a run meets an
// entry's first token the held rows are replaced by the request's kept rows.
template <typename TC> __device__ __forceinline__ void store4(TC* p, const float (&v)[4]);
template <> __device__ __forceinline__ void store4<float>(float* p, const float (&v)[4]) {
    *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
}
template <> __device__ __forceinline__ void store4<__nv_bfloat16>(__nv_bfloat16* p, const float (&v)[4]) {
    const __nv_bfloat162 lo = __floats2bfloat162_rn(v[0], v[1]), hi = __floats2bfloat162_rn(v[2], v[3]);
    uint2 packed;
    packed.x = *reinterpret_cast<const uint32_t*>(&lo);
    packed.y = *reinterpret_cast<const uint32_t*>(&hi);
    *reinterpret_cast<uint2*>(p) = packed;
}

__device__ __forceinline__ float4 load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 load4(const __nv_bfloat16* p) {
    const uint2 raw = *reinterpret_cast<const uint2*>(p);
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
    const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
    return make_float4(a.x, a.y, b.x, b.y);
}

constexpr int SHORT_CONV_THREADS = 128;

// FORM: 0 plain, 1 rows multiplied by row_scale, 2 a bias and silu
template <typename TI, typename TC, int TAPS, int FORM>
__global__ void __launch_bounds__(SHORT_CONV_THREADS)
short_conv_runs_kernel(const TI* __restrict__ u, long long u_stride, const float* __restrict__ weight,
                       int conv_channels, int channels, const float* __restrict__ row_scale, float* kept,
                       long long kept_stride, const int* __restrict__ token_item, const int* __restrict__ q_start,
                       const int* __restrict__ item_slot, TC* __restrict__ out, long long out_stride, int mode, int mix_lo,
                       int mix_heads, int head_slot, int head_values, float* __restrict__ shared_values,
                       const float* __restrict__ mix, const float* __restrict__ bias, int tokens, int run) {
    const int c = 4 * (blockIdx.x * SHORT_CONV_THREADS + threadIdx.x);
    const int t0 = blockIdx.y * run, t1 = min(t0 + run, tokens);
    const bool convolved = c < conv_channels;
    // the taps of the thread's four channels: static for the step, fetched before the wait
    float w[4][TAPS];
    if (convolved && c < channels) {
        // (4 * TAPS neighbouring numbers)
        float flat[4 * TAPS];
#pragma unroll
        for (int p = 0; p < TAPS; ++p) {
            const float4 v = *reinterpret_cast<const float4*>(weight + (size_t)c * TAPS + 4 * p);
            flat[4 * p] = v.x; flat[4 * p + 1] = v.y; flat[4 * p + 2] = v.z; flat[4 * p + 3] = v.w;
        }
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
            for (int j = 0; j < TAPS; ++j) w[i][j] = flat[i * TAPS + j];
    }
    float4 shift = make_float4(0.f, 0.f, 0.f, 0.f);
    if constexpr (FORM == 2) {
        if (convolved && c < channels) shift = *reinterpret_cast<const float4*>(bias + c);
    }
    const float blend = mode == 2 ? *mix : 0.f;
    // which entry the run lies in is static for the step too
    const int item0 = convolved ? token_item[t0] : 0, item1 = convolved ? token_item[t1 - 1] : 0;
    const int start0 = convolved ? q_start[item0] : 0;
    pdl_prologue();
    u = pdl_fresh(u);
    row_scale = pdl_fresh(row_scale);
    shared_values = pdl_fresh(shared_values);
    auto scaled = [&](int t) {
        float4 v = load4(u + (size_t)t * u_stride + c);
        if constexpr (FORM == 1) {
            const float f = row_scale[t];
            v.x *= f; v.y *= f; v.z *= f; v.w *= f;
        }
        return v;
    };
    if (c >= channels) return;
    constexpr int AHEAD = sizeof(TI) == 2 ? 8 : 4;                // tokens whose rows are fetched together
    if (!convolved) {
        for (int t = t0; t < t1; t += AHEAD) {
            float4 rows[AHEAD];
#pragma unroll
            for (int a = 0; a < AHEAD; ++a)
                if (t + a < t1) rows[a] = scaled(t + a);
#pragma unroll
            for (int a = 0; a < AHEAD; ++a) {
                if (t + a < t1) {
                    const float y[4] = {rows[a].x, rows[a].y, rows[a].z, rows[a].w};
                    store4<TC>(out + (size_t)(t + a) * out_stride + c, y);
                }
            }
        }
        return;
    }
    // where the values that are blended lie among the thread's channels (whole quads: the launcher sees to that)
    int common = -1;
    if (mode) {
        const int local = c - mix_lo;
        if (local >= 0 && local < mix_heads * head_slot) {
            const int head = local / head_slot, place = local - head * head_slot;
            if (place < head_values) common = head * head_values + place;
        }
    }
    constexpr int OLD = TAPS > 1 ? TAPS - 1 : 1;
    float4 held[OLD];                                             // held[k]: the row k + 1 tokens back
    // one token: its output, and its row becomes the newest of the held ones
    auto emit = [&](int t, const float4& now) {
        float y[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
        for (int j = 0; j < TAPS - 1; ++j) {                      // tap j reads the row TAPS - 1 - j tokens back
            const float4 v = held[TAPS - 2 - j];
            y[0] = fmaf(w[0][j], v.x, y[0]); y[1] = fmaf(w[1][j], v.y, y[1]);
            y[2] = fmaf(w[2][j], v.z, y[2]); y[3] = fmaf(w[3][j], v.w, y[3]);
        }
        y[0] = fmaf(w[0][TAPS - 1], now.x, y[0]); y[1] = fmaf(w[1][TAPS - 1], now.y, y[1]);
        y[2] = fmaf(w[2][TAPS - 1], now.z, y[2]); y[3] = fmaf(w[3][TAPS - 1], now.w, y[3]);
#pragma unroll
        for (int k = TAPS - 2; k > 0; --k) held[k] = held[k - 1];
        if (TAPS > 1) held[0] = now;
        if constexpr (FORM == 2) {
            auto gate = [](float v) { return sizeof(TC) == 2 ? silu_fast(v) : silu(v); };
            y[0] = gate(y[0] + shift.x); y[1] = gate(y[1] + shift.y);
            y[2] = gate(y[2] + shift.z); y[3] = gate(y[3] + shift.w);
        }
        if (common >= 0) {
            float* place = shared_values + (size_t)t * mix_heads * head_values + common;
            if (mode == 1) {
                *reinterpret_cast<float4*>(place) = make_float4(y[0], y[1], y[2], y[3]);
            } else {
                const float4 other = *reinterpret_cast<const float4*>(place);
                y[0] = (1.0f - blend) * y[0] + blend * other.x; y[1] = (1.0f - blend) * y[1] + blend * other.y;
                y[2] = (1.0f - blend) * y[2] + blend * other.z; y[3] = (1.0f - blend) * y[3] + blend * other.w;
            }
        }
        store4<TC>(out + (size_t)t * out_stride + c, y);
    };
    if (item0 == item1 && t0 - start0 >= TAPS - 1) {
        // the run lies inside one entry, behind its first TAPS - 1 tokens: no kept rows
#pragma unroll
        for (int k = 0; k < TAPS - 1; ++k) held[k] = scaled(t0 - 1 - k);
        for (int t = t0; t < t1; t += AHEAD) {
            float4 rows[AHEAD];
#pragma unroll
            for (int a = 0; a < AHEAD; ++a)
                if (t + a < t1) rows[a] = scaled(t + a);
#pragma unroll
            for (int a = 0; a < AHEAD; ++a)
                if (t + a < t1) emit(t + a, rows[a]);
        }
        return;
    }
    bool fresh = true;
    // a token among its entry's first TAPS - 1 belongs to the run that holds the entry's first token (see the top): the
    // run before this one may have taken this one's first tokens, and this one may take some behind its end
    const int limit = min(t1 + (TAPS > 1 ? TAPS - 2 : 0), tokens);
#pragma unroll 1
    for (int t = t0; t < limit; ++t) {
        const int item = token_item[t], start = q_start[item];
        const int anchor = t - start < TAPS - 1 ? start : t;
        if (anchor < t0 || anchor >= t1) continue;
        const float4 now = scaled(t);
        if (TAPS > 1 && t == start) {
            float* old = kept + (size_t)item_slot[item] * kept_stride + c;
#pragma unroll
            for (int k = 0; k < TAPS - 1; ++k)
                held[k] = *reinterpret_cast<const float4*>(old + (size_t)(TAPS - 2 - k) * conv_channels);
            // new row k is the token at place count - (TAPS - 1) + k of the entry, or the old row k + count
            const int count = q_start[item + 1] - start;
#pragma unroll
            for (int k = 0; k < TAPS - 1; ++k) {
                const int place = count - (TAPS - 1) + k;
                float4 v = now;
                if (place > 0) v = scaled(start + place);
#pragma unroll
                for (int j = 0; j < TAPS - 1; ++j)
                    if (TAPS - 2 - j == k + count) v = held[j];
                *reinterpret_cast<float4*>(old + (size_t)k * conv_channels) = v;
            }
        } else if (TAPS > 1 && fresh) {                           // all of these lie in the entry
#pragma unroll
            for (int k = 0; k < TAPS - 1; ++k) held[k] = scaled(t - 1 - k);
        }
        fresh = false;
        emit(t, now);
    }
}

}  // namespace ps

// u [T, channels] rows (u_stride apart), float32 or (u_dtype) of `dtype`; row_scale float32 [T] or null; weight float32
// [conv_channels, taps]; kept float32 [slots, (taps - 1) * conv_channels] rows (kept_stride apart; may be null when taps = 1);
// out [T, channels] rows of `dtype`.  mode 0: no blending; 1: store the convolved values; 2: blend with the stored ones by
// *mix.  bias float32 [conv_channels] or null, act an activation code: behind the convolution.
PS_EXPORT int ps_short_conv(const void* u, int u_dtype, long long u_stride, const float* weight, int taps, int conv_channels,
                            int channels, const float* row_scale, float* kept, long long kept_stride, const int* token_item,
                            const int* q_start, const int* item_slot, void* out, long long out_stride, int mode,
                            int mix_lo, int mix_heads, int head_slot, int head_values, float* shared_values,
                            const float* mix, const float* bias, int act, int T, int dtype, void* stream) {
    if (T <= 0 || channels <= 0) return PS_OK;
    if (!u || !out || conv_channels < 0 || conv_channels > channels || taps < 1) return PS_ERR_BAD_ARGUMENT;
    if (conv_channels && (!weight || !token_item || !q_start || !item_slot || (taps > 1 && !kept)))
        return PS_ERR_BAD_ARGUMENT;
    if (mode < 0 || mode > 2 || (mode && (!shared_values || head_slot <= 0 || head_values <= 0 || head_values > head_slot)))
        return PS_ERR_BAD_ARGUMENT;
    if (mode == 2 && !mix) return PS_ERR_BAD_ARGUMENT;
    if ((dtype != PS_F32 && dtype != PS_BF16) || (u_dtype != PS_F32 && u_dtype != dtype)) return PS_ERR_UNSUPPORTED;
    if (taps > ps::SHORT_CONV_MAX_TAPS) return PS_ERR_UNSUPPORTED;
    cudaStream_t s = (cudaStream_t)stream;
    using bf = __nv_bfloat16;
    // quads of channels over runs of tokens, where every boundary between kinds of channels falls between quads
    const int elem = dtype == PS_F32 ? 4 : 2, in_elem = u_dtype == PS_F32 ? 4 : 2;
    const int form = row_scale ? 1 : (bias && act == PS_ACT_SILU) ? 2 : 0;
    const bool plain = bias == nullptr && act == PS_ACT_NONE;
    const bool quads = taps <= 4 && conv_channels > 0 && channels % 4 == 0 && conv_channels % 4 == 0 && u_stride % 4 == 0 &&
                       out_stride % 4 == 0 && kept_stride % 4 == 0 && !((uintptr_t)u & (uintptr_t)(4 * in_elem - 1)) &&
                       !((uintptr_t)kept & 15) && !((uintptr_t)weight & 15) && !((uintptr_t)bias & 15) &&
                       !((uintptr_t)out & (uintptr_t)(4 * elem - 1)) && (plain || form == 2) &&
                       (u_dtype == PS_F32 || form == 2) &&
                       (!mode || (mix_lo % 4 == 0 && head_slot % 4 == 0 && head_values % 4 == 0 &&
                                  !((uintptr_t)shared_values & 15)));
    if (quads) {
        // runs of 16 tokens re-read (taps - 1) / 16 of the rows; shorter runs where the step has too few for the SMs
        const int columns = (channels / 4 + ps::SHORT_CONV_THREADS - 1) / ps::SHORT_CONV_THREADS;
        int run = 16;
        // (rows of two bytes a number: as many bytes on their way as with four take twice the tokens a thread)
        const long long enough = in_elem == 2 ? 1000 : 1200;
        while (run > 1 && (long long)columns * ((T + run - 1) / run) < enough) run >>= 1;
        const dim3 grid(columns, (T + run - 1) / run), block(ps::SHORT_CONV_THREADS);
#define PS_CONV_RUNS(TI, TC, TAPS, FORM)                                                                              \
    return ps::launch_pdl(ps::short_conv_runs_kernel<TI, TC, TAPS, FORM>, grid, block, 0, s, (const TI*)u, u_stride,    \
                          weight, conv_channels, channels, row_scale, kept, kept_stride, token_item, q_start, item_slot, \
                          (TC*)out, out_stride, mode, mix_lo, mix_heads, head_slot, head_values, shared_values, mix,     \
                          bias, T, run)
#define PS_CONV_TAPS(TI, TC, FORM)                                                                                    \
    switch (taps) {                                                                                                   \
        case 1: PS_CONV_RUNS(TI, TC, 1, FORM);                                                                        \
        case 2: PS_CONV_RUNS(TI, TC, 2, FORM);                                                                        \
        case 3: PS_CONV_RUNS(TI, TC, 3, FORM);                                                                        \
        default: PS_CONV_RUNS(TI, TC, 4, FORM);                                                                       \
    }
        if (form == 2) {
            if (dtype == PS_F32) PS_CONV_TAPS(float, float, 2)
            if (u_dtype == PS_F32) PS_CONV_TAPS(float, bf, 2)
            PS_CONV_TAPS(bf, bf, 2)
        }
        if (dtype == PS_F32) {
            if (form == 1) PS_CONV_TAPS(float, float, 1)
            PS_CONV_TAPS(float, float, 0)
        }
        if (form == 1) PS_CONV_TAPS(float, bf, 1)
        PS_CONV_TAPS(float, bf, 0)
#undef PS_CONV_TAPS
#undef PS_CONV_RUNS
    }
    const long long total = (long long)T * channels;
    const long long blocks = (total + 255) / 256;
    const dim3 grid((unsigned)(blocks < 4736 ? blocks : 4736));
#define PS_CONV(TI, TC)                                                                                               \
    return ps::launch_pdl(ps::short_conv_kernel<TI, TC>, grid, dim3(256), 0, s, (const TI*)u, u_stride, weight, taps,   \
                          conv_channels, channels, row_scale, kept, kept_stride, token_item, q_start, item_slot,        \
                          (TC*)out, out_stride, mode, mix_lo, mix_heads, head_slot, head_values, shared_values, mix,     \
                          bias, act, T)
    if (dtype == PS_F32) PS_CONV(float, float);
    if (u_dtype == PS_F32) PS_CONV(float, bf);
    PS_CONV(bf, bf);
#undef PS_CONV
}
