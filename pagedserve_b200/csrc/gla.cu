// Gated linear attention: a matrix state per head whose rows (key channels) decay by a gate of the current token.
//
// Per request the mixer keeps, in the request's slot, S [heads][dk][dv] (float32, zeros before a sequence's first
// token).  One stacked product has left, per token, a row with q | k [heads * dk], v | g [heads * dv] and
// low [rank] somewhere in it (offsets in elements; the compute type).  Per head, everything float32:
//     z_t     = A2 low_t + b                                       (dk numbers; A2 [heads * dk, rank])
//     alpha_t = sigmoid(z_t)^(1 / tau) = exp(log sigmoid(z_t) / tau)
//     S_t[i][j] = alpha_t[i] S_(t-1)[i][j] + k_t[i] v_t[j]
//     o_t[j]  = q_scale * sum_i q_t[i] S_t[i][j]
//     out_t[j] = o_t[j] / sqrt(mean_j o_t[j]^2 + eps) * gain[j] * silu(g_t[j]) * out_scale        (compute type)
// An entry of one token is a decode step.
//
// gla_recurrence_kernel: one CTA per (entry, head, segment); thread (group, part) holds eight rows (part) of four
// columns (group) of S in registers.  Tokens come in chunks of CH through shared memory; inside a chunk nothing but
// registers is written, and the sums over the parts are formed for all tokens of a chunk at once.
// The recurrence is linear in S, so the entries from `first_cut` on (prompt portions) are cut into `segments` runs of
// tokens that are worked on side by side: a first launch (STATE_ONLY) leaves every run's own contribution to S
// (started from zero) and its product of alphas in scratch, and a copy of the slot's S; in the second launch a run
// starts from the fold of what lies before it, in order.  Sums run in a fixed order that depends on the entry's
// length alone.
// gla_wide_kernel: any head size, S in the slot's memory throughout; for heads of more than 128 numbers.
#include "common.cuh"

namespace ps {

struct GlaInputs {
    long long ld;                          // elements between rows of the stacked product
    int q, k, v, g, low;                   // where the parts of a row begin
    const float* a2;                       // [heads * dk, rank]
    const float* bias;                     // [heads * dk]
    int rank;
    float inv_tau, q_scale;
    const float* gain;                     // [dv]
    float eps, out_scale;
    int heads, dk, dv;
};

// log(sigmoid(z)) without overflow at either end
__device__ __forceinline__ float log_sigmoid(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }

template <int DK, int DV>
struct GlaLayout {
    static constexpr int ROWS = 8, COLS = 4;                     // the block of S of one thread
    static constexpr int PARTS = DK / ROWS;                      // threads that share a group of columns
    static constexpr int THREADS = (DV / COLS) * PARTS;
    static constexpr int RUN = ROWS + 4;                         // a part's run of a row, padded against bank conflicts
    static constexpr int ROW = PARTS * RUN;
    static constexpr int CH = DK > 64 ? 8 : 16;                  // tokens of a chunk
    static constexpr int VALUES = CH * COLS / PARTS;             // sums a thread ends up with
    // floats: q, k, alpha in padded rows, v, sums, gain; then low [CH][rank], and A2 of the head [rank][DK] if it fits
    static constexpr int Q = 0, K = CH * ROW, A = 2 * CH * ROW, V = 3 * CH * ROW, Y = V + CH * DV, GAIN = Y + CH * DV,
                         LOW = GAIN + DV;
    static_assert(PARTS >= 4 && PARTS <= 16 && THREADS % 32 == 0 && THREADS % DK == 0 && VALUES >= 1, "layout");
    __host__ __device__ static bool a2_staged(int rank) { return rank <= 64; }
    __host__ __device__ static size_t bytes(int rank) {
        return (size_t)(LOW + CH * rank + (a2_staged(rank) ? rank * DK : 0)) * sizeof(float);
    }
};

// elements of one 16-byte access, as floats
__device__ __forceinline__ void gla_load16(const float* p, float (&x)[4]) {
    const float4 v = *reinterpret_cast<const float4*>(p);
    x[0] = v.x; x[1] = v.y; x[2] = v.z; x[3] = v.w;
}
__device__ __forceinline__ void gla_load16(const __nv_bfloat16* p, float (&x)[8]) {
    const uint4 raw = *reinterpret_cast<const uint4*>(p);
    const __nv_bfloat162* pair = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const float2 f = __bfloat1622float2(pair[i]);
        x[2 * i] = f.x;
        x[2 * i + 1] = f.y;
    }
}

template <typename T, int DK, int DV, bool STATE_ONLY>
__global__ void __launch_bounds__(GlaLayout<DK, DV>::THREADS)
gla_recurrence_kernel(const T* __restrict__ rows, const GlaInputs in, int wide, float* __restrict__ state,
                      long long state_stride, const int* __restrict__ q_start, const int* __restrict__ item_slot,
                      int first_item, int first_cut, int segments, float* __restrict__ run_state,
                      float* __restrict__ run_decay, T* __restrict__ out, long long out_stride) {
    using L = GlaLayout<DK, DV>;
    constexpr int PARTS = L::PARTS, ROW = L::ROW, RUN = L::RUN, CH = L::CH, THREADS = L::THREADS, VEC = 16 / sizeof(T);
    extern __shared__ __align__(16) float gla_smem[];
    float* const s_q = gla_smem + L::Q;
    float* const s_k = gla_smem + L::K;
    float* const s_a = gla_smem + L::A;
    float* const s_v = gla_smem + L::V;
    float* const s_y = gla_smem + L::Y;
    float* const s_gain = gla_smem + L::GAIN;
    float* const s_low = gla_smem + L::LOW;
    float* const s_a2 = s_low + CH * in.rank;
    const int item = first_item + blockIdx.x, h = blockIdx.y, segment = blockIdx.z, tid = threadIdx.x;
    const int dk = in.dk, dv = in.dv, rank = in.rank;
    const int begin = q_start[item], count = q_start[item + 1] - begin;
    // how this entry is cut (a rule of its length): runs of whole chunks
    const bool cut = segments > 1 && item >= first_cut;
    const int per = cut ? ((count + segments - 1) / segments + CH - 1) / CH * CH : count;
    const int runs = cut && count > 0 ? (count + per - 1) / per : 1;
    if (count <= 0 || segment >= (STATE_ONLY ? runs - 1 : runs)) return;
    const int lo = begin + segment * per, hi = min(lo + per, begin + count);
    const int part = tid % PARTS, j0 = (tid / PARTS) * 4, i0 = part * 8;
    const int lane = tid & 31, warp = tid >> 5;

    // what no kernel of this step writes: before the wait
    if (dk < DK || dv < DV)                                      // channels past dk and dv stay zero
        for (int e = tid; e < L::Y; e += THREADS) gla_smem[e] = 0.f;
    for (int j = tid; j < DV; j += THREADS) s_gain[j] = j < dv ? in.gain[j] * in.out_scale : 0.f;
    const float* a2 = in.a2 + (size_t)h * dk * rank;
    const bool a2_staged = L::a2_staged(rank);
    if (a2_staged)
        for (int e = tid; e < dk * rank; e += THREADS) s_a2[(e % rank) * DK + e / rank] = a2[e];
    const int channel = tid % DK;
    const float z_bias = channel < dk ? in.bias[h * dk + channel] : 0.f;
    // S of the slot: only this kernel of an earlier step wrote it, and that one is done
    float* S = state + (size_t)item_slot[item] * state_stride + (size_t)h * dk * dv;
    const size_t block = (size_t)dk * dv;
    // scratch entry e of (entry, head): e = 0 the slot's S at the start, e > 0 what run e - 1 adds; decays likewise
    const size_t cut_base = cut ? ((size_t)(item - first_cut) * in.heads + h) * segments : 0;
    const bool wide_state = (dv & 3) == 0 && (((uintptr_t)S | (uintptr_t)run_state) & 15) == 0;
    auto load_block = [&](const float* from, float (&to)[8][4]) {
#pragma unroll
        for (int r = 0; r < 8; ++r) {
            const int i = i0 + r;
            if (wide_state && i < dk && j0 < dv) {
                const float4 v = *reinterpret_cast<const float4*>(from + (size_t)i * dv + j0);
                to[r][0] = v.x; to[r][1] = v.y; to[r][2] = v.z; to[r][3] = v.w;
            } else {
#pragma unroll
                for (int c = 0; c < 4; ++c) to[r][c] = (i < dk && j0 + c < dv) ? from[(size_t)i * dv + j0 + c] : 0.f;
            }
        }
    };
    auto store_block = [&](float* to, const float (&from)[8][4]) {
#pragma unroll
        for (int r = 0; r < 8; ++r) {
            const int i = i0 + r;
            if (wide_state && i < dk && j0 < dv) {
                *reinterpret_cast<float4*>(to + (size_t)i * dv + j0) = make_float4(from[r][0], from[r][1], from[r][2], from[r][3]);
            } else {
#pragma unroll
                for (int c = 0; c < 4; ++c)
                    if (i < dk && j0 + c < dv) to[(size_t)i * dv + j0 + c] = from[r][c];
            }
        }
    };
    float s[8][4];
    if (STATE_ONLY ? segment == 0 : runs == 1) load_block(S, s);
    pdl_prologue();
    rows = pdl_fresh(rows);
    if (STATE_ONLY) {
        if (segment == 0) store_block(run_state + cut_base * block, s);
#pragma unroll
        for (int r = 0; r < 8; ++r) s[r][0] = s[r][1] = s[r][2] = s[r][3] = 0.f;
    } else if (runs > 1) {
        const float* kept = pdl_fresh(run_state) + cut_base * block;
        const float* decay = pdl_fresh(run_decay) + cut_base * dk;
        load_block(kept, s);
        for (int e = 1; e <= segment; ++e) {
            float add[8][4];
            load_block(kept + (size_t)e * block, add);
#pragma unroll
            for (int r = 0; r < 8; ++r) {
                const float d = i0 + r < dk ? decay[(size_t)e * dk + i0 + r] : 0.f;
#pragma unroll
                for (int c = 0; c < 4; ++c) s[r][c] = fmaf(d, s[r][c], add[r][c]);
            }
        }
    }
    float product[8];                                            // STATE_ONLY: the run's product of alphas
#pragma unroll
    for (int r = 0; r < 8; ++r) product[r] = 1.f;
    const float inv_dv = 1.0f / (float)dv;
    __syncthreads();                                             // the zeros are in place

    for (int t0 = lo; t0 < hi; t0 += CH) {
        const int n = min(CH, hi - t0);
        // ---- the chunk's rows into shared memory, as floats
        const T* base = rows + (size_t)t0 * in.ld;
        if (wide) {
            const int kp = dk / VEC, vp = dv / VEC;
            for (int e = tid; e < n * kp; e += THREADS) {
                const int tt = e / kp, i = (e - tt * kp) * VEC;
                const T* at = base + (size_t)tt * in.ld + h * dk + i;
                float x[VEC];
                gla_load16(at + in.k, x);
#pragma unroll
                for (int w = 0; w < VEC; w += 4)
                    *reinterpret_cast<float4*>(s_k + tt * ROW + ((i + w) >> 3) * RUN + ((i + w) & 7)) =
                        make_float4(x[w], x[w + 1], x[w + 2], x[w + 3]);
                if (!STATE_ONLY) {
                    gla_load16(at + in.q, x);
#pragma unroll
                    for (int w = 0; w < VEC; w += 4)
                        *reinterpret_cast<float4*>(s_q + tt * ROW + ((i + w) >> 3) * RUN + ((i + w) & 7)) =
                            make_float4(x[w], x[w + 1], x[w + 2], x[w + 3]);
                }
            }
            for (int e = tid; e < n * vp; e += THREADS) {
                const int tt = e / vp, j = (e - tt * vp) * VEC;
                float x[VEC];
                gla_load16(base + (size_t)tt * in.ld + in.v + h * dv + j, x);
#pragma unroll
                for (int w = 0; w < VEC; w += 4)
                    *reinterpret_cast<float4*>(s_v + tt * DV + j + w) = make_float4(x[w], x[w + 1], x[w + 2], x[w + 3]);
            }
        } else {
            for (int e = tid; e < n * dk; e += THREADS) {
                const int tt = e / dk, i = e - tt * dk, place = tt * ROW + (i >> 3) * RUN + (i & 7);
                const T* at = base + (size_t)tt * in.ld + h * dk + i;
                s_k[place] = to_float(at[in.k]);
                if (!STATE_ONLY) s_q[place] = to_float(at[in.q]);
            }
            for (int e = tid; e < n * dv; e += THREADS) {
                const int tt = e / dv, j = e - tt * dv;
                s_v[tt * DV + j] = to_float(base[(size_t)tt * in.ld + in.v + h * dv + j]);
            }
        }
        for (int e = tid; e < n * rank; e += THREADS) {
            const int tt = e / rank;
            s_low[e] = to_float(base[(size_t)tt * in.ld + in.low + (e - tt * rank)]);
        }
        __syncthreads();
        // ---- the decays: a thread's channel is fixed, its tokens are THREADS / DK apart
        {
            constexpr int STEP = THREADS / DK, MINE = CH / STEP > 0 ? CH / STEP : 1;
            const int first = tid / DK;
            float z[MINE];
#pragma unroll
            for (int m = 0; m < MINE; ++m) z[m] = 0.f;
            if (channel < dk && first < n) {
                for (int r = 0; r < rank; ++r) {
                    const float w = a2_staged ? s_a2[r * DK + channel] : a2[(size_t)channel * rank + r];
#pragma unroll
                    for (int m = 0; m < MINE; ++m)
                        if (first + m * STEP < n) z[m] = fmaf(w, s_low[(first + m * STEP) * rank + r], z[m]);
                }
#pragma unroll
                for (int m = 0; m < MINE; ++m) {
                    const int tt = first + m * STEP;
                    if (tt < n) s_a[tt * ROW + (channel >> 3) * RUN + (channel & 7)] = expf(log_sigmoid(z[m] + z_bias) * in.inv_tau);
                }
            }
        }
        __syncthreads();
        // ---- the chunk's tokens in order
        float y[CH * 4];
        auto token = [&](int tt) {
            const float4 vv = *reinterpret_cast<const float4*>(s_v + tt * DV + j0);
            const float v[4] = {vv.x, vv.y, vv.z, vv.w};
            if (!STATE_ONLY) y[tt * 4] = y[tt * 4 + 1] = y[tt * 4 + 2] = y[tt * 4 + 3] = 0.f;
#pragma unroll
            for (int half = 0; half < 2; ++half) {
                const int place = tt * ROW + part * RUN + 4 * half;
                const float4 kk = *reinterpret_cast<const float4*>(s_k + place);
                const float4 aa = *reinterpret_cast<const float4*>(s_a + place);
                const float k[4] = {kk.x, kk.y, kk.z, kk.w}, a[4] = {aa.x, aa.y, aa.z, aa.w};
                float q[4] = {0.f, 0.f, 0.f, 0.f};
                if (!STATE_ONLY) {
                    const float4 qq = *reinterpret_cast<const float4*>(s_q + place);
                    q[0] = qq.x; q[1] = qq.y; q[2] = qq.z; q[3] = qq.w;
                }
#pragma unroll
                for (int e = 0; e < 4; ++e) {
#pragma unroll
                    for (int c = 0; c < 4; ++c) {
                        s[4 * half + e][c] = fmaf(a[e], s[4 * half + e][c], k[e] * v[c]);
                        if (!STATE_ONLY) y[tt * 4 + c] = fmaf(q[e], s[4 * half + e][c], y[tt * 4 + c]);
                    }
                    if (STATE_ONLY) product[4 * half + e] *= a[e];
                }
            }
        };
        if (n == CH) {
#pragma unroll
            for (int tt = 0; tt < CH; ++tt) token(tt);
        } else {
#pragma unroll
            for (int tt = 0; tt < CH; ++tt) {
                if (tt < n) token(tt);
                else if (!STATE_ONLY) y[tt * 4] = y[tt * 4 + 1] = y[tt * 4 + 2] = y[tt * 4 + 3] = 0.f;
            }
        }
        if (STATE_ONLY) {
            __syncthreads();                                     // before the next chunk's rows arrive
            continue;
        }
        // ---- the sums over the parts: at every step a thread passes half of what it holds to a neighbour
        int first_sum = 0;
#pragma unroll
        for (int m = 1; m < PARTS; m <<= 1) {
            const int half = CH * 4 / (2 * m);
            const bool upper = part & m;
            if (upper) first_sum += half;
#pragma unroll
            for (int i = 0; i < half; ++i) {
                const float keep = upper ? y[half + i] : y[i], send = upper ? y[i] : y[half + i];
                y[i] = keep + __shfl_xor_sync(0xffffffffu, send, m);
            }
        }
#pragma unroll
        for (int i = 0; i < L::VALUES; ++i) {
            const int index = first_sum + i;
            s_y[(index >> 2) * DV + j0 + (index & 3)] = y[i] * in.q_scale;
        }
        __syncthreads();
        // ---- head norm, gain and gate: sixteen lanes per token (the chunk's other buffers are free from here on)
        constexpr int WARPS = THREADS / 32;
        for (int pair = 2 * warp; pair < n; pair += 2 * WARPS) {
            const int tt = pair + (lane >> 4);
            const bool valid = tt < n;
            const T* gate = base + (size_t)(valid ? tt : 0) * in.ld + in.g + h * dv;
            float o[DV / 16], factor[DV / 16], sq = 0.f;
#pragma unroll
            for (int m = 0; m < DV / 16; ++m) {
                const int j = (lane & 15) + 16 * m;
                const bool here = valid && j < dv;
                o[m] = here ? s_y[tt * DV + j] : 0.f;
                factor[m] = here ? s_gain[j] * silu(to_float(gate[j])) : 0.f;
                sq = fmaf(o[m], o[m], sq);
            }
#pragma unroll
            for (int x = 8; x > 0; x >>= 1) sq += __shfl_xor_sync(0xffffffffu, sq, x);
            const float inverse = 1.0f / sqrtf(sq * inv_dv + in.eps);
            if (valid) {
                T* target = out + (size_t)(t0 + tt) * out_stride + h * dv;
#pragma unroll
                for (int m = 0; m < DV / 16; ++m) {
                    const int j = (lane & 15) + 16 * m;
                    if (j < dv) target[j] = from_float<T>(o[m] * inverse * factor[m]);
                }
            }
        }
    }
    if (STATE_ONLY) {
        const size_t entry = cut_base + segment + 1;
        store_block(run_state + entry * block, s);
        if (tid < PARTS) {
#pragma unroll
            for (int r = 0; r < 8; ++r)
                if (i0 + r < dk) run_decay[entry * dk + i0 + r] = product[r];
        }
    } else if (segment == runs - 1) {
        store_block(S, s);
    }
}

// Any head size: one CTA per (entry, head), a thread per value column, S updated in the slot's memory.
constexpr int GLA_WIDE_THREADS = 256;

template <typename T>
__global__ void __launch_bounds__(GLA_WIDE_THREADS)
gla_wide_kernel(const T* __restrict__ rows, const GlaInputs in, float* __restrict__ state, long long state_stride,
                const int* __restrict__ q_start, const int* __restrict__ item_slot, T* __restrict__ out,
                long long out_stride) {
    extern __shared__ __align__(16) float gla_smem[];
    const int dk = in.dk, dv = in.dv, rank = in.rank;
    float* const s_q = gla_smem;
    float* const s_k = s_q + dk;
    float* const s_a = s_k + dk;
    float* const s_y = s_a + dk;
    float* const s_low = s_y + dv;
    __shared__ float partial[GLA_WIDE_THREADS / 32];
    const int item = blockIdx.x, h = blockIdx.y, tid = threadIdx.x;
    const int begin = q_start[item], end = q_start[item + 1];
    if (begin >= end) return;
    pdl_prologue();
    rows = pdl_fresh(rows);
    float* S = state + (size_t)item_slot[item] * state_stride + (size_t)h * dk * dv;
    for (int t = begin; t < end; ++t) {
        const T* row = rows + (size_t)t * in.ld;
        for (int r = tid; r < rank; r += GLA_WIDE_THREADS) s_low[r] = to_float(row[in.low + r]);
        for (int i = tid; i < dk; i += GLA_WIDE_THREADS) {
            s_q[i] = to_float(row[in.q + h * dk + i]);
            s_k[i] = to_float(row[in.k + h * dk + i]);
        }
        __syncthreads();
        for (int i = tid; i < dk; i += GLA_WIDE_THREADS) {
            const float* w = in.a2 + (size_t)(h * dk + i) * rank;
            float z = 0.f;
            for (int r = 0; r < rank; ++r) z = fmaf(w[r], s_low[r], z);
            s_a[i] = expf(log_sigmoid(z + in.bias[h * dk + i]) * in.inv_tau);
        }
        __syncthreads();
        float sq = 0.f;
        for (int j = tid; j < dv; j += GLA_WIDE_THREADS) {
            const float v = to_float(row[in.v + h * dv + j]);
            float y = 0.f;
            for (int i = 0; i < dk; ++i) {
                const float s = fmaf(s_a[i], S[(size_t)i * dv + j], s_k[i] * v);
                S[(size_t)i * dv + j] = s;
                y = fmaf(s_q[i], s, y);
            }
            y *= in.q_scale;
            s_y[j] = y;
            sq = fmaf(y, y, sq);
        }
        sq = warp_sum(sq);
        if ((tid & 31) == 0) partial[tid >> 5] = sq;
        __syncthreads();
        float total = 0.f;
        for (int w = 0; w < GLA_WIDE_THREADS / 32; ++w) total += partial[w];
        const float inverse = 1.0f / sqrtf(total / (float)dv + in.eps);
        for (int j = tid; j < dv; j += GLA_WIDE_THREADS)
            out[(size_t)t * out_stride + h * dv + j] =
                from_float<T>(s_y[j] * inverse * in.gain[j] * in.out_scale * silu(to_float(row[in.g + h * dv + j])));
        __syncthreads();
    }
}

template <typename T, int DK, int DV>
int launch_gla(const T* rows, const GlaInputs& in, int wide, float* state, long long state_stride, const int* q_start,
               const int* item_slot, int n_items, int first_cut, int segments, float* run_state, float* run_decay, T* out,
               long long out_stride, cudaStream_t s) {
    using L = GlaLayout<DK, DV>;
    const size_t smem = L::bytes(in.rank);
    if (smem > 200 * 1024) return PS_ERR_UNSUPPORTED;
    if (segments > 1) {
        auto kernel = gla_recurrence_kernel<T, DK, DV, true>;
        static size_t raised[MAX_DEVICES] = {0};
        if (!ensure_dynamic_smem((const void*)kernel, smem, raised)) return PS_ERR_LAUNCH;
        const int status = launch_pdl(kernel, dim3(n_items - first_cut, in.heads, segments - 1), dim3(L::THREADS), smem, s,
                                      rows, in, wide, state, state_stride, q_start, item_slot, first_cut, first_cut,
                                      segments, run_state, run_decay, out, out_stride);
        if (status != PS_OK) return status;
    }
    auto kernel = gla_recurrence_kernel<T, DK, DV, false>;
    static size_t raised[MAX_DEVICES] = {0};
    if (!ensure_dynamic_smem((const void*)kernel, smem, raised)) return PS_ERR_LAUNCH;
    return launch_pdl(kernel, dim3(n_items, in.heads, segments), dim3(L::THREADS), smem, s, rows, in, wide, state,
                      state_stride, q_start, item_slot, 0, first_cut, segments, run_state, run_decay, out, out_stride);
}

template <typename T>
int pick_gla(const T* rows, const GlaInputs& in, float* state, long long state_stride, const int* q_start,
             const int* item_slot, int n_items, int first_cut, int segments, float* run_state, float* run_decay, T* out,
             long long out_stride, cudaStream_t s) {
    if (in.dk > 128 || in.dv > 128 || in.rank > 256) {
        auto kernel = gla_wide_kernel<T>;
        const size_t smem = (size_t)(3 * in.dk + in.dv + in.rank) * sizeof(float);
        if (smem > 200 * 1024) return PS_ERR_UNSUPPORTED;
        static size_t raised[MAX_DEVICES] = {0};
        if (!ensure_dynamic_smem((const void*)kernel, smem, raised)) return PS_ERR_LAUNCH;
        return launch_pdl(kernel, dim3(n_items, in.heads), dim3(GLA_WIDE_THREADS), smem, s, rows, in, state, state_stride,
                          q_start, item_slot, out, out_stride);
    }
    constexpr int VEC = 16 / sizeof(T);
    const int wide = in.dk % VEC == 0 && in.dv % VEC == 0 && in.ld % VEC == 0 && in.q % VEC == 0 && in.k % VEC == 0 &&
                     in.v % VEC == 0 && !((uintptr_t)rows & 15);
#define PS_GLA(DK, DV)                                                                                             \
    return launch_gla<T, DK, DV>(rows, in, wide, state, state_stride, q_start, item_slot, n_items, first_cut, segments, \
                                 run_state, run_decay, out, out_stride, s)
#define PS_GLA_DV(DK)              \
    do {                           \
        if (in.dv <= 32) PS_GLA(DK, 32);  \
        if (in.dv <= 64) PS_GLA(DK, 64);  \
        PS_GLA(DK, 128);           \
    } while (0)
    if (in.dk <= 32) PS_GLA_DV(32);
    if (in.dk <= 64) PS_GLA_DV(64);
    PS_GLA_DV(128);
#undef PS_GLA_DV
#undef PS_GLA
}

}  // namespace ps

// rows: [T] rows of `dtype`, ld elements apart, in which q | k | v | g | low begin at the five offsets.  state: float32
// [slots] rows of state_stride, of which the first heads * dk * dv numbers are S.  Entries [first_cut, n_items) are cut
// into up to `segments` runs: run_state float32 [(n_items - first_cut) * heads * segments][dk * dv] and run_decay
// [...][dk] are scratch (null when segments is 1).  out: rows of heads * dv numbers, out_stride apart.
PS_EXPORT int ps_gla_recurrence(const void* rows, long long ld, const int* offsets, const float* a2, const float* bias,
                                int rank, float inv_tau, float q_scale, const float* gain, float eps, float out_scale,
                                float* state, long long state_stride, const int* q_start, const int* item_slot,
                                int n_items, int first_cut, int segments, float* run_state, float* run_decay, void* out,
                                long long out_stride, int heads, int dk, int dv, int dtype, void* stream) {
    if (n_items <= 0) return PS_OK;
    if (!rows || !offsets || !a2 || !bias || !gain || !state || !q_start || !item_slot || !out) return PS_ERR_BAD_ARGUMENT;
    if (rank <= 0 || heads <= 0 || heads > 65535 || dk <= 0 || dv <= 0 || first_cut < 0 || first_cut > n_items)
        return PS_ERR_BAD_ARGUMENT;
    if (segments < 1 || segments > 65535 || (segments > 1 && (!run_state || !run_decay))) return PS_ERR_BAD_ARGUMENT;
    if (first_cut == n_items) segments = 1;
    const ps::GlaInputs in{ld, offsets[0], offsets[1], offsets[2], offsets[3], offsets[4], a2, bias, rank, inv_tau, q_scale,
                           gain, eps, out_scale, heads, dk, dv};
    cudaStream_t s = (cudaStream_t)stream;
    if (dtype == PS_F32)
        return ps::pick_gla<float>((const float*)rows, in, state, state_stride, q_start, item_slot, n_items, first_cut,
                                   segments, run_state, run_decay, (float*)out, out_stride, s);
    if (dtype == PS_BF16)
        return ps::pick_gla<__nv_bfloat16>((const __nv_bfloat16*)rows, in, state, state_stride, q_start, item_slot, n_items,
                                           first_cut, segments, run_state, run_decay, (__nv_bfloat16*)out, out_stride, s);
    return PS_ERR_UNSUPPORTED;
}
