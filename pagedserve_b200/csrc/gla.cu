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
//
// gla_step_kernel:   steps in which every entry brings one token (decode).  One CTA per (entry, head); S, the decay's
//                    matrix and the constants are fetched before the wait for the product that makes the token's row.
// gla_recurrence_kernel: everything else.  One CTA per (entry, head, segment); thread (group, part) holds eight rows
//                    (part) of four columns (group) of S in registers, two rows to a packed pair.  Tokens come in chunks of
//                    CH, the next chunk's rows on their way into registers while one is worked on; inside a chunk nothing
//                    but registers is written, and the sums over the parts are formed for all tokens of a chunk at once.
// The recurrence is linear in S, so the entries from `first_cut` on (prompt portions) are cut into `segments` runs of
// tokens that are worked on side by side: gla_decay_kernel forms every token's alphas once; a first launch of the
// recurrence (STATE_ONLY) leaves every run's own contribution to S (started from zero) and its product of alphas in
// scratch, and a copy of the slot's S; gla_fold_kernel folds them in order into the S that every run starts from; the
// second launch of the recurrence does the rest.
// Sums run in a fixed order that depends on the entry's length alone.
// gla_wide_kernel:   any head size, S in the slot's memory throughout; for heads of more than 128 numbers.
#include "common.cuh"

#include <type_traits>

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

// x / (1 + exp(-x)), for the gate on the result (nothing of it is carried on)
__device__ __forceinline__ float gla_silu(float x) { return __fdividef(x, 1.0f + __expf(-x)); }
// log(sigmoid(z)) without overflow at either end
__device__ __forceinline__ float log_sigmoid(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }

// elements of one 16-byte access, as floats
__device__ __forceinline__ void gla_unpack(const uint4& raw, float (&x)[4]) {
    x[0] = __uint_as_float(raw.x); x[1] = __uint_as_float(raw.y); x[2] = __uint_as_float(raw.z); x[3] = __uint_as_float(raw.w);
}
__device__ __forceinline__ void gla_unpack(const uint4& raw, float (&x)[8]) {
    const __nv_bfloat162* pair = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const float2 f = __bfloat1622float2(pair[i]);
        x[2 * i] = f.x;
        x[2 * i + 1] = f.y;
    }
}

template <typename T, int DK, int DV>
struct GlaLayout {
    static constexpr int ROWS = 8, COLS = 4;                     // the block of S of one thread
    static constexpr int PARTS = DK / ROWS;                      // threads that share a group of columns
    static constexpr int THREADS = (DV / COLS) * PARTS;
    static constexpr int RUN = ROWS + 4;                         // a part's run of a row, padded against bank conflicts
    static constexpr int ROW = PARTS * RUN;
    static constexpr int CH = 8;                                 // tokens of a chunk
    static constexpr int CTAS = THREADS >= 512 ? 1 : 512 / THREADS;                // resident ones that registers allow
    static constexpr int VALUES = CH * COLS / PARTS;             // sums a thread ends up with
    static constexpr int VEC = 16 / (int)sizeof(T);
    // 16-byte pieces of a chunk that a thread fetches: of q (as of k), of v (as of g), of the alphas
    static constexpr int up(int a, int b) { return (a + b - 1) / b; }
    static constexpr int K_PIECES = up(CH * DK / VEC, THREADS), V_PIECES = up(CH * DV / VEC, THREADS),
                         A_PIECES = up(CH * DK / 4, THREADS);
    // floats: q, k, alpha in padded rows, v, g (two chunks of it), sums, gain; then low [CH][rank], and A2 of the head [rank][DK] if it fits
    static constexpr int Q = 0, K = CH * ROW, A = 2 * CH * ROW, V = 3 * CH * ROW, G = V + CH * DV, Y = G + 2 * CH * DV,
                         GAIN = Y + CH * DV, LOW = GAIN + DV;
    static_assert(PARTS >= 4 && PARTS <= 16 && THREADS % 32 == 0 && THREADS % DK == 0 && VALUES >= 1, "layout");
    __host__ __device__ static bool a2_staged(int rank) { return rank <= 64; }
    // (with the alphas formed beforehand neither low nor A2 has a place)
    __host__ __device__ static size_t bytes(int rank, bool decays) {
        return (size_t)(LOW + (decays ? 0 : CH * rank + (a2_staged(rank) ? rank * DK : 0))) * sizeof(float);
    }
};

// alpha[t][channel] for all heads' channels, GLA_DECAY_TOKENS tokens a CTA
constexpr int GLA_DECAY_THREADS = 256, GLA_DECAY_TOKENS = 16;

template <typename T>
__global__ void __launch_bounds__(GLA_DECAY_THREADS)
gla_decay_kernel(const T* __restrict__ rows, const GlaInputs in, float* __restrict__ alpha, int tokens) {
    extern __shared__ __align__(16) float gla_smem[];               // low, [rank][GLA_DECAY_TOKENS]
    const int channel = blockIdx.x * GLA_DECAY_THREADS + threadIdx.x, channels = in.heads * in.dk, rank = in.rank;
    const int t0 = blockIdx.y * GLA_DECAY_TOKENS, n = min(GLA_DECAY_TOKENS, tokens - t0);
    pdl_prologue();
    rows = pdl_fresh(rows);
    for (int e = threadIdx.x; e < GLA_DECAY_TOKENS * rank; e += GLA_DECAY_THREADS) {
        const int tt = e / rank, r = e - tt * rank;
        gla_smem[r * GLA_DECAY_TOKENS + tt] = tt < n ? to_float(rows[(size_t)(t0 + tt) * in.ld + in.low + r]) : 0.f;
    }
    __syncthreads();
    if (channel >= channels) return;
    const float* w = in.a2 + (size_t)channel * rank;
    const float b = in.bias[channel];
    float z[GLA_DECAY_TOKENS];
#pragma unroll
    for (int t = 0; t < GLA_DECAY_TOKENS; ++t) z[t] = 0.f;
    auto take = [&](int r, float wr) {
#pragma unroll
        for (int t = 0; t < GLA_DECAY_TOKENS; t += 4) {
            const float4 low = *reinterpret_cast<const float4*>(gla_smem + r * GLA_DECAY_TOKENS + t);
            z[t] = fmaf(wr, low.x, z[t]);
            z[t + 1] = fmaf(wr, low.y, z[t + 1]);
            z[t + 2] = fmaf(wr, low.z, z[t + 2]);
            z[t + 3] = fmaf(wr, low.w, z[t + 3]);
        }
    };
    if ((rank & 3) == 0 && !((uintptr_t)in.a2 & 15)) {
#pragma unroll 4
        for (int r = 0; r < rank; r += 4) {
            const float4 four = *reinterpret_cast<const float4*>(w + r);
            take(r, four.x); take(r + 1, four.y); take(r + 2, four.z); take(r + 3, four.w);
        }
    } else {
        for (int r = 0; r < rank; ++r) take(r, w[r]);
    }
#pragma unroll
    for (int t = 0; t < GLA_DECAY_TOKENS; ++t)
        if (t < n) alpha[(size_t)(t0 + t) * channels + channel] = expf(log_sigmoid(z[t] + b) * in.inv_tau);
}

// DECAYS: the alphas are read from `alpha` [tokens][heads * dk]; else they are formed here.
template <typename T, int DK, int DV, bool STATE_ONLY, bool DECAYS>
__global__ void __launch_bounds__(GlaLayout<T, DK, DV>::THREADS, GlaLayout<T, DK, DV>::CTAS)
gla_recurrence_kernel(const T* __restrict__ rows, const GlaInputs in, int wide, const float* __restrict__ alpha,
                      float* __restrict__ state, long long state_stride, const int* __restrict__ q_start,
                      const int* __restrict__ item_slot, int first_item, int first_cut, int segments,
                      float* __restrict__ run_state, float* __restrict__ run_decay, T* __restrict__ out,
                      long long out_stride) {
    using L = GlaLayout<T, DK, DV>;
    constexpr int PARTS = L::PARTS, ROW = L::ROW, RUN = L::RUN, CH = L::CH, THREADS = L::THREADS, VEC = L::VEC;
    extern __shared__ __align__(16) float gla_smem[];
    float* const s_q = gla_smem + L::Q;
    float* const s_k = gla_smem + L::K;
    float* const s_a = gla_smem + L::A;
    float* const s_v = gla_smem + L::V;
    float* s_g = gla_smem + L::G;                                // the chunk's; the other buffer is the chunk's before
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
    for (int j = tid; j < DV; j += THREADS) s_gain[j] = j < dv ? in.gain[j] * in.out_scale : 0.f;
    const float* a2 = in.a2 + (size_t)h * dk * rank;
    const bool a2_staged = L::a2_staged(rank);
    if (!DECAYS && a2_staged)
        for (int e = tid; e < dk * rank; e += THREADS) s_a2[(e % rank) * DK + e / rank] = a2[e];
    const int channel = tid % DK;
    const float z_bias = !DECAYS && channel < dk ? in.bias[h * dk + channel] : 0.f;
    // S of the slot: only this kernel of an earlier step wrote it, and that one is done
    float* S = state + (size_t)item_slot[item] * state_stride + (size_t)h * dk * dv;
    const size_t block = (size_t)dk * dv;
    // scratch entry e of (entry, head): e = 0 the slot's S at the start, e > 0 what run e - 1 adds (and its product of
    // alphas); gla_fold_kernel turns entry e into the S that run e starts from
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
    float start[8][4];
#pragma unroll
    for (int r = 0; r < 8; ++r) start[r][0] = start[r][1] = start[r][2] = start[r][3] = 0.f;
    if (STATE_ONLY ? segment == 0 : runs == 1) load_block(S, start);
    pdl_prologue();
    rows = pdl_fresh(rows);
    alpha = pdl_fresh(alpha);

    // ---- the rows of a chunk: 16-byte pieces on their way in registers (wide), or straight into shared memory
    uint4 in_q[L::K_PIECES], in_k[L::K_PIECES], in_v[L::V_PIECES], in_g[L::V_PIECES], in_a[L::A_PIECES];
    const uint4 zero = make_uint4(0, 0, 0, 0);
    auto fetch = [&](int t0) {
        const int n = min(CH, hi - t0);
        const T* base = rows + (size_t)t0 * in.ld;
#pragma unroll
        for (int p = 0; p < L::K_PIECES; ++p) {
            const int e = tid + p * THREADS, tt = e / (DK / VEC), i = (e % (DK / VEC)) * VEC;
            const bool here = tt < n && i < dk;
            const T* at = base + (size_t)tt * in.ld + h * dk + i;
            in_k[p] = here ? *reinterpret_cast<const uint4*>(at + in.k) : zero;
            if (!STATE_ONLY) in_q[p] = here ? *reinterpret_cast<const uint4*>(at + in.q) : zero;
        }
#pragma unroll
        for (int p = 0; p < L::V_PIECES; ++p) {
            const int e = tid + p * THREADS, tt = e / (DV / VEC), j = (e % (DV / VEC)) * VEC;
            const bool here = tt < n && j < dv;
            const T* at = base + (size_t)tt * in.ld + h * dv + j;
            in_v[p] = here ? *reinterpret_cast<const uint4*>(at + in.v) : zero;
            if (!STATE_ONLY) in_g[p] = here ? *reinterpret_cast<const uint4*>(at + in.g) : zero;
        }
        if (DECAYS) {
#pragma unroll
            for (int p = 0; p < L::A_PIECES; ++p) {
                const int e = tid + p * THREADS, tt = e / (DK / 4), i = (e % (DK / 4)) * 4;
                const bool here = tt < n && i < dk;
                in_a[p] = here ? *reinterpret_cast<const uint4*>(alpha + (size_t)(t0 + tt) * in.heads * dk + h * dk + i) : zero;
            }
        }
    };
    auto place = [&](int tt, int i) { return tt * ROW + (i >> 3) * RUN + (i & 7); };
    auto settle = [&](int t0) {
        const int n = min(CH, hi - t0);
        const T* base = rows + (size_t)t0 * in.ld;
        if (wide) {
#pragma unroll
            for (int p = 0; p < L::K_PIECES; ++p) {
                const int e = tid + p * THREADS, tt = e / (DK / VEC), i = (e % (DK / VEC)) * VEC;
                if (tt < CH) {
                    float x[VEC];
                    gla_unpack(in_k[p], x);
#pragma unroll
                    for (int w = 0; w < VEC; w += 4)
                        *reinterpret_cast<float4*>(s_k + place(tt, i + w)) = make_float4(x[w], x[w + 1], x[w + 2], x[w + 3]);
                    if (!STATE_ONLY) {
                        gla_unpack(in_q[p], x);
#pragma unroll
                        for (int w = 0; w < VEC; w += 4)
                            *reinterpret_cast<float4*>(s_q + place(tt, i + w)) = make_float4(x[w], x[w + 1], x[w + 2], x[w + 3]);
                    }
                }
            }
#pragma unroll
            for (int p = 0; p < L::V_PIECES; ++p) {
                const int e = tid + p * THREADS, tt = e / (DV / VEC), j = (e % (DV / VEC)) * VEC;
                if (tt < CH) {
                    float x[VEC];
                    gla_unpack(in_v[p], x);
#pragma unroll
                    for (int w = 0; w < VEC; w += 4)
                        *reinterpret_cast<float4*>(s_v + tt * DV + j + w) = make_float4(x[w], x[w + 1], x[w + 2], x[w + 3]);
                    if (!STATE_ONLY) {
                        gla_unpack(in_g[p], x);
#pragma unroll
                        for (int w = 0; w < VEC; w += 4)
                            *reinterpret_cast<float4*>(s_g + tt * DV + j + w) = make_float4(x[w], x[w + 1], x[w + 2], x[w + 3]);
                    }
                }
            }
            if (DECAYS) {
#pragma unroll
                for (int p = 0; p < L::A_PIECES; ++p) {
                    const int e = tid + p * THREADS, tt = e / (DK / 4), i = (e % (DK / 4)) * 4;
                    if (tt < CH) *reinterpret_cast<uint4*>(s_a + place(tt, i)) = in_a[p];
                }
            }
        } else {
            for (int e = tid; e < CH * DK; e += THREADS) {
                const int tt = e / DK, i = e % DK;
                const bool here = tt < n && i < dk;
                const T* at = base + (size_t)tt * in.ld + h * dk + i;
                s_k[place(tt, i)] = here ? to_float(at[in.k]) : 0.f;
                if (!STATE_ONLY) s_q[place(tt, i)] = here ? to_float(at[in.q]) : 0.f;
                if (DECAYS) s_a[place(tt, i)] = here ? alpha[(size_t)(t0 + tt) * in.heads * dk + h * dk + i] : 0.f;
            }
            for (int e = tid; e < CH * DV; e += THREADS) {
                const int tt = e / DV, j = e % DV;
                const bool here = tt < n && j < dv;
                const T* at = base + (size_t)tt * in.ld + h * dv + j;
                s_v[e] = here ? to_float(at[in.v]) : 0.f;
                if (!STATE_ONLY) s_g[e] = here ? to_float(at[in.g]) : 0.f;
            }
        }
        if (!DECAYS) {
            for (int e = tid; e < n * rank; e += THREADS) {
                const int tt = e / rank;
                s_low[e] = to_float(base[(size_t)tt * in.ld + in.low + (e - tt * rank)]);
            }
        }
    };
    if (wide) fetch(lo);

    if (STATE_ONLY) {
        if (segment == 0) store_block(run_state + cut_base * block, start);
#pragma unroll
        for (int r = 0; r < 8; ++r) start[r][0] = start[r][1] = start[r][2] = start[r][3] = 0.f;
    } else if (runs > 1) {
        load_block(pdl_fresh(run_state) + (cut_base + segment) * block, start);
    }
    unsigned long long s[4][4];                                  // s[p][c]: rows i0 + 2p and + 1 of column j0 + c
#pragma unroll
    for (int p = 0; p < 4; ++p)
#pragma unroll
        for (int c = 0; c < 4; ++c) s[p][c] = pair_of(start[2 * p][c], start[2 * p + 1][c]);
    unsigned long long product[4];                               // STATE_ONLY: the run's product of alphas
#pragma unroll
    for (int p = 0; p < 4; ++p) product[p] = pair_of(1.f, 1.f);
    const float inv_dv = 1.0f / (float)dv;

    for (int t0 = lo; t0 < hi; t0 += CH) {
        const int n = min(CH, hi - t0);
        // q, k, v and the alphas of the chunk before were last read ahead of its second barrier; its gates, which the head
        // norm may still be reading, lie in the other buffer; its sums are overwritten behind the next barrier only
        settle(t0);
        __syncthreads();
        if (wide && t0 + CH < hi) fetch(t0 + CH);
        // ---- the decays: a thread's channel is fixed, its tokens are THREADS / DK apart
        if (!DECAYS) {
            constexpr int STEP = THREADS / DK, MINE = CH / STEP > 0 ? CH / STEP : 1;
            const int first = tid / DK;
            float z[MINE];
#pragma unroll
            for (int m = 0; m < MINE; ++m) z[m] = 0.f;
            if (first < CH) {
                if (channel < dk) {
                    for (int r = 0; r < rank; ++r) {
                        const float w = a2_staged ? s_a2[r * DK + channel] : a2[(size_t)channel * rank + r];
#pragma unroll
                        for (int m = 0; m < MINE; ++m)
                            if (first + m * STEP < n) z[m] = fmaf(w, s_low[(first + m * STEP) * rank + r], z[m]);
                    }
                }
#pragma unroll
                for (int m = 0; m < MINE; ++m) {
                    const int tt = first + m * STEP;
                    if (tt < n) s_a[place(tt, channel)] = channel < dk ? expf(log_sigmoid(z[m] + z_bias) * in.inv_tau) : 0.f;
                }
            }
            __syncthreads();
        }
        // ---- the chunk's tokens in order
        float y[CH * 4];
        auto token = [&](int tt) {
            const float4 vv = *reinterpret_cast<const float4*>(s_v + tt * DV + j0);
            const unsigned long long v[4] = {pair_of(vv.x, vv.x), pair_of(vv.y, vv.y), pair_of(vv.z, vv.z), pair_of(vv.w, vv.w)};
            unsigned long long sum[4];
#pragma unroll
            for (int half = 0; half < 2; ++half) {
                const int at = tt * ROW + part * RUN + 4 * half;
                const ulonglong2 kk = *reinterpret_cast<const ulonglong2*>(s_k + at);
                const ulonglong2 aa = *reinterpret_cast<const ulonglong2*>(s_a + at);
                const unsigned long long k[2] = {kk.x, kk.y}, a[2] = {aa.x, aa.y};
                unsigned long long q[2] = {0, 0};
                if (!STATE_ONLY) {
                    const ulonglong2 qq = *reinterpret_cast<const ulonglong2*>(s_q + at);
                    q[0] = qq.x; q[1] = qq.y;
                }
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    const int p = 2 * half + e;
#pragma unroll
                    for (int c = 0; c < 4; ++c) {
                        s[p][c] = pair_fma(a[e], s[p][c], pair_mul(k[e], v[c]));
                        if (!STATE_ONLY) sum[c] = p == 0 ? pair_mul(q[e], s[p][c]) : pair_fma(q[e], s[p][c], sum[c]);
                    }
                    if (STATE_ONLY) product[p] = pair_mul(product[p], a[e]);
                }
            }
            if (!STATE_ONLY) {
#pragma unroll
                for (int c = 0; c < 4; ++c) {
                    float even, odd;
                    pair_split(sum[c], even, odd);
                    y[tt * 4 + c] = even + odd;
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
        // ---- head norm, gain and gate: sixteen lanes per token
        constexpr int WARPS = THREADS / 32;
        for (int pair = 2 * warp; pair < n; pair += 2 * WARPS) {
            const int tt = pair + (lane >> 4);
            const bool valid = tt < n;
            float o[DV / 16], factor[DV / 16], sq = 0.f;
#pragma unroll
            for (int m = 0; m < DV / 16; ++m) {
                const int j = (lane & 15) + 16 * m;
                const bool here = valid && j < dv;
                o[m] = here ? s_y[tt * DV + j] : 0.f;
                factor[m] = here ? s_gain[j] * gla_silu(s_g[tt * DV + j]) : 0.f;
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
        s_g = gla_smem + L::G + (s_g == gla_smem + L::G ? CH * DV : 0);
    }
    float end[8][4];
#pragma unroll
    for (int p = 0; p < 4; ++p)
#pragma unroll
        for (int c = 0; c < 4; ++c) pair_split(s[p][c], end[2 * p][c], end[2 * p + 1][c]);
    if (STATE_ONLY) {
        const size_t entry = cut_base + segment + 1;
        store_block(run_state + entry * block, end);
        if (tid < PARTS) {
#pragma unroll
            for (int p = 0; p < 4; ++p) {
                float even, odd;
                pair_split(product[p], even, odd);
                if (i0 + 2 * p < dk) run_decay[entry * dk + i0 + 2 * p] = even;
                if (i0 + 2 * p + 1 < dk) run_decay[entry * dk + i0 + 2 * p + 1] = odd;
            }
        }
    } else if (segment == runs - 1) {
        store_block(S, end);
    }
}

// run_state[e] <- run_decay[e] * run_state[e - 1] + run_state[e] for e = 1 .. runs - 1, element by element.
constexpr int GLA_FOLD_THREADS = 128, GLA_FOLD_AHEAD = 8;

template <int V>
__global__ void __launch_bounds__(GLA_FOLD_THREADS)
gla_fold_kernel(float* __restrict__ run_state, const float* __restrict__ run_decay, const int* __restrict__ q_start,
                int first_cut, int segments, int chunk, int heads, int dk, int dv) {
    const int unit = (blockIdx.x * GLA_FOLD_THREADS + threadIdx.x) * V, item = first_cut + blockIdx.z;
    const int count = q_start[item + 1] - q_start[item];
    pdl_prologue();
    if (count <= 0 || unit >= dk * dv) return;
    const int per = ((count + segments - 1) / segments + chunk - 1) / chunk * chunk, runs = (count + per - 1) / per;
    const size_t base = ((size_t)blockIdx.z * heads + blockIdx.y) * segments, block = (size_t)dk * dv;
    float* at = pdl_fresh(run_state) + base * block + unit;
    const float* decay = pdl_fresh(run_decay) + base * dk + unit / dv;
    using Pack = typename std::conditional<V == 4, float4, float>::type;
    Pack s = *reinterpret_cast<const Pack*>(at);
    for (int e0 = 1; e0 < runs; e0 += GLA_FOLD_AHEAD) {
        Pack add[GLA_FOLD_AHEAD];
        float d[GLA_FOLD_AHEAD];
#pragma unroll
        for (int a = 0; a < GLA_FOLD_AHEAD; ++a) {
            if (e0 + a < runs) {
                add[a] = *reinterpret_cast<const Pack*>(at + (size_t)(e0 + a) * block);
                d[a] = decay[(size_t)(e0 + a) * dk];
            }
        }
#pragma unroll
        for (int a = 0; a < GLA_FOLD_AHEAD; ++a) {
            if (e0 + a < runs) {
                if constexpr (V == 4) {
                    s.x = fmaf(d[a], s.x, add[a].x); s.y = fmaf(d[a], s.y, add[a].y);
                    s.z = fmaf(d[a], s.z, add[a].z); s.w = fmaf(d[a], s.w, add[a].w);
                } else {
                    s = fmaf(d[a], s, add[a]);
                }
                *reinterpret_cast<Pack*>(at + (size_t)(e0 + a) * block) = s;
            }
        }
    }
}

// One token per entry.  The same blocks of S per thread; every thread reads its own q, k and v from the token's row.
template <typename T, int DK, int DV>
__global__ void __launch_bounds__(GlaLayout<T, DK, DV>::THREADS)
gla_step_kernel(const T* __restrict__ rows, const GlaInputs in, int wide, float* __restrict__ state, long long state_stride,
                const int* __restrict__ q_start, const int* __restrict__ item_slot, T* __restrict__ out,
                long long out_stride) {
    using L = GlaLayout<T, DK, DV>;
    constexpr int PARTS = L::PARTS, THREADS = L::THREADS, SHARE = THREADS / DK;     // SHARE threads form one alpha
    extern __shared__ __align__(16) float gla_smem[];                             // A2 of the head, as it lies
    __shared__ __align__(16) float s_a[DK];
    __shared__ float s_low[256];
    __shared__ float s_sq[THREADS / 32];
    const int item = blockIdx.x, h = blockIdx.y, tid = threadIdx.x;
    const int dk = in.dk, dv = in.dv, rank = in.rank;
    const int t = q_start[item];
    if (q_start[item + 1] <= t) return;
    const int part = tid % PARTS, j0 = (tid / PARTS) * 4, i0 = part * 8;
    float* S = state + (size_t)item_slot[item] * state_stride + (size_t)h * dk * dv;
    const bool wide_state = (dv & 3) == 0 && ((uintptr_t)S & 15) == 0;
    // ---- before the wait: S (only this kernel of an earlier step wrote it, and that one is done) and the constants
    float s[8][4];
#pragma unroll
    for (int r = 0; r < 8; ++r) {
        const int i = i0 + r;
        if (wide_state && i < dk && j0 < dv) {
            const float4 v = *reinterpret_cast<const float4*>(S + (size_t)i * dv + j0);
            s[r][0] = v.x; s[r][1] = v.y; s[r][2] = v.z; s[r][3] = v.w;
        } else {
#pragma unroll
            for (int c = 0; c < 4; ++c) s[r][c] = (i < dk && j0 + c < dv) ? S[(size_t)i * dv + j0 + c] : 0.f;
        }
    }
    const float* a2 = in.a2 + (size_t)h * dk * rank;
    for (int e = tid; e < dk * rank; e += THREADS) gla_smem[e] = a2[e];
    const int channel = tid / SHARE;
    const float z_bias = channel < dk ? in.bias[h * dk + channel] : 0.f;
    const int mine = j0 + (part & 3);                            // the column this thread writes (parts 0 to 3)
    const float gain = mine < dv ? in.gain[mine] * in.out_scale : 0.f;
    pdl_prologue();
    rows = pdl_fresh(rows);
    // ---- the token's row
    const T* row = rows + (size_t)t * in.ld;
    for (int r = tid; r < rank; r += THREADS) s_low[r] = to_float(row[in.low + r]);
    float q[8], k[8], v[4];
    if (wide && i0 < dk) {
#pragma unroll
        for (int w = 0; w < 8; w += L::VEC) {
            float x[L::VEC];
            gla_unpack(*reinterpret_cast<const uint4*>(row + in.q + h * dk + i0 + w), x);
#pragma unroll
            for (int e = 0; e < L::VEC; ++e) q[w + e] = i0 + w + e < dk ? x[e] : 0.f;
            gla_unpack(*reinterpret_cast<const uint4*>(row + in.k + h * dk + i0 + w), x);
#pragma unroll
            for (int e = 0; e < L::VEC; ++e) k[w + e] = i0 + w + e < dk ? x[e] : 0.f;
        }
    } else {
#pragma unroll
        for (int r = 0; r < 8; ++r) {
            q[r] = i0 + r < dk ? to_float(row[in.q + h * dk + i0 + r]) : 0.f;
            k[r] = i0 + r < dk ? to_float(row[in.k + h * dk + i0 + r]) : 0.f;
        }
    }
#pragma unroll
    for (int c = 0; c < 4; ++c) v[c] = j0 + c < dv ? to_float(row[in.v + h * dv + j0 + c]) : 0.f;
    const float gate = mine < dv ? to_float(row[in.g + h * dv + mine]) : 0.f;
    __syncthreads();
    // ---- the decays
    {
        float z = 0.f;
        if (channel < dk)
            for (int r = tid % SHARE; r < rank; r += SHARE) z = fmaf(gla_smem[channel * rank + r], s_low[r], z);
#pragma unroll
        for (int x = 1; x < SHARE; x <<= 1) z += __shfl_xor_sync(0xffffffffu, z, x);
        if (tid % SHARE == 0) s_a[channel] = channel < dk ? expf(log_sigmoid(z + z_bias) * in.inv_tau) : 0.f;
    }
    __syncthreads();
    // ---- S and the sums over the key channels
    const float4 a_lo = *reinterpret_cast<const float4*>(s_a + i0), a_hi = *reinterpret_cast<const float4*>(s_a + i0 + 4);
    const float a[8] = {a_lo.x, a_lo.y, a_lo.z, a_lo.w, a_hi.x, a_hi.y, a_hi.z, a_hi.w};
    float y[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
    for (int r = 0; r < 8; ++r) {
#pragma unroll
        for (int c = 0; c < 4; ++c) {
            s[r][c] = fmaf(a[r], s[r][c], k[r] * v[c]);
            y[c] = fmaf(q[r], s[r][c], y[c]);
        }
        const int i = i0 + r;
        if (wide_state && i < dk && j0 < dv) {
            *reinterpret_cast<float4*>(S + (size_t)i * dv + j0) = make_float4(s[r][0], s[r][1], s[r][2], s[r][3]);
        } else {
#pragma unroll
            for (int c = 0; c < 4; ++c)
                if (i < dk && j0 + c < dv) S[(size_t)i * dv + j0 + c] = s[r][c];
        }
    }
#pragma unroll
    for (int x = 1; x < PARTS; x <<= 1)
#pragma unroll
        for (int c = 0; c < 4; ++c) y[c] += __shfl_xor_sync(0xffffffffu, y[c], x);
#pragma unroll
    for (int c = 0; c < 4; ++c) y[c] *= in.q_scale;
    // ---- head norm, gain and gate (columns past dv hold zeros)
    float sq = part == 0 ? fmaf(y[0], y[0], y[1] * y[1]) + fmaf(y[2], y[2], y[3] * y[3]) : 0.f;
    sq = warp_sum(sq);
    if ((tid & 31) == 0) s_sq[tid >> 5] = sq;
    __syncthreads();
    float total = 0.f;
#pragma unroll
    for (int w = 0; w < THREADS / 32; ++w) total += s_sq[w];
    const float inverse = 1.0f / sqrtf(total / (float)dv + in.eps);
    const float own = (part & 3) == 0 ? y[0] : (part & 3) == 1 ? y[1] : (part & 3) == 2 ? y[2] : y[3];
    if (part < 4 && mine < dv) out[(size_t)t * out_stride + h * dv + mine] = from_float<T>(own * inverse * gain * silu(gate));
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

template <typename T, int DK, int DV, bool STATE_ONLY, bool DECAYS>
int launch_gla_recurrence(dim3 grid, size_t smem, cudaStream_t s, const T* rows, const GlaInputs& in, int wide,
                          const float* alpha, float* state, long long state_stride, const int* q_start, const int* item_slot,
                          int first_item, int first_cut, int segments, float* run_state, float* run_decay, T* out,
                          long long out_stride) {
    auto kernel = gla_recurrence_kernel<T, DK, DV, STATE_ONLY, DECAYS>;
    static size_t raised[MAX_DEVICES] = {0};
    if (!ensure_dynamic_smem((const void*)kernel, smem, raised)) return PS_ERR_LAUNCH;
    return launch_pdl(kernel, grid, dim3(GlaLayout<T, DK, DV>::THREADS), smem, s, rows, in, wide, alpha, state, state_stride,
                      q_start, item_slot, first_item, first_cut, segments, run_state, run_decay, out, out_stride);
}

template <typename T, int DK, int DV>
int launch_gla(const T* rows, const GlaInputs& in, int wide, int tokens, int single, float* state, long long state_stride,
               const int* q_start, const int* item_slot, int n_items, int first_cut, int segments, float* alpha,
               float* run_state, float* run_decay, T* out, long long out_stride, cudaStream_t s) {
    using L = GlaLayout<T, DK, DV>;
    if (single && (size_t)in.dk * in.rank * sizeof(float) <= 64 * 1024) {
        auto kernel = gla_step_kernel<T, DK, DV>;
        const size_t smem = (size_t)in.dk * in.rank * sizeof(float);
        static size_t raised[MAX_DEVICES] = {0};
        if (!ensure_dynamic_smem((const void*)kernel, smem, raised)) return PS_ERR_LAUNCH;
        return launch_pdl(kernel, dim3(n_items, in.heads), dim3(L::THREADS), smem, s, rows, in, wide, state, state_stride,
                          q_start, item_slot, out, out_stride);
    }
    if (segments > 1) {
        int status = launch_pdl(gla_decay_kernel<T>,
                                dim3((in.heads * in.dk + GLA_DECAY_THREADS - 1) / GLA_DECAY_THREADS,
                                     (tokens + GLA_DECAY_TOKENS - 1) / GLA_DECAY_TOKENS),
                                dim3(GLA_DECAY_THREADS), (size_t)in.rank * GLA_DECAY_TOKENS * sizeof(float), s, rows, in, alpha,
                                tokens);
        if (status != PS_OK) return status;
        const size_t smem = L::bytes(in.rank, true);
        status = launch_gla_recurrence<T, DK, DV, true, true>(dim3(n_items - first_cut, in.heads, segments - 1), smem, s, rows,
                                                              in, wide, alpha, state, state_stride, q_start, item_slot,
                                                              first_cut, first_cut, segments, run_state, run_decay, out,
                                                              out_stride);
        if (status != PS_OK) return status;
        // (a unit of four numbers lies in one row of S where dv is a multiple of four)
        const bool by4 = in.dv % 4 == 0 && !((uintptr_t)run_state & 15);
        const int units = by4 ? in.dk * in.dv / 4 : in.dk * in.dv;
        status = launch_pdl(by4 ? gla_fold_kernel<4> : gla_fold_kernel<1>,
                            dim3((units + GLA_FOLD_THREADS - 1) / GLA_FOLD_THREADS, in.heads, n_items - first_cut),
                            dim3(GLA_FOLD_THREADS), 0, s, run_state, (const float*)run_decay, q_start, first_cut, segments,
                            (int)L::CH, in.heads, in.dk, in.dv);
        if (status != PS_OK) return status;
        return launch_gla_recurrence<T, DK, DV, false, true>(dim3(n_items, in.heads, segments), smem, s, rows, in, wide, alpha,
                                                             state, state_stride, q_start, item_slot, 0, first_cut, segments,
                                                             run_state, run_decay, out, out_stride);
    }
    const size_t smem = L::bytes(in.rank, false);
    if (smem > 200 * 1024) return PS_ERR_UNSUPPORTED;
    return launch_gla_recurrence<T, DK, DV, false, false>(dim3(n_items, in.heads), smem, s, rows, in, wide, alpha, state,
                                                          state_stride, q_start, item_slot, 0, first_cut, 1, run_state,
                                                          run_decay, out, out_stride);
}

template <typename T>
int pick_gla(const T* rows, const GlaInputs& in, int tokens, int single, float* state, long long state_stride,
             const int* q_start, const int* item_slot, int n_items, int first_cut, int segments, float* alpha,
             float* run_state, float* run_decay, T* out, long long out_stride, cudaStream_t s) {
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
                     in.v % VEC == 0 && in.g % VEC == 0 && !((uintptr_t)rows & 15) && !((uintptr_t)alpha & 15);
#define PS_GLA(DK, DV)                                                                                                \
    return launch_gla<T, DK, DV>(rows, in, wide, tokens, single, state, state_stride, q_start, item_slot, n_items, first_cut, \
                                 segments, alpha, run_state, run_decay, out, out_stride, s)
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
// [slots] rows of state_stride, of which the first heads * dk * dv numbers are S.  single: every entry brings exactly one
// token.  Entries [first_cut, n_items) are cut into up to `segments` runs: alpha float32 [T][heads * dk], run_state float32
// [(n_items - first_cut) * heads * segments][dk * dv] and run_decay [...][dk] are scratch (null when segments is 1).
// out: rows of heads * dv numbers, out_stride apart.
PS_EXPORT int ps_gla_recurrence(const void* rows, long long ld, const int* offsets, const float* a2, const float* bias,
                                int rank, float inv_tau, float q_scale, const float* gain, float eps, float out_scale,
                                float* state, long long state_stride, const int* q_start, const int* item_slot,
                                int n_items, int T, int single, int first_cut, int segments, float* alpha, float* run_state,
                                float* run_decay, void* out, long long out_stride, int heads, int dk, int dv, int dtype,
                                void* stream) {
    if (n_items <= 0 || T <= 0) return PS_OK;
    if (!rows || !offsets || !a2 || !bias || !gain || !state || !q_start || !item_slot || !out) return PS_ERR_BAD_ARGUMENT;
    if (rank <= 0 || heads <= 0 || heads > 65535 || dk <= 0 || dv <= 0 || first_cut < 0 || first_cut > n_items)
        return PS_ERR_BAD_ARGUMENT;
    if (segments < 1 || segments > 65535 || (segments > 1 && (!alpha || !run_state || !run_decay))) return PS_ERR_BAD_ARGUMENT;
    if (first_cut == n_items) segments = 1;
    const ps::GlaInputs in{ld, offsets[0], offsets[1], offsets[2], offsets[3], offsets[4], a2, bias, rank, inv_tau, q_scale,
                           gain, eps, out_scale, heads, dk, dv};
    cudaStream_t s = (cudaStream_t)stream;
    if (dtype == PS_F32)
        return ps::pick_gla<float>((const float*)rows, in, T, single, state, state_stride, q_start, item_slot, n_items,
                                   first_cut, segments, alpha, run_state, run_decay, (float*)out, out_stride, s);
    if (dtype == PS_BF16)
        return ps::pick_gla<__nv_bfloat16>((const __nv_bfloat16*)rows, in, T, single, state, state_stride, q_start, item_slot,
                                           n_items, first_cut, segments, alpha, run_state, run_decay, (__nv_bfloat16*)out,
                                           out_stride, s);
    return PS_ERR_UNSUPPORTED;
}
