// State-space recurrence with one decay per head and token (a matrix state that shrinks by a number).
//
// Per request the mixer keeps, in the request's slot, S [heads][N][P] (float32, zeros before a sequence's first token).  Of a
// token the kernels read x [heads][P], B [groups][N], C [groups][N] (side by side in one row of the compute type, behind their
// convolution) and z [heads][P], dt [heads] (in the row of the projection).  Per head, everything float32, head h with the B
// and C of group h / (heads / groups):
//     d_t    = softplus(dt_t + bias_h)
//     S_t    = exp(-exp(A_h) d_t) S_(t-1) + d_t B_t x_t^T
//     out_t  = (S_t^T C_t + D_h x_t) * silu(z_t)                    (rows of heads * P numbers; the norm behind is another kernel)
//
// ssd_step_kernel: entries of few tokens (decode).  One CTA per (entry, head); S goes through registers, four columns an
//                  access, the first rows on their way before the wait for the kernel that makes the token's row.
// ssd_prompt_kernel: prompt portions in bfloat16, on tensor cores to float32 accuracy.  One CTA per (entry, head, tile of
//                  columns, run of tokens), chunks of 64 tokens (copied in by cp.async, the next chunk's on their way), S as
//                  float32 mma accumulators that stay in registers.  The equations are those of the next kernel; every matrix
//                  product has one operand that is bfloat16 as it comes (x, B, C) and one float32 operand, which is cut into
//                  three bfloat16 pieces (together its 24 bits), so that the products are those of float32 numbers.
// ssd_scan_kernel: all other portions, float32 arithmetic on CUDA cores, any size.  One CTA per (entry, head, tile of columns, run
//                  of tokens): a lane holds one or two columns, a warp N / 8 rows of S in registers, two rows to a packed pair.
//                  Tokens come in chunks of 16, the next chunk's rows on their way in registers while one is worked on.  With
//                  S the state ahead of a chunk and L_t the sum of the chunk's -exp(A_h) d up to and including token t,
//                      y_t = exp(L_t) C_t S + sum over s <= t of exp(L_t - L_s) d_s (C_t . B_s) x_s,
//                      S  <- exp(L_end) S + sum over s of exp(L_end - L_s) d_s B_s x_s^T,
//                  so that a state element takes one multiply-add per token for the result and one for the update.  (Exponents
//                  are never positive: nothing overflows however fast a head forgets.)  The 16 x 16 products C_t . B_s come
//                  from mma.sync where B and C are bfloat16 (exact products, float32 sums).
// The recurrence is linear in S, so the entries from `first_cut` on (prompt portions) are cut into `segments` runs of tokens that
// are worked on side by side: a first launch (STATE_ONLY) leaves every run's own contribution to S (started from zero) and the
// product of its decays in scratch, ssd_fold_kernel folds them in order into the S that every run starts from, the second
// launch does the rest.  Sums run in a fixed order that depends on the entry's length alone.
#include "common.cuh"

namespace ps {

struct SsdInputs {
    long long ld_conv, ld_raw;             // elements between rows of the convolved and of the projected rows
    int x, b, c, z, dt;                    // where the parts begin: x, B, C in a convolved row, z and dt in a projected one
    const float* a_log;                    // [heads]
    const float* dt_bias;                  // [heads]
    const float* d;                        // [heads]
    int heads, groups, N, P;
};

__device__ __forceinline__ float softplus(float v) { return fmaxf(v, 0.f) + log1pf(expf(-fabsf(v))); }

constexpr int SSD_THREADS = 256, SSD_WARPS = 8, SSD_CHUNK = 16;

// how an entry of `count` tokens is cut into runs of whole chunks
__host__ __device__ __forceinline__ int ssd_run_length(int count, int segments, int chunk) {
    return ((count + segments - 1) / segments + chunk - 1) / chunk * chunk;
}

// elements of one 16-byte access, as floats
__device__ __forceinline__ void ssd_unpack(const uint4& raw, float (&x)[4]) {
    x[0] = __uint_as_float(raw.x); x[1] = __uint_as_float(raw.y); x[2] = __uint_as_float(raw.z); x[3] = __uint_as_float(raw.w);
}
__device__ __forceinline__ void ssd_unpack(const uint4& raw, float (&x)[8]) {
    const __nv_bfloat162* pair = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const float2 f = __bfloat1622float2(pair[i]);
        x[2 * i] = f.x;
        x[2 * i + 1] = f.y;
    }
}

// R: rows of S of a warp (N <= 8 R); CPL: columns of a lane
template <typename T, int R, int CPL>
struct SsdLayout {
    static constexpr int CH = SSD_CHUNK, NP = SSD_WARPS * R, COLS = 32 * CPL, ROW = NP + 4;      // ROW: padded against bank conflicts
    static constexpr int VEC = 16 / (int)sizeof(T);
    static constexpr int up(int a, int b) { return (a + b - 1) / b; }
    static constexpr int N_PIECES = up(CH * NP / VEC, SSD_THREADS), P_PIECES = up(CH * COLS / VEC, SSD_THREADS);
    // floats: B, C (padded rows), x, z, the warps' sums, the chunk's weights W; then B and C as they came (bfloat16 only)
    static constexpr int B = 0, C = CH * ROW, X = 2 * CH * ROW, Z = X + CH * COLS, Y = Z + CH * COLS, W = Y + SSD_WARPS * CH * COLS,
                         TYPED = W + CH * (CH + 4);
    static constexpr int TROW = NP + 8;                          // a row of the typed tiles, in elements
    static constexpr size_t BYTES = (size_t)TYPED * 4 + (sizeof(T) == 2 ? (size_t)2 * CH * TROW * 2 : 0);
};

template <typename T, typename TO, int R, int CPL, bool STATE_ONLY>
__global__ void __launch_bounds__(SSD_THREADS, R * CPL <= 32 ? 2 : 1)
ssd_scan_kernel(const T* __restrict__ conv, const T* __restrict__ raw, const SsdInputs in, int wide, float* __restrict__ state,
                long long state_stride, const int* __restrict__ q_start, const int* __restrict__ item_slot, int first_item,
                int last_item, int first_cut, int segments, float* __restrict__ run_state, float* __restrict__ run_decay,
                TO* __restrict__ out, long long out_stride) {
    using L = SsdLayout<T, R, CPL>;
    constexpr int CH = L::CH, NP = L::NP, COLS = L::COLS, ROW = L::ROW, VEC = L::VEC, TROW = L::TROW;
    extern __shared__ __align__(16) float ssd_smem[];
    float* const s_b = ssd_smem + L::B;
    float* const s_c = ssd_smem + L::C;
    float* const s_x = ssd_smem + L::X;
    float* const s_z = ssd_smem + L::Z;
    float* const s_y = ssd_smem + L::Y;
    float* const s_w = ssd_smem + L::W;                          // [CH][CH + 4]
    T* const t_b = reinterpret_cast<T*>(ssd_smem + L::TYPED);
    T* const t_c = t_b + CH * TROW;
    // of the chunk's tokens: step size, sum of the decays' logarithms so far, its exponential, weight in the update
    __shared__ float s_dt[CH], s_log[CH], s_from[CH], s_to[CH];
    const int item = first_item + blockIdx.x, h = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int col_tiles = (in.P + COLS - 1) / COLS;
    const int p0 = (blockIdx.z % col_tiles) * COLS, segment = blockIdx.z / col_tiles, p = p0 + CPL * lane;
    if (item >= last_item) return;
    const int begin = q_start[item], count = q_start[item + 1] - begin;
    const bool cut = segments > 1 && item >= first_cut;
    const int per = cut ? ssd_run_length(count, segments, CH) : count;
    const int runs = cut && count > 0 ? (count + per - 1) / per : 1;
    if (count <= 0 || segment >= (STATE_ONLY ? runs - 1 : runs)) return;
    const int lo = begin + segment * per, hi = min(lo + per, begin + count);
    const int N = in.N, P = in.P, n0 = warp * R, g = h / (in.heads / in.groups);
    const float rate = -expf(in.a_log[h]), bias = in.dt_bias[h], skip = in.d[h];
    const size_t block = (size_t)N * P;
    float* S = state + (size_t)item_slot[item] * state_stride + (size_t)h * block;
    const size_t cut_base = cut ? ((size_t)(item - first_cut) * in.heads + h) * segments : 0;

    unsigned long long s[R / 2][CPL];                            // s[r][c]: rows n0 + 2r and + 1 of column p + c
    auto load_state = [&](const float* from) {
#pragma unroll
        for (int r = 0; r < R / 2; ++r)
#pragma unroll
            for (int c = 0; c < CPL; ++c) {
                const int n = n0 + 2 * r;
                const float a = (p + c < P && n < N) ? from[(size_t)n * P + p + c] : 0.f;
                const float b = (p + c < P && n + 1 < N) ? from[(size_t)(n + 1) * P + p + c] : 0.f;
                s[r][c] = pair_of(a, b);
            }
    };
    auto store_state = [&](float* to) {
#pragma unroll
        for (int r = 0; r < R / 2; ++r)
#pragma unroll
            for (int c = 0; c < CPL; ++c) {
                const int n = n0 + 2 * r;
                float a, b;
                pair_split(s[r][c], a, b);
                if (p + c < P && n < N) to[(size_t)n * P + p + c] = a;
                if (p + c < P && n + 1 < N) to[(size_t)(n + 1) * P + p + c] = b;
            }
    };
    // S of the slot: only this kernel of an earlier step wrote it, and that one is done
    if (STATE_ONLY ? segment == 0 : runs == 1) load_state(S);
    pdl_prologue();
    conv = pdl_fresh(conv);
    raw = pdl_fresh(raw);

    // ---- the rows of a chunk: 16-byte pieces on their way in registers (wide), or straight into shared memory
    uint4 in_b[L::N_PIECES], in_c[L::N_PIECES], in_x[L::P_PIECES], in_z[L::P_PIECES];
    const uint4 zero = make_uint4(0, 0, 0, 0);
    float in_dt = 0.f;
    auto fetch = [&](int t0) {
        const int n = min(CH, hi - t0);
        if (tid < n) in_dt = to_float(raw[(size_t)(t0 + tid) * in.ld_raw + in.dt + h]);
        if (!wide) return;
#pragma unroll
        for (int q = 0; q < L::N_PIECES; ++q) {
            const int e = tid + q * SSD_THREADS, tt = e / (NP / VEC), i = (e % (NP / VEC)) * VEC;
            const bool here = tt < n && i < N;
            const T* at = conv + (size_t)(t0 + tt) * in.ld_conv + (size_t)g * N + i;
            in_b[q] = here ? *reinterpret_cast<const uint4*>(at + in.b) : zero;
            if (!STATE_ONLY) in_c[q] = here ? *reinterpret_cast<const uint4*>(at + in.c) : zero;
        }
#pragma unroll
        for (int q = 0; q < L::P_PIECES; ++q) {
            const int e = tid + q * SSD_THREADS, tt = e / (COLS / VEC), j = (e % (COLS / VEC)) * VEC;
            const bool here = tt < n && p0 + j < P;
            in_x[q] = here ? *reinterpret_cast<const uint4*>(conv + (size_t)(t0 + tt) * in.ld_conv + in.x + (size_t)h * P + p0 + j) : zero;
            if (!STATE_ONLY)
                in_z[q] = here ? *reinterpret_cast<const uint4*>(raw + (size_t)(t0 + tt) * in.ld_raw + in.z + (size_t)h * P + p0 + j) : zero;
        }
    };
    auto place = [&](float* to, const uint4& piece) {
        float x[VEC];
        ssd_unpack(piece, x);
#pragma unroll
        for (int w = 0; w < VEC; w += 4) *reinterpret_cast<float4*>(to + w) = make_float4(x[w], x[w + 1], x[w + 2], x[w + 3]);
    };
    auto settle = [&](int t0) {
        const int n = min(CH, hi - t0);
        if (wide) {
#pragma unroll
            for (int q = 0; q < L::N_PIECES; ++q) {
                const int e = tid + q * SSD_THREADS, tt = e / (NP / VEC), i = (e % (NP / VEC)) * VEC;
                if (tt < CH) {
                    place(s_b + tt * ROW + i, in_b[q]);
                    if (!STATE_ONLY) place(s_c + tt * ROW + i, in_c[q]);
                    if constexpr (sizeof(T) == 2 && !STATE_ONLY) {
                        *reinterpret_cast<uint4*>(t_b + tt * TROW + i) = in_b[q];
                        *reinterpret_cast<uint4*>(t_c + tt * TROW + i) = in_c[q];
                    }
                }
            }
#pragma unroll
            for (int q = 0; q < L::P_PIECES; ++q) {
                const int e = tid + q * SSD_THREADS, tt = e / (COLS / VEC), j = (e % (COLS / VEC)) * VEC;
                if (tt < CH) {
                    place(s_x + tt * COLS + j, in_x[q]);
                    if (!STATE_ONLY) place(s_z + tt * COLS + j, in_z[q]);
                }
            }
        } else {
            for (int e = tid; e < CH * NP; e += SSD_THREADS) {
                const int tt = e / NP, i = e - tt * NP;
                const bool here = tt < n && i < N;
                const T* at = conv + (size_t)(t0 + tt) * in.ld_conv + (size_t)g * N + i;
                const T b = here ? at[in.b] : from_float<T>(0.f), c = here ? at[in.c] : from_float<T>(0.f);
                s_b[tt * ROW + i] = to_float(b);
                s_c[tt * ROW + i] = to_float(c);
                if constexpr (sizeof(T) == 2) {
                    t_b[tt * TROW + i] = b;
                    t_c[tt * TROW + i] = c;
                }
            }
            for (int e = tid; e < CH * COLS; e += SSD_THREADS) {
                const int tt = e / COLS, j = p0 + e % COLS;
                const bool here = tt < n && j < P;
                s_x[e] = here ? to_float(conv[(size_t)(t0 + tt) * in.ld_conv + in.x + (size_t)h * P + j]) : 0.f;
                s_z[e] = here ? to_float(raw[(size_t)(t0 + tt) * in.ld_raw + in.z + (size_t)h * P + j]) : 0.f;
            }
        }
        if (warp == 0) {                                         // (tokens behind the last: no step, nothing decays)
            const float dt = lane < n ? softplus(in_dt + bias) : 0.f;
            float sum = rate * dt;
#pragma unroll
            for (int o = 1; o < CH; o <<= 1) {
                const float other = __shfl_up_sync(0xffffffffu, sum, o);
                if (lane >= o) sum += other;
            }
            const float end = __shfl_sync(0xffffffffu, sum, CH - 1);
            if (lane < CH) {
                s_dt[lane] = dt;
                s_log[lane] = sum;
                s_from[lane] = expf(sum);
                s_to[lane] = expf(end - sum) * dt;
            }
        }
    };
    fetch(lo);
    if (STATE_ONLY) {
        if (segment == 0) store_state(run_state + cut_base * block);         // the first run's start is the slot's state
#pragma unroll
        for (int r = 0; r < R / 2; ++r)
#pragma unroll
            for (int c = 0; c < CPL; ++c) s[r][c] = pair_of(0.f, 0.f);
    } else if (runs > 1) {
        load_state(pdl_fresh(run_state) + (cut_base + segment) * block);
    }
    float exponent = 0.f;                                        // STATE_ONLY: the sum of the run's logarithms of decays
    for (int t0 = lo; t0 < hi; t0 += CH) {
        const int n = min(CH, hi - t0);
        settle(t0);
        __syncthreads();
        if (t0 + CH < hi) fetch(t0 + CH);
        if constexpr (!STATE_ONLY) {
            // ---- the weights W[t][s] of the chunk's own tokens
            if constexpr (sizeof(T) == 2) {
                if (warp < 2) {
                    float acc[4] = {0.f, 0.f, 0.f, 0.f};
                    const uint32_t a_at = (uint32_t)__cvta_generic_to_shared(t_c + (lane & 15) * TROW + (lane >> 4) * 8);
                    const uint32_t b_at = (uint32_t)__cvta_generic_to_shared(t_b + (8 * warp + (lane & 7)) * TROW + ((lane >> 3) & 1) * 8);
#pragma unroll
                    for (int k = 0; k < NP / 16; ++k) {
                        uint32_t a[4], b[2];
                        asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
                                     : "=r"(a[0]), "=r"(a[1]), "=r"(a[2]), "=r"(a[3]) : "r"(a_at + 32 * k) : "memory");
                        asm volatile("ldmatrix.sync.aligned.m8n8.x2.shared.b16 {%0,%1}, [%2];"
                                     : "=r"(b[0]), "=r"(b[1]) : "r"(b_at + 32 * k) : "memory");
                        asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                                     : "+f"(acc[0]), "+f"(acc[1]), "+f"(acc[2]), "+f"(acc[3])
                                     : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b[0]), "r"(b[1]));
                    }
#pragma unroll
                    for (int i = 0; i < 4; ++i) {
                        const int t = (lane >> 2) + 8 * (i >> 1), u = 8 * warp + 2 * (lane & 3) + (i & 1);
                        s_w[t * (CH + 4) + u] = u <= t ? acc[i] * expf(s_log[t] - s_log[u]) * s_dt[u] : 0.f;
                    }
                }
            } else {
                const int t = tid >> 4, u = tid & 15;
                float dot = 0.f;
                if (u <= t) {
                    for (int i = 0; i < NP; i += 4) {
                        const float4 a = *reinterpret_cast<const float4*>(s_c + t * ROW + i);
                        const float4 b = *reinterpret_cast<const float4*>(s_b + u * ROW + i);
                        dot = fmaf(a.x, b.x, dot); dot = fmaf(a.y, b.y, dot);
                        dot = fmaf(a.z, b.z, dot); dot = fmaf(a.w, b.w, dot);
                    }
                    dot *= expf(s_log[t] - s_log[u]) * s_dt[u];
                }
                s_w[t * (CH + 4) + u] = dot;
            }
            // ---- what the state ahead of the chunk gives to its tokens
#pragma unroll
            for (int tt = 0; tt < CH; ++tt) {
                unsigned long long sum[CPL];
#pragma unroll
                for (int r = 0; r < R / 2; r += 2) {
                    const ulonglong2 cc = *reinterpret_cast<const ulonglong2*>(s_c + tt * ROW + n0 + 2 * r);
#pragma unroll
                    for (int c = 0; c < CPL; ++c) {
                        sum[c] = r == 0 ? pair_mul(cc.x, s[r][c]) : pair_fma(cc.x, s[r][c], sum[c]);
                        sum[c] = pair_fma(cc.y, s[r + 1][c], sum[c]);
                    }
                }
                float y[CPL];
#pragma unroll
                for (int c = 0; c < CPL; ++c) {
                    float even, odd;
                    pair_split(sum[c], even, odd);
                    y[c] = even + odd;
                }
                float* to = s_y + (warp * CH + tt) * COLS + CPL * lane;
                if constexpr (CPL == 2) *reinterpret_cast<float2*>(to) = make_float2(y[0], y[1]);
                else *to = y[0];
            }
        }
        // ---- the state behind the chunk
        {
            const float keep = s_from[CH - 1];
            const unsigned long long k2 = pair_of(keep, keep);
            if (STATE_ONLY) exponent += s_log[CH - 1];
#pragma unroll
            for (int r = 0; r < R / 2; ++r)
#pragma unroll
                for (int c = 0; c < CPL; ++c) s[r][c] = pair_mul(k2, s[r][c]);
#pragma unroll 4
            for (int tt = 0; tt < CH; ++tt) {
                const float weight = s_to[tt];
                unsigned long long x2[CPL];
                if constexpr (CPL == 2) {
                    const float2 x = *reinterpret_cast<const float2*>(s_x + tt * COLS + 2 * lane);
                    x2[0] = pair_of(x.x * weight, x.x * weight);
                    x2[1] = pair_of(x.y * weight, x.y * weight);
                } else {
                    const float x = s_x[tt * COLS + lane] * weight;
                    x2[0] = pair_of(x, x);
                }
#pragma unroll
                for (int r = 0; r < R / 2; r += 2) {
                    const ulonglong2 bb = *reinterpret_cast<const ulonglong2*>(s_b + tt * ROW + n0 + 2 * r);
#pragma unroll
                    for (int c = 0; c < CPL; ++c) {
                        s[r][c] = pair_fma(bb.x, x2[c], s[r][c]);
                        s[r + 1][c] = pair_fma(bb.y, x2[c], s[r + 1][c]);
                    }
                }
            }
        }
        __syncthreads();
        if constexpr (!STATE_ONLY) {
            // ---- the sums over the warps, the chunk's own tokens, the skip and the gate: CPL neighbouring columns at a time
            for (int e = tid; e < CH * 32; e += SSD_THREADS) {
                const int tt = e >> 5, col = (e & 31) * CPL;
                if (tt >= n || p0 + col >= P) continue;
                float total[CPL], own[CPL];
#pragma unroll
                for (int c = 0; c < CPL; ++c) total[c] = own[c] = 0.f;
                auto take = [&](const float* from, float weight, float (&to)[CPL]) {
                    if constexpr (CPL == 2) {
                        const float2 f = *reinterpret_cast<const float2*>(from);
                        to[0] = fmaf(weight, f.x, to[0]);
                        to[1] = fmaf(weight, f.y, to[1]);
                    } else {
                        to[0] = fmaf(weight, *from, to[0]);
                    }
                };
#pragma unroll
                for (int w = 0; w < SSD_WARPS; ++w) take(s_y + (w * CH + tt) * COLS + col, 1.f, total);
#pragma unroll
                for (int u = 0; u < CH; u += 4) {
                    const float4 w = *reinterpret_cast<const float4*>(s_w + tt * (CH + 4) + u);
                    take(s_x + u * COLS + col, w.x, own);
                    take(s_x + (u + 1) * COLS + col, w.y, own);
                    take(s_x + (u + 2) * COLS + col, w.z, own);
                    take(s_x + (u + 3) * COLS + col, w.w, own);
                }
                take(s_x + tt * COLS + col, skip, own);
                TO* to = out + (size_t)(t0 + tt) * out_stride + (size_t)h * P + p0 + col;
#pragma unroll
                for (int c = 0; c < CPL; ++c)
                    if (p0 + col + c < P) to[c] = from_float<TO>(fmaf(s_from[tt], total[c], own[c]) * silu(s_z[tt * COLS + col + c]));
            }
            __syncthreads();                                     // before the next chunk's rows arrive
        }
    }
    if (STATE_ONLY) {
        const size_t entry = cut_base + segment + 1;
        store_state(run_state + entry * block);
        if (tid == 0 && p0 == 0) run_decay[entry] = expf(exponent);
    } else if (segment == runs - 1) {
        store_state(S);
    }
}

// run_state[e] <- run_decay[e] * run_state[e - 1] + run_state[e] for e = 1 .. runs - 1, element by element.
constexpr int SSD_FOLD_THREADS = 128, SSD_FOLD_AHEAD = 8;

template <int V>
__global__ void __launch_bounds__(SSD_FOLD_THREADS)
ssd_fold_kernel(float* __restrict__ run_state, const float* __restrict__ run_decay, const int* __restrict__ q_start,
                int first_cut, int segments, int chunk_unit, int heads, int block) {
    const int unit = (blockIdx.x * SSD_FOLD_THREADS + threadIdx.x) * V, item = first_cut + blockIdx.z;
    const int count = q_start[item + 1] - q_start[item];
    pdl_prologue();
    if (count <= 0 || unit >= block) return;
    const int per = ssd_run_length(count, segments, chunk_unit), runs = (count + per - 1) / per;
    const size_t base = ((size_t)blockIdx.z * heads + blockIdx.y) * segments;
    float* at = pdl_fresh(run_state) + base * block + unit;
    const float* decay = pdl_fresh(run_decay) + base;
    float s[V];
#pragma unroll
    for (int v = 0; v < V; ++v) s[v] = at[v];
    for (int e0 = 1; e0 < runs; e0 += SSD_FOLD_AHEAD) {
        float add[SSD_FOLD_AHEAD][V], d[SSD_FOLD_AHEAD];
#pragma unroll
        for (int a = 0; a < SSD_FOLD_AHEAD; ++a) {
            if (e0 + a < runs) {
                if constexpr (V == 4) {
                    const float4 f = *reinterpret_cast<const float4*>(at + (size_t)(e0 + a) * block);
                    add[a][0] = f.x; add[a][1] = f.y; add[a][2] = f.z; add[a][3] = f.w;
                } else {
                    add[a][0] = at[(size_t)(e0 + a) * block];
                }
                d[a] = decay[e0 + a];
            }
        }
#pragma unroll
        for (int a = 0; a < SSD_FOLD_AHEAD; ++a) {
            if (e0 + a < runs) {
#pragma unroll
                for (int v = 0; v < V; ++v) s[v] = fmaf(d[a], s[v], add[a][v]);
                if constexpr (V == 4) *reinterpret_cast<float4*>(at + (size_t)(e0 + a) * block) = make_float4(s[0], s[1], s[2], s[3]);
                else at[(size_t)(e0 + a) * block] = s[0];
            }
        }
    }
}

// Entries [0, gridDim.x) of few tokens, token by token.  Thread (part, group) works on the columns [V group, V group + V) of the rows part, part + parts, ...;
// `lanes` (a power of two, at least P / V) threads share a row.
constexpr int SSD_STEP_ROWS = 8;                                 // rows of a thread that are on their way together

template <typename T, typename TO, int V>
__global__ void __launch_bounds__(SSD_THREADS, 4)
ssd_step_kernel(const T* __restrict__ conv, const T* __restrict__ raw, const SsdInputs in, float* __restrict__ state,
                long long state_stride, const int* __restrict__ q_start, const int* __restrict__ item_slot, int lanes,
                TO* __restrict__ out, long long out_stride) {
    extern __shared__ __align__(16) float ssd_smem[];             // B [N], C [N], then the sums [warps or parts][P]
    const int item = blockIdx.x, h = blockIdx.y, tid = threadIdx.x;
    const int begin = q_start[item], end = q_start[item + 1];
    if (end <= begin) return;
    const int N = in.N, P = in.P, g = h / (in.heads / in.groups);
    const int parts = SSD_THREADS / lanes, part = tid / lanes, col = (tid - part * lanes) * V;
    const bool mine = col < P;
    float* const s_b = ssd_smem;
    float* const s_c = s_b + N;
    float* const s_y = s_c + N;
    float* S = state + (size_t)item_slot[item] * state_stride + (size_t)h * N * P + col;
    float s[SSD_STEP_ROWS][V];
    // (S was last written by this kernel of an earlier step, and that one is done)
    auto fetch = [&](int first) {
#pragma unroll
        for (int r = 0; r < SSD_STEP_ROWS; ++r) {
            const int n = first + part + r * parts;
            if (mine && n < N) {
                if constexpr (V == 4) {
                    const float4 f = *reinterpret_cast<const float4*>(S + (size_t)n * P);
                    s[r][0] = f.x; s[r][1] = f.y; s[r][2] = f.z; s[r][3] = f.w;
                } else {
                    s[r][0] = S[(size_t)n * P];
                }
            }
        }
    };
    fetch(0);
    const float rate = -expf(in.a_log[h]), bias = in.dt_bias[h], skip = in.d[h];
    pdl_prologue();
    conv = pdl_fresh(conv) + (size_t)begin * in.ld_conv;
    raw = pdl_fresh(raw) + (size_t)begin * in.ld_raw;
    for (int t = begin; t < end; ++t, conv += in.ld_conv, raw += in.ld_raw) {
        if (t > begin) {                                             // (S: what this thread has just stored)
            __syncthreads();
            fetch(0);
        }
        for (int i = tid; i < N; i += SSD_THREADS) {
            s_b[i] = to_float(conv[in.b + g * N + i]);
            s_c[i] = to_float(conv[in.c + g * N + i]);
        }
        float x[V], y[V];
        const float dt = softplus(to_float(raw[in.dt + h]) + bias), keep = expf(rate * dt);
#pragma unroll
        for (int v = 0; v < V; ++v) {
            x[v] = mine && col + v < P ? to_float(conv[in.x + (size_t)h * P + col + v]) * dt : 0.f;
            y[v] = 0.f;
        }
        __syncthreads();
        for (int first = 0; first < N; first += SSD_STEP_ROWS * parts) {
            if (first) fetch(first);
#pragma unroll
            for (int r = 0; r < SSD_STEP_ROWS; ++r) {
                const int n = first + part + r * parts;
                if (mine && n < N) {
                    const float b = s_b[n], c = s_c[n];
#pragma unroll
                    for (int v = 0; v < V; ++v) {
                        s[r][v] = fmaf(b, x[v], keep * s[r][v]);
                        y[v] = fmaf(c, s[r][v], y[v]);
                    }
                    if constexpr (V == 4) *reinterpret_cast<float4*>(S + (size_t)n * P) = make_float4(s[r][0], s[r][1], s[r][2], s[r][3]);
                    else S[(size_t)n * P] = s[r][0];
                }
            }
        }
        // the sums over the parts: first inside a warp, then between its rows in shared memory
        for (int o = lanes; o < 32; o <<= 1)
#pragma unroll
            for (int v = 0; v < V; ++v) y[v] += __shfl_xor_sync(0xffffffffu, y[v], o);
        const int rows = lanes < 32 ? SSD_WARPS : parts, own = lanes < 32 ? tid >> 5 : part;
        if (mine && (lanes >= 32 || (tid & 31) < lanes)) {
#pragma unroll
            for (int v = 0; v < V; ++v)
                if (col + v < P) s_y[own * P + col + v] = y[v];
        }
        __syncthreads();
        for (int j = tid; j < P; j += SSD_THREADS) {
            float total = 0.f;
            for (int w = 0; w < rows; ++w) total += s_y[w * P + j];
            total = fmaf(skip, to_float(conv[in.x + (size_t)h * P + j]), total);
            out[(size_t)t * out_stride + (size_t)h * P + j] = from_float<TO>(total * silu(to_float(raw[in.z + (size_t)h * P + j])));
        }
    }
}

// ---- prompt portions on tensor cores
constexpr int SSD_PROMPT_CHUNK = 64, SSD_PIECES = 3;

__device__ __forceinline__ void ssd_ldm(uint32_t (&r)[4], uint32_t at) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(at) : "memory");
}
__device__ __forceinline__ void ssd_ldm_t(uint32_t (&r)[4], uint32_t at) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(at) : "memory");
}
__device__ __forceinline__ void ssd_mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// two float32 numbers as three pairs of bfloat16 numbers that add up to them
__device__ __forceinline__ void ssd_split(float x, float y, uint32_t (&piece)[SSD_PIECES]) {
#pragma unroll
    for (int i = 0; i < SSD_PIECES; ++i) {
        const __nv_bfloat162 rounded = __floats2bfloat162_rn(x, y);
        piece[i] = *reinterpret_cast<const uint32_t*>(&rounded);
        const float2 back = __bfloat1622float2(rounded);
        x -= back.x;
        y -= back.y;
    }
}

// NT: rows of S, PT: columns of S of a CTA (both padded with zeros)
template <int NT, int PT>
struct SsdPromptLayout {
    static constexpr int CH = SSD_PROMPT_CHUNK, TROW = NT + 8, PROW = PT + 8;           // padded rows, in elements
    static constexpr int B = 0, C = CH * TROW, X = 2 * CH * TROW, Z = X + CH * PROW, STAGE = Z + CH * PROW;
    static constexpr int WX = 2 * STAGE, S = WX + SSD_PIECES * CH * PROW, END = S + SSD_PIECES * NT * PROW;
    static constexpr size_t BYTES = (size_t)END * 2;
    // warps as tiles of 16 rows of S by groups of 8-column tiles (the update), and as tiles of 16 tokens by halves (the result)
    static constexpr int NTILES = NT / 16, P_SPLITS = SSD_WARPS / NTILES, UPDATE = PT / 8 / P_SPLITS, RESULT = PT / 8 / 2;
    static_assert(NTILES * P_SPLITS == SSD_WARPS && UPDATE >= 1 && RESULT >= 2, "layout");
};

template <typename TO, int NT, int PT, bool STATE_ONLY>
__global__ void __launch_bounds__(SSD_THREADS, 1)
ssd_prompt_kernel(const __nv_bfloat16* __restrict__ conv, const __nv_bfloat16* __restrict__ raw, const SsdInputs in,
                  float* __restrict__ state, long long state_stride, const int* __restrict__ q_start,
                  const int* __restrict__ item_slot, int first_item, int segments, float* __restrict__ run_state,
                  float* __restrict__ run_decay, TO* __restrict__ out, long long out_stride) {
    using L = SsdPromptLayout<NT, PT>;
    constexpr int CH = L::CH, TROW = L::TROW, PROW = L::PROW;
    extern __shared__ __align__(16) __nv_bfloat16 ssd_tiles[];
    __shared__ float s_dt[CH], s_log[CH], s_from[CH], s_to[CH];
    const int item = first_item + blockIdx.x, h = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int col_tiles = (in.P + PT - 1) / PT, p0 = (blockIdx.z % col_tiles) * PT, segment = blockIdx.z / col_tiles;
    const int begin = q_start[item], count = q_start[item + 1] - begin;
    const int per = ssd_run_length(count, segments, CH), runs = count > 0 ? (count + per - 1) / per : 1;
    if (count <= 0 || segment >= (STATE_ONLY ? runs - 1 : runs)) return;
    const int lo = begin + segment * per, hi = min(lo + per, begin + count);
    const int N = in.N, P = in.P, g = h / (in.heads / in.groups);
    const float rate = -expf(in.a_log[h]), bias = in.dt_bias[h], skip = in.d[h];
    const size_t block = (size_t)N * P;
    float* S = state + (size_t)item_slot[item] * state_stride + (size_t)h * block;
    const size_t cut_base = ((size_t)blockIdx.x * in.heads + h) * segments;

    // ---- S as accumulators: rows n_row and n_row + 8, columns p0 + 8 (u_first + j) + 2 (lane & 3) and the next
    const int n_tile = warp % L::NTILES, u_first = warp / L::NTILES * L::UPDATE;
    const int n_row = 16 * n_tile + (lane >> 2), s_col = 8 * u_first + 2 * (lane & 3);
    float s[L::UPDATE][4];
    auto each_pair = [&](auto&& visit) {
#pragma unroll
        for (int j = 0; j < L::UPDATE; ++j)
#pragma unroll
            for (int half = 0; half < 2; ++half) {
                const int n = n_row + 8 * half, p = p0 + s_col + 8 * j;
                visit(j, 2 * half, n < N && p < P, (size_t)n * P + p);
            }
    };
    auto load_state = [&](const float* from) {
        each_pair([&](int j, int i, bool here, size_t at) {
            const float2 v = here ? *reinterpret_cast<const float2*>(from + at) : make_float2(0.f, 0.f);
            s[j][i] = v.x;
            s[j][i + 1] = v.y;
        });
    };
    auto store_state = [&](float* to) {
        each_pair([&](int j, int i, bool here, size_t at) {
            if (here) *reinterpret_cast<float2*>(to + at) = make_float2(s[j][i], s[j][i + 1]);
        });
    };
    // S of the slot: only these kernels of an earlier step wrote it, and they are done
    if (STATE_ONLY ? segment == 0 : runs == 1) load_state(S);
    pdl_prologue();
    conv = pdl_fresh(conv);
    raw = pdl_fresh(raw);

    const uint32_t tiles = (uint32_t)__cvta_generic_to_shared(ssd_tiles);
    auto copy = [&](int to, const __nv_bfloat16* from, bool here) {
        const int bytes = here ? 16 : 0;                                       // 0: sixteen bytes of zeros
        asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(tiles + 2 * to), "l"(here ? from : conv), "r"(bytes) : "memory");
    };
    float dt_next[2] = {0.f, 0.f};                                             // warp 0: the tokens 2 lane and 2 lane + 1
    auto fetch = [&](int t0, int stage) {
        const int n = min(CH, hi - t0), base = stage * L::STAGE;
        for (int e = tid; e < CH * (NT / 8); e += SSD_THREADS) {
            const int tt = e / (NT / 8), i = (e % (NT / 8)) * 8;
            const bool here = tt < n && i < N;
            const __nv_bfloat16* at = conv + (size_t)(t0 + tt) * in.ld_conv + (size_t)g * N + i;
            copy(base + L::B + tt * TROW + i, at + in.b, here);
            if (!STATE_ONLY) copy(base + L::C + tt * TROW + i, at + in.c, here);
        }
        for (int e = tid; e < CH * (PT / 8); e += SSD_THREADS) {
            const int tt = e / (PT / 8), j = (e % (PT / 8)) * 8;
            const bool here = tt < n && p0 + j < P;
            copy(base + L::X + tt * PROW + j, conv + (size_t)(t0 + tt) * in.ld_conv + in.x + (size_t)h * P + p0 + j, here);
            if (!STATE_ONLY) copy(base + L::Z + tt * PROW + j, raw + (size_t)(t0 + tt) * in.ld_raw + in.z + (size_t)h * P + p0 + j, here);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
        if (warp == 0) {
#pragma unroll
            for (int i = 0; i < 2; ++i)
                if (2 * lane + i < n) dt_next[i] = to_float(raw[(size_t)(t0 + 2 * lane + i) * in.ld_raw + in.dt + h]);
        }
    };
    fetch(lo, 0);
    if (STATE_ONLY) {
        if (segment == 0) store_state(run_state + cut_base * block);           // the first run's start is the slot's state
#pragma unroll
        for (int j = 0; j < L::UPDATE; ++j) s[j][0] = s[j][1] = s[j][2] = s[j][3] = 0.f;
    } else if (runs > 1) {
        load_state(pdl_fresh(run_state) + (cut_base + segment) * block);
    }
    // lane addresses (bytes) of the fragments: rows of a tile as they lie, and transposed
    const uint32_t straight_row = (lane & 15), straight_col = (lane >> 4) * 8;            // A: [row][k]
    const uint32_t pair_row = (lane & 7) + ((lane >> 4) & 1) * 8, pair_col = ((lane >> 3) & 1) * 8;    // B from [n][k]; A from [k][row]
    const uint32_t trans_row = (lane & 7) + ((lane >> 3) & 1) * 8, trans_col = ((lane >> 4) & 1) * 8;  // B from [k][n]
    float exponent = 0.f;                                                      // STATE_ONLY: the sum of the run's logarithms of decays
    int stage = 0;
    for (int t0 = lo; t0 < hi; t0 += CH, stage ^= 1) {
        const int n = min(CH, hi - t0);
        const uint32_t here = tiles + 2 * stage * L::STAGE;
        const __nv_bfloat16* x_tile = ssd_tiles + stage * L::STAGE + L::X;
        // ---- step sizes and decays; the state's pieces
        if (warp == 0) {
            float dt[2], v[2];
#pragma unroll
            for (int i = 0; i < 2; ++i) {
                dt[i] = 2 * lane + i < n ? softplus(dt_next[i] + bias) : 0.f;
                v[i] = rate * dt[i];
            }
            float sum = v[0] + v[1];
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const float other = __shfl_up_sync(0xffffffffu, sum, o);
                if (lane >= o) sum += other;
            }
            const float end = __shfl_sync(0xffffffffu, sum, 31), mid = sum - v[1];
            s_dt[2 * lane] = dt[0];             s_dt[2 * lane + 1] = dt[1];
            s_log[2 * lane] = mid;              s_log[2 * lane + 1] = sum;
            s_from[2 * lane] = expf(mid);       s_from[2 * lane + 1] = expf(sum);
            s_to[2 * lane] = expf(end - mid) * dt[0];
            s_to[2 * lane + 1] = expf(end - sum) * dt[1];
        }
        if (!STATE_ONLY) {
#pragma unroll
            for (int j = 0; j < L::UPDATE; ++j)
#pragma unroll
                for (int half = 0; half < 2; ++half) {
                    uint32_t piece[SSD_PIECES];
                    ssd_split(s[j][2 * half], s[j][2 * half + 1], piece);
#pragma unroll
                    for (int q = 0; q < SSD_PIECES; ++q)
                        *reinterpret_cast<uint32_t*>(ssd_tiles + L::S + (q * NT + n_row + 8 * half) * PROW + s_col + 8 * j) = piece[q];
                }
        }
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();
        if (t0 + CH < hi) fetch(t0 + CH, stage ^ 1);
        // ---- the pieces of the weighted x
        for (int e = tid; e < CH * (PT / 2); e += SSD_THREADS) {
            const int tt = e / (PT / 2), j = (e % (PT / 2)) * 2;
            const float2 x = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(x_tile + tt * PROW + j));
            const float weight = s_to[tt];
            uint32_t piece[SSD_PIECES];
            ssd_split(x.x * weight, x.y * weight, piece);
#pragma unroll
            for (int q = 0; q < SSD_PIECES; ++q)
                *reinterpret_cast<uint32_t*>(ssd_tiles + L::WX + (q * CH + tt) * PROW + j) = piece[q];
        }
        if constexpr (!STATE_ONLY) {
            const int m_tile = warp & 3, r_first = (warp >> 2) * L::RESULT;    // 16 tokens, half of the columns
            const int row = 16 * m_tile + (lane >> 2);
            float y[L::RESULT][4];
#pragma unroll
            for (int j = 0; j < L::RESULT; ++j) y[j][0] = y[j][1] = y[j][2] = y[j][3] = 0.f;
            uint32_t c_frag[NT / 16][4];
#pragma unroll
            for (int k = 0; k < NT / 16; ++k)
                ssd_ldm(c_frag[k], here + 2 * (L::C + (16 * m_tile + straight_row) * TROW + 16 * k + straight_col));
            // what the state ahead of the chunk gives
#pragma unroll
            for (int k = 0; k < NT / 16; ++k)
#pragma unroll
                for (int q = 0; q < SSD_PIECES; ++q)
#pragma unroll
                    for (int j = 0; j < L::RESULT; j += 2) {
                        uint32_t b[4];
                        ssd_ldm_t(b, tiles + 2 * (L::S + (q * NT + 16 * k + trans_row) * PROW + 8 * (r_first + j) + trans_col));
                        ssd_mma(y[j], c_frag[k], b[0], b[1]);
                        ssd_mma(y[j + 1], c_frag[k], b[2], b[3]);
                    }
            const float from[2] = {s_from[row], s_from[row + 8]};
#pragma unroll
            for (int j = 0; j < L::RESULT; ++j) {
                y[j][0] *= from[0]; y[j][1] *= from[0];
                y[j][2] *= from[1]; y[j][3] *= from[1];
            }
            // the chunk's own tokens, 16 at a time
            const float log_row[2] = {s_log[row], s_log[row + 8]};
#pragma unroll
            for (int kk = 0; kk < CH / 16; ++kk) {
                if (kk > m_tile) continue;
                float w[2][4];
#pragma unroll
                for (int j = 0; j < 2; ++j) w[j][0] = w[j][1] = w[j][2] = w[j][3] = 0.f;
#pragma unroll
                for (int k = 0; k < NT / 16; ++k) {
                    uint32_t b[4];
                    ssd_ldm(b, here + 2 * (L::B + (16 * kk + pair_row) * TROW + 16 * k + pair_col));
                    ssd_mma(w[0], c_frag[k], b[0], b[1]);
                    ssd_mma(w[1], c_frag[k], b[2], b[3]);
                }
                uint32_t a[SSD_PIECES][4];
#pragma unroll
                for (int j = 0; j < 2; ++j) {
                    const int u = 16 * kk + 8 * j + 2 * (lane & 3);
                    const float2 log_u = *reinterpret_cast<const float2*>(s_log + u), dt_u = *reinterpret_cast<const float2*>(s_dt + u);
#pragma unroll
                    for (int half = 0; half < 2; ++half) {
                        const int t = row + 8 * half;
                        const float v0 = u <= t ? w[j][2 * half] * expf(log_row[half] - log_u.x) * dt_u.x : 0.f;
                        const float v1 = u + 1 <= t ? w[j][2 * half + 1] * expf(log_row[half] - log_u.y) * dt_u.y : 0.f;
                        uint32_t piece[SSD_PIECES];
                        ssd_split(v0, v1, piece);
#pragma unroll
                        for (int q = 0; q < SSD_PIECES; ++q) a[q][2 * j + half] = piece[q];
                    }
                }
#pragma unroll
                for (int j = 0; j < L::RESULT; j += 2) {
                    uint32_t b[4];
                    ssd_ldm_t(b, here + 2 * (L::X + (16 * kk + trans_row) * PROW + 8 * (r_first + j) + trans_col));
#pragma unroll
                    for (int q = 0; q < SSD_PIECES; ++q) {
                        ssd_mma(y[j], a[q], b[0], b[1]);
                        ssd_mma(y[j + 1], a[q], b[2], b[3]);
                    }
                }
            }
            // skip, gate, out
            const __nv_bfloat16* z_tile = ssd_tiles + stage * L::STAGE + L::Z;
#pragma unroll
            for (int half = 0; half < 2; ++half) {
                const int tt = row + 8 * half;
                if (tt >= n) continue;
                TO* to = out + (size_t)(t0 + tt) * out_stride + (size_t)h * P + p0;
#pragma unroll
                for (int j = 0; j < L::RESULT; ++j) {
                    const int col = 8 * (r_first + j) + 2 * (lane & 3);
                    if (p0 + col >= P) continue;
                    const float2 x = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(x_tile + tt * PROW + col));
                    const float2 z = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(z_tile + tt * PROW + col));
                    const float v0 = fmaf(skip, x.x, y[j][2 * half]) * silu_fast(z.x), v1 = fmaf(skip, x.y, y[j][2 * half + 1]) * silu_fast(z.y);
                    if constexpr (sizeof(TO) == 4) *reinterpret_cast<float2*>(to + col) = make_float2(v0, v1);
                    else *reinterpret_cast<__nv_bfloat162*>(to + col) = __floats2bfloat162_rn(v0, v1);
                }
            }
        }
        // (the decays are read ahead of the barrier: behind it the first warp may already form the next chunk's)
        const float keep = s_from[CH - 1];
        if (STATE_ONLY) exponent += s_log[CH - 1];
        __syncthreads();
        // ---- the state behind the chunk
#pragma unroll
        for (int j = 0; j < L::UPDATE; ++j) {
            s[j][0] *= keep; s[j][1] *= keep; s[j][2] *= keep; s[j][3] *= keep;
        }
#pragma unroll
        for (int k = 0; k < CH / 16; ++k) {
            uint32_t a[4];
            ssd_ldm_t(a, here + 2 * (L::B + (16 * k + pair_row) * TROW + 16 * n_tile + pair_col));
#pragma unroll
            for (int q = 0; q < SSD_PIECES; ++q) {
                if constexpr (L::UPDATE == 1) {
                    uint32_t b[4];                                             // (the neighbouring tile's fragments are not used)
                    ssd_ldm_t(b, tiles + 2 * (L::WX + (q * CH + 16 * k + trans_row) * PROW + 8 * (u_first & ~1) + trans_col));
                    if (u_first & 1) ssd_mma(s[0], a, b[2], b[3]);
                    else ssd_mma(s[0], a, b[0], b[1]);
                } else {
#pragma unroll
                    for (int j = 0; j < L::UPDATE; j += 2) {
                        uint32_t b[4];
                        ssd_ldm_t(b, tiles + 2 * (L::WX + (q * CH + 16 * k + trans_row) * PROW + 8 * (u_first + j) + trans_col));
                        ssd_mma(s[j], a, b[0], b[1]);
                        ssd_mma(s[j + 1], a, b[2], b[3]);
                    }
                }
            }
        }
    }
    if (STATE_ONLY) {
        const size_t entry = cut_base + segment + 1;
        store_state(run_state + entry * block);
        if (tid == 0 && p0 == 0) run_decay[entry] = expf(exponent);
    } else if (segment == runs - 1) {
        store_state(S);
    }
}

template <typename T, typename TO, int R, int CPL, bool STATE_ONLY>
int launch_ssd_scan_rows(const T* conv, const T* raw, const SsdInputs& in, float* state, long long state_stride,
                         const int* q_start, const int* item_slot, int first_item, int last_item, int first_cut, int segments,
                         int depth, float* run_state, float* run_decay, TO* out, long long out_stride, cudaStream_t s) {
    using L = SsdLayout<T, R, CPL>;
    auto kernel = ssd_scan_kernel<T, TO, R, CPL, STATE_ONLY>;
    const int tiles = (in.P + L::COLS - 1) / L::COLS;
    static size_t raised[MAX_DEVICES] = {0};
    if (!ensure_dynamic_smem((const void*)kernel, L::BYTES, raised)) return PS_ERR_LAUNCH;
    if ((long long)tiles * depth > 65535) return PS_ERR_UNSUPPORTED;
    constexpr int V = L::VEC;
    const int wide = in.N % V == 0 && in.P % V == 0 && in.ld_conv % V == 0 && in.ld_raw % V == 0 && in.x % V == 0 && in.b % V == 0 &&
                     in.c % V == 0 && in.z % V == 0 && !(((uintptr_t)conv | (uintptr_t)raw) & 15);
    return launch_pdl(kernel, dim3(last_item - first_item, in.heads, tiles * depth), dim3(SSD_THREADS), L::BYTES, s, conv, raw, in,
                      wide, state, state_stride, q_start, item_slot, first_item, last_item, first_cut, segments, run_state,
                      run_decay, out, out_stride);
}

template <typename T, typename TO, bool STATE_ONLY>
int launch_ssd_scan(const T* conv, const T* raw, const SsdInputs& in, float* state, long long state_stride, const int* q_start,
                    const int* item_slot, int first_item, int last_item, int first_cut, int segments, int depth,
                    float* run_state, float* run_decay, TO* out, long long out_stride, cudaStream_t s) {
#define PS_SSD_ROWS(R, CPL)                                                                                             \
    return launch_ssd_scan_rows<T, TO, R, CPL, STATE_ONLY>(conv, raw, in, state, state_stride, q_start, item_slot, first_item, \
                                                           last_item, first_cut, segments, depth, run_state, run_decay, out, \
                                                           out_stride, s)
    const bool two = in.P > 32;                                  // columns of a lane
    if (in.N <= 32) {
        if (two) PS_SSD_ROWS(4, 2);
        PS_SSD_ROWS(4, 1);
    }
    if (in.N <= 64) {
        if (two) PS_SSD_ROWS(8, 2);
        PS_SSD_ROWS(8, 1);
    }
    if (in.N <= 128) {
        if (two) PS_SSD_ROWS(16, 2);
        PS_SSD_ROWS(16, 1);
    }
    if (in.N <= 256) PS_SSD_ROWS(32, 1);
    PS_SSD_ROWS(64, 1);
#undef PS_SSD_ROWS
}

template <typename TO, int NT, int PT, bool STATE_ONLY>
int launch_ssd_prompt(const __nv_bfloat16* conv, const __nv_bfloat16* raw, const SsdInputs& in, float* state,
                      long long state_stride, const int* q_start, const int* item_slot, int n_items, int first_item,
                      int segments, int depth, float* run_state, float* run_decay, TO* out, long long out_stride, cudaStream_t s) {
    using L = SsdPromptLayout<NT, PT>;
    auto kernel = ssd_prompt_kernel<TO, NT, PT, STATE_ONLY>;
    static size_t raised[MAX_DEVICES] = {0};
    if (!ensure_dynamic_smem((const void*)kernel, L::BYTES, raised)) return PS_ERR_LAUNCH;
    const int tiles = (in.P + PT - 1) / PT;
    if ((long long)tiles * depth > 65535) return PS_ERR_UNSUPPORTED;
    return launch_pdl(kernel, dim3(n_items - first_item, in.heads, tiles * depth), dim3(SSD_THREADS), L::BYTES, s, conv, raw, in,
                      state, state_stride, q_start, item_slot, first_item, segments, run_state, run_decay, out, out_stride);
}

template <typename TO, bool STATE_ONLY>
int pick_ssd_prompt(const __nv_bfloat16* conv, const __nv_bfloat16* raw, const SsdInputs& in, float* state,
                    long long state_stride, const int* q_start, const int* item_slot, int n_items, int first_item,
                    int segments, int depth, float* run_state, float* run_decay, TO* out, long long out_stride, cudaStream_t s) {
#define PS_SSD_PROMPT(NT, PT)                                                                                           \
    return launch_ssd_prompt<TO, NT, PT, STATE_ONLY>(conv, raw, in, state, state_stride, q_start, item_slot, n_items, first_item, \
                                                     segments, depth, run_state, run_decay, out, out_stride, s)
    if (in.P <= 32) {
        if (in.N <= 32) PS_SSD_PROMPT(32, 32);
        if (in.N <= 64) PS_SSD_PROMPT(64, 32);
        PS_SSD_PROMPT(128, 32);
    }
    if (in.N <= 32) PS_SSD_PROMPT(32, 64);
    if (in.N <= 64) PS_SSD_PROMPT(64, 64);
    PS_SSD_PROMPT(128, 64);
#undef PS_SSD_PROMPT
}

template <typename T, typename TO>
int pick_ssd(const T* conv, const T* raw, const SsdInputs& in, float* state, long long state_stride, const int* q_start,
             const int* item_slot, int n_items, int first_cut, int segments, float* run_state, float* run_decay, TO* out,
             long long out_stride, cudaStream_t s) {
    int status = PS_OK, first = 0;                                // entries [0, first) are done
    const bool by4 = in.P % 4 == 0 && state_stride % 4 == 0 && !((uintptr_t)state & 15);
    const int V = by4 ? 4 : 1;
    int lanes = 1;
    while (lanes < SSD_THREADS && lanes * V < in.P) lanes <<= 1;
    if (first_cut > 0 && lanes * V >= in.P) {
        const int parts = SSD_THREADS / lanes, rows = lanes < 32 ? SSD_WARPS : parts;
        const size_t smem = (size_t)(2 * in.N + rows * in.P) * sizeof(float);
        auto kernel = by4 ? ssd_step_kernel<T, TO, 4> : ssd_step_kernel<T, TO, 1>;
        if (smem > 48 * 1024) return PS_ERR_UNSUPPORTED;
        status = launch_pdl(kernel, dim3(first_cut, in.heads), dim3(SSD_THREADS), smem, s, conv, raw, in, state, state_stride,
                            q_start, item_slot, lanes, out, out_stride);
        if (status != PS_OK) return status;
        first = first_cut;
    }
    if (first == n_items) return PS_OK;
    const bool prompt = sizeof(T) == 2 && first == first_cut && in.N <= 128 && in.N % 8 == 0 && in.P % 8 == 0 && in.ld_conv % 8 == 0 &&
                        in.ld_raw % 8 == 0 && in.x % 8 == 0 && in.b % 8 == 0 && in.c % 8 == 0 && in.z % 8 == 0 &&
                        !(((uintptr_t)conv | (uintptr_t)raw) & 15) && out_stride % 2 == 0 && !((uintptr_t)out & 7) &&
                        state_stride % 2 == 0 && !((uintptr_t)state & 7) && !((uintptr_t)run_state & 7);
    if (segments > 1) {
        if constexpr (sizeof(T) == 2) {
            if (prompt)
                status = pick_ssd_prompt<TO, true>(conv, raw, in, state, state_stride, q_start, item_slot, n_items, first_cut,
                                                   segments, segments - 1, run_state, run_decay, out, out_stride, s);
        }
        if (!prompt)
            status = launch_ssd_scan<T, TO, true>(conv, raw, in, state, state_stride, q_start, item_slot, first_cut, n_items,
                                                  first_cut, segments, segments - 1, run_state, run_decay, out, out_stride, s);
        if (status != PS_OK) return status;
        const int block = in.N * in.P;
        const bool quads = block % 4 == 0 && !((uintptr_t)run_state & 15);
        const int units = quads ? block / 4 : block;
        status = launch_pdl(quads ? ssd_fold_kernel<4> : ssd_fold_kernel<1>,
                            dim3((units + SSD_FOLD_THREADS - 1) / SSD_FOLD_THREADS, in.heads, n_items - first_cut),
                            dim3(SSD_FOLD_THREADS), 0, s, run_state, (const float*)run_decay, q_start, first_cut, segments,
                            (int)(prompt ? SSD_PROMPT_CHUNK : SSD_CHUNK), in.heads, block);
        if (status != PS_OK) return status;
    }
    if constexpr (sizeof(T) == 2) {
        if (prompt)
            return pick_ssd_prompt<TO, false>(conv, raw, in, state, state_stride, q_start, item_slot, n_items, first_cut, segments,
                                              segments, run_state, run_decay, out, out_stride, s);
    }
    return launch_ssd_scan<T, TO, false>(conv, raw, in, state, state_stride, q_start, item_slot, first, n_items, first_cut, segments,
                                         segments, run_state, run_decay, out, out_stride, s);
}

}  // namespace ps

// conv, raw: rows of `dtype`, ld_conv / ld_raw elements apart; offsets: where x, B, C (in conv), z and dt (in raw) begin.
// state: float32 [slots] rows of state_stride, of which the first heads * N * P numbers are S.  Entries [0, first_cut) bring
// few tokens and run token by token; entries [first_cut, n_items) are cut into up to `segments` runs: run_state float32
// [(n_items - first_cut) * heads * segments][N * P] and run_decay [...] are scratch (null when segments is 1).  out: rows of
// heads * P numbers of out_dtype (`dtype` or float32), out_stride apart.
PS_EXPORT int ps_ssd(const void* conv, long long ld_conv, const void* raw, long long ld_raw, const int* offsets,
                     const float* a_log, const float* dt_bias, const float* d, float* state, long long state_stride,
                     const int* q_start, const int* item_slot, int n_items, int T, int first_cut, int segments,
                     float* run_state, float* run_decay, void* out, long long out_stride, int heads, int groups, int N, int P,
                     int dtype, int out_dtype, void* stream) {
    if (n_items <= 0 || T <= 0) return PS_OK;
    if (!conv || !raw || !offsets || !a_log || !dt_bias || !d || !state || !q_start || !item_slot || !out)
        return PS_ERR_BAD_ARGUMENT;
    if (heads <= 0 || heads > 65535 || groups <= 0 || heads % groups || N <= 0 || P <= 0 || first_cut < 0 || first_cut > n_items)
        return PS_ERR_BAD_ARGUMENT;
    if (N > 512 || P > 1024) return PS_ERR_UNSUPPORTED;
    if (segments < 1 || (segments > 1 && (!run_state || !run_decay))) return PS_ERR_BAD_ARGUMENT;
    if (first_cut == n_items) segments = 1;
    const ps::SsdInputs in{ld_conv, ld_raw, offsets[0], offsets[1], offsets[2], offsets[3], offsets[4], a_log, dt_bias, d,
                           heads, groups, N, P};
    cudaStream_t s = (cudaStream_t)stream;
    using bf = __nv_bfloat16;
    if (dtype == PS_F32 && out_dtype == PS_F32)
        return ps::pick_ssd<float, float>((const float*)conv, (const float*)raw, in, state, state_stride, q_start,
                                          item_slot, n_items, first_cut, segments, run_state, run_decay, (float*)out, out_stride, s);
    if (dtype == PS_BF16 && out_dtype == PS_F32)
        return ps::pick_ssd<bf, float>((const bf*)conv, (const bf*)raw, in, state, state_stride, q_start, item_slot,
                                       n_items, first_cut, segments, run_state, run_decay, (float*)out, out_stride, s);
    if (dtype == PS_BF16 && out_dtype == PS_BF16)
        return ps::pick_ssd<bf, bf>((const bf*)conv, (const bf*)raw, in, state, state_stride, q_start, item_slot, n_items,
                                    first_cut, segments, run_state, run_decay, (bf*)out, out_stride, s);
    return PS_ERR_UNSUPPORTED;
}
