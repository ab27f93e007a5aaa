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
// ssd_step_kernel: steps in which every entry brings one token (decode).  One CTA per (entry, head); S goes through registers,
//                  four columns an access, the first rows on their way before the wait for the kernel that makes the token's row.
// ssd_scan_kernel: everything else, on CUDA cores, any size.  One CTA per (entry, head, 32 columns, run of tokens): a lane is a
//                  column, a warp holds N / 8 rows of S in registers, two rows to a packed pair; tokens come in chunks of
//                  SSD_CHUNK through shared memory, the sums over the warps are formed for a whole chunk at once.
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

constexpr int SSD_THREADS = 256, SSD_WARPS = 8, SSD_CHUNK = 16, SSD_COLS = 32;

// how an entry of `count` tokens is cut into runs of whole chunks
__host__ __device__ __forceinline__ int ssd_run_length(int count, int segments, int chunk) {
    return ((count + segments - 1) / segments + chunk - 1) / chunk * chunk;
}

// R: rows of S of a warp (N <= 8 R)
template <typename T, typename TO, int R, bool STATE_ONLY>
__global__ void __launch_bounds__(SSD_THREADS)
ssd_scan_kernel(const T* __restrict__ conv, const T* __restrict__ raw, const SsdInputs in, float* __restrict__ state,
                long long state_stride, const int* __restrict__ q_start, const int* __restrict__ item_slot, int first_item,
                int last_item, int first_cut, int segments, int chunk_unit, float* __restrict__ run_state,
                float* __restrict__ run_decay, TO* __restrict__ out, long long out_stride) {
    constexpr int NP = SSD_WARPS * R, CH = SSD_CHUNK;
    extern __shared__ __align__(16) float ssd_smem[];
    float* const s_b = ssd_smem;                                 // [CH][NP]
    float* const s_c = s_b + CH * NP;                            // [CH][NP]
    float* const s_x = s_c + CH * NP;                            // [CH][32]
    float* const s_y = s_x + CH * SSD_COLS;                      // [WARPS][CH][32]
    __shared__ float s_dt[CH], s_keep[CH];
    const int item = first_item + blockIdx.x, h = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int col_tiles = (in.P + SSD_COLS - 1) / SSD_COLS;
    const int p0 = (blockIdx.z % col_tiles) * SSD_COLS, segment = blockIdx.z / col_tiles, p = p0 + lane;
    if (item >= last_item) return;
    const int begin = q_start[item], count = q_start[item + 1] - begin;
    const bool cut = segments > 1 && item >= first_cut;
    const int per = cut ? ssd_run_length(count, segments, chunk_unit) : count;
    const int runs = cut && count > 0 ? (count + per - 1) / per : 1;
    if (count <= 0 || segment >= (STATE_ONLY ? runs - 1 : runs)) return;
    const int lo = begin + segment * per, hi = min(lo + per, begin + count);
    const int N = in.N, P = in.P, n0 = warp * R, g = h / (in.heads / in.groups);
    const float rate = -expf(in.a_log[h]), bias = in.dt_bias[h], skip = in.d[h];
    const size_t block = (size_t)N * P;
    float* S = state + (size_t)item_slot[item] * state_stride + (size_t)h * block;
    const size_t cut_base = cut ? ((size_t)(item - first_cut) * in.heads + h) * segments : 0;
    pdl_prologue();
    conv = pdl_fresh(conv);
    raw = pdl_fresh(raw);

    unsigned long long s[R / 2];
    auto load_state = [&](const float* from) {
#pragma unroll
        for (int r = 0; r < R / 2; ++r) {
            const int n = n0 + 2 * r;
            const float a = (p < P && n < N) ? from[(size_t)n * P + p] : 0.f;
            const float b = (p < P && n + 1 < N) ? from[(size_t)(n + 1) * P + p] : 0.f;
            s[r] = pair_of(a, b);
        }
    };
    auto store_state = [&](float* to) {
#pragma unroll
        for (int r = 0; r < R / 2; ++r) {
            const int n = n0 + 2 * r;
            float a, b;
            pair_split(s[r], a, b);
            if (p < P && n < N) to[(size_t)n * P + p] = a;
            if (p < P && n + 1 < N) to[(size_t)(n + 1) * P + p] = b;
        }
    };
    if (STATE_ONLY) {
        if (segment == 0) {                                      // the first run's start is the slot's state
            load_state(S);
            store_state(run_state + cut_base * block);
        }
#pragma unroll
        for (int r = 0; r < R / 2; ++r) s[r] = pair_of(0.f, 0.f);
    } else if (runs > 1) {
        load_state(pdl_fresh(run_state) + (cut_base + segment) * block);
    } else {
        load_state(S);
    }
    float exponent = 0.f;                                        // STATE_ONLY: the sum of the run's logarithms of decays
    for (int t0 = lo; t0 < hi; t0 += CH) {
        const int n = min(CH, hi - t0);
        __syncthreads();                                         // the chunk before is done with shared memory
        for (int e = tid; e < CH * NP; e += SSD_THREADS) {
            const int tt = e / NP, i = e - tt * NP;
            const bool here = tt < n && i < N;
            const T* at = conv + (size_t)(t0 + tt) * in.ld_conv + (size_t)g * N + i;
            s_b[e] = here ? to_float(at[in.b]) : 0.f;
            if (!STATE_ONLY) s_c[e] = here ? to_float(at[in.c]) : 0.f;
        }
        for (int e = tid; e < CH * SSD_COLS; e += SSD_THREADS) {
            const int tt = e / SSD_COLS, j = p0 + (e & (SSD_COLS - 1));
            s_x[e] = tt < n && j < P ? to_float(conv[(size_t)(t0 + tt) * in.ld_conv + in.x + (size_t)h * P + j]) : 0.f;
        }
        if (tid < CH) {
            const float dt = tid < n ? softplus(to_float(raw[(size_t)(t0 + tid) * in.ld_raw + in.dt + h]) + bias) : 0.f;
            s_dt[tid] = dt;
            s_keep[tid] = expf(rate * dt);                       // (1 behind the last token)
        }
        __syncthreads();
        float y[CH];
        auto token = [&](int tt) {
            const float xd = s_x[tt * SSD_COLS + lane] * s_dt[tt], keep = s_keep[tt];
            const unsigned long long x2 = pair_of(xd, xd), k2 = pair_of(keep, keep);
            unsigned long long sum = pair_of(0.f, 0.f);
#pragma unroll
            for (int r = 0; r < R / 2; r += 2) {
                const ulonglong2 bb = *reinterpret_cast<const ulonglong2*>(s_b + tt * NP + n0 + 2 * r);
                s[r] = pair_fma(bb.x, x2, pair_mul(k2, s[r]));
                s[r + 1] = pair_fma(bb.y, x2, pair_mul(k2, s[r + 1]));
                if (!STATE_ONLY) {
                    const ulonglong2 cc = *reinterpret_cast<const ulonglong2*>(s_c + tt * NP + n0 + 2 * r);
                    sum = pair_fma(cc.x, s[r], sum);
                    sum = pair_fma(cc.y, s[r + 1], sum);
                }
            }
            float even, odd;
            pair_split(sum, even, odd);
            y[tt] = even + odd;
        };
        if (STATE_ONLY) {
#pragma unroll 1
            for (int tt = 0; tt < n; ++tt) {
                const float xd = s_x[tt * SSD_COLS + lane] * s_dt[tt], keep = s_keep[tt];
                exponent = fmaf(rate, s_dt[tt], exponent);
                const unsigned long long x2 = pair_of(xd, xd), k2 = pair_of(keep, keep);
#pragma unroll
                for (int r = 0; r < R / 2; r += 2) {
                    const ulonglong2 bb = *reinterpret_cast<const ulonglong2*>(s_b + tt * NP + n0 + 2 * r);
                    s[r] = pair_fma(bb.x, x2, pair_mul(k2, s[r]));
                    s[r + 1] = pair_fma(bb.y, x2, pair_mul(k2, s[r + 1]));
                }
            }
            continue;
        }
#pragma unroll
        for (int tt = 0; tt < CH; ++tt) {
            if (tt < n) token(tt);
            else y[tt] = 0.f;
        }
#pragma unroll
        for (int tt = 0; tt < CH; ++tt) s_y[(warp * CH + tt) * SSD_COLS + lane] = y[tt];
        __syncthreads();
        for (int e = tid; e < n * SSD_COLS; e += SSD_THREADS) {
            const int tt = e / SSD_COLS, col = e & (SSD_COLS - 1), j = p0 + col;
            if (j >= P) continue;
            float total = 0.f;
#pragma unroll
            for (int w = 0; w < SSD_WARPS; ++w) total += s_y[(w * CH + tt) * SSD_COLS + col];
            total = fmaf(skip, s_x[e], total);
            const float z = to_float(raw[(size_t)(t0 + tt) * in.ld_raw + in.z + (size_t)h * P + j]);
            out[(size_t)(t0 + tt) * out_stride + (size_t)h * P + j] = from_float<TO>(total * silu(z));
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

// One token per entry.  Thread (part, group) works on the columns [V group, V group + V) of the rows part, part + parts, ...;
// `lanes` (a power of two, at least P / V) threads share a row.
constexpr int SSD_STEP_ROWS = 8;                                 // rows of a thread that are on their way together

template <typename T, typename TO, int V>
__global__ void __launch_bounds__(SSD_THREADS)
ssd_step_kernel(const T* __restrict__ conv, const T* __restrict__ raw, const SsdInputs in, float* __restrict__ state,
                long long state_stride, const int* __restrict__ q_start, const int* __restrict__ item_slot, int lanes,
                TO* __restrict__ out, long long out_stride) {
    extern __shared__ __align__(16) float ssd_smem[];             // B [N], C [N], then the sums [warps or parts][P]
    const int item = blockIdx.x, h = blockIdx.y, tid = threadIdx.x;
    const int t = q_start[item];
    if (q_start[item + 1] <= t) return;
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
    conv = pdl_fresh(conv) + (size_t)t * in.ld_conv;
    raw = pdl_fresh(raw) + (size_t)t * in.ld_raw;
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

template <typename T, typename TO, int R, bool STATE_ONLY>
int launch_ssd_scan_rows(const T* conv, const T* raw, const SsdInputs& in, float* state, long long state_stride,
                         const int* q_start, const int* item_slot, int first_item, int last_item, int first_cut, int segments,
                         int chunk_unit, int depth, float* run_state, float* run_decay, TO* out, long long out_stride,
                         cudaStream_t s) {
    auto kernel = ssd_scan_kernel<T, TO, R, STATE_ONLY>;
    const int tiles = (in.P + SSD_COLS - 1) / SSD_COLS;
    const size_t smem = (size_t)(2 * SSD_CHUNK * SSD_WARPS * R + SSD_CHUNK * SSD_COLS + SSD_WARPS * SSD_CHUNK * SSD_COLS) * sizeof(float);
    static size_t raised[MAX_DEVICES] = {0};
    if (!ensure_dynamic_smem((const void*)kernel, smem, raised)) return PS_ERR_LAUNCH;
    if ((long long)tiles * depth > 65535) return PS_ERR_UNSUPPORTED;
    return launch_pdl(kernel, dim3(last_item - first_item, in.heads, tiles * depth), dim3(SSD_THREADS), smem, s, conv, raw, in,
                      state, state_stride, q_start, item_slot, first_item, last_item, first_cut, segments, chunk_unit, run_state,
                      run_decay, out, out_stride);
}

template <typename T, typename TO, bool STATE_ONLY>
int launch_ssd_scan(const T* conv, const T* raw, const SsdInputs& in, float* state, long long state_stride, const int* q_start,
                    const int* item_slot, int first_item, int last_item, int first_cut, int segments, int chunk_unit, int depth,
                    float* run_state, float* run_decay, TO* out, long long out_stride, cudaStream_t s) {
#define PS_SSD_ROWS(R)                                                                                                  \
    return launch_ssd_scan_rows<T, TO, R, STATE_ONLY>(conv, raw, in, state, state_stride, q_start, item_slot, first_item, last_item, \
                                                      first_cut, segments, chunk_unit, depth, run_state, run_decay, out, out_stride, s)
    if (in.N <= 32) PS_SSD_ROWS(4);
    if (in.N <= 64) PS_SSD_ROWS(8);
    if (in.N <= 128) PS_SSD_ROWS(16);
    if (in.N <= 256) PS_SSD_ROWS(32);
    PS_SSD_ROWS(64);
#undef PS_SSD_ROWS
}

template <typename T, typename TO>
int pick_ssd(const T* conv, const T* raw, const SsdInputs& in, int single, float* state, long long state_stride,
             const int* q_start, const int* item_slot, int n_items, int first_cut, int segments, float* run_state,
             float* run_decay, TO* out, long long out_stride, cudaStream_t s) {
    if (single) {
        const bool by4 = in.P % 4 == 0 && state_stride % 4 == 0 && !((uintptr_t)state & 15);
        const int V = by4 ? 4 : 1;
        int lanes = 1;
        while (lanes < SSD_THREADS && lanes * V < in.P) lanes <<= 1;
        if (lanes * V < in.P) return PS_ERR_UNSUPPORTED;
        const int parts = SSD_THREADS / lanes, rows = lanes < 32 ? SSD_WARPS : parts;
        const size_t smem = (size_t)(2 * in.N + rows * in.P) * sizeof(float);
        if (by4) {
            auto kernel = ssd_step_kernel<T, TO, 4>;
            static size_t raised[MAX_DEVICES] = {0};
            if (!ensure_dynamic_smem((const void*)kernel, smem, raised)) return PS_ERR_LAUNCH;
            return launch_pdl(kernel, dim3(n_items, in.heads), dim3(SSD_THREADS), smem, s, conv, raw, in, state, state_stride,
                              q_start, item_slot, lanes, out, out_stride);
        }
        auto kernel = ssd_step_kernel<T, TO, 1>;
        static size_t raised[MAX_DEVICES] = {0};
        if (!ensure_dynamic_smem((const void*)kernel, smem, raised)) return PS_ERR_LAUNCH;
        return launch_pdl(kernel, dim3(n_items, in.heads), dim3(SSD_THREADS), smem, s, conv, raw, in, state, state_stride, q_start,
                          item_slot, lanes, out, out_stride);
    }
    if (segments > 1) {
        int status = launch_ssd_scan<T, TO, true>(conv, raw, in, state, state_stride, q_start, item_slot, first_cut, n_items,
                                                  first_cut, segments, SSD_CHUNK, segments - 1, run_state, run_decay, out,
                                                  out_stride, s);
        if (status != PS_OK) return status;
        const int block = in.N * in.P;
        const bool by4 = block % 4 == 0 && !((uintptr_t)run_state & 15);
        const int units = by4 ? block / 4 : block;
        status = launch_pdl(by4 ? ssd_fold_kernel<4> : ssd_fold_kernel<1>,
                            dim3((units + SSD_FOLD_THREADS - 1) / SSD_FOLD_THREADS, in.heads, n_items - first_cut),
                            dim3(SSD_FOLD_THREADS), 0, s, run_state, (const float*)run_decay, q_start, first_cut, segments,
                            (int)SSD_CHUNK, in.heads, block);
        if (status != PS_OK) return status;
    }
    return launch_ssd_scan<T, TO, false>(conv, raw, in, state, state_stride, q_start, item_slot, 0, n_items, first_cut, segments,
                                         SSD_CHUNK, segments, run_state, run_decay, out, out_stride, s);
}

}  // namespace ps

// conv, raw: rows of `dtype`, ld_conv / ld_raw elements apart; offsets: where x, B, C (in conv), z and dt (in raw) begin.
// state: float32 [slots] rows of state_stride, of which the first heads * N * P numbers are S.  single: every entry brings
// exactly one token.  Entries [first_cut, n_items) are cut into up to `segments` runs: run_state float32
// [(n_items - first_cut) * heads * segments][N * P] and run_decay [...] are scratch (null when segments is 1).  out: rows of
// heads * P numbers of out_dtype (`dtype` or float32), out_stride apart.
PS_EXPORT int ps_ssd(const void* conv, long long ld_conv, const void* raw, long long ld_raw, const int* offsets,
                     const float* a_log, const float* dt_bias, const float* d, float* state, long long state_stride,
                     const int* q_start, const int* item_slot, int n_items, int T, int single, int first_cut, int segments,
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
        return ps::pick_ssd<float, float>((const float*)conv, (const float*)raw, in, single, state, state_stride, q_start,
                                          item_slot, n_items, first_cut, segments, run_state, run_decay, (float*)out, out_stride, s);
    if (dtype == PS_BF16 && out_dtype == PS_F32)
        return ps::pick_ssd<bf, float>((const bf*)conv, (const bf*)raw, in, single, state, state_stride, q_start, item_slot,
                                       n_items, first_cut, segments, run_state, run_decay, (float*)out, out_stride, s);
    if (dtype == PS_BF16 && out_dtype == PS_BF16)
        return ps::pick_ssd<bf, bf>((const bf*)conv, (const bf*)raw, in, single, state, state_stride, q_start, item_slot, n_items,
                                    first_cut, segments, run_state, run_decay, (bf*)out, out_stride, s);
    return PS_ERR_UNSUPPORTED;
}
