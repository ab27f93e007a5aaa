// Attention of single tokens with the query heads of a token as the rows of one tensor-core tile (bfloat16).
//
// Heads that share a key/value head read the same keys: the split-key kernel (attention_decode.cu) fetches them once per
// head, this one once per group of up to 16 heads.  Two forms:
//   plain: one cluster per (token, key/value head); the rows are the heads / kv_heads query heads of the group.
//   mixed: one cluster per token; the rows are all (up to 16) query heads, the tile meets the keys and the values of every
//          key/value head, and the heads' results are mixed at the end.  For a layer that mixes its heads' weights before
//          they meet the values, w'_h = sum_g M[h][g] w_g, and hence result_h = sum_g M[h][g] all[g][G(h)] with
//          all[g][e] = sum_j w_g(j) v_e(j), G(h) = h / (heads / kv_heads).
// Every warp walks key tiles of 16 on its own (tile numbers first + warp, + warps of the cluster, ...), with its own double
// buffer, its own running maximum and sum and its own unnormalised results:
//   S = Q K^T and O += P V with mma.sync.m16n8k16 (float32 accumulation), online softmax in float32 with exp2.
// The warps of a CTA merge through shared memory; the CTAs of a cluster then read one another's merged states, each for a
// share of the result's columns (all rows of a column are in one CTA, which is what the mixing needs).  A sink joins the
// denominator at the very end.  Sums run in an order fixed by the token's position and the grid.
// Keys older than this step are fetched before the wait for the kernel that writes the step's own.
#include "common.cuh"

namespace ps {
namespace rows {

constexpr int WARPS = 4, THREADS = WARPS * 32, M = 16, TILE = 16, MAX_CLUSTER = 8;

__device__ __forceinline__ uint32_t smem_u32(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void copy16(void* dst, const void* src, bool valid) {
    const int bytes = valid ? 16 : 0;                                   // 0: fill the 16 bytes with zeros
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(dst)), "l"(src), "r"(bytes) : "memory");
}
__device__ __forceinline__ void copy_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void copy_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }
__device__ __forceinline__ void ldm_x4(uint32_t (&r)[4], const void* p) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(p)) : "memory");
}
__device__ __forceinline__ void ldm_x4_trans(uint32_t (&r)[4], const void* p) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(p)) : "memory");
}
__device__ __forceinline__ void mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile(
        "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
        : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
        : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ uint32_t pack(float lo, float hi) {
    const __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
    return *reinterpret_cast<const uint32_t*>(&v);
}

// D: head size; NG: key/value heads that a CTA works on (at least the actual count)
template <int D, int NG>
struct Layout {
    static constexpr int WIDE = NG * D, RS = WIDE + 8;                  // a key's (or value's) row in shared memory, padded
    static constexpr int QS = D + 8;
    static constexpr int STAGE = 2 * TILE * RS;                         // K and V of one tile, elements
    static constexpr size_t Q_BYTES = (size_t)M * QS * 2, KV_BYTES = (size_t)WARPS * 2 * STAGE * 2;
    // after the tiles: every warp's sums [M][WIDE], then the CTA's, (max, sum) of warps and CTA
    static constexpr size_t SUM_BYTES = (size_t)M * WIDE * 4;
    static constexpr size_t MERGE_BYTES = (WARPS + 1) * SUM_BYTES;
    static constexpr size_t BYTES = Q_BYTES + (KV_BYTES > MERGE_BYTES ? KV_BYTES : MERGE_BYTES);
};

template <int D, int NG>
__global__ void __launch_bounds__(THREADS)
attention_rows_kernel(const __nv_bfloat16* __restrict__ q, int q_stride, __nv_bfloat16* __restrict__ out, int out_stride,
                      const __nv_bfloat16* __restrict__ k_pool, const __nv_bfloat16* __restrict__ v_pool,
                      long long page_stride, const int* __restrict__ token_item, const int* __restrict__ token_row,
                      const int* __restrict__ positions, const int* __restrict__ block_table, int bt_stride,
                      const int* __restrict__ q_start, const int* __restrict__ kv_len, int n_heads, int n_kv_heads,
                      int page_size, int window, float scale_log2, SoftmaxExtras extras, const float* __restrict__ mix) {
    using L = Layout<D, NG>;
    constexpr int WIDE = L::WIDE, RS = L::RS, QS = L::QS, KS = D / 16, PIECES = D / 8;
    extern __shared__ __align__(16) unsigned char smem_raw[];
    __shared__ float s_m[WARPS][M], s_l[WARPS][M], cta_m[M], cta_l[M];
    __nv_bfloat16* q_s = reinterpret_cast<__nv_bfloat16*>(smem_raw);
    unsigned char* shared_part = smem_raw + L::Q_BYTES;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, gq = lane >> 2, tq = lane & 3;
    __nv_bfloat16* stages = reinterpret_cast<__nv_bfloat16*>(shared_part) + (size_t)warp * 2 * L::STAGE;

    const int t = blockIdx.x, split = blockIdx.z, splits = gridDim.z;
    const bool mixed = mix != nullptr;
    const int per = n_heads / n_kv_heads;
    const int group0 = mixed ? 0 : blockIdx.y, groups = mixed ? n_kv_heads : 1;
    const int head0 = mixed ? 0 : group0 * per, rows = mixed ? n_heads : per;
    const int p = positions[t], item = token_item[t];
    const int lo = first_visible_key(p, window);
    const int* bt = block_table + (size_t)(token_row ? token_row[t] : item) * bt_stride;
    const int first_new = (q_start && kv_len) ? kv_len[item] - (q_start[item + 1] - q_start[item]) : 0;
    const int first = lo / TILE + split * WARPS + warp, last = p / TILE, step = splits * WARPS;
    const int page_log2 = 31 - __clz(page_size);

    auto load_tile = [&](int tile, int buf) {
        __nv_bfloat16* k_s = stages + (size_t)buf * L::STAGE;
        __nv_bfloat16* v_s = k_s + TILE * RS;
        // lane: key of the tile and, for the two lanes of a key, every other piece
        const int r = lane >> 1, key = tile * TILE + r;
        const bool ok = key >= lo && key <= p;
        const long long page = ok ? bt[key >> page_log2] : 0;
        const long long base = page * page_stride + ((long long)group0 * page_size + (key & (page_size - 1))) * D;
#pragma unroll
        for (int e = 0; e < NG; ++e) {
            if (e < groups) {
                const long long at = base + (long long)e * page_size * D;
#pragma unroll
                for (int c = 0; c < PIECES / 2; ++c) {
                    const int piece = 2 * c + (lane & 1);
                    copy16(k_s + r * RS + e * D + piece * 8, k_pool + (ok ? at + piece * 8 : 0), ok);
                    copy16(v_s + r * RS + e * D + piece * 8, v_pool + (ok ? at + piece * 8 : 0), ok);
                }
            }
        }
    };
    // a first tile of older keys only goes out before the wait
    const bool early = first <= last && (first + 1) * TILE <= first_new;
    if (early) load_tile(first, 0);
    pdl_prologue();
    q = pdl_fresh(q);
    k_pool = pdl_fresh(k_pool);
    v_pool = pdl_fresh(v_pool);
    if (!early && first <= last) load_tile(first, 0);
    copy_commit();
    for (int c = threadIdx.x; c < M * PIECES; c += THREADS) {
        const int r = c / PIECES, piece = c % PIECES;
        uint4 v = make_uint4(0, 0, 0, 0);
        if (r < rows) v = *reinterpret_cast<const uint4*>(q + (size_t)t * q_stride + (head0 + r) * D + piece * 8);
        *reinterpret_cast<uint4*>(q_s + r * QS + piece * 8) = v;
    }
    __syncthreads();
    uint32_t qf[KS][4];
#pragma unroll
    for (int ks = 0; ks < KS; ++ks) ldm_x4(qf[ks], q_s + (lane & 15) * QS + (ks * 2 + (lane >> 4)) * 8);

    const int row0 = gq, row1 = gq + 8;
    const int own0 = mixed ? row0 / per : 0, own1 = mixed ? row1 / per : 0;       // the rows' own key heads
    float o[WIDE / 8][4];
#pragma unroll
    for (int i = 0; i < WIDE / 8; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
    float m0 = -INFINITY, m1 = -INFINITY, l0 = 0.f, l1 = 0.f;
    int buf = 0;
    for (int tile = first; tile <= last; tile += step, buf ^= 1) {
        if (tile + step <= last) load_tile(tile + step, buf ^ 1);
        copy_commit();
        copy_wait<1>();
        __syncwarp();
        const __nv_bfloat16* k_s = stages + (size_t)buf * L::STAGE;
        const __nv_bfloat16* v_s = k_s + TILE * RS;
        float s[2][4];
#pragma unroll
        for (int e = 0; e < NG; ++e) {
            if (e < groups) {
                float c[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
#pragma unroll
                for (int ks = 0; ks < KS; ++ks) {
                    uint32_t b[4];
                    ldm_x4(b, k_s + (8 * (lane >> 4) + (lane & 7)) * RS + e * D + (ks * 2 + ((lane >> 3) & 1)) * 8);
                    mma(c[0], qf[ks], b[0], b[1]);
                    mma(c[1], qf[ks], b[2], b[3]);
                }
#pragma unroll
                for (int nt = 0; nt < 2; ++nt) {
                    if (e == 0 || own0 == e) { s[nt][0] = c[nt][0]; s[nt][1] = c[nt][1]; }
                    if (e == 0 || own1 == e) { s[nt][2] = c[nt][2]; s[nt][3] = c[nt][3]; }
                }
            }
        }
        float mx0 = -INFINITY, mx1 = -INFINITY;
#pragma unroll
        for (int nt = 0; nt < 2; ++nt) {
#pragma unroll
            for (int x = 0; x < 4; ++x) {
                const int key = tile * TILE + nt * 8 + tq * 2 + (x & 1);
                const float v = key >= lo && key <= p ? score_log2(s[nt][x], scale_log2, extras) : -INFINITY;
                s[nt][x] = v;
            }
            mx0 = fmaxf(mx0, fmaxf(s[nt][0], s[nt][1]));
            mx1 = fmaxf(mx1, fmaxf(s[nt][2], s[nt][3]));
        }
        mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 1));
        mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 2));
        mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 1));
        mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 2));
        // (a tile of the walk holds at least one visible key, so the new maxima are finite)
        const float n0 = fmaxf(m0, mx0), n1 = fmaxf(m1, mx1);
        const float corr0 = exp2f(m0 - n0), corr1 = exp2f(m1 - n1);
        m0 = n0;
        m1 = n1;
        float sum0 = 0.f, sum1 = 0.f;
#pragma unroll
        for (int nt = 0; nt < 2; ++nt) {
            s[nt][0] = exp2f(s[nt][0] - n0); s[nt][1] = exp2f(s[nt][1] - n0);
            s[nt][2] = exp2f(s[nt][2] - n1); s[nt][3] = exp2f(s[nt][3] - n1);
            sum0 += s[nt][0] + s[nt][1];
            sum1 += s[nt][2] + s[nt][3];
        }
        l0 = l0 * corr0 + sum0;
        l1 = l1 * corr1 + sum1;
#pragma unroll
        for (int i = 0; i < WIDE / 8; ++i) { o[i][0] *= corr0; o[i][1] *= corr0; o[i][2] *= corr1; o[i][3] *= corr1; }
        uint32_t a[4];
        a[0] = pack(s[0][0], s[0][1]);
        a[1] = pack(s[0][2], s[0][3]);
        a[2] = pack(s[1][0], s[1][1]);
        a[3] = pack(s[1][2], s[1][3]);
#pragma unroll
        for (int e = 0; e < NG; ++e) {
            if (e < groups) {
#pragma unroll
                for (int dn = 0; dn < D / 8; dn += 2) {
                    uint32_t b[4];
                    ldm_x4_trans(b, v_s + ((lane & 7) + ((lane >> 3) & 1) * 8) * RS + e * D + (dn + (lane >> 4)) * 8);
                    mma(o[e * (D / 8) + dn], a, b[0], b[1]);
                    mma(o[e * (D / 8) + dn + 1], a, b[2], b[3]);
                }
            }
        }
        __syncwarp();                                             // this buffer is refilled two tiles on
    }
    copy_wait<0>();
    l0 += __shfl_xor_sync(0xffffffffu, l0, 1);
    l0 += __shfl_xor_sync(0xffffffffu, l0, 2);
    l1 += __shfl_xor_sync(0xffffffffu, l1, 1);
    l1 += __shfl_xor_sync(0xffffffffu, l1, 2);
    __syncthreads();                                              // the tile buffers of all warps are free
    float* sums = reinterpret_cast<float*>(shared_part);          // [WARPS][M][WIDE], then the CTA's [M][WIDE]
    float* merged = sums + WARPS * M * WIDE;
    float* mine = sums + warp * M * WIDE;
#pragma unroll
    for (int i = 0; i < WIDE / 8; ++i) {
        const int d = i * 8 + tq * 2;
        *reinterpret_cast<float2*>(mine + row0 * WIDE + d) = make_float2(o[i][0], o[i][1]);
        *reinterpret_cast<float2*>(mine + row1 * WIDE + d) = make_float2(o[i][2], o[i][3]);
    }
    if (tq == 0) {
        s_m[warp][row0] = m0; s_l[warp][row0] = l0;
        s_m[warp][row1] = m1; s_l[warp][row1] = l1;
    }
    __syncthreads();
    // ---- the warps' states become the CTA's
    for (int idx = threadIdx.x; idx < M * WIDE / 4; idx += THREADS) {
        const int r = idx / (WIDE / 4), d = (idx % (WIDE / 4)) * 4;
        float top = -INFINITY;
#pragma unroll
        for (int w = 0; w < WARPS; ++w) top = fmaxf(top, s_m[w][r]);
        const float floor_ = top == -INFINITY ? 0.f : top;
        float4 total = make_float4(0.f, 0.f, 0.f, 0.f);
        float sum = 0.f;
#pragma unroll
        for (int w = 0; w < WARPS; ++w) {
            const float weight = exp2f(s_m[w][r] - floor_);
            const float4 v = *reinterpret_cast<const float4*>(sums + (w * M + r) * WIDE + d);
            total.x = fmaf(weight, v.x, total.x); total.y = fmaf(weight, v.y, total.y);
            total.z = fmaf(weight, v.z, total.z); total.w = fmaf(weight, v.w, total.w);
            sum = fmaf(weight, s_l[w][r], sum);
        }
        *reinterpret_cast<float4*>(merged + r * WIDE + d) = total;
        if (d == 0) { cta_m[r] = top; cta_l[r] = sum; }
    }
    __syncthreads();
    if (splits > 1) cluster_sync_all();
    // ---- the CTAs' states become the token's, every CTA for its share of the columns (whole quads)
    const int quads = groups * D / 4, share = (quads + splits - 1) / splits;
    const int quad0 = split * share, quad1 = min(quad0 + share, quads);
    float* final_rows = sums;                                     // [M][WIDE]: the warps' states have been read
    for (int idx = threadIdx.x; idx < M * share; idx += THREADS) {
        const int r = idx / share, quad = quad0 + idx % share;
        if (quad >= quad1 || r >= rows) continue;
        const int d = quad * 4;
        float mc[MAX_CLUSTER], lc[MAX_CLUSTER];
        float4 vc[MAX_CLUSTER];
#pragma unroll
        for (int c = 0; c < MAX_CLUSTER; ++c) {
            mc[c] = -INFINITY;
            lc[c] = 0.f;
            vc[c] = make_float4(0.f, 0.f, 0.f, 0.f);
            if (c < splits) {
                if (splits > 1) {
                    mc[c] = ld_cluster_f32(&cta_m[r], c);
                    lc[c] = ld_cluster_f32(&cta_l[r], c);
                    vc[c] = ld_cluster_f32x4(merged + r * WIDE + d, c);
                } else {
                    mc[c] = cta_m[r];
                    lc[c] = cta_l[r];
                    vc[c] = *reinterpret_cast<const float4*>(merged + r * WIDE + d);
                }
            }
        }
        float top = extras.sink ? extras.sink[head0 + r] * 1.4426950408889634f : -INFINITY, sum = extras.sink ? 1.f : 0.f;
        const float sink_score = top;
#pragma unroll
        for (int c = 0; c < MAX_CLUSTER; ++c) top = fmaxf(top, mc[c]);
        sum = extras.sink ? exp2f(sink_score - top) : 0.f;
        float4 total = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
        for (int c = 0; c < MAX_CLUSTER; ++c) {
            const float weight = c < splits ? exp2f(mc[c] - top) : 0.f;
            total.x = fmaf(weight, vc[c].x, total.x); total.y = fmaf(weight, vc[c].y, total.y);
            total.z = fmaf(weight, vc[c].z, total.z); total.w = fmaf(weight, vc[c].w, total.w);
            sum = fmaf(weight, lc[c], sum);
        }
        const float inverse = sum > 0.f ? 1.f / sum : 0.f;
        total.x *= inverse; total.y *= inverse; total.z *= inverse; total.w *= inverse;
        if (mixed) {
            *reinterpret_cast<float4*>(final_rows + r * WIDE + d) = total;
        } else {
            store_result4(out, (size_t)t * out_stride + (head0 + r) * D + d, total, extras);
        }
    }
    __syncthreads();
    if (splits > 1) asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory");    // the others' states have been read
    if (mixed) {
        // ---- result_h = sum_g M[h][g] all[g][G(h)]: a thread per head and quad of its own key head
        for (int idx = threadIdx.x; idx < share * per; idx += THREADS) {
            const int quad = quad0 + idx / per;
            if (quad >= quad1) continue;
            const int e = quad / (D / 4), d = (quad % (D / 4)) * 4, h = e * per + idx % per;
            float4 total = make_float4(0.f, 0.f, 0.f, 0.f);
            for (int g = 0; g < n_heads; ++g) {
                const float weight = mix[h * n_heads + g];
                const float4 v = *reinterpret_cast<const float4*>(final_rows + g * WIDE + quad * 4);
                total.x = fmaf(weight, v.x, total.x); total.y = fmaf(weight, v.y, total.y);
                total.z = fmaf(weight, v.z, total.z); total.w = fmaf(weight, v.w, total.w);
            }
            store_result4(out, (size_t)t * out_stride + h * D + d, total, extras);
        }
    }
    // nobody's shared memory goes away before it was read
    __syncwarp();
    if (splits > 1) asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory");
}

template <int D, int NG>
int launch(const void* q, int q_stride, void* out, int out_stride, const void* k_pool, const void* v_pool, long long page_stride,
           const int* token_item, const int* token_row, const int* positions, const int* block_table, int bt_stride,
           const int* q_start, const int* kv_len, int T, int n_heads, int n_kv_heads, int page_size, int window, float scale,
           int splits, float softcap, const float* sink, const float* mix, int wide, cudaStream_t s) {
    auto kernel = attention_rows_kernel<D, NG>;
    static size_t raised[MAX_DEVICES] = {0};
    if (!ensure_dynamic_smem((const void*)kernel, Layout<D, NG>::BYTES, raised)) return PS_ERR_LAUNCH;
    return launch_pdl_cluster(kernel, dim3(T, mix ? 1 : n_kv_heads, splits), dim3(THREADS), Layout<D, NG>::BYTES, s, splits,
                              (const __nv_bfloat16*)q, q_stride, (__nv_bfloat16*)out, out_stride, (const __nv_bfloat16*)k_pool,
                              (const __nv_bfloat16*)v_pool, page_stride, token_item, token_row, positions, block_table,
                              bt_stride, q_start, kv_len, n_heads, n_kv_heads, page_size, window,
                              scale * 1.4426950408889634f, softmax_extras(scale, softcap, sink, wide), mix);
}

}  // namespace rows
}  // namespace ps

// Token t's query heads (q [T, n_heads * head_dim], row stride q_stride) against the keys up to positions[t] of the request
// in block-table row token_row[t] (null: token_item[t]); out likewise.  mix null: plain attention, groups of at most 16 heads.
// mix float32 [n_heads][n_heads]: the heads' weights are mixed by it; at most 16 heads, and n_kv_heads rounded up to a power
// of two times head_dim at most 256.  Head sizes: multiples of 16 up to 128.  splits: 1, 2, 4 or 8 CTAs share a token's keys.
// q_start / kv_len (per item, both or neither): which keys are older than this step.  softcap, sink, wide (out is
// float32): see common.cuh.
PS_EXPORT int ps_attention_rows(const void* q, int q_stride, void* out, int out_stride, const void* k_pool, const void* v_pool,
                                long long page_stride, const int* token_item, const int* token_row, const int* positions,
                                const int* block_table, int bt_stride, const int* q_start, const int* kv_len, int T,
                                int n_heads, int n_kv_heads, int head_dim, int page_size, int window, float scale, int splits,
                                float softcap, const float* sink, const float* mix, int wide, void* stream) {
    if (T <= 0) return PS_OK;
    if (!q || !out || !k_pool || !v_pool || !token_item || !positions || !block_table) return PS_ERR_BAD_ARGUMENT;
    if ((q_start == nullptr) != (kv_len == nullptr)) return PS_ERR_BAD_ARGUMENT;
    if (n_heads <= 0 || n_kv_heads <= 0 || n_heads % n_kv_heads != 0 || n_kv_heads > 65535) return PS_ERR_BAD_ARGUMENT;
    if (splits != 1 && splits != 2 && splits != 4 && splits != 8) return PS_ERR_BAD_ARGUMENT;
    if (head_dim <= 0 || head_dim % 16 != 0 || head_dim > 128) return PS_ERR_UNSUPPORTED;
    if (page_size <= 0 || page_size > 64 || (page_size & (page_size - 1))) return PS_ERR_UNSUPPORTED;
    if ((mix ? n_heads : n_heads / n_kv_heads) > ps::rows::M) return PS_ERR_UNSUPPORTED;
    if (q_stride % 8 != 0 || out_stride % 4 != 0 || page_stride % 8 != 0) return PS_ERR_UNSUPPORTED;
    if (((uintptr_t)q & 15) || ((uintptr_t)out & (wide ? 15 : 7)) || ((uintptr_t)k_pool & 15) || ((uintptr_t)v_pool & 15))
        return PS_ERR_UNSUPPORTED;
    cudaStream_t s = (cudaStream_t)stream;
    const int ng = mix ? n_kv_heads : 1;
#define PS_ROWS(D, NG)                                                                                                 \
    return ps::rows::launch<D, NG>(q, q_stride, out, out_stride, k_pool, v_pool, page_stride, token_item, token_row,    \
                                   positions, block_table, bt_stride, q_start, kv_len, T, n_heads, n_kv_heads, page_size, \
                                   window, scale, splits, softcap, sink, mix, wide, s)
#define PS_ROWS_2(D)                \
    case D:                         \
        if (ng <= 1) PS_ROWS(D, 1); \
        if (ng <= 2) PS_ROWS(D, 2); \
        break;
#define PS_ROWS_4(D)                \
    case D:                         \
        if (ng <= 1) PS_ROWS(D, 1); \
        if (ng <= 2) PS_ROWS(D, 2); \
        if (ng <= 4) PS_ROWS(D, 4); \
        break;
#define PS_ROWS_8(D)                \
    case D:                         \
        if (ng <= 1) PS_ROWS(D, 1); \
        if (ng <= 2) PS_ROWS(D, 2); \
        if (ng <= 4) PS_ROWS(D, 4); \
        if (ng <= 8) PS_ROWS(D, 8); \
        break;
    switch (head_dim) {
        PS_ROWS_8(16) PS_ROWS_8(32) PS_ROWS_4(48) PS_ROWS_4(64)
        PS_ROWS_2(80) PS_ROWS_2(96) PS_ROWS_2(112) PS_ROWS_2(128)
    }
#undef PS_ROWS_2
#undef PS_ROWS_4
#undef PS_ROWS_8
#undef PS_ROWS
    return PS_ERR_UNSUPPORTED;
}
