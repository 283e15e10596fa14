// Causal (or windowed) attention of all heads over one cached row per token whose first entries are the value - latent
// attention, and any layer with one kv head and its values inside its keys - for portions of prompts and decode steps, on
// the 5th-generation tensor cores.
//
// The (token, head) pairs of a segment are one run of rows: a CTA owns 128 of them (UMMA M), whatever the number of heads,
// and walks the keys in tiles of 64.  Roles as in attention_tcgen05.cu (warp 0 TMA producer, warp 1 MMA issue, warps 2-5
// softmax with thread = row = tensor-memory lane), with these differences:
//   * a key tile is brought once and read twice: K-major for S = Q K^T over all of its entries, MN-major for O += P V over
//     the first `dv`; its stage is free after the second;
//   * the softmax's weights are float32 quantities by the models' definition, so P enters P V as two bf16 terms, hi + lo
//     (16 mantissa bits): the two take exactly the place of the 64 scores in tensor memory;
//   * a sink (one more term in the softmax's denominator) joins at the end;
//   * scores of two tiles and up to 256 output columns take most of tensor memory: one CTA per SM, three key stages.
// Key rows beyond the last visible key (or before the window) are zeroed in shared memory between the two products, so
// nothing unwritten in a page can reach the result.  Every mbarrier wait is bounded; on expiry all roles leave through
// the common exit.
#include "tcgen05_attention.cuh"

namespace prism {
namespace tca {

constexpr int LQ = 128;              // rows per CTA
constexpr int LK = 64;               // keys per tile
constexpr int L_THREADS = 192;
constexpr int L_STAGES = 3;
constexpr int L_TMEM = 512;          // S0, S1 (64 each), O (up to 256)
constexpr int L_OCOL = 2 * LK;
constexpr float L_RESCALE_STEP = 8.f;

struct LatentAttn {
    __nv_bfloat16* out;              // [T nh, dv]
    const int* block_table;
    int bt_width;
    const int* seg_start;
    const int* cached_len;
    int nh, dv, page_size, num_pages, window;
    float scale_log2;
    const void* sink;
    int sink_bf16;
    int* err;
    int nsplit;                      // CTAs that share the key tiles of 128 rows
    float* part_o;                   // [T nh, nsplit, dv]  their partial outputs (not normalised) ...
    float* part_ml;                  // [T nh, nsplit, 2]   ... with reference exponent and sum
};

template <int HALVES>                // 64-entry (128-byte) boxes per key row
__global__ void __launch_bounds__(L_THREADS, 1)
attn_latent_tc_kernel(const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_k, const LatentAttn a) {
    constexpr int Q_BYTES = LQ * HALVES * 128, K_BYTES = LK * HALVES * 128;
    const int seg = blockIdx.y;
    const int s0 = a.seg_start[seg], nrows = (a.seg_start[seg + 1] - s0) * a.nh;
    const int split = blockIdx.x % a.nsplit;
    const int r0 = ((int)gridDim.x / a.nsplit - 1 - (int)blockIdx.x / a.nsplit) * LQ;     // later rows see more keys: first
    if (r0 >= nrows) return;

    extern __shared__ unsigned char smem_raw[];
    unsigned char* tiles = reinterpret_cast<unsigned char*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
    unsigned char* Qs = tiles;                                   // [half][128 rows][128 B]
    unsigned char* Ks = Qs + Q_BYTES;                            // [stage][half][64 keys][128 B]
    uint64_t* q_full = reinterpret_cast<uint64_t*>(Ks + L_STAGES * K_BYTES);
    uint64_t* k_full = q_full + 1;               // [3]
    uint64_t* k_empty = k_full + L_STAGES;       // [3]
    uint64_t* s_full = k_empty + L_STAGES;       // [2]
    uint64_t* p_full = s_full + 2;               // [2]
    uint64_t* pv_done = p_full + 2;              // [2], by tile parity
    uint64_t* o_done = pv_done + 2;
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(o_done + 1);
    __shared__ int abort_flag;

    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int rows = min(LQ, nrows - r0);
    const long long row0 = (long long)s0 * a.nh + r0;            // the CTA's first row among all tokens' rows
    const int cached = a.cached_len[seg];
    const int pos0 = cached + r0 / a.nh, hi = cached + (r0 + rows - 1) / a.nh;      // positions of the first and the last row
    const int* bt = a.block_table + (size_t)seg * a.bt_width;
    const int window = a.window;
    const int lo = (window > 0 && pos0 - window + 1 > 0) ? pos0 - window + 1 : 0;   // first key any row sees
    int t0 = lo / LK, n = hi / LK + 1 - t0;
    if (a.nsplit > 1) {
        const int per = (n + a.nsplit - 1) / a.nsplit;
        t0 += split * per;
        n = min(per, n - split * per);
        if (n <= 0) {                 // no key tile for this split: an empty partial
            pdl_wait();
            for (int i = threadIdx.x; i < rows * a.dv; i += L_THREADS)
                a.part_o[((size_t)(row0 + i / a.dv) * a.nsplit + split) * a.dv + i % a.dv] = 0.f;
            for (int r = threadIdx.x; r < rows; r += L_THREADS) {
                float* ml = a.part_ml + ((size_t)(row0 + r) * a.nsplit + split) * 2;
                ml[0] = -INFINITY;
                ml[1] = 0.f;
            }
            return;
        }
    }

    // key tile j of this CTA into its stage (one thread)
    auto load_keys = [&](int j) {
        const int s = j % L_STAGES, key0 = (t0 + j) * LK;
        int page = bt[key0 / a.page_size];
        if (page < 0 || page >= a.num_pages) {
            report_error(a.err, PRISM_ERR_PAGE_RANGE);
            page = 0;                                    // the result is flagged; read something that exists
        }
        const int row = page * a.page_size + key0 % a.page_size;
        mbar_expect_tx(&k_full[s], K_BYTES);
#pragma unroll
        for (int hh = 0; hh < HALVES; ++hh) tma_load_2d(Ks + s * K_BYTES + hh * LK * 128, &map_k, &k_full[s], hh * 64, row);
    };
    int early = 0;
    if (threadIdx.x == 0) {
        abort_flag = 0;
        mbar_init(q_full, 1);
        for (int s = 0; s < L_STAGES; ++s) { mbar_init(&k_full[s], 1); mbar_init(&k_empty[s], 1); }
        for (int s = 0; s < 2; ++s) { mbar_init(&s_full[s], 1); mbar_init(&p_full[s], 128); mbar_init(&pv_done[s], 1); }
        mbar_init(o_done, 1);
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
        // The step's descriptor is there before its first kernel starts, and keys of earlier steps are in the cache: the
        // first tiles, as far as they hold no key of this step, are asked for before the kernels before this one have ended.
        while (early < min(n, L_STAGES) && (t0 + early + 1) * LK <= cached) load_keys(early++);
    }
    pdl_wait();
    if (warp == 1) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_addr(tmem_slot)), "r"(L_TMEM));
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::);
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem_base = *tmem_slot;
    volatile int* abortp = &abort_flag;
    pdl_trigger();       // not earlier: this CTA holds its tensor memory now (see attention_tcgen05.cu)

    if (warp == 0) {
        // ---- TMA producer ---------------------------------------------------------
        if (lane == 0) {
            mbar_expect_tx(q_full, Q_BYTES);
#pragma unroll
            for (int hh = 0; hh < HALVES; ++hh) tma_load_2d(Qs + hh * LQ * 128, &map_q, q_full, hh * 64, (int)row0);
            int issued = early;
            for (int j = early; j < n; ++j) {
                if (j >= L_STAGES && !mbar_wait(&k_empty[j % L_STAGES], ((j / L_STAGES) - 1) & 1, abortp)) break;
                load_keys(j);
                issued = j + 1;
            }
            if (*abortp) {
                // give the copies already in flight a bounded chance to land before the CTA's memory is reused
                mbar_wait(q_full, 0, abortp);
                for (int j = max(0, issued - L_STAGES); j < issued; ++j) mbar_wait(&k_full[j % L_STAGES], (j / L_STAGES) & 1, abortp);
            }
        }
    } else if (warp == 1) {
        // ---- MMA issue ------------------------------------------------------------
        if (lane == 0) {
            constexpr uint32_t idesc_s = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(LK >> 3) << 17) | ((uint32_t)(LQ >> 4) << 24);
            const uint32_t npv = (uint32_t)(a.dv + 15) / 16 * 16;                    // columns beyond dv are never stored
            const uint32_t idesc_pv = (1u << 4) | (1u << 7) | (1u << 10) | (1u << 16) /* B is MN-major */ | ((npv >> 3) << 17) |
                                      ((uint32_t)(LQ >> 4) << 24);
            const uint32_t q_addr = smem_addr(Qs), k_addr = smem_addr(Ks);
            bool ok = mbar_wait(q_full, 0, abortp);
            for (int j = 0; j <= n && ok; ++j) {
                if (j < n) {
                    const int s = j % L_STAGES;
                    ok = mbar_wait(&k_full[s], (j / L_STAGES) & 1, abortp);
                    if (!ok) break;
                    tc_fence_after();
#pragma unroll
                    for (int k = 0; k < HALVES * 4; ++k) {
                        const int hh = k / 4, kk = k % 4;
                        const uint64_t da = umma_desc(q_addr + hh * LQ * 128) + (uint64_t)(kk * 2);
                        const uint64_t db = umma_desc(k_addr + s * K_BYTES + hh * LK * 128) + (uint64_t)(kk * 2);
                        umma_bf16(tmem_base + (j & 1) * LK, da, db, idesc_s, k > 0 ? 1u : 0u);
                    }
                    umma_commit(&s_full[j & 1]);
                }
                if (j >= 1) {
                    const int jj = j - 1, s = jj % L_STAGES, b = jj & 1;
                    ok = mbar_wait(&p_full[b], (jj >> 1) & 1, abortp);
                    if (!ok) break;
                    tc_fence_after();
#pragma unroll
                    for (int k = 0; k < LK / UMMA_K; ++k) {
                        const uint64_t db = umma_desc_mn(k_addr + s * K_BYTES + k * (UMMA_K * 128), LK * 128);
                        const uint32_t p = tmem_base + b * LK + k * (UMMA_K / 2);
                        umma_bf16_ts(tmem_base + L_OCOL, p, db, idesc_pv, (jj > 0 || k > 0) ? 1u : 0u);       // hi
                        umma_bf16_ts(tmem_base + L_OCOL, p + LK / 2, db, idesc_pv, 1u);                       // lo
                    }
                    umma_commit(&k_empty[s]);
                    umma_commit(&pv_done[b]);
                    if (jj == n - 1) umma_commit(o_done);
                }
            }
        }
    } else {
        // ---- softmax: warps 2..5, thread = row = tensor-memory lane ---------------------
        const int qd = warp & 3;
        const int r = qd * 32 + lane;
        const uint32_t lane_base = tmem_base + ((uint32_t)(qd * 32) << 16);
        const int pos_r = min(cached + (r0 + r) / a.nh, hi);       // rows past the end behave like the last one
        const int lo_r = (window > 0 && pos_r - window + 1 > 0) ? pos_r - window + 1 : 0;
        const int chunks = (a.dv + 31) / 32;
        float m_run = -INFINITY, l_run = 0.f;
        bool ok = true;
        for (int j = 0; j < n && ok; ++j) {
            const int s = j & 1, key0 = (t0 + j) * LK;
            ok = __all_sync(0xffffffffu, mbar_wait(&s_full[s], (j >> 1) & 1, abortp));
            if (!ok) break;
            tc_fence_after();
            uint32_t sa[32], sb[32];
            tmem_ld32(lane_base + s * LK, sa);
            tmem_ld32(lane_base + s * LK + 32, sb);
            tmem_wait_ld();
            // some row of the CTA has a masked key in this tile: the causal edge, or the window's start
            if (key0 + LK - 1 > pos0 || (window > 0 && key0 < hi - window + 1)) {
#pragma unroll
                for (int i = 0; i < 32; ++i) {
                    const int ka = key0 + i, kb = key0 + 32 + i;
                    if (ka > pos_r || ka < lo_r) sa[i] = 0xff800000u;          // -inf
                    if (kb > pos_r || kb < lo_r) sb[i] = 0xff800000u;
                }
            }
            float mx4[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};      // four chains side by side: a warp has its scheduler alone
#pragma unroll
            for (int i = 0; i < 32; ++i) mx4[i & 3] = max3(mx4[i & 3], __uint_as_float(sa[i]), __uint_as_float(sb[i]));
            const float mx = fmaxf(fmaxf(mx4[0], mx4[1]), fmaxf(mx4[2], mx4[3]));
            // the exponent's reference follows the row maximum lazily (attention_tcgen05.cu)
            const float m_tile = mx * a.scale_log2;                    // scale_log2 > 0
            const bool move = m_tile - m_run > L_RESCALE_STEP;         // also the first visible key (m_run = -inf)
            const float m_new = move ? m_tile : m_run;
            const float mu = m_new == -INFINITY ? 0.f : m_new;
            const float corr = move ? ex2(m_run - mu) : 1.f;           // 0 for a row that saw nothing yet
            const uint64_t scale2 = f2_pack(a.scale_log2, a.scale_log2), neg_mu2 = f2_pack(-mu, -mu);
            uint64_t sum_a = f2_pack(0.f, 0.f), sum_b = sum_a, sum_c = sum_a, sum_d = sum_a;
            // a weight's two terms, hi = bf16(p) and lo = bf16(p - hi): hi over the scores' first half, lo over the second
            uint32_t hv[32], lv[32];
#pragma unroll
            for (int i = 0; i < 16; ++i) {
                float p0, p1, p2, p3;
                f2_unpack(f2_fma(f2_pack(__uint_as_float(sa[2 * i]), __uint_as_float(sa[2 * i + 1])), scale2, neg_mu2), p0, p1);
                f2_unpack(f2_fma(f2_pack(__uint_as_float(sb[2 * i]), __uint_as_float(sb[2 * i + 1])), scale2, neg_mu2), p2, p3);
                p0 = ex2(p0), p1 = ex2(p1), p2 = ex2(p2), p3 = ex2(p3);
                if (i & 1) {
                    sum_a = f2_add(sum_a, f2_pack(p0, p1));
                    sum_b = f2_add(sum_b, f2_pack(p2, p3));
                } else {
                    sum_c = f2_add(sum_c, f2_pack(p0, p1));
                    sum_d = f2_add(sum_d, f2_pack(p2, p3));
                }
                const uint32_t h0 = pack2(p0, p1), h1 = pack2(p2, p3);
                hv[i] = h0;
                hv[16 + i] = h1;
                lv[i] = pack2(p0 - __uint_as_float(h0 << 16), p1 - __uint_as_float(h0 & 0xffff0000u));
                lv[16 + i] = pack2(p2 - __uint_as_float(h1 << 16), p3 - __uint_as_float(h1 & 0xffff0000u));
            }
            float l0, l1;
            f2_unpack(f2_add(f2_add(sum_a, sum_b), f2_add(sum_c, sum_d)), l0, l1);
            l_run = l_run * corr + (l0 + l1);
            m_run = m_new;
            // O holds the sum up to tile j-1 relative to the old reference: rescale this row when it moved
            if (j > 0 && __any_sync(0xffffffffu, corr != 1.f)) {
                ok = __all_sync(0xffffffffu, mbar_wait(&pv_done[(j - 1) & 1], ((j - 1) >> 1) & 1, abortp));
                if (!ok) break;
                tc_fence_after();
                for (int c = 0; c < chunks; ++c) {
                    uint32_t o[32];
                    tmem_ld32(lane_base + L_OCOL + c * 32, o);
                    tmem_wait_ld();
#pragma unroll
                    for (int i = 0; i < 32; ++i) o[i] = __float_as_uint(__uint_as_float(o[i]) * corr);
                    tmem_st32(lane_base + L_OCOL + c * 32, o);
                }
            }
            // rows of keys that no row of the CTA may see are zeroed (their scores are made) before P V reads them
            if (key0 + LK - 1 > hi || key0 < lo) {
                const int ks = j % L_STAGES;
                ok = __all_sync(0xffffffffu, mbar_wait(&k_full[ks], (j / L_STAGES) & 1, abortp));
                if (!ok) break;
                if (r < LK && (key0 + r > hi || key0 + r < lo)) {
#pragma unroll
                    for (int hh = 0; hh < HALVES; ++hh) {
                        uint4* row = reinterpret_cast<uint4*>(Ks + ks * K_BYTES + hh * LK * 128 + r * 128);
#pragma unroll
                        for (int c = 0; c < 8; ++c) row[c] = make_uint4(0u, 0u, 0u, 0u);
                    }
                }
                asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
            }
            tmem_st32(lane_base + s * LK, hv);
            tmem_st32(lane_base + s * LK + 32, lv);
            tmem_wait_st();
            tc_fence_before();
            mbar_arrive(&p_full[s]);
        }
        if (ok) ok = __all_sync(0xffffffffu, mbar_wait(o_done, 0, abortp));
        if (ok) {
            tc_fence_after();
            const bool mine = r < rows;
            float inv = 1.f;
            if (a.nsplit > 1) {
                if (mine) {
                    float* ml = a.part_ml + ((size_t)(row0 + r) * a.nsplit + split) * 2;
                    ml[0] = m_run;
                    ml[1] = l_run;
                }
            } else {
                float l = l_run;
                if (a.sink != nullptr)
                    l += ex2(load_param(a.sink, a.sink_bf16, (r0 + r) % a.nh) * 1.4426950408889634f - (m_run == -INFINITY ? 0.f : m_run));
                inv = l > 0.f ? 1.f / l : 0.f;
            }
            for (int c = 0; c < chunks; ++c) {
                uint32_t o[32];
                __syncwarp();                              // the load is a warp's, whoever stored before
                tmem_ld32(lane_base + L_OCOL + c * 32, o);
                tmem_wait_ld();
                if (mine && a.nsplit > 1) {
                    float* prow = a.part_o + ((size_t)(row0 + r) * a.nsplit + split) * a.dv + c * 32;
#pragma unroll
                    for (int v4 = 0; v4 < 8; ++v4)
                        if (c * 32 + v4 * 4 < a.dv)
                            *reinterpret_cast<uint4*>(prow + v4 * 4) = make_uint4(o[v4 * 4], o[v4 * 4 + 1], o[v4 * 4 + 2], o[v4 * 4 + 3]);
                } else if (mine) {
                    __nv_bfloat16* orow = a.out + (size_t)(row0 + r) * a.dv + c * 32;
#pragma unroll
                    for (int v8 = 0; v8 < 4; ++v8)
                        if (c * 32 + v8 * 8 < a.dv) {
                            uint4 w;
                            w.x = pack2(__uint_as_float(o[v8 * 8 + 0]) * inv, __uint_as_float(o[v8 * 8 + 1]) * inv);
                            w.y = pack2(__uint_as_float(o[v8 * 8 + 2]) * inv, __uint_as_float(o[v8 * 8 + 3]) * inv);
                            w.z = pack2(__uint_as_float(o[v8 * 8 + 4]) * inv, __uint_as_float(o[v8 * 8 + 5]) * inv);
                            w.w = pack2(__uint_as_float(o[v8 * 8 + 6]) * inv, __uint_as_float(o[v8 * 8 + 7]) * inv);
                            *reinterpret_cast<uint4*>(orow + v8 * 8) = w;
                        }
                }
            }
        }
    }
    tc_fence_before();
    __syncthreads();
    if (threadIdx.x == 0 && abort_flag) report_error(a.err, PRISM_ERR_WAIT_TIMEOUT);
    if (warp == 1) {
        tc_fence_after();
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem_base), "r"(L_TMEM));
    }
}

template <int HALVES>
static int launch_latent(const LatentAttn& a, const void* q, long long q_rows, const void* kc, long long k_rows, int dk, int S,
                         int max_q_len, cudaStream_t stream) {
    CUtensorMap mq, mk;
    int rc = make_map(&mq, q, q_rows, dk, dk, LQ);
    if (rc) return rc;
    rc = make_map(&mk, kc, k_rows, dk, dk, LK);
    if (rc) return rc;
    const size_t smem = (size_t)HALVES * 128 * (LQ + L_STAGES * LK) + 1024 /*alignment*/ + 256 /*barriers*/;
    auto kern = attn_latent_tc_kernel<HALVES>;
    cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    const int tiles = (int)(((long long)max_q_len * a.nh + LQ - 1) / LQ);
    return (int)launch_kernel(kern, dim3(tiles * a.nsplit, S), dim3(L_THREADS), smem, stream, mq, mk, a);
}

}  // namespace tca
}  // namespace prism

// 1 if the kernel takes these sizes: key rows of whole 16-byte pieces up to 320 entries, values (their first dv entries) in
// whole 16-byte pieces up to 256, key tiles that lie in one page.
PRISM_EXPORT int prism_attention_latent_tc_supported(int dk, int dv, int page_size) {
    return dk >= 8 && dk % 8 == 0 && dk <= 320 && dv >= 8 && dv % 8 == 0 && dv <= dk && dv <= 256 && page_size > 0 &&
           page_size % prism::tca::LK == 0;
}

// q [T, nh, dk] bf16 contiguous; out [T, nh, dv] bf16 contiguous; kc bf16 [cache_pages, page_size, dk] contiguous; window <= 0:
// every key up to the query's own; sink [nh] or null.  nsplit > 1: partial results in part_o [T, nh, nsplit, dv] and part_ml
// [T, nh, nsplit, 2] (float32) for prism_attention_masked_merge; `out` is then not written here.
PRISM_EXPORT int prism_attention_latent_tc(const void* q, int T, void* out, const void* kc, int cache_pages, const int* block_table,
                                           int bt_width, const int* seg_start, const int* cached_len, int S, int max_q_len, int nh,
                                           int dk, int dv, int page_size, int num_pages, int window, float scale, const void* sink,
                                           int sink_dtype, int nsplit, float* part_o, float* part_ml, int* err, cudaStream_t stream) {
    using namespace prism::tca;
    if (S <= 0 || max_q_len <= 0 || T <= 0) return 0;
    if (!prism_attention_latent_tc_supported(dk, dv, page_size) || nh < 1 || S > 65535 || (long long)T * nh > (1LL << 30) ||
        ((uintptr_t)q & 15) || ((uintptr_t)out & 15) || ((uintptr_t)kc & 15) || num_pages > cache_pages || !(scale > 0.f) || nsplit < 1 ||
        nsplit > 64 || (nsplit > 1 && (part_o == nullptr || part_ml == nullptr || ((uintptr_t)part_o & 15))))
        return (int)cudaErrorInvalidValue;
    LatentAttn a;
    a.out = (__nv_bfloat16*)out; a.block_table = block_table; a.bt_width = bt_width; a.seg_start = seg_start; a.cached_len = cached_len;
    a.nh = nh; a.dv = dv; a.page_size = page_size; a.num_pages = num_pages; a.window = window;
    a.scale_log2 = scale * 1.4426950408889634f; a.sink = sink; a.sink_bf16 = sink_dtype == PRISM_DTYPE_BF16; a.err = err;
    a.nsplit = nsplit; a.part_o = part_o; a.part_ml = part_ml;
    const long long q_rows = (long long)T * nh, k_rows = (long long)cache_pages * page_size;
    switch ((dk + 63) / 64) {
        case 1: return launch_latent<1>(a, q, q_rows, kc, k_rows, dk, S, max_q_len, stream);
        case 2: return launch_latent<2>(a, q, q_rows, kc, k_rows, dk, S, max_q_len, stream);
        case 3: return launch_latent<3>(a, q, q_rows, kc, k_rows, dk, S, max_q_len, stream);
        case 4: return launch_latent<4>(a, q, q_rows, kc, k_rows, dk, S, max_q_len, stream);
        case 5: return launch_latent<5>(a, q, q_rows, kc, k_rows, dk, S, max_q_len, stream);
    }
    return (int)cudaErrorInvalidValue;
}
