// Query/key norm, rotation and cache store for attention layers that norm each head of q and k before they
// rotate it.  From the float32 result of the input projection, per token:
//   q_h <- rotate(q_h / sqrt(mean(q_h^2) + eps) * wq)      into q_out [T, nh, dk] (compute dtype)
//   k_g <- rotate(k_g / sqrt(mean(k_g^2) + eps) * wk)      into the key plane, at the token's slot
//   v_g times a constant                                   into the value plane, at the token's slot
// wq, wk: one weight vector of dk entries each, shared by the heads (null: no norm).  With `whole` the norm runs
// over the whole projection instead, all heads of q (of k) at once, q <- q / sqrt(mean over nh dk (q^2) + eps) * wq
// with wq of nh dk entries (wk: nkv dk).  The rotation turns the
// first `rot` entries of a head, entry 2i paired with entry 2i + 1 (interleaved pairs) or, with `halves`, entry i
// with entry i + rot / 2: the pair (a, b) at
// position p becomes (a cos t - b sin t, b cos t + a sin t), t = p * freq[i]; `freq` is a float32 table
// of rot / 2 entries (any frequency scaling is in the table), the angle and sincosf are float32.  The slot of
// position p of request seg is block_table[seg][p / page_size] * page_size + p % page_size.
// One warp per (token, head); one more warp per token copies the values.  With `whole` one CTA takes a token: it reads q and k
// once into shared memory, sums both, and norms and turns them from there.
#include "common.cuh"

namespace prism {

template <typename T>
__global__ void qk_norm_rope_store_kernel(const float* __restrict__ q_in, const float* __restrict__ k_in,
                                          const float* __restrict__ v_in, long long ps, const void* __restrict__ wq,
                                          int wq_bf16, const void* __restrict__ wk, int wk_bf16, float eps,
                                          const float* __restrict__ freq, int rot, T* __restrict__ q_out,
                                          T* __restrict__ k_plane, T* __restrict__ v_plane,
                                          const int* __restrict__ block_table, int bt_width,
                                          const int* __restrict__ positions, const int* __restrict__ tok_seg, int nh, int nkv,
                                          int dk, int dv, int page_size, int num_pages, int max_pos, int* err, int whole,
                                          int halves, float v_scale) {
    __shared__ float red[33];
    pdl_trigger();
    pdl_wait();
    const int t = blockIdx.x;
    const float* q = pdl_fresh(q_in) + (size_t)t * ps;
    const float* k = pdl_fresh(k_in) + (size_t)t * ps;
    const float* v = pdl_fresh(v_in) + (size_t)t * ps;
    const int pos = positions[t];
    float inv_q = 1.f, inv_k = 1.f;           // whole: every CTA of the token forms both sums itself
    if (whole && (wq != nullptr || wk != nullptr)) {
        float sq = 0.f, sk = 0.f;
        for (int c = threadIdx.x; c < nh * dk; c += blockDim.x) sq += q[c] * q[c];
        if (k_plane != nullptr)
            for (int c = threadIdx.x; c < nkv * dk; c += blockDim.x) sk += k[c] * k[c];
        sq = block_sum(sq, red);
        sk = block_sum(sk, red);
        inv_q = 1.f / sqrtf(sq / (float)(nh * dk) + eps);
        inv_k = 1.f / sqrtf(sk / (float)(nkv * dk) + eps);
    }
    if (pos < 0 || pos >= max_pos) {
        if (threadIdx.x == 0) report_error(err, PRISM_ERR_POSITION_RANGE);
        return;
    }
    // a layer without planes of its own stores nothing and looks up no page
    const int page = k_plane != nullptr ? block_table[(size_t)tok_seg[t] * bt_width + pos / page_size] : 0;
    const bool page_ok = page >= 0 && page < num_pages;
    if (!page_ok && threadIdx.x == 0) report_error(err, PRISM_ERR_PAGE_RANGE);
    const size_t slot = page_ok ? (size_t)page * page_size + pos % page_size : 0;
    const int lane = threadIdx.x & 31;
    const int unit = blockIdx.y * (blockDim.x >> 5) + (threadIdx.x >> 5);      // q heads, k heads, then the values
    if (unit == nh + nkv && page_ok && v_plane != nullptr)
        for (int c = lane; c < nkv * dv; c += 32) v_plane[slot * nkv * dv + c] = from_float<T>(v[c] * v_scale);
    const int half = rot >> 1;
    for (int hh = unit; hh < nh + nkv; hh += nh + nkv) {
        const bool is_q = hh < nh;
        if (!is_q && k_plane == nullptr) continue;          // a layer that reads another layer's keys and values
        const float* row = is_q ? q + (size_t)hh * dk : k + (size_t)(hh - nh) * dk;
        const void* w = is_q ? wq : wk;
        const int wb = is_q ? wq_bf16 : wk_bf16;
        const size_t w0 = whole ? (size_t)(is_q ? hh : hh - nh) * dk : 0;      // the head's first weight
        float inv = is_q ? inv_q : inv_k;
        if (w != nullptr && !whole) {
            float ss = 0.f;
            for (int d = lane; d < dk; d += 32) ss += row[d] * row[d];
            ss = warp_sum(ss);
            inv = 1.f / sqrtf(ss / (float)dk + eps);
        }
        if (!is_q && !page_ok) continue;
        T* dst = is_q ? q_out + ((size_t)t * nh + hh) * dk : k_plane + (slot * nkv + (hh - nh)) * dk;
        for (int d = lane; d < dk; d += 32) {
            float a = row[d] * inv * (w != nullptr ? load_param(w, wb, w0 + d) : 1.f);
            if (d < rot) {
                const int e = halves ? (d < half ? d + half : d - half) : d ^ 1;
                const bool second = halves ? d >= half : (d & 1);
                const float b = row[e] * inv * (w != nullptr ? load_param(w, wb, w0 + e) : 1.f);
                float sn, cs;
                sincosf((float)pos * freq[halves ? (second ? e : d) : d >> 1], &sn, &cs);
                a = second ? a * cs + b * sn : a * cs - b * sn;
            }
            dst[d] = from_float<T>(a);
        }
    }
}

// The whole-projection form: dynamic shared memory [(nh + nkv) dk] floats, then cosines and sines [rot / 2] each.  VEC 4: q, k, v
// rows and outputs are read and written four entries at a time.
template <typename T, int VEC>
__global__ void __launch_bounds__(256) qk_norm_whole_kernel(
    const float* __restrict__ q_in, const float* __restrict__ k_in, const float* __restrict__ v_in, long long ps,
    const void* __restrict__ wq, int wq_bf16, const void* __restrict__ wk, int wk_bf16, float eps, const float* __restrict__ freq, int rot,
    T* __restrict__ q_out, T* __restrict__ k_plane, T* __restrict__ v_plane, const int* __restrict__ block_table, int bt_width,
    const int* __restrict__ positions, const int* __restrict__ tok_seg, int nh, int nkv, int dk, int dv, int page_size, int num_pages,
    int max_pos, int* err, int halves, float v_scale) {
    pdl_trigger();
    extern __shared__ __align__(16) float row[];
    __shared__ float red[33];
    const bool own = k_plane != nullptr;
    const int t = blockIdx.x, pos = positions[t], nq = nh * dk, nk = own ? nkv * dk : 0, half = rot >> 1;
    float *cs = row + (nh + nkv) * dk, *sn = cs + half;
    for (int i = threadIdx.x; i < half; i += blockDim.x) sincosf((float)pos * freq[i], sn + i, cs + i);
    if (pos < 0 || pos >= max_pos) {
        if (threadIdx.x == 0) report_error(err, PRISM_ERR_POSITION_RANGE);
        return;
    }
    const int page = own ? block_table[(size_t)tok_seg[t] * bt_width + pos / page_size] : 0;
    const bool page_ok = page >= 0 && page < num_pages;
    if (!page_ok && threadIdx.x == 0) report_error(err, PRISM_ERR_PAGE_RANGE);
    const size_t slot = page_ok ? (size_t)page * page_size + pos % page_size : 0;
    pdl_wait();
    const float* q = pdl_fresh(q_in) + (size_t)t * ps;
    const float* k = pdl_fresh(k_in) + (size_t)t * ps;
    const float* v = pdl_fresh(v_in) + (size_t)t * ps;
    auto load = [](const float* p, float (&x)[VEC]) {
        if constexpr (VEC == 4) {
            const float4 a = *reinterpret_cast<const float4*>(p);
            x[0] = a.x; x[1] = a.y; x[2] = a.z; x[3] = a.w;
        } else {
            x[0] = *p;
        }
    };
    auto store = [](T* p, const float (&x)[VEC]) {
        if constexpr (VEC == 4 && sizeof(T) == 2) {
            const __nv_bfloat162 a = __floats2bfloat162_rn(x[0], x[1]), b = __floats2bfloat162_rn(x[2], x[3]);
            *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&a), *reinterpret_cast<const uint32_t*>(&b));
        } else if constexpr (VEC == 4) {
            *reinterpret_cast<float4*>(p) = make_float4(x[0], x[1], x[2], x[3]);
        } else {
            *p = from_float<T>(x[0]);
        }
    };
    float sq = 0.f, sk = 0.f;
    for (int c = threadIdx.x * VEC; c < nq + nk; c += blockDim.x * VEC) {
        float x[VEC];
        load(c < nq ? q + c : k + (c - nq), x);
        float ss = 0.f;
#pragma unroll
        for (int i = 0; i < VEC; ++i) {
            row[c + i] = x[i];
            ss += x[i] * x[i];
        }
        if (c < nq) sq += ss; else sk += ss;
    }
    if (own && page_ok)
        for (int c = threadIdx.x * VEC; c < nkv * dv; c += blockDim.x * VEC) {
            float x[VEC];
            load(v + c, x);
#pragma unroll
            for (int i = 0; i < VEC; ++i) x[i] *= v_scale;
            store(v_plane + slot * nkv * dv + c, x);
        }
    sq = block_sum(sq, red);
    sk = own ? block_sum(sk, red) : 0.f;
    const float inv_q = 1.f / sqrtf(sq / (float)nq + eps), inv_k = own ? 1.f / sqrtf(sk / (float)nk + eps) : 0.f;
    for (int c = threadIdx.x * VEC; c < nq + nk; c += blockDim.x * VEC) {
        const bool is_q = c < nq;
        if (!is_q && !page_ok) continue;
        const int g = is_q ? c : c - nq;                       // place in its projection
        const void* w = is_q ? wq : wk;
        const int wb = is_q ? wq_bf16 : wk_bf16;
        const float inv = is_q ? inv_q : inv_k;
        float x[VEC];
#pragma unroll
        for (int i = 0; i < VEC; ++i) {
            const int d = (g + i) % dk;
            float a = row[c + i] * inv * load_param(w, wb, g + i);
            if (d < rot) {
                const int e = halves ? (d < half ? half : -half) : ((d & 1) ? -1 : 1);
                const bool second = halves ? d >= half : (d & 1);
                const int f = halves ? (second ? d - half : d) : d >> 1;
                const float b = row[c + i + e] * inv * load_param(w, wb, g + i + e);
                a = second ? a * cs[f] + b * sn[f] : a * cs[f] - b * sn[f];
            }
            x[i] = a;
        }
        store(is_q ? q_out + (size_t)t * nq + g : k_plane + slot * nk + g, x);
    }
}

}  // namespace prism

// q, k, v: float32 rows with one row stride `ps` (column blocks of one product); planes [slots, nkv, dk] and
// [slots, nkv, dv] of `dtype` (both null: only q is made), q_out [T, nh, dk] of `dtype`; rot even, <= dk.
PRISM_EXPORT int prism_qk_norm_rope_store(const float* q, const float* k, const float* v, long long ps, const void* wq,
                                          int wq_dtype, const void* wk, int wk_dtype, float eps, const float* freq, int rot,
                                          void* q_out, void* k_plane, void* v_plane, int dtype, const int* block_table,
                                          int bt_width, const int* positions, const int* tok_seg, int T, int nh, int nkv, int dk,
                                          int dv, int page_size, int num_pages, int max_pos, int* err, int whole, int halves,
                                          float v_scale, cudaStream_t stream) {
    if (T <= 0) return 0;
    if (rot < 0 || rot > dk || rot % 2 || (rot > 0 && freq == nullptr) || nh < 1 || nkv < 1 || dk < 1 || dv < 1)
        return (int)cudaErrorInvalidValue;
    const int units = nh + nkv + 1;
    const int threads = units >= 4 ? 128 : 32 * units;
    const dim3 grid(T, (units + threads / 32 - 1) / (threads / 32));
    if (T > 65535 * 32) return (int)cudaErrorInvalidValue;
    const int qb = wq_dtype == PRISM_DTYPE_BF16, kb = wk_dtype == PRISM_DTYPE_BF16;
    const size_t row_bytes = ((size_t)(nh + nkv) * dk + rot) * sizeof(float);
    if (whole && wq != nullptr && (wk != nullptr || k_plane == nullptr) && row_bytes <= 160 * 1024) {
        const int esz = dtype == PRISM_DTYPE_BF16 ? 2 : 4;
        const bool vec = dk % 4 == 0 && dv % 4 == 0 && ps % 4 == 0 && (uintptr_t)q % 16 == 0 && (uintptr_t)k % 16 == 0 && (uintptr_t)v % 16 == 0 &&
                         (uintptr_t)q_out % (4 * esz) == 0 && (uintptr_t)k_plane % (4 * esz) == 0 && (uintptr_t)v_plane % (4 * esz) == 0;
#define PRISM_QW(TT, V)                                                                                                      \
    do {                                                                                                                     \
        auto kern = prism::qk_norm_whole_kernel<TT, V>;                                                                      \
        if (row_bytes > 40 * 1024) cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)row_bytes);  \
        return (int)prism::launch_kernel(kern, dim3(T), dim3(256), row_bytes, stream, q, k, v, ps, wq, qb, wk, kb, eps, freq, rot, \
                                         (TT*)q_out, (TT*)k_plane, (TT*)v_plane, block_table, bt_width, positions, tok_seg, nh, nkv, \
                                         dk, dv, page_size, num_pages, max_pos, err, halves, v_scale);                       \
    } while (0)
        if (dtype == PRISM_DTYPE_BF16) {
            if (vec) PRISM_QW(__nv_bfloat16, 4);
            PRISM_QW(__nv_bfloat16, 1);
        }
        if (vec) PRISM_QW(float, 4);
        PRISM_QW(float, 1);
#undef PRISM_QW
    }
    if (dtype == PRISM_DTYPE_BF16)
        return (int)prism::launch_kernel(prism::qk_norm_rope_store_kernel<__nv_bfloat16>, grid, dim3(threads), 0, stream, q, k,
                                         v, ps, wq, qb, wk, kb, eps, freq, rot, (__nv_bfloat16*)q_out, (__nv_bfloat16*)k_plane,
                                         (__nv_bfloat16*)v_plane, block_table, bt_width, positions, tok_seg, nh, nkv, dk, dv,
                                         page_size, num_pages, max_pos, err, whole, halves, v_scale);
    return (int)prism::launch_kernel(prism::qk_norm_rope_store_kernel<float>, grid, dim3(threads), 0, stream, q, k, v, ps, wq,
                                     qb, wk, kb, eps, freq, rot, (float*)q_out, (float*)k_plane, (float*)v_plane, block_table,
                                     bt_width, positions, tok_seg, nh, nkv, dk, dv, page_size, num_pages, max_pos, err, whole, halves,
                                     v_scale);
}
