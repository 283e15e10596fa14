// Residual add fused with RMSNorm.
//
//   residual[r, :] += sum_s delta[s, r, :]          (float32, in place)
//   out[i, :] = residual[r, :] * rsqrt(mean(residual[r, :]^2) + eps) * w
//
// which is andre-fu/prism's `residual + F.linear(...)` followed by
// `fused_rms_norm` (engine/executor.py:122-124; formula
// engine/fused_kernels.py:41-49), with the sum and the norm in float32 and a
// single rounding at the store of `out`.  `rows` (optional) lists the rows to
// process, so that the final norm touches only the rows whose logits are
// wanted (executor.py:130).  One block per row; the order of additions is
// fixed by the block size, so a row's result does not depend on the batch.
#include "common.cuh"
#include "vec.cuh"

namespace prism {

template <typename TD, typename TO>
__global__ void add_rmsnorm_kernel(float* __restrict__ residual, const TD* __restrict__ delta_in,
                                   int nsplit, size_t split_stride,
                                   const void* __restrict__ weight, int weight_bf16, float eps,
                                   TO* __restrict__ out, const int* __restrict__ rows, int H) {
    pdl_trigger();
    pdl_wait();
    const TD* delta = pdl_fresh(delta_in);          // the previous kernel's output
    __shared__ float scratch[33];
    const int i = blockIdx.x;
    const int r = rows ? rows[i] : i;
    float* res = residual + (size_t)r * H;
    float ss = 0.f;
    for (int c = threadIdx.x; c < H; c += blockDim.x) {
        float v = res[c];
        if (delta != nullptr) {
            for (int s = 0; s < nsplit; ++s)
                v += to_float(delta[(size_t)s * split_stride + (size_t)r * H + c]);
            res[c] = v;
        }
        ss += v * v;
    }
    ss = block_sum(ss, scratch);
    const float inv = rsqrtf(ss / (float)H + eps);
    TO* o = out + (size_t)i * H;
    for (int c = threadIdx.x; c < H; c += blockDim.x)
        o[c] = from_float<TO>(res[c] * inv * load_param(weight, weight_bf16, c));
}

// Vector version for H % 8 == 0 and H <= 8 * 1024 * ITERS: a thread keeps its
// 8 * ITERS values in registers between the sum of squares and the store, so
// the row is read once.  One block per row, as above.
template <typename TD, typename TO, int ITERS>
__global__ void __launch_bounds__(1024) add_rmsnorm_vec_kernel(float* __restrict__ residual, const TD* __restrict__ delta_in,
                                       int nsplit, size_t split_stride,
                                       const void* __restrict__ weight, int weight_bf16, float eps,
                                       TO* __restrict__ out, const int* __restrict__ rows, int H) {
    pdl_trigger();
    // the norm's weight is a constant: it is in registers before the kernels before this one have ended
    float w[ITERS][8];
#pragma unroll
    for (int it = 0; it < ITERS; ++it) {
        const int c = (threadIdx.x + it * blockDim.x) * 8;
        if (c < H) load_param8(weight, weight_bf16, c, w[it]);
    }
    pdl_wait();
    const TD* delta = pdl_fresh(delta_in);          // the previous kernel's output
    __shared__ float scratch[33];
    const int i = blockIdx.x;
    const int r = rows ? rows[i] : i;
    float* res = residual + (size_t)r * H;
    float v[ITERS][8];
    float ss = 0.f;
#pragma unroll
    for (int it = 0; it < ITERS; ++it) {
        const int c = (threadIdx.x + it * blockDim.x) * 8;
        if (c < H) {
            load8(res + c, v[it]);
            if (delta != nullptr) {
                for (int s = 0; s < nsplit; ++s) {
                    float d[8];
                    load8(delta + (size_t)s * split_stride + (size_t)r * H + c, d);
#pragma unroll
                    for (int k = 0; k < 8; ++k) v[it][k] += d[k];
                }
                store8(res + c, v[it]);
            }
#pragma unroll
            for (int k = 0; k < 8; ++k) ss += v[it][k] * v[it][k];
        }
    }
    ss = block_sum(ss, scratch);
    const float inv = rsqrtf(ss / (float)H + eps);
    TO* o = out + (size_t)i * H;
#pragma unroll
    for (int it = 0; it < ITERS; ++it) {
        const int c = (threadIdx.x + it * blockDim.x) * 8;
        if (c < H) {
#pragma unroll
            for (int k = 0; k < 8; ++k) w[it][k] *= v[it][k] * inv;
            store8(o + c, w[it]);
        }
    }
}

// Norm after the sum, for layers whose residual stream is itself normed:
//   x[r, :] <- (alpha x[r, :] + sum_s delta[s, r, :]) * rsqrt(mean((..)^2) + eps) * w        (float32, in place)
//   copy[r, :] = x[r, :] in the compute dtype (optional: what the next sublayer's matrix products read)
// One block per row; a thread touches only its own columns, so the row can be rewritten in place.
template <typename TD, typename TO>
__global__ void scale_add_rmsnorm_kernel(float* __restrict__ x, float alpha, const TD* __restrict__ delta_in, int nsplit,
                                         size_t split_stride, const void* __restrict__ weight, int weight_bf16, float eps,
                                         TO* __restrict__ copy, int H) {
    pdl_trigger();
    pdl_wait();
    const TD* delta = pdl_fresh(delta_in);
    __shared__ float scratch[33];
    const int r = blockIdx.x;
    float* row = x + (size_t)r * H;
    float ss = 0.f;
    for (int c = threadIdx.x; c < H; c += blockDim.x) {
        float v = alpha * row[c];
        if (delta != nullptr)
            for (int s = 0; s < nsplit; ++s) v += to_float(delta[(size_t)s * split_stride + (size_t)r * H + c]);
        row[c] = v;
        ss += v * v;
    }
    ss = block_sum(ss, scratch);
    const float inv = 1.f / sqrtf(ss / (float)H + eps);
    for (int c = threadIdx.x; c < H; c += blockDim.x) {
        const float v = row[c] * inv * load_param(weight, weight_bf16, c);
        row[c] = v;
        if (copy != nullptr) copy[(size_t)r * H + c] = from_float<TO>(v);
    }
}

// Vector version for H % 8 == 0 and H <= 8 * 1024 * ITERS: a thread keeps its 8 * ITERS values in registers, the
// partial sums' loads are independent of one another (four in flight per pass), the weight is read before the wait.
template <typename TD, typename TO, int ITERS>
__global__ void __launch_bounds__(1024) scale_add_rmsnorm_vec_kernel(float* __restrict__ x, float alpha, const TD* __restrict__ delta_in,
                                                                     int nsplit, size_t split_stride, const void* __restrict__ weight,
                                                                     int weight_bf16, float eps, TO* __restrict__ copy, int H) {
    pdl_trigger();
    float w[ITERS][8];
#pragma unroll
    for (int it = 0; it < ITERS; ++it) {
        const int c = (threadIdx.x + it * blockDim.x) * 8;
        if (c < H) load_param8(weight, weight_bf16, c, w[it]);
    }
    pdl_wait();
    const TD* delta = pdl_fresh(delta_in);
    __shared__ float scratch[33];
    const int r = blockIdx.x;
    float* row = x + (size_t)r * H;
    float v[ITERS][8];
    float ss = 0.f;
#pragma unroll
    for (int it = 0; it < ITERS; ++it) {
        const int c = (threadIdx.x + it * blockDim.x) * 8;
        if (c < H) {
            load8(row + c, v[it]);
#pragma unroll
            for (int k = 0; k < 8; ++k) v[it][k] *= alpha;
            if (delta != nullptr) {
                const TD* d0 = delta + (size_t)r * H + c;
                int s = 0;
                for (; s + 4 <= nsplit; s += 4) {
                    float d[4][8];
#pragma unroll
                    for (int j = 0; j < 4; ++j) load8(d0 + (size_t)(s + j) * split_stride, d[j]);
#pragma unroll
                    for (int j = 0; j < 4; ++j)
#pragma unroll
                        for (int k = 0; k < 8; ++k) v[it][k] += d[j][k];
                }
                for (; s < nsplit; ++s) {
                    float d[8];
                    load8(d0 + (size_t)s * split_stride, d);
#pragma unroll
                    for (int k = 0; k < 8; ++k) v[it][k] += d[k];
                }
            }
#pragma unroll
            for (int k = 0; k < 8; ++k) ss += v[it][k] * v[it][k];
        }
    }
    ss = block_sum(ss, scratch);
    const float inv = 1.f / sqrtf(ss / (float)H + eps);
#pragma unroll
    for (int it = 0; it < ITERS; ++it) {
        const int c = (threadIdx.x + it * blockDim.x) * 8;
        if (c < H) {
#pragma unroll
            for (int k = 0; k < 8; ++k) v[it][k] *= inv * w[it][k];
            store8(row + c, v[it]);
            if (copy != nullptr) store8(copy + (size_t)r * H + c, v[it]);
        }
    }
}

// The residual sum alone, for a sublayer that reads the stream itself rather than its norm:
//   residual[r, :] += sum_s delta[s, r, :]   (float32, in place);   copy[r, :] = residual[r, :] in the compute dtype.
template <typename TD, typename TO>
__global__ void add_rows_kernel(float* __restrict__ residual, const TD* __restrict__ delta_in, int nsplit, size_t split_stride,
                                TO* __restrict__ copy, int H) {
    pdl_trigger();
    pdl_wait();
    const TD* delta = pdl_fresh(delta_in);
    const int r = blockIdx.x;
    float* res = residual + (size_t)r * H;
    for (int c = threadIdx.x; c < H; c += blockDim.x) {
        float v = res[c];
        if (delta != nullptr) {
            for (int s = 0; s < nsplit; ++s) v += to_float(delta[(size_t)s * split_stride + (size_t)r * H + c]);
            res[c] = v;
        }
        if (copy != nullptr) copy[(size_t)r * H + c] = from_float<TO>(v);
    }
}

// A sublayer between two norms: its result is normed before it joins the residual stream, and the next sublayer's norm
// follows at once.  Per row, one block, one launch:
//   d = sum_s delta[s, r, :];   x = residual[r, :] + d * rsqrt(mean(d^2) + eps_d) * wd;   residual[r, :] = x  (float32)
//   out[i, :] = x * rsqrt(mean(x^2) + eps) * w
// rows (optional): only these rows, and the residual rows are then left alone (nothing reads them afterwards).
template <typename TD, typename TO>
__global__ void add_normed_rmsnorm_kernel(float* __restrict__ residual, const TD* __restrict__ delta_in, int nsplit,
                                          size_t split_stride, const void* __restrict__ wd, int wd_bf16, float eps_d,
                                          const void* __restrict__ weight, int weight_bf16, float eps, TO* __restrict__ out,
                                          const int* __restrict__ rows, int H) {
    pdl_trigger();
    pdl_wait();
    const TD* delta = pdl_fresh(delta_in);
    extern __shared__ float row[];                 // [H]: the summed delta, then the new residual row
    __shared__ float scratch[33];
    const int i = blockIdx.x;
    const int r = rows ? rows[i] : i;
    float* res = pdl_fresh(residual) + (size_t)r * H;
    float ss = 0.f;
    for (int c = threadIdx.x; c < H; c += blockDim.x) {
        float v = 0.f;
        for (int s = 0; s < nsplit; ++s) v += to_float(delta[(size_t)s * split_stride + (size_t)r * H + c]);
        row[c] = v;
        ss += v * v;
    }
    ss = block_sum(ss, scratch);
    const float inv_d = 1.f / sqrtf(ss / (float)H + eps_d);
    ss = 0.f;
    for (int c = threadIdx.x; c < H; c += blockDim.x) {
        const float v = res[c] + row[c] * inv_d * load_param(wd, wd_bf16, c);
        row[c] = v;
        if (rows == nullptr) res[c] = v;
        ss += v * v;
    }
    if (out == nullptr) return;
    TO* o = out + (size_t)i * H;
    if (weight == nullptr) {                       // the rows themselves
        for (int c = threadIdx.x; c < H; c += blockDim.x) o[c] = from_float<TO>(row[c]);
        return;
    }
    ss = block_sum(ss, scratch);
    const float inv = 1.f / sqrtf(ss / (float)H + eps);
    for (int c = threadIdx.x; c < H; c += blockDim.x) o[c] = from_float<TO>(row[c] * inv * load_param(weight, weight_bf16, c));
}

// Vector version for H % 8 == 0 and H <= 8 * 1024 * ITERS: everything in registers, both weights read before the wait.
template <typename TD, typename TO, int ITERS>
__global__ void __launch_bounds__(1024) add_normed_rmsnorm_vec_kernel(float* __restrict__ residual, const TD* __restrict__ delta_in,
                                                                      int nsplit, size_t split_stride, const void* __restrict__ wd,
                                                                      int wd_bf16, float eps_d, const void* __restrict__ weight,
                                                                      int weight_bf16, float eps, TO* __restrict__ out,
                                                                      const int* __restrict__ rows, int H) {
    pdl_trigger();
    float a[ITERS][8], w[ITERS][8];
#pragma unroll
    for (int it = 0; it < ITERS; ++it) {
        const int c = (threadIdx.x + it * blockDim.x) * 8;
        if (c < H) {
            load_param8(wd, wd_bf16, c, a[it]);
            if (weight != nullptr) load_param8(weight, weight_bf16, c, w[it]);
        }
    }
    pdl_wait();
    const TD* delta = pdl_fresh(delta_in);
    __shared__ float scratch[33];
    const int i = blockIdx.x;
    const int r = rows ? rows[i] : i;
    float* res = pdl_fresh(residual) + (size_t)r * H;
    float x[ITERS][8], d[ITERS][8];
    float ss = 0.f;
#pragma unroll
    for (int it = 0; it < ITERS; ++it) {
        const int c = (threadIdx.x + it * blockDim.x) * 8;
        if (c < H) {
            load8(res + c, x[it]);                 // on its way while the delta is summed
            const TD* d0 = delta + (size_t)r * H + c;
            load8(d0, d[it]);
            for (int s = 1; s < nsplit; ++s) {
                float e[8];
                load8(d0 + (size_t)s * split_stride, e);
#pragma unroll
                for (int k = 0; k < 8; ++k) d[it][k] += e[k];
            }
#pragma unroll
            for (int k = 0; k < 8; ++k) ss += d[it][k] * d[it][k];
        }
    }
    ss = block_sum(ss, scratch);
    const float inv_d = 1.f / sqrtf(ss / (float)H + eps_d);
    ss = 0.f;
#pragma unroll
    for (int it = 0; it < ITERS; ++it) {
        const int c = (threadIdx.x + it * blockDim.x) * 8;
        if (c < H) {
#pragma unroll
            for (int k = 0; k < 8; ++k) {
                x[it][k] += d[it][k] * inv_d * a[it][k];
                ss += x[it][k] * x[it][k];
            }
            if (rows == nullptr) store8(res + c, x[it]);
            if (weight == nullptr && out != nullptr) store8(out + (size_t)i * H + c, x[it]);      // the rows themselves
        }
    }
    if (weight == nullptr) return;
    ss = block_sum(ss, scratch);
    const float inv = 1.f / sqrtf(ss / (float)H + eps);
    TO* o = out + (size_t)i * H;
#pragma unroll
    for (int it = 0; it < ITERS; ++it) {
        const int c = (threadIdx.x + it * blockDim.x) * 8;
        if (c < H) {
#pragma unroll
            for (int k = 0; k < 8; ++k) w[it][k] *= x[it][k] * inv;
            store8(o + c, w[it]);
        }
    }
}

}  // namespace prism

// residual float32 [T, H] in place; delta [nsplit, T, H] of delta_dtype, normed with wd and eps_d before it is added; out
// [nrows, H] of out_dtype: the norm (weight, eps) of the new rows, for all of them or for `rows` (the residual is then
// not written).  weight null: out receives the new rows themselves (null: nothing does).
PRISM_EXPORT int prism_add_normed_rmsnorm(float* residual, const void* delta, int delta_dtype, int nsplit, long long split_stride,
                                          const void* wd, int wd_dtype, float eps_d, const void* weight, int weight_dtype,
                                          float eps, void* out, int out_dtype, const int* rows, int nrows, int H,
                                          cudaStream_t stream) {
    if (nrows <= 0) return 0;
    if (nsplit < 1 || delta == nullptr || wd == nullptr || H < 1 || H > 50000 || (weight != nullptr && out == nullptr))
        return (int)cudaErrorInvalidValue;
    const int db = wd_dtype == PRISM_DTYPE_BF16, wb = weight_dtype == PRISM_DTYPE_BF16;
    const int chunks = H / 8;
    const bool vec = H % 8 == 0 && chunks <= 2048 && split_stride % 8 == 0 && (uintptr_t)residual % 32 == 0 &&
                     (uintptr_t)delta % 32 == 0 && (uintptr_t)out % 32 == 0 && (uintptr_t)weight % 32 == 0 && (uintptr_t)wd % 32 == 0;
    const int iters = chunks > 1024 ? 2 : 1;
    const int threads = vec ? ((chunks + iters - 1) / iters + 31) / 32 * 32 : (H >= 4096 ? 512 : (H >= 1024 ? 256 : 128));
    const size_t smem = vec ? 0 : (size_t)H * sizeof(float);
#define ARGS residual, (const TD*)delta, nsplit, (size_t)split_stride, wd, db, eps_d, weight, wb, eps, (TO*)out, rows, H
#define LAUNCH(TDx, TOx)                                                                                                  \
    do {                                                                                                                  \
        using TD = TDx; using TO = TOx;                                                                                   \
        auto plain = prism::add_normed_rmsnorm_kernel<TD, TO>;                                                            \
        if (smem > 40 * 1024) cudaFuncSetAttribute(plain, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);        \
        if (vec && iters == 1)                                                                                            \
            return (int)prism::launch_kernel(prism::add_normed_rmsnorm_vec_kernel<TD, TO, 1>, dim3(nrows), dim3(threads), 0, stream, ARGS); \
        if (vec)                                                                                                          \
            return (int)prism::launch_kernel(prism::add_normed_rmsnorm_vec_kernel<TD, TO, 2>, dim3(nrows), dim3(threads), 0, stream, ARGS); \
        return (int)prism::launch_kernel(plain, dim3(nrows), dim3(threads), smem, stream, ARGS);                          \
    } while (0)
    if (delta_dtype == PRISM_DTYPE_BF16) {
        if (out_dtype == PRISM_DTYPE_BF16) LAUNCH(__nv_bfloat16, __nv_bfloat16);
        LAUNCH(__nv_bfloat16, float);
    }
    if (out_dtype == PRISM_DTYPE_BF16) LAUNCH(float, __nv_bfloat16);
    LAUNCH(float, float);
#undef LAUNCH
#undef ARGS
}

// x float32 [rows, H] in place; delta (null: none) [nsplit, rows, H] of delta_dtype; copy (null: none) [rows, H] of
// copy_dtype.
PRISM_EXPORT int prism_scale_add_rmsnorm(float* x, float alpha, const void* delta, int delta_dtype, int nsplit,
                                         long long split_stride, const void* weight, int weight_dtype, float eps,
                                         void* copy, int copy_dtype, int rows, int H, cudaStream_t stream) {
    if (rows <= 0) return 0;
    const int wb = weight_dtype == PRISM_DTYPE_BF16;
    const int chunks = H / 8;
    const bool vec = H % 8 == 0 && chunks <= 2048 && split_stride % 8 == 0 && (uintptr_t)x % 32 == 0 &&
                     (uintptr_t)delta % 32 == 0 && (uintptr_t)copy % 32 == 0 && (uintptr_t)weight % 32 == 0;
    const int iters = chunks > 1024 ? 2 : 1;
    const int threads = vec ? ((chunks + iters - 1) / iters + 31) / 32 * 32 : (H >= 4096 ? 512 : (H >= 1024 ? 256 : 128));
#define LAUNCH(TD, TO)                                                                                              \
    do {                                                                                                            \
        if (vec && iters == 1)                                                                                      \
            return (int)prism::launch_kernel(prism::scale_add_rmsnorm_vec_kernel<TD, TO, 1>, dim3(rows), dim3(threads), 0, stream, \
                                             x, alpha, (const TD*)delta, nsplit, (size_t)split_stride, weight, wb, eps, (TO*)copy, H); \
        if (vec)                                                                                                    \
            return (int)prism::launch_kernel(prism::scale_add_rmsnorm_vec_kernel<TD, TO, 2>, dim3(rows), dim3(threads), 0, stream, \
                                             x, alpha, (const TD*)delta, nsplit, (size_t)split_stride, weight, wb, eps, (TO*)copy, H); \
        return (int)prism::launch_kernel(prism::scale_add_rmsnorm_kernel<TD, TO>, dim3(rows), dim3(threads), 0, stream, x,  \
                                         alpha, (const TD*)delta, nsplit, (size_t)split_stride, weight, wb, eps, (TO*)copy, H); \
    } while (0)
    if (delta_dtype == PRISM_DTYPE_BF16) {
        if (copy_dtype == PRISM_DTYPE_BF16) LAUNCH(__nv_bfloat16, __nv_bfloat16);
        LAUNCH(__nv_bfloat16, float);
    }
    if (copy_dtype == PRISM_DTYPE_BF16) LAUNCH(float, __nv_bfloat16);
    LAUNCH(float, float);
#undef LAUNCH
}

// delta_dtype / out_dtype: PRISM_DTYPE_*.  delta may be null (plain norm).
PRISM_EXPORT int prism_add_rmsnorm(float* residual, const void* delta, int delta_dtype, int nsplit,
                                   long long split_stride, const void* weight, int weight_dtype,
                                   float eps, void* out, int out_dtype, const int* rows, int nrows,
                                   int H, cudaStream_t stream) {
    if (nrows <= 0) return 0;
    const int wb = weight_dtype == PRISM_DTYPE_BF16;
    const int chunks = H / 8;
    const bool vec = (H % 8 == 0) && chunks <= 2048;
    const int iters = chunks > 1024 ? 2 : 1;
    const int threads = vec ? ((chunks + iters - 1) / iters + 31) / 32 * 32
                            : (H >= 2048 ? 256 : (H >= 512 ? 128 : 64));
    cudaError_t rc = cudaSuccess;
#define ARGS residual, (const TD*)delta, nsplit, (size_t)split_stride, weight, wb, eps, (TO*)out, rows, H
#define LAUNCH(TDx, TOx)                                                                          \
    do {                                                                                          \
        using TD = TDx; using TO = TOx;                                                           \
        if (vec && iters == 1) rc = prism::launch_kernel(prism::add_rmsnorm_vec_kernel<TD, TO, 1>, dim3(nrows), dim3(threads), 0, stream, ARGS); \
        else if (vec) rc = prism::launch_kernel(prism::add_rmsnorm_vec_kernel<TD, TO, 2>, dim3(nrows), dim3(threads), 0, stream, ARGS);          \
        else rc = prism::launch_kernel(prism::add_rmsnorm_kernel<TD, TO>, dim3(nrows), dim3(threads), 0, stream, ARGS);              \
    } while (0)
    if (delta_dtype == PRISM_DTYPE_BF16) {
        if (out_dtype == PRISM_DTYPE_BF16) LAUNCH(__nv_bfloat16, __nv_bfloat16);
        else LAUNCH(__nv_bfloat16, float);
    } else {
        if (out_dtype == PRISM_DTYPE_BF16) LAUNCH(float, __nv_bfloat16);
        else LAUNCH(float, float);
    }
#undef LAUNCH
#undef ARGS
    return (int)rc;
}

// residual [T, H] float32 += delta (nsplit planes [T, H] of delta_dtype, plane stride split_stride; null: nothing);
// copy [T, H] of copy_dtype (null: none) receives the new rows.
PRISM_EXPORT int prism_add_rows(float* residual, const void* delta, int delta_dtype, int nsplit, long long split_stride,
                                void* copy, int copy_dtype, int T, int H, cudaStream_t stream) {
    if (T <= 0 || H <= 0) return 0;
    const int threads = H >= 2048 ? 512 : (H >= 512 ? 256 : 128);
#define PRISM_AR(TD, TO)                                                                                              \
    return (int)prism::launch_kernel(prism::add_rows_kernel<TD, TO>, dim3(T), dim3(threads), 0, stream, residual,      \
                                     (const TD*)delta, nsplit, (size_t)split_stride, (TO*)copy, H)
    if (delta_dtype == PRISM_DTYPE_BF16) {
        if (copy_dtype == PRISM_DTYPE_BF16) PRISM_AR(__nv_bfloat16, __nv_bfloat16);
        PRISM_AR(__nv_bfloat16, float);
    }
    if (copy_dtype == PRISM_DTYPE_BF16) PRISM_AR(float, __nv_bfloat16);
    PRISM_AR(float, float);
#undef PRISM_AR
}
