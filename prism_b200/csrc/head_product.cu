// Per-head products of a few tokens, y[t, h, :] = W_h x[t, h, :], with what surrounds them in latent attention:
//
//   * query side:  out[t, h, 0 .. N) = W_h q[t, h, 0 .. K)  (the key up-projection moved to the query), and the rotated
//     part q[t, h, K .. K + r) turned by the token's position into out[t, h, N .. N + r) - one launch;
//   * value side:  out[t, h, :] = (W_h x[t, h, :]) * sigmoid(gate[t, h, :])  (the value up-projection behind the
//     attention, and the output gate) - one launch.
//
// A step of few tokens is bound by latency and by the weights' way from memory: a warp takes eight output columns of one
// head, asks for its piece of W_h before the dependency wait (16-byte loads; a thread's eight neighbouring k are spread
// over two m16n8k16 MMAs, the same way in both operands), then for the tokens' rows, sixteen at a time.
#include "mma_helpers.cuh"

namespace prism {

struct HeadProduct {
    const __nv_bfloat16* x;      // [T, nh, >= K]: token and head strides
    long long x_tok;
    int x_head;
    const __nv_bfloat16* w;      // [nh, N, K] contiguous
    __nv_bfloat16* out;          // [T, nh, N]: token and head strides
    long long out_tok;
    int out_head;
    const float* gate;           // [T, nh * N] (row stride gate_tok), or null
    long long gate_tok;
    int T, nh, N, K;
    int ntiles, ctas;            // tiles of eight columns per head; CTAs of products (the rest rotate)
    const float* freq;           // rotation of x[.., K .. K + r) into out[.., N .. N + r); r 0: none
    const int* positions;
    int r, rot, pairs;
    float amp;
};

constexpr int HP_WARPS = 4;

template <int KB>      // blocks of 32 k: K <= 32 KB
__global__ void __launch_bounds__(HP_WARPS * 32) head_product_kernel(const HeadProduct a) {
    pdl_trigger();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    if ((int)blockIdx.x >= a.ctas) {           // rotation: a warp per (token, head)
        const int unit = ((int)blockIdx.x - a.ctas) * HP_WARPS + warp;
        const bool ok = unit < a.T * a.nh;
        const int t = ok ? unit / a.nh : 0, h = ok ? unit % a.nh : 0;
        const float pos = (float)a.positions[t];
        const int half = a.rot >> 1;
        float sn = 0.f, cs = 0.f;
        if (lane < half) sincosf(pos * a.freq[lane], &sn, &cs);
        pdl_wait();
        if (!ok) return;
        const __nv_bfloat16* src = pdl_fresh(a.x) + (size_t)t * a.x_tok + (size_t)h * a.x_head + a.K;
        __nv_bfloat16* dst = a.out + (size_t)t * a.out_tok + (size_t)h * a.out_head + a.N;
        for (int i = lane; i < half; i += 32) {
            if (i != lane) sincosf(pos * a.freq[i], &sn, &cs);
            const int p = a.pairs ? 2 * i : i, q = a.pairs ? 2 * i + 1 : i + half;
            const float u = to_float(src[p]), v = to_float(src[q]), c = cs * a.amp, s = sn * a.amp;
            dst[p] = from_float<__nv_bfloat16>(u * c - v * s);
            dst[q] = from_float<__nv_bfloat16>(v * c + u * s);
        }
        for (int c = a.rot + lane; c < a.r; c += 32) dst[c] = src[c];
        return;
    }
    const int unit = blockIdx.x * HP_WARPS + warp;
    const bool ok = unit < a.nh * a.ntiles;
    const int h = ok ? unit / a.ntiles : 0, n0 = ok ? (unit % a.ntiles) * 8 : 0;
    const int g = lane >> 2, q = lane & 3;
    uint4 b[KB];
    const bool row_ok = ok && n0 + g < a.N;
    const __nv_bfloat16* wr = a.w + ((size_t)h * a.N + (row_ok ? n0 + g : 0)) * a.K + q * 8;
#pragma unroll
    for (int kb = 0; kb < KB; ++kb)
        b[kb] = row_ok && kb * 32 + q * 8 < a.K ? *reinterpret_cast<const uint4*>(wr + kb * 32) : make_uint4(0u, 0u, 0u, 0u);
    pdl_wait();
    if (!ok) return;
    const __nv_bfloat16* x = pdl_fresh(a.x) + (size_t)h * a.x_head + q * 8;
    for (int t0 = 0; t0 < a.T; t0 += 16) {
        float acc[4] = {0.f, 0.f, 0.f, 0.f};
        const int ta = t0 + g, tb = t0 + g + 8;
        uint4 xa[KB], xb[KB];
#pragma unroll
        for (int kb = 0; kb < KB; ++kb) {
            const bool in = kb * 32 + q * 8 < a.K;
            xa[kb] = in && ta < a.T ? *reinterpret_cast<const uint4*>(x + (size_t)ta * a.x_tok + kb * 32) : make_uint4(0u, 0u, 0u, 0u);
            xb[kb] = in && tb < a.T ? *reinterpret_cast<const uint4*>(x + (size_t)tb * a.x_tok + kb * 32) : make_uint4(0u, 0u, 0u, 0u);
        }
#pragma unroll
        for (int kb = 0; kb < KB; ++kb) {
            const uint32_t lo[4] = {xa[kb].x, xb[kb].x, xa[kb].y, xb[kb].y}, hi[4] = {xa[kb].z, xb[kb].z, xa[kb].w, xb[kb].w};
            mma_bf16_16816(acc, lo, b[kb].x, b[kb].y);
            mma_bf16_16816(acc, hi, b[kb].z, b[kb].w);
        }
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int t = e < 2 ? ta : tb, n = n0 + q * 2 + (e & 1);
            if (t >= a.T || n >= a.N) continue;
            float v = acc[e];
            if (a.gate != nullptr) v *= 1.f / (1.f + expf(-pdl_fresh(a.gate)[(size_t)t * a.gate_tok + (size_t)h * a.N + n]));
            a.out[(size_t)t * a.out_tok + (size_t)h * a.out_head + n] = __float2bfloat16_rn(v);
        }
    }
}

}  // namespace prism

// 1 if the kernel takes these sizes: rows of whole 16-byte pieces, K up to 256.
PRISM_EXPORT int prism_head_product_supported(int T, int N, int K) {
    return T >= 1 && T <= 64 && N >= 1 && K >= 8 && K % 8 == 0 && K <= 256;
}

// x [T, nh, *] bf16 (token and head strides in elements, multiples of 8), w [nh, N, K] bf16, out [T, nh, N (+ r)] bf16;
// gate float32 [T, nh N] or null; r > 0: x[.., K .. K + r) rotated (rot entries; pairs, amp as elsewhere) into
// out[.., N .. N + r).
PRISM_EXPORT int prism_head_product(const void* x, long long x_tok, int x_head, const void* w, void* out, long long out_tok,
                                    int out_head, const float* gate, long long gate_tok, int T, int nh, int N, int K,
                                    const float* freq, const int* positions, int r, int rot, int pairs, float amp,
                                    cudaStream_t stream) {
    using namespace prism;
    if (T <= 0 || nh <= 0) return 0;
    if (!prism_head_product_supported(T, N, K) || x_tok % 8 || x_head % 8 || (uintptr_t)x % 16 || (uintptr_t)w % 16 || r < 0 || rot < 0 ||
        rot > r || rot % 2 || (rot > 0 && freq == nullptr) || (r > 0 && positions == nullptr))
        return (int)cudaErrorInvalidValue;
    HeadProduct a;
    a.x = (const __nv_bfloat16*)x; a.x_tok = x_tok; a.x_head = x_head; a.w = (const __nv_bfloat16*)w;
    a.out = (__nv_bfloat16*)out; a.out_tok = out_tok; a.out_head = out_head; a.gate = gate; a.gate_tok = gate_tok;
    a.T = T; a.nh = nh; a.N = N; a.K = K; a.ntiles = (N + 7) / 8; a.ctas = (nh * a.ntiles + HP_WARPS - 1) / HP_WARPS;
    a.freq = freq; a.positions = positions; a.r = r; a.rot = rot; a.pairs = pairs; a.amp = amp;
    const int turns = r > 0 ? (T * nh + HP_WARPS - 1) / HP_WARPS : 0;
    const dim3 grid(a.ctas + turns), block(HP_WARPS * 32);
    if (K <= 64) return (int)launch_kernel(head_product_kernel<2>, grid, block, 0, stream, a);
    if (K <= 128) return (int)launch_kernel(head_product_kernel<4>, grid, block, 0, stream, a);
    return (int)launch_kernel(head_product_kernel<8>, grid, block, 0, stream, a);
}
