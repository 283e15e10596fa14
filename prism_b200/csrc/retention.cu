// Retention: S <- g S + k v^T, o = S^T q per head, with one constant decay g per head, q and k rotated by the token's
// position and k times dk^-1/2, then o / rms(o) times silu(gate).  S is kept as [slot][head][value channel][key channel],
// float32.  Everything reads the float32 result of the input projections, proj [T, *] = q | k | v | gate.
//
//   * prism_retention_step   a step of single tokens: one CTA per (head, request) rotates, updates the state, reads it
//     out, norms and gates - the whole mixer between its two projections in one launch.  The state of earlier steps is
//     requested before the dependency wait.
//   * prism_retention_chunks stretches of many tokens, in chunks of 64 (counted from the segment's first token), three
//     launches: what each chunk adds to the state, U = sum_j g^(n-1-j) k_j v_j^T (all chunks side by side); the state
//     each chunk starts from (a walk over the chunks per state entry, in place over U, and the new state to the slot);
//     the outputs, o_i = g^(i+1) S^T q_i + sum_{j<=i} g^(i-j) (q_i . k_j) v_j, with norm and gate.  The products run on
//     tensor cores with both operands as two bf16 terms, x = hi + lo, hi*hi + hi*lo + lo*hi, accumulated in float32: 16
//     mantissa bits of every operand.  The powers of g come from a table made on the host.
#include "mma_helpers.cuh"

namespace prism {

constexpr int RET_CHUNK = 64;

__device__ __forceinline__ float ret_silu(float z) { return z / (1.f + expf(-z)); }

// ---------------------------------------------------------------------------------------------------------
// one token per request
// ---------------------------------------------------------------------------------------------------------
// LANES neighbouring lanes share a column of S (its dk entries, QPL quads a lane), a warp takes 32 / LANES columns at a
// time and NB times as many in one batch, all of whose loads are in flight together.
constexpr int RET_STEP_THREADS = 256;

template <typename T, int LANES, int QPL, int NB>
__global__ void __launch_bounds__(RET_STEP_THREADS)
retention_step_kernel(const float* __restrict__ proj_in, long long ps, int ko, int vo, int go, int H, int dk, int dv,
                      const float* __restrict__ freq, int rot, int pairs, float amp, float kmul, const float* __restrict__ decay,
                      float* __restrict__ state, const int* __restrict__ positions, const int* __restrict__ slots, float eps,
                      T* __restrict__ out, long long os) {
    pdl_trigger();
    extern __shared__ __align__(16) float sm[];        // q [dk] | k [dk] | v [dv] | gate [dv] | o [dv]
    __shared__ float scratch[33];
    float *q_s = sm, *k_s = sm + dk, *v_s = k_s + dk, *g_s = v_s + dv, *o_s = g_s + dv;
    const int h = blockIdx.x, t = blockIdx.y;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    constexpr int CPW = 32 / LANES, WARPS = RET_STEP_THREADS / 32;
    const int part = lane % LANES, sub = lane / LANES;
    const float g = decay[h];
    float* st = state + ((size_t)slots[t] * H + h) * (size_t)dv * dk;
    float4 S[NB][QPL];
    auto column = [&](int b, int j) { return b + (j * WARPS + warp) * CPW + sub; };
    auto fetch = [&](int b) {
#pragma unroll
        for (int j = 0; j < NB; ++j)
#pragma unroll
            for (int m = 0; m < QPL; ++m) {
                const int c = column(b, j), i = 4 * (part + LANES * m);
                S[j][m] = (c < dv && i < dk) ? *reinterpret_cast<const float4*>(st + (size_t)c * dk + i) : make_float4(0.f, 0.f, 0.f, 0.f);
            }
    };
    fetch(0);
    const float pos = (float)positions[t];
    pdl_wait();
    const float* row = pdl_fresh(proj_in) + (size_t)t * ps;
    const int half = rot >> 1;
    for (int i = threadIdx.x; i < 2 * dk; i += RET_STEP_THREADS) {
        const bool is_k = i >= dk;
        const int d = is_k ? i - dk : i;
        const float* x = row + (is_k ? ko : 0) + (size_t)h * dk;
        float a = x[d];
        if (d < rot) {
            const int e = pairs ? (d ^ 1) : (d < half ? d + half : d - half);
            const bool second = pairs ? (d & 1) : d >= half;
            float sn, cs;
            sincosf(pos * freq[pairs ? d >> 1 : (second ? e : d)], &sn, &cs);
            sn *= amp;
            cs *= amp;
            a = second ? a * cs + x[e] * sn : a * cs - x[e] * sn;
        }
        sm[i] = is_k ? a * kmul : a;
    }
    for (int c = threadIdx.x; c < dv; c += RET_STEP_THREADS) {
        v_s[c] = row[vo + (size_t)h * dv + c];
        g_s[c] = row[go + (size_t)h * dv + c];
    }
    __syncthreads();
    float4 qq[QPL], kk[QPL];
#pragma unroll
    for (int m = 0; m < QPL; ++m) {
        const int i = 4 * (part + LANES * m);
        qq[m] = i < dk ? *reinterpret_cast<const float4*>(q_s + i) : make_float4(0.f, 0.f, 0.f, 0.f);
        kk[m] = i < dk ? *reinterpret_cast<const float4*>(k_s + i) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    for (int b = 0; b < dv; b += NB * WARPS * CPW) {
        if (b > 0) fetch(b);
#pragma unroll
        for (int j = 0; j < NB; ++j) {
            const int c = column(b, j);
            const bool ok = c < dv;
            const float v = ok ? v_s[c] : 0.f;
            float o = 0.f;
#pragma unroll
            for (int m = 0; m < QPL; ++m) {
                float4 s = S[j][m];
                s.x = g * s.x + kk[m].x * v;
                s.y = g * s.y + kk[m].y * v;
                s.z = g * s.z + kk[m].z * v;
                s.w = g * s.w + kk[m].w * v;
                o += (s.x * qq[m].x + s.y * qq[m].y) + (s.z * qq[m].z + s.w * qq[m].w);
                const int i = 4 * (part + LANES * m);
                if (ok && i < dk) *reinterpret_cast<float4*>(st + (size_t)c * dk + i) = s;
            }
#pragma unroll
            for (int w = LANES / 2; w > 0; w >>= 1) o += __shfl_xor_sync(0xffffffffu, o, w);
            if (ok && part == 0) o_s[c] = o;
        }
    }
    __syncthreads();
    float ss = 0.f;
    for (int c = threadIdx.x; c < dv; c += RET_STEP_THREADS) ss += o_s[c] * o_s[c];
    ss = block_sum(ss, scratch);
    const float inv = 1.f / sqrtf(ss / (float)dv + eps);
    T* dst = out + (size_t)t * os + (size_t)h * dv;
    for (int c = threadIdx.x; c < dv; c += RET_STEP_THREADS) dst[c] = from_float<T>(o_s[c] * inv * ret_silu(g_s[c]));
}

// ---------------------------------------------------------------------------------------------------------
// chunks
// ---------------------------------------------------------------------------------------------------------
struct RetChunks {
    const float* proj;       // q | k | v | gate rows
    long long ps;
    int ko, vo, go, H, dk, dv, S;
    const float2* table;     // [T, half] cosine and sine of position * frequency, or null (no rotation)
    int rot, pairs;
    float amp, kmul, eps;
    const float* pw;         // [H, RET_CHUNK + 1] powers of the heads' decays
    float* state;            // [slots, H, dv, dk]
    const int* seg_start;
    const int* slots;
    float* ws;               // [chunks, H, dv, dk]: U, then the incoming state as two bf16 terms in one word
    __nv_bfloat16* out;
    long long os;
};

// Chunk x of the step: its segment, first token and length.  The chunks of segment s are numbered from
// seg_start[s] / 64 + s on, so every segment has room for its own; numbers in between have no chunk (n <= 0).
__device__ __forceinline__ void ret_chunk(const RetChunks& a, int x, int& t0, int& n) {
    int lo = 0, hi = a.S - 1;
    while (lo < hi) {
        const int mid = (lo + hi + 1) >> 1;
        if (a.seg_start[mid] / RET_CHUNK + mid <= x) lo = mid; else hi = mid - 1;
    }
    const int s0 = a.seg_start[lo];
    t0 = s0 + (x - (s0 / RET_CHUNK + lo)) * RET_CHUNK;
    n = min(RET_CHUNK, a.seg_start[lo + 1] - t0);
}

// four floats as hi and lo bf16 terms, at the same place of two arrays
__device__ __forceinline__ void ret_split4(float4 v, __nv_bfloat16* hi, __nv_bfloat16* lo) {
    const __nv_bfloat162 h0 = __floats2bfloat162_rn(v.x, v.y), h1 = __floats2bfloat162_rn(v.z, v.w);
    const float2 f0 = __bfloat1622float2(h0), f1 = __bfloat1622float2(h1);
    *reinterpret_cast<uint2*>(hi) = make_uint2(*reinterpret_cast<const uint32_t*>(&h0), *reinterpret_cast<const uint32_t*>(&h1));
    *reinterpret_cast<uint2*>(lo) = make_uint2(pack_bf16(v.x - f0.x, v.y - f0.y), pack_bf16(v.z - f1.x, v.w - f1.y));
}

// What a rotated quad is made of: the quad at column d (a multiple of 4) of token t's q or k, its partner, and the cosines
// and sines.  Loads only, all of them in any case (from a legal place where they are not needed), so that a batch of
// quads has all its loads on their way together; the arithmetic follows in ret_turn.
struct RetQuad {
    float4 u, w, c0, c1;
};
__device__ __forceinline__ RetQuad ret_quad(const RetChunks& a, const float* __restrict__ x, int t, int d) {
    const int half = a.rot >> 1;
    const bool turns = d < a.rot, second = d >= half;
    const int e = !turns || a.pairs ? d : (second ? d - half : d + half);
    const int ti = !turns ? 0 : (a.pairs ? d >> 1 : (second ? d - half : d));
    const float* tb = a.rot > 0 ? reinterpret_cast<const float*>(a.table + (size_t)t * half + ti) : x;
    RetQuad q;
    q.u = *reinterpret_cast<const float4*>(x + d);
    q.w = *reinterpret_cast<const float4*>(x + e);
    q.c0 = *reinterpret_cast<const float4*>(tb);
    q.c1 = *reinterpret_cast<const float4*>(tb + (a.pairs || a.rot == 0 ? 0 : 4));
    return q;
}
// the quad, rotated and times f
__device__ __forceinline__ float4 ret_turn(const RetChunks& a, const RetQuad& q, int d, float f) {
    const float4 u = q.u, w = q.w, c0 = q.c0, c1 = q.c1;
    const float g = d < a.rot ? a.amp * f : f;
    float4 r = u;
    if (d < a.rot) {
        if (a.pairs) r = make_float4(u.x * c0.x - u.y * c0.y, u.y * c0.x + u.x * c0.y, u.z * c0.z - u.w * c0.w, u.w * c0.z + u.z * c0.w);
        else {
            const float s = d >= (a.rot >> 1) ? 1.f : -1.f;
            r = make_float4(u.x * c0.x + w.x * (c0.y * s), u.y * c0.z + w.y * (c0.w * s), u.z * c1.x + w.z * (c1.y * s),
                            u.w * c1.z + w.w * (c1.w * s));
        }
    }
    return make_float4(r.x * g, r.y * g, r.z * g, r.w * g);
}
__device__ __forceinline__ float4 ret_zero4() { return make_float4(0.f, 0.f, 0.f, 0.f); }

// The quads of a [rows, 4 cols] tile, dealt out to the threads in turn, in batches of U: all of a batch's loads are on their
// way before its first store (past the end the tile's last row is loaded again instead of branching).  A thread walks its
// (row, quad) pairs by adding, it divides once.
template <int U, int THREADS, typename V, typename Load, typename Store>
__device__ __forceinline__ void ret_batches(int rows, int cols, Load load, Store store) {
    const int dr = THREADS / cols, dc = THREADS - dr * cols;
    int r = threadIdx.x / cols, c = threadIdx.x - r * cols;
    while (r < rows) {
        V v[U];
        int rr[U], cc[U];
#pragma unroll
        for (int u = 0; u < U; ++u) {
            rr[u] = r;
            cc[u] = c;
            r += dr;
            c += dc;
            if (c >= cols) { c -= cols; ++r; }
            v[u] = load(min(rr[u], rows - 1), cc[u] * 4);
        }
#pragma unroll
        for (int u = 0; u < U; ++u)
            if (rr[u] < rows) store(rr[u], cc[u] * 4, v[u]);
    }
}

constexpr int RET_STATE_THREADS = 256;

// U[c][i] = sum_j g^(n-1-j) v_j[c] k_j[i] of one chunk and head: m = c, n = i, k = j.
__global__ void __launch_bounds__(RET_STATE_THREADS) retention_chunk_state_kernel(const RetChunks a) {
    pdl_trigger();
    int t0, n;
    ret_chunk(a, blockIdx.x, t0, n);
    if (n <= 0) return;
    pdl_wait();
    extern __shared__ __align__(16) unsigned char raw[];
    const int h = blockIdx.y, dk = a.dk, dv = a.dv, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int ks = (dk + 63) / 64 * 64 + 8, vs = (dv + 31) / 32 * 32 + 8;          // whole units of the warps below, zeros beyond
    __nv_bfloat16* kh = reinterpret_cast<__nv_bfloat16*>(raw);
    __nv_bfloat16 *kl = kh + RET_CHUNK * ks, *vh = kl + RET_CHUNK * ks, *vl = vh + RET_CHUNK * vs;
    const float* proj = pdl_fresh(a.proj);
    const float* pw = a.pw + (size_t)h * (RET_CHUNK + 1);
    const int kq = (ks - 8) / 4, vq = (vs - 8) / 4;
    ret_batches<4, RET_STATE_THREADS, RetQuad>(RET_CHUNK, kq, [&](int r, int d) {
        const int t = t0 + min(r, n - 1);
        return ret_quad(a, proj + (size_t)t * a.ps + a.ko + (size_t)h * dk, t, d < dk ? d : 0);
    }, [&](int r, int d, const RetQuad& q) {
        ret_split4(r < n && d < dk ? ret_turn(a, q, d, a.kmul * pw[n - 1 - r]) : ret_zero4(), kh + r * ks + d, kl + r * ks + d);
    });
    ret_batches<8, RET_STATE_THREADS, float4>(RET_CHUNK, vq, [&](int r, int d) {
        return *reinterpret_cast<const float4*>(proj + (size_t)(t0 + min(r, n - 1)) * a.ps + a.vo + (size_t)h * dv + (d < dv ? d : 0));
    }, [&](int r, int d, float4 v) {
        ret_split4(r < n && d < dv ? v : ret_zero4(), vh + r * vs + d, vl + r * vs + d);
    });
    __syncthreads();
    float* U = a.ws + ((size_t)blockIdx.x * a.H + h) * (size_t)dv * dk;
    const int mat = lane >> 3, lr = lane & 7;
    const int mu = (dv + 31) / 32, nu = (dk + 63) / 64;
    const int steps = (n + 15) / 16;                                                // rows of tokens beyond n are zeros
    for (int u = warp; u < mu * nu; u += RET_STATE_THREADS / 32) {
        const int m0 = (u % mu) * 32, n0 = (u / mu) * 64;
        float acc[2][8][4];
#pragma unroll
        for (int i = 0; i < 2; ++i)
#pragma unroll
            for (int j = 0; j < 8; ++j) acc[i][j][0] = acc[i][j][1] = acc[i][j][2] = acc[i][j][3] = 0.f;
        for (int kk = 0; kk < steps; ++kk) {
            uint32_t ah[2][4], al[2][4];
#pragma unroll
            for (int i = 0; i < 2; ++i) {
                const int at = (kk * 16 + (mat >> 1) * 8 + lr) * vs + m0 + i * 16 + (mat & 1) * 8;
                ldmatrix_x4_trans(ah[i], vh + at);
                ldmatrix_x4_trans(al[i], vl + at);
            }
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                uint32_t bh[4], bl[4];
                const int at = (kk * 16 + (mat & 1) * 8 + lr) * ks + n0 + j * 16 + (mat >> 1) * 8;
                ldmatrix_x4_trans(bh, kh + at);
                ldmatrix_x4_trans(bl, kl + at);
#pragma unroll
                for (int i = 0; i < 2; ++i)
#pragma unroll
                    for (int e = 0; e < 2; ++e) {
                        float(&c)[4] = acc[i][2 * j + e];
                        mma_bf16_16816(c, ah[i], bh[2 * e], bh[2 * e + 1]);
                        mma_bf16_16816(c, ah[i], bl[2 * e], bl[2 * e + 1]);
                        mma_bf16_16816(c, al[i], bh[2 * e], bh[2 * e + 1]);
                    }
            }
        }
#pragma unroll
        for (int i = 0; i < 2; ++i)
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const int c = m0 + i * 16 + (lane >> 2) + e * 8;
                if (c >= dv) continue;
#pragma unroll
                for (int j = 0; j < 8; ++j) {
                    const int d = n0 + j * 8 + (lane & 3) * 2;
                    if (d < dk) *reinterpret_cast<float2*>(U + (size_t)c * dk + d) = make_float2(acc[i][j][2 * e], acc[i][j][2 * e + 1]);
                }
            }
    }
}

// a float as its two bf16 terms in one word
__device__ __forceinline__ uint32_t ret_pack(float x) {
    const __nv_bfloat16 h = __float2bfloat16_rn(x), l = __float2bfloat16_rn(x - __bfloat162float(h));
    return (uint32_t)__bfloat16_as_ushort(h) | ((uint32_t)__bfloat16_as_ushort(l) << 16);
}

// Per segment, head and quad of state entries: the state each chunk starts from, over the chunk's U, and the state after
// the last one to the slot.
__global__ void __launch_bounds__(256) retention_carry_kernel(const RetChunks a) {
    pdl_trigger();
    const int seg = blockIdx.z, h = blockIdx.y;
    const int s0 = a.seg_start[seg], qlen = a.seg_start[seg + 1] - s0;
    const int nc = (qlen + RET_CHUNK - 1) / RET_CHUNK, x0 = s0 / RET_CHUNK + seg;
    const int e4 = a.dv * a.dk / 4, i = blockIdx.x * blockDim.x + threadIdx.x;
    const float* pw = a.pw + (size_t)h * (RET_CHUNK + 1);
    const float whole = pw[RET_CHUNK], rest = pw[qlen - (nc - 1) * RET_CHUNK];
    pdl_wait();
    if (i >= e4) return;
    float4* st = reinterpret_cast<float4*>(pdl_fresh(a.state)) + ((size_t)a.slots[seg] * a.H + h) * e4 + i;
    float4* u = reinterpret_cast<float4*>(pdl_fresh(a.ws)) + ((size_t)x0 * a.H + h) * e4 + i;
    const size_t stride = (size_t)a.H * e4;
    float4 s = *st;
    constexpr int AHEAD = 8;
    for (int c0 = 0; c0 < nc; c0 += AHEAD) {
        float4 v[AHEAD];
#pragma unroll
        for (int j = 0; j < AHEAD; ++j) v[j] = u[(size_t)min(c0 + j, nc - 1) * stride];
#pragma unroll
        for (int j = 0; j < AHEAD; ++j) {
            if (c0 + j >= nc) continue;
            *reinterpret_cast<uint4*>(u + (size_t)(c0 + j) * stride) = make_uint4(ret_pack(s.x), ret_pack(s.y), ret_pack(s.z), ret_pack(s.w));
            const float f = c0 + j + 1 < nc ? whole : rest;
            s.x = f * s.x + v[j].x;
            s.y = f * s.y + v[j].y;
            s.z = f * s.z + v[j].z;
            s.w = f * s.w + v[j].w;
        }
    }
    *st = s;
}

constexpr int RET_OUT_THREADS = 128;

// The outputs of one chunk and head.  Warp w owns tokens 16 w .. 16 w + 15 of the chunk; the operand on the other side
// (64 value channels of the incoming state, the chunk's keys, its values) passes through one shared buffer.
template <int DVP>
__global__ void __launch_bounds__(RET_OUT_THREADS, DVP <= 128 ? 3 : 1) retention_chunk_out_kernel(const RetChunks a) {
    pdl_trigger();
    int t0, n;
    ret_chunk(a, blockIdx.x, t0, n);
    if (n <= 0) return;
    pdl_wait();
    extern __shared__ __align__(16) unsigned char raw[];
    const int h = blockIdx.y, dk = a.dk, dv = a.dv, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int dkp = (dk + 15) / 16 * 16, qs = dkp + 8;
    constexpr int VS = DVP + 8;
    const int bs = qs > VS ? qs : VS;
    __nv_bfloat16* qh = reinterpret_cast<__nv_bfloat16*>(raw);
    __nv_bfloat16 *ql = qh + RET_CHUNK * qs, *bh = ql + RET_CHUNK * qs, *bl = bh + RET_CHUNK * bs;
    const float* proj = pdl_fresh(a.proj);
    const float* pw = a.pw + (size_t)h * (RET_CHUNK + 1);
    const int kq = dkp / 4, mat = lane >> 3, lr = lane & 7, row0 = warp * 16;
    const bool mine = row0 < n;                            // this warp has tokens
    // q (is_k 0) or k rows of the chunk, rotated, as two terms
    auto load_rows = [&](int off, float mul, __nv_bfloat16* hi, __nv_bfloat16* lo) {
        ret_batches<4, RET_OUT_THREADS, RetQuad>(RET_CHUNK, kq, [&](int r, int d) {
            const int t = t0 + min(r, n - 1);
            return ret_quad(a, proj + (size_t)t * a.ps + off + (size_t)h * dk, t, d < dk ? d : 0);
        }, [&](int r, int d, const RetQuad& q) {
            ret_split4(r < n && d < dk ? ret_turn(a, q, d, mul) : ret_zero4(), hi + r * qs + d, lo + r * qs + d);
        });
    };
    load_rows(0, 1.f, qh, ql);
    float o[DVP / 8][4];
#pragma unroll
    for (int i = 0; i < DVP / 8; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;

    // S^T q: the incoming state [c][i], 64 value channels at a time
    const uint32_t* sin = reinterpret_cast<const uint32_t*>(pdl_fresh(a.ws)) + ((size_t)blockIdx.x * a.H + h) * (size_t)dv * dk;
    constexpr int SB = DVP < 64 ? DVP : 64;
#pragma unroll
    for (int n0 = 0; n0 < DVP; n0 += SB) {
        if (n0 < dv) {
            ret_batches<8, RET_OUT_THREADS, uint4>(SB, kq, [&](int r, int d) {
                return *reinterpret_cast<const uint4*>(sin + (size_t)min(n0 + r, dv - 1) * dk + (d < dk ? d : 0));
            }, [&](int r, int d, uint4 v) {
                if (n0 + r >= dv || d >= dk) v = make_uint4(0u, 0u, 0u, 0u);
                *reinterpret_cast<uint2*>(bh + r * qs + d) = make_uint2(__byte_perm(v.x, v.y, 0x5410), __byte_perm(v.z, v.w, 0x5410));
                *reinterpret_cast<uint2*>(bl + r * qs + d) = make_uint2(__byte_perm(v.x, v.y, 0x7632), __byte_perm(v.z, v.w, 0x7632));
            });
            __syncthreads();
            if (mine)
                for (int ks = 0; ks < dkp / 16; ++ks) {
                    uint32_t ah[4], al[4];
                    const int at = (row0 + lr + (mat & 1) * 8) * qs + ks * 16 + (mat >> 1) * 8;
                    ldmatrix_x4(ah, qh + at);
                    ldmatrix_x4(al, ql + at);
#pragma unroll
                    for (int np = 0; np < SB / 16; ++np) {
                        uint32_t xh[4], xl[4];
                        const int bt = (np * 16 + (mat >> 1) * 8 + lr) * qs + ks * 16 + (mat & 1) * 8;
                        ldmatrix_x4(xh, bh + bt);
                        ldmatrix_x4(xl, bl + bt);
#pragma unroll
                        for (int e = 0; e < 2; ++e) {
                            float(&c)[4] = o[n0 / 8 + 2 * np + e];
                            mma_bf16_16816(c, ah, xh[2 * e], xh[2 * e + 1]);
                            mma_bf16_16816(c, ah, xl[2 * e], xl[2 * e + 1]);
                            mma_bf16_16816(c, al, xh[2 * e], xh[2 * e + 1]);
                        }
                    }
                }
            __syncthreads();
        }
    }
    const int r0 = row0 + (lane >> 2), r1 = r0 + 8;        // the two tokens this thread holds entries of
    {
        const float f0 = pw[r0 + 1], f1 = pw[r1 + 1];
#pragma unroll
        for (int i = 0; i < DVP / 8; ++i) { o[i][0] *= f0; o[i][1] *= f0; o[i][2] *= f1; o[i][3] *= f1; }
    }
    // scores against the chunk's own keys, decayed by distance
    load_rows(a.ko, a.kmul, bh, bl);
    __syncthreads();
    float s[RET_CHUNK / 8][4];
#pragma unroll
    for (int i = 0; i < RET_CHUNK / 8; ++i) s[i][0] = s[i][1] = s[i][2] = s[i][3] = 0.f;
    if (mine)
        for (int ks = 0; ks < dkp / 16; ++ks) {
            uint32_t ah[4], al[4];
            const int at = (row0 + lr + (mat & 1) * 8) * qs + ks * 16 + (mat >> 1) * 8;
            ldmatrix_x4(ah, qh + at);
            ldmatrix_x4(al, ql + at);
#pragma unroll
            for (int np = 0; np < RET_CHUNK / 16; ++np) {
                if (np > warp) continue;                   // keys after this warp's last token
                uint32_t xh[4], xl[4];
                const int bt = (np * 16 + (mat >> 1) * 8 + lr) * qs + ks * 16 + (mat & 1) * 8;
                ldmatrix_x4(xh, bh + bt);
                ldmatrix_x4(xl, bl + bt);
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    mma_bf16_16816(s[2 * np + e], ah, xh[2 * e], xh[2 * e + 1]);
                    mma_bf16_16816(s[2 * np + e], ah, xl[2 * e], xl[2 * e + 1]);
                    mma_bf16_16816(s[2 * np + e], al, xh[2 * e], xh[2 * e + 1]);
                }
            }
        }
#pragma unroll
    for (int nt = 0; nt < RET_CHUNK / 8; ++nt)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int back = (e < 2 ? r0 : r1) - (nt * 8 + (lane & 3) * 2 + (e & 1));
            s[nt][e] = back >= 0 ? s[nt][e] * pw[back] : 0.f;
        }
    __syncthreads();
    ret_batches<8, RET_OUT_THREADS, float4>(RET_CHUNK, DVP / 4, [&](int r, int d) {
        return *reinterpret_cast<const float4*>(proj + (size_t)(t0 + min(r, n - 1)) * a.ps + a.vo + (size_t)h * dv + (d < dv ? d : 0));
    }, [&](int r, int d, float4 v) {
        ret_split4(r < n && d < dv ? v : ret_zero4(), bh + r * VS + d, bl + r * VS + d);
    });
    __syncthreads();
    if (!mine) return;
#pragma unroll
    for (int kk = 0; kk < RET_CHUNK / 16; ++kk) {
        if (kk > warp) continue;
        uint32_t ph[4], pl[4];
#pragma unroll
        for (int u = 0; u < 4; ++u) {
            const float x0 = s[2 * kk + (u >> 1)][(u & 1) * 2], x1 = s[2 * kk + (u >> 1)][(u & 1) * 2 + 1];
            const __nv_bfloat162 hh = __floats2bfloat162_rn(x0, x1);
            const float2 hf = __bfloat1622float2(hh);
            ph[u] = *reinterpret_cast<const uint32_t*>(&hh);
            pl[u] = pack_bf16(x0 - hf.x, x1 - hf.y);
        }
#pragma unroll
        for (int j = 0; j < DVP / 16; ++j) {
            uint32_t xh[4], xl[4];
            const int bt = (kk * 16 + (mat & 1) * 8 + lr) * VS + j * 16 + (mat >> 1) * 8;
            ldmatrix_x4_trans(xh, bh + bt);
            ldmatrix_x4_trans(xl, bl + bt);
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                mma_bf16_16816(o[2 * j + e], ph, xh[2 * e], xh[2 * e + 1]);
                mma_bf16_16816(o[2 * j + e], ph, xl[2 * e], xl[2 * e + 1]);
                mma_bf16_16816(o[2 * j + e], pl, xh[2 * e], xh[2 * e + 1]);
            }
        }
    }
    // head norm and gate
    float ss[2] = {0.f, 0.f};
#pragma unroll
    for (int i = 0; i < DVP / 8; ++i) {
        ss[0] += o[i][0] * o[i][0] + o[i][1] * o[i][1];
        ss[1] += o[i][2] * o[i][2] + o[i][3] * o[i][3];
    }
#pragma unroll
    for (int e = 0; e < 2; ++e) {
        ss[e] += __shfl_xor_sync(0xffffffffu, ss[e], 1);
        ss[e] += __shfl_xor_sync(0xffffffffu, ss[e], 2);
        const int r = e ? r1 : r0;
        if (r >= n) continue;
        const float inv = 1.f / sqrtf(ss[e] / (float)dv + a.eps);
        const float* gate = proj + (size_t)(t0 + r) * a.ps + a.go + (size_t)h * dv;
        __nv_bfloat16* dst = a.out + (size_t)(t0 + r) * a.os + (size_t)h * dv;
#pragma unroll
        for (int i = 0; i < DVP / 8; ++i) {
            const int d = i * 8 + (lane & 3) * 2;
            if (d >= dv) continue;
            const float2 gz = *reinterpret_cast<const float2*>(gate + d);
            *reinterpret_cast<uint32_t*>(dst + d) = pack_bf16(o[i][2 * e] * inv * ret_silu(gz.x), o[i][2 * e + 1] * inv * ret_silu(gz.y));
        }
    }
}

template <int DVP> static int launch_chunk_out(const RetChunks& a, int chunks, cudaStream_t stream) {
    const int qs = (a.dk + 15) / 16 * 16 + 8, bs = qs > DVP + 8 ? qs : DVP + 8;
    const size_t smem = (size_t)RET_CHUNK * (2 * qs + 2 * bs) * sizeof(__nv_bfloat16);
    auto kern = retention_chunk_out_kernel<DVP>;
    cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    return (int)launch_kernel(kern, dim3(chunks, a.H), dim3(RET_OUT_THREADS), smem, stream, a);
}

}  // namespace prism

// 1 if the one-token kernel takes these sizes.
PRISM_EXPORT int prism_retention_step_supported(int dk, int dv) { return dk >= 4 && dk % 4 == 0 && dk <= 256 && dv >= 1 && dv <= 4096; }

// 1 if the chunked kernels take these sizes: whole quads everywhere (rot: entries that turn, pairs or halves of them).
PRISM_EXPORT int prism_retention_chunks_supported(int dk, int dv, int rot, int pairs) {
    return dk >= 8 && dk % 8 == 0 && dk <= 256 && dv >= 8 && dv % 8 == 0 && dv <= 256 && rot % (pairs ? 4 : 8) == 0;
}

// proj float32 [T, *] (row stride ps, q at 0, k at ko, v at vo, gate at go), one token per request; freq [rot / 2] (null
// with rot 0), pairs: entries (2i, 2i + 1) turn together instead of halves, amp: a factor on cosine and sine; kmul: a
// factor on k; decay [H]; state [slots, H, dv, dk]; out [T, H dv] of out_dtype.
PRISM_EXPORT int prism_retention_step(const float* proj, long long ps, int ko, int vo, int go, int T, int H, int dk, int dv,
                                      const float* freq, int rot, int pairs, float amp, float kmul, const float* decay,
                                      float* state, const int* positions, const int* slots, float eps, void* out, int out_dtype,
                                      long long os, cudaStream_t stream) {
    using namespace prism;
    if (T <= 0) return 0;
    if (!prism_retention_step_supported(dk, dv) || H < 1 || T > 65535 || rot < 0 || rot > dk || rot % 2 || (rot && freq == nullptr) ||
        (uintptr_t)state % 16)
        return (int)cudaErrorInvalidValue;
    const size_t smem = (size_t)(2 * dk + 3 * dv) * sizeof(float);
    if (smem > 48 * 1024) return (int)cudaErrorInvalidValue;
#define PRISM_RS(TT, L, Q, N)                                                                                                  \
    return (int)launch_kernel(retention_step_kernel<TT, L, Q, N>, dim3(H, T), dim3(RET_STEP_THREADS), smem, stream, proj, ps, ko, vo, \
                              go, H, dk, dv, freq, rot, pairs, amp, kmul, decay, state, positions, slots, eps, (TT*)out, os)
#define PRISM_RS_SIZE(TT)                       \
    do {                                        \
        if (dk <= 32) PRISM_RS(TT, 8, 1, 4);    \
        if (dk <= 64) PRISM_RS(TT, 16, 1, 8);   \
        if (dk <= 128) PRISM_RS(TT, 32, 1, 16); \
        PRISM_RS(TT, 32, 2, 8);                 \
    } while (0)
    if (out_dtype == PRISM_DTYPE_BF16) PRISM_RS_SIZE(__nv_bfloat16);
    PRISM_RS_SIZE(float);
#undef PRISM_RS_SIZE
#undef PRISM_RS
}

// As above for segments of any length, bf16 out; table [T, rot / 2, 2] float32: cosine and sine of position * frequency;
// pw [H, 65]: powers 0 .. 64 of the heads' decays; ws: (T / 64 + S) * H * dv * dk floats.
PRISM_EXPORT int prism_retention_chunks(const float* proj, long long ps, int ko, int vo, int go, int T, int S, int H, int dk, int dv,
                                        const float* table, int rot, int pairs, float amp, float kmul, const float* pw, float* state,
                                        const int* seg_start, const int* slots, float eps, float* ws, void* out, long long os,
                                        cudaStream_t stream) {
    using namespace prism;
    if (T <= 0 || S <= 0) return 0;
    if (!prism_retention_chunks_supported(dk, dv, rot, pairs) || H < 1 || H > 65535 || S > 65535 || rot < 0 || rot > dk ||
        (rot && table == nullptr) || ps % 4 || ko % 4 || vo % 4 || go % 4 || os % 2 || (uintptr_t)proj % 16 || (uintptr_t)table % 16 ||
        (uintptr_t)state % 16 || (uintptr_t)ws % 16 || (uintptr_t)out % 4)
        return (int)cudaErrorInvalidValue;
    RetChunks a;
    a.proj = proj; a.ps = ps; a.ko = ko; a.vo = vo; a.go = go; a.H = H; a.dk = dk; a.dv = dv; a.S = S;
    a.table = reinterpret_cast<const float2*>(table); a.rot = rot; a.pairs = pairs; a.amp = amp; a.kmul = kmul; a.eps = eps; a.pw = pw;
    a.state = state; a.seg_start = seg_start; a.slots = slots; a.ws = ws; a.out = (__nv_bfloat16*)out; a.os = os;
    const int chunks = T / RET_CHUNK + S;
    const int ks = (dk + 63) / 64 * 64 + 8, vs = (dv + 31) / 32 * 32 + 8;
    const size_t smem = (size_t)RET_CHUNK * 2 * (ks + vs) * sizeof(__nv_bfloat16);
    cudaFuncSetAttribute(retention_chunk_state_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    cudaError_t rc = launch_kernel(retention_chunk_state_kernel, dim3(chunks, H), dim3(RET_STATE_THREADS), smem, stream, a);
    if (rc != cudaSuccess) return (int)rc;
    rc = launch_kernel(retention_carry_kernel, dim3((dv * dk / 4 + 255) / 256, H, S), dim3(256), 0, stream, a);
    if (rc != cudaSuccess) return (int)rc;
    if (dv <= 32) return launch_chunk_out<32>(a, chunks, stream);
    if (dv <= 64) return launch_chunk_out<64>(a, chunks, stream);
    if (dv <= 128) return launch_chunk_out<128>(a, chunks, stream);
    return launch_chunk_out<256>(a, chunks, stream);
}
