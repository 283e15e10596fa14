// Sums of outer products under a decay, S <- D S + k v^T, o = S^T q per head, the recurrence of the linear-attention mixers,
// with what lies between a mixer's two projections around it.  Three kinds of decay D:
//
//   DS_HEAD      one constant g per head                        (retention, lightning attention)
//   DS_TOKEN     g_t = exp(-exp(a_log) d_t) per head and token, d_t = softplus(dt_t + bias), and d_t k v^T is added; the
//                read-out has a skip path, o = S^T q + D v      (state-space mixers)
//   DS_CHANNEL   one decay per key channel and token            (gated linear attention)
//
// q, k and v are float32 rows; q and k may be rotated by the token's position (DS_HEAD), all three may go through silu, q and k
// have constant factors.  Several heads may share a q/k head.  S is kept as [slot][head][value channel][key channel], float32.
// The result: o / rms(o) * weight * silu(gate) per head, in the compute dtype, or o itself in float32 for mixers whose norm
// runs over more than one head.
//
//   * prism_decay_step    a step of single tokens: one CTA per (head, request) prepares q, k and the decay (the low-rank
//     product of DS_CHANNEL included), updates the state, reads it out, norms and gates in one launch.  The state of earlier
//     steps is requested before the dependency wait.
//   * prism_decay_chunks  stretches of many tokens, in chunks of 64 (counted from the segment's first token), three
//     launches: what each chunk adds to the state, U = sum_j D_(j+1) .. D_(n-1) k_j v_j^T (all chunks side by side); the state
//     each chunk starts from (a walk over the chunks per state entry, in place over U, and the new state to the slot);
//     the outputs, o_i = (D_0 .. D_i S)^T q_i + sum_{j<=i} (q_i . D_(j+1) .. D_i k_j) v_j.  The products run on
//     tensor cores with both operands as two bf16 terms, x = hi + lo, hi*hi + hi*lo + lo*hi, accumulated in float32: 16
//     mantissa bits of every operand.  Products of decays: a table of powers made on the host (DS_HEAD), or exp of differences
//     of the sums b_i of log decays from the chunk's first token on (the others), always of later minus earlier, so that no
//     factor exceeds one: with a decay per channel a query row meets the keys of an earlier sub-chunk of 16 as q_i exp(b_i - e)
//     and k_j exp(e - b_j), e the sums at that sub-chunk's end.  Inside a sub-chunk the first factor does exceed one; where
//     the decay across it is too strong for that, its scores are formed term by term.
#include "mma_helpers.cuh"

#define PRISM_DS_HEAD 0
#define PRISM_DS_TOKEN 1
#define PRISM_DS_CHANNEL 2

namespace prism {

constexpr int DS_CHUNK = 64;
constexpr int DS_SUB = 16;                 // a sub-chunk: the rows a pair of warps of the output kernel owns
constexpr float DS_LEAST_LOG2 = -160.f;    // a decay below 2^-160 is zero in float32 (as is one below e^-160): its logarithm need not go lower,
                                           // which keeps the sums, and so the digits of their differences, small
constexpr float DS_MAX_SPAN = 80.f;        // the most a sub-chunk's log decays (in units of ln 2) may sum to before its scores are formed
                                           // term by term

__device__ __forceinline__ float ds_silu(float z) { return z / (1.f + expf(-z)); }
// 2^x by the special-function unit (results below 2^-126 are zero)
__device__ __forceinline__ float ds_exp2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
// log2 of sigmoid(z), with e = 2^-|z|/ln 2: where e is small log2(1 + e) comes from the series of ln(1 + e), which keeps its
// leading digits
__device__ __forceinline__ float ds_log2_sigmoid(float z) {
    const float y = -fabsf(z) * 1.44269504f, e = ds_exp2(y);
    float l;
    asm("lg2.approx.ftz.f32 %0, %1;" : "=f"(l) : "f"(1.f + e));
    const float series = e * (1.f - e * (0.5f - e * (0.33333333f - e * (0.25f - e * 0.2f)))) * 1.44269504f;
    return (z < 0.f ? y : 0.f) - (e < 0.05f ? series : l);
}
__device__ __forceinline__ float ds_softplus(float z) { return z > 20.f ? z : log1pf(expf(z)); }

// ---------------------------------------------------------------------------------------------------------
// one token per request
// ---------------------------------------------------------------------------------------------------------
struct DecayStep {
    const float *q, *k, *v;  // rows with stride xs; head h: q and k at (h / rep) dk, v at h dv
    long long xs;
    int H, rep, dk, dv, act; // act: q, k and v through silu
    const float* freq;       // rotation of q and k (rot 0: none)
    int rot, pairs;
    float amp, qmul, kmul;
    const float* decay;      // DS_HEAD: [H]
    const float* dt;         // DS_TOKEN: [T, H] (row stride dts)
    long long dts;
    const void *dt_bias, *a_log, *skip;
    int dt_bias_bf16, a_log_bf16, skip_bf16;
    const float* low;        // DS_CHANNEL: [T, R] (row stride ls); w = sigmoid(low a2t + a2_bias)^rate, a2t [R, H dk]
    long long ls;
    int R;
    const float* a2t;
    const void* a2_bias;
    int a2_bias_bf16;
    float rate;
    float* state;
    const int *positions, *slots;
    const float* gate;       // [T, H dv] (row stride gs), or null: o itself
    long long gs;
    const void* weight;      // [dv], or null
    int weight_bf16;
    float eps;
    void* out;
    long long os;
};

// LANES neighbouring lanes share a column of S (its dk entries, QPL quads a lane), a warp takes 32 / LANES columns at a
// time and NB times as many in one batch, all of whose loads are in flight together.
constexpr int DS_STEP_THREADS = 256;
constexpr int DS_STEP_RANK = 16;           // rows of the low-rank product's second matrix that are asked for before the wait

template <typename T, int LANES, int QPL, int NB, int DECAY>
__global__ void __launch_bounds__(DS_STEP_THREADS) decay_step_kernel(const DecayStep a) {
    pdl_trigger();
    extern __shared__ __align__(16) float sm[];        // q [dk] | k [dk] | w [dk] | v [dv] | gate [dv] | o [dv]
    __shared__ float scratch[33];
    const int dk = a.dk, dv = a.dv;
    float *q_s = sm, *k_s = sm + dk, *w_s = k_s + dk, *v_s = w_s + dk, *g_s = v_s + dv, *o_s = g_s + dv;
    const int h = blockIdx.x, t = blockIdx.y;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    constexpr int CPW = 32 / LANES, WARPS = DS_STEP_THREADS / 32;
    const int part = lane % LANES, sub = lane / LANES;
    float* st = a.state + ((size_t)a.slots[t] * a.H + h) * (size_t)dv * dk;
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
    const float pos = (float)a.positions[t];
    float g = DECAY == PRISM_DS_HEAD ? a.decay[h] : 0.f, rate = 0.f, bias = 0.f, skip = 0.f;
    float aw[DECAY == PRISM_DS_CHANNEL ? DS_STEP_RANK : 1];
    if (DECAY == PRISM_DS_TOKEN) {
        rate = expf(load_param(a.a_log, a.a_log_bf16, h));
        bias = load_param(a.dt_bias, a.dt_bias_bf16, h);
        skip = a.skip != nullptr ? load_param(a.skip, a.skip_bf16, h) : 0.f;
    }
    if (DECAY == PRISM_DS_CHANNEL && threadIdx.x < dk) {
        bias = a.a2_bias != nullptr ? load_param(a.a2_bias, a.a2_bias_bf16, (size_t)h * dk + threadIdx.x) : 0.f;
#pragma unroll
        for (int r = 0; r < DS_STEP_RANK; ++r) aw[r] = r < a.R ? a.a2t[(size_t)r * a.H * dk + (size_t)h * dk + threadIdx.x] : 0.f;
    }
    pdl_wait();
    const size_t row = (size_t)t * a.xs;
    const float* q_row = pdl_fresh(a.q) + row + (size_t)(h / a.rep) * dk;
    const float* k_row = pdl_fresh(a.k) + row + (size_t)(h / a.rep) * dk;
    const float* v_row = pdl_fresh(a.v) + row + (size_t)h * dv;
    float kmul = a.kmul;
    if (DECAY == PRISM_DS_TOKEN) {
        const float d = ds_softplus(pdl_fresh(a.dt)[(size_t)t * a.dts + h] + bias);
        g = expf(-rate * d);
        kmul *= d;
    }
    const int half = a.rot >> 1;
    for (int i = threadIdx.x; i < 2 * dk; i += DS_STEP_THREADS) {
        const bool is_k = i >= dk;
        const int d = is_k ? i - dk : i;
        const float* x = is_k ? k_row : q_row;
        float y = x[d];
        if (a.act) y = ds_silu(y);
        if (DECAY == PRISM_DS_HEAD && d < a.rot) {
            const int e = a.pairs ? (d ^ 1) : (d < half ? d + half : d - half);
            const bool second = a.pairs ? (d & 1) : d >= half;
            const float z = a.act ? ds_silu(x[e]) : x[e];
            float sn, cs;
            sincosf(pos * a.freq[a.pairs ? d >> 1 : (second ? e : d)], &sn, &cs);
            sn *= a.amp;
            cs *= a.amp;
            y = second ? y * cs + z * sn : y * cs - z * sn;
        }
        sm[i] = y * (is_k ? kmul : a.qmul);
    }
    if (DECAY == PRISM_DS_CHANNEL) {
        const float* low = pdl_fresh(a.low) + (size_t)t * a.ls;
        if (threadIdx.x < dk) {
            float z = 0.f;
#pragma unroll
            for (int r = 0; r < DS_STEP_RANK; ++r)
                if (r < a.R) z += low[r] * aw[r];
            for (int r = DS_STEP_RANK; r < a.R; ++r) z += low[r] * a.a2t[(size_t)r * a.H * dk + (size_t)h * dk + threadIdx.x];
            w_s[threadIdx.x] = expf(-a.rate * ds_softplus(-(z + bias)));
        }
    }
    const float* gate = a.gate != nullptr ? pdl_fresh(a.gate) + (size_t)t * a.gs + (size_t)h * dv : nullptr;
    for (int c = threadIdx.x; c < dv; c += DS_STEP_THREADS) {
        v_s[c] = a.act ? ds_silu(v_row[c]) : v_row[c];
        if (gate != nullptr) g_s[c] = gate[c];
    }
    __syncthreads();
    float4 qq[QPL], kk[QPL], ww[QPL];
#pragma unroll
    for (int m = 0; m < QPL; ++m) {
        const int i = 4 * (part + LANES * m);
        qq[m] = i < dk ? *reinterpret_cast<const float4*>(q_s + i) : make_float4(0.f, 0.f, 0.f, 0.f);
        kk[m] = i < dk ? *reinterpret_cast<const float4*>(k_s + i) : make_float4(0.f, 0.f, 0.f, 0.f);
        ww[m] = DECAY != PRISM_DS_CHANNEL ? make_float4(g, g, g, g)
                                          : (i < dk ? *reinterpret_cast<const float4*>(w_s + i) : make_float4(0.f, 0.f, 0.f, 0.f));
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
                s.x = ww[m].x * s.x + kk[m].x * v;
                s.y = ww[m].y * s.y + kk[m].y * v;
                s.z = ww[m].z * s.z + kk[m].z * v;
                s.w = ww[m].w * s.w + kk[m].w * v;
                o += (s.x * qq[m].x + s.y * qq[m].y) + (s.z * qq[m].z + s.w * qq[m].w);
                const int i = 4 * (part + LANES * m);
                if (ok && i < dk) *reinterpret_cast<float4*>(st + (size_t)c * dk + i) = s;
            }
#pragma unroll
            for (int w = LANES / 2; w > 0; w >>= 1) o += __shfl_xor_sync(0xffffffffu, o, w);
            if (ok && part == 0) o_s[c] = DECAY == PRISM_DS_TOKEN ? o + skip * v : o;
        }
    }
    __syncthreads();
    if (gate == nullptr) {
        float* dst = reinterpret_cast<float*>(a.out) + (size_t)t * a.os + (size_t)h * dv;
        for (int c = threadIdx.x; c < dv; c += DS_STEP_THREADS) dst[c] = o_s[c];
        return;
    }
    float ss = 0.f;
    for (int c = threadIdx.x; c < dv; c += DS_STEP_THREADS) ss += o_s[c] * o_s[c];
    ss = block_sum(ss, scratch);
    const float inv = 1.f / sqrtf(ss / (float)dv + a.eps);
    T* dst = reinterpret_cast<T*>(a.out) + (size_t)t * a.os + (size_t)h * dv;
    for (int c = threadIdx.x; c < dv; c += DS_STEP_THREADS) {
        const float w = a.weight != nullptr ? load_param(a.weight, a.weight_bf16, c) : 1.f;
        dst[c] = from_float<T>(o_s[c] * inv * w * ds_silu(g_s[c]));
    }
}

// ---------------------------------------------------------------------------------------------------------
// chunks
// ---------------------------------------------------------------------------------------------------------
struct DecayChunks {
    const float *q, *k, *v;  // rows with stride xs; head h: q and k at (h / rep) dk, v at h dv
    long long xs;
    int H, rep, dk, dv, S, act;
    const float2* table;     // [T, half] cosine and sine of position * frequency, or null (no rotation)
    int rot, pairs;
    float amp, qmul, kmul;
    const float* pw;         // DS_HEAD: [H, DS_CHUNK + 1] powers of the heads' decays
    const float* dt;         // DS_TOKEN: [T, H] (row stride dts)
    long long dts;
    const void *dt_bias, *a_log, *skip;
    int dt_bias_bf16, a_log_bf16, skip_bf16;
    const float* low;        // DS_CHANNEL: [T, R] (row stride ls); log decay = rate log sigmoid(low a2t + a2_bias), a2t [R, H dk]
    long long ls;
    int R;
    const float* a2t;
    const void* a2_bias;
    int a2_bias_bf16;
    float rate;
    float* cum;              // DS_CHANNEL: [T, H dk]: the first kernel leaves the log decays' sums from each chunk's start on here,
                             // in units of ln 2
    float* state;            // [slots, H, dv, dk]
    const int* seg_start;
    const int* slots;
    float* ws;               // [chunks, H, dv, dk]: U, then the incoming state as two bf16 terms in one word
    float* fac;              // DS_TOKEN: [chunks, H] the decay across a chunk
    const float* gate;       // [T, H dv] (row stride gs), or null: o itself
    long long gs;
    const void* weight;      // [dv], or null
    int weight_bf16;
    float eps;
    void* out;               // bf16 (float32 without a gate)
    long long os;
};

// Chunk x of the step: its segment, first token and length.  The chunks of segment s are numbered from
// seg_start[s] / 64 + s on, so every segment has room for its own; numbers in between have no chunk (n <= 0).
__device__ __forceinline__ void ds_chunk(const DecayChunks& a, int x, int& t0, int& n) {
    int lo = 0, hi = a.S - 1;
    while (lo < hi) {
        const int mid = (lo + hi + 1) >> 1;
        if (a.seg_start[mid] / DS_CHUNK + mid <= x) lo = mid; else hi = mid - 1;
    }
    const int s0 = a.seg_start[lo];
    t0 = s0 + (x - (s0 / DS_CHUNK + lo)) * DS_CHUNK;
    n = min(DS_CHUNK, a.seg_start[lo + 1] - t0);
}

// four floats as hi and lo bf16 terms, at the same place of two arrays
__device__ __forceinline__ void ds_split4(float4 v, __nv_bfloat16* hi, __nv_bfloat16* lo) {
    const __nv_bfloat162 h0 = __floats2bfloat162_rn(v.x, v.y), h1 = __floats2bfloat162_rn(v.z, v.w);
    const float2 f0 = __bfloat1622float2(h0), f1 = __bfloat1622float2(h1);
    *reinterpret_cast<uint2*>(hi) = make_uint2(*reinterpret_cast<const uint32_t*>(&h0), *reinterpret_cast<const uint32_t*>(&h1));
    *reinterpret_cast<uint2*>(lo) = make_uint2(pack_bf16(v.x - f0.x, v.y - f0.y), pack_bf16(v.z - f1.x, v.w - f1.y));
}

// What a rotated quad is made of: the quad at column d (a multiple of 4) of token t's q or k, its partner, and the cosines
// and sines.  Loads only, all of them in any case (from a legal place where they are not needed), so that a batch of
// quads has all its loads on their way together; the arithmetic follows in ds_turn.
struct DsRotQuad {
    float4 u, w, c0, c1;
};
__device__ __forceinline__ DsRotQuad ds_rot_quad(const DecayChunks& a, const float* __restrict__ x, int t, int d) {
    const int half = a.rot >> 1;
    const bool turns = d < a.rot, second = d >= half;
    const int e = !turns || a.pairs ? d : (second ? d - half : d + half);
    const int ti = !turns ? 0 : (a.pairs ? d >> 1 : (second ? d - half : d));
    const float* tb = a.rot > 0 ? reinterpret_cast<const float*>(a.table + (size_t)t * half + ti) : x;
    DsRotQuad q;
    q.u = *reinterpret_cast<const float4*>(x + d);
    q.w = *reinterpret_cast<const float4*>(x + e);
    q.c0 = *reinterpret_cast<const float4*>(tb);
    q.c1 = *reinterpret_cast<const float4*>(tb + (a.pairs || a.rot == 0 ? 0 : 4));
    return q;
}
// the quad, rotated and times f
__device__ __forceinline__ float4 ds_turn(const DecayChunks& a, const DsRotQuad& q, int d, float f) {
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
// a quad without rotation, through the activation where there is one, times f
__device__ __forceinline__ float4 ds_turn(const DecayChunks& a, float4 q, int, float f) {
    if (a.act) q = make_float4(ds_silu(q.x), ds_silu(q.y), ds_silu(q.z), ds_silu(q.w));
    return make_float4(q.x * f, q.y * f, q.z * f, q.w * f);
}
template <bool ROT> struct DsQuad { using type = float4; };
template <> struct DsQuad<true> { using type = DsRotQuad; };
template <bool ROT> __device__ __forceinline__ typename DsQuad<ROT>::type ds_quad(const DecayChunks& a, const float* __restrict__ x, int t, int d) {
    if constexpr (ROT) return ds_rot_quad(a, x, t, d);
    else return *reinterpret_cast<const float4*>(x + d);
}

// DS_TOKEN: of one chunk and head, by the first warp: step sizes into d [64] and the sums of the log decays, from the chunk's
// first token up to each, into b [64]; rows beyond n: step size 0, sums as at the last token.
__device__ __forceinline__ void ds_token_sums(const DecayChunks& a, int h, int t0, int n, float* b, float* d) {
    const int lane = threadIdx.x;
    if (lane >= 32) return;
    const float rate = expf(load_param(a.a_log, a.a_log_bf16, h)), bias = load_param(a.dt_bias, a.dt_bias_bf16, h);
    const float* dt = pdl_fresh(a.dt);
    float x[2];
#pragma unroll
    for (int i = 0; i < 2; ++i) {
        const int r = lane + 32 * i;
        const float s = r < n ? ds_softplus(dt[(size_t)(t0 + r) * a.dts + h] + bias) : 0.f;
        d[r] = s;
        x[i] = fmaxf(-rate * s, DS_LEAST_LOG2);
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float y = __shfl_up_sync(0xffffffffu, x[i], o);
            if (lane >= o) x[i] += y;
        }
    }
    x[1] += __shfl_sync(0xffffffffu, x[0], 31);
    b[lane] = x[0];
    b[lane + 32] = x[1];
}

__device__ __forceinline__ float4 ds_zero4() { return make_float4(0.f, 0.f, 0.f, 0.f); }

// The quads of a [rows, 4 cols] tile, dealt out to the threads in turn, in batches of U: all of a batch's loads are on their
// way before its first store (past the end the tile's last row is loaded again instead of branching).  A thread walks its
// (row, quad) pairs by adding, it divides once.
template <int U, int THREADS, typename V, typename Load, typename Store>
__device__ __forceinline__ void ds_batches(int rows, int cols, Load load, Store store) {
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

constexpr int DS_STATE_THREADS = 256;

// U[c][i] = sum_j (D_(j+1) .. D_(n-1))[i] v_j[c] k_j[i] of one chunk and head: m = c, n = i, k = j.
template <int DECAY, bool ROT>
__global__ void __launch_bounds__(DS_STATE_THREADS) decay_chunk_state_kernel(const DecayChunks a) {
    pdl_trigger();
    int t0, n;
    ds_chunk(a, blockIdx.x, t0, n);
    if (n <= 0) return;
    pdl_wait();
    extern __shared__ __align__(16) unsigned char raw[];
    const int h = blockIdx.y, dk = a.dk, dv = a.dv, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int ks = (dk + 63) / 64 * 64 + 8, vs = (dv + 31) / 32 * 32 + 8;          // whole units of the warps below, zeros beyond
    __nv_bfloat16* kh = reinterpret_cast<__nv_bfloat16*>(raw);
    __nv_bfloat16 *kl = kh + DS_CHUNK * ks, *vh = kl + DS_CHUNK * ks, *vl = vh + DS_CHUNK * vs;
    __shared__ float s_b[DS_CHUNK], s_d[DS_CHUNK];             // DS_TOKEN
    __shared__ float s_part[DS_STATE_THREADS];                  // DS_CHANNEL
    const float* kx = pdl_fresh(a.k) + (size_t)(h / a.rep) * dk;
    const float* vx = pdl_fresh(a.v) + (size_t)h * dv;
    const float* pw = DECAY == PRISM_DS_HEAD ? a.pw + (size_t)h * (DS_CHUNK + 1) : nullptr;
    const int kq = (ks - 8) / 4, vq = (vs - 8) / 4;
    if (DECAY == PRISM_DS_TOKEN) {
        ds_token_sums(a, h, t0, n, s_b, s_d);
        __syncthreads();
        if (tid == 0) a.fac[(size_t)blockIdx.x * a.H + h] = expf(s_b[DS_CHUNK - 1]);
    }
    if (DECAY == PRISM_DS_CHANNEL) {
        // a thread owns one key channel of a run of rows: first the runs' sums, then the sums up to each row
        const int dkw = (dk + 31) / 32 * 32, runs = DS_STATE_THREADS / dkw, per = (DS_CHUNK + runs - 1) / runs;
        const int g = tid / dkw, d = tid - g * dkw, r0 = g * per, r1 = min(n, r0 + per);
        const bool on = g < runs && d < dk;
        float* cum = pdl_fresh(a.cum) + (size_t)t0 * a.H * dk + (size_t)h * dk + d;
        const size_t cs = (size_t)a.H * dk;
        float sum = 0.f;
        constexpr int U = 8;
        {
            // the chunk's low-rank rows lie where the values' tile will be; eight tokens' products side by side
            float* s_low = reinterpret_cast<float*>(vh);
            const int RT = min(a.R, vs);                                  // entries of a row that fit (all of them but for large ranks)
            const float* low = pdl_fresh(a.low) + (size_t)t0 * a.ls;
            for (int i = tid; i < DS_CHUNK * RT; i += DS_STATE_THREADS) {
                const int r = i / RT, c = i - r * RT;
                s_low[c * DS_CHUNK + r] = r < n ? low[(size_t)r * a.ls + c] : 0.f;
            }
            __syncthreads();
            const float* w2 = a.a2t + (size_t)h * dk + d;
            const float bias = on && a.a2_bias != nullptr ? load_param(a.a2_bias, a.a2_bias_bf16, (size_t)h * dk + d) : 0.f;
            float wr[DS_STEP_RANK];
#pragma unroll
            for (int c = 0; c < DS_STEP_RANK; ++c) wr[c] = on && c < RT ? w2[(size_t)c * cs] : 0.f;
            if (on)
                for (int r = r0; r < r1; r += U) {
                    float z[U];
#pragma unroll
                    for (int u = 0; u < U; ++u) z[u] = bias;
                    auto add = [&](int c, float w) {
                        const float4 x0 = *reinterpret_cast<const float4*>(s_low + c * DS_CHUNK + r);
                        const float4 x1 = *reinterpret_cast<const float4*>(s_low + c * DS_CHUNK + r + 4);
                        z[0] += w * x0.x; z[1] += w * x0.y; z[2] += w * x0.z; z[3] += w * x0.w;
                        z[4] += w * x1.x; z[5] += w * x1.y; z[6] += w * x1.z; z[7] += w * x1.w;
                    };
#pragma unroll
                    for (int c = 0; c < DS_STEP_RANK; ++c)
                        if (c < RT) add(c, wr[c]);
                    for (int c = DS_STEP_RANK; c < RT; ++c) add(c, w2[(size_t)c * cs]);
                    for (int c = RT; c < a.R; ++c) {
                        const float w = w2[(size_t)c * cs];
#pragma unroll
                        for (int u = 0; u < U; ++u)
                            if (r + u < r1) z[u] += w * low[(size_t)(r + u) * a.ls + c];
                    }
#pragma unroll
                    for (int u = 0; u < U; ++u)
                        if (r + u < r1) {
                            sum += fmaxf(a.rate * ds_log2_sigmoid(z[u]), DS_LEAST_LOG2);
                            cum[(size_t)(r + u) * cs] = sum;                 // so far: from the run's first row on
                        }
                }
        }
        s_part[tid] = sum;
        __syncthreads();
        if (on) {
            float before = 0.f, total = 0.f;
            for (int i = 0; i < runs; ++i) {
                const float s = s_part[i * dkw + d];
                if (i < g) before += s;
                total += s;
            }
            for (int r = r0; r < min(DS_CHUNK, r0 + per); r += U) {
                float x[U], y[U];
#pragma unroll
                for (int u = 0; u < U; ++u) {
                    const bool in = r + u < r1;
                    x[u] = in ? cum[(size_t)(r + u) * cs] : 0.f;
                    y[u] = in ? kx[(size_t)(t0 + r + u) * a.xs + d] : 0.f;
                }
#pragma unroll
                for (int u = 0; u < U; ++u) {
                    if (r + u >= min(DS_CHUNK, r0 + per)) continue;
                    const float acc = before + x[u];
                    if (r + u < r1) cum[(size_t)(r + u) * cs] = acc;
                    const float w = r + u < r1 ? (a.act ? ds_silu(y[u]) : y[u]) * a.kmul * ds_exp2(total - acc) : 0.f;
                    const __nv_bfloat16 hi = __float2bfloat16_rn(w);
                    kh[(r + u) * ks + d] = hi;
                    kl[(r + u) * ks + d] = __float2bfloat16_rn(w - __bfloat162float(hi));
                }
            }
        }
        for (int i = tid; i < DS_CHUNK * (ks - 8 - dk); i += DS_STATE_THREADS) {        // columns beyond dk
            const int r = i / (ks - 8 - dk), c = dk + i - r * (ks - 8 - dk);
            kh[r * ks + c] = kl[r * ks + c] = __float2bfloat16_rn(0.f);
        }
    } else {
        ds_batches<ROT ? 4 : 8, DS_STATE_THREADS, typename DsQuad<ROT>::type>(DS_CHUNK, kq, [&](int r, int d) {
            const int t = t0 + min(r, n - 1);
            return ds_quad<ROT>(a, kx + (size_t)t * a.xs, t, d < dk ? d : 0);
        }, [&](int r, int d, const typename DsQuad<ROT>::type& q) {
            if (r < n && d < dk) {
                const float w = DECAY == PRISM_DS_HEAD ? pw[n - 1 - r] : expf(s_b[n - 1] - s_b[r]) * s_d[r];
                ds_split4(ds_turn(a, q, d, a.kmul * w), kh + r * ks + d, kl + r * ks + d);
            } else {
                ds_split4(ds_zero4(), kh + r * ks + d, kl + r * ks + d);
            }
        });
    }
    ds_batches<8, DS_STATE_THREADS, float4>(DS_CHUNK, vq, [&](int r, int d) {
        return *reinterpret_cast<const float4*>(vx + (size_t)(t0 + min(r, n - 1)) * a.xs + (d < dv ? d : 0));
    }, [&](int r, int d, float4 v) {
        ds_split4(r < n && d < dv ? (ROT ? v : ds_turn(a, v, d, 1.f)) : ds_zero4(), vh + r * vs + d, vl + r * vs + d);
    });
    __syncthreads();
    float* U = a.ws + ((size_t)blockIdx.x * a.H + h) * (size_t)dv * dk;
    const int mat = lane >> 3, lr = lane & 7;
    const int mu = (dv + 31) / 32, nu = (dk + 63) / 64;
    const int steps = (n + 15) / 16;                                                // rows of tokens beyond n are zeros
    for (int u = warp; u < mu * nu; u += DS_STATE_THREADS / 32) {
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
__device__ __forceinline__ uint32_t ds_pack(float x) {
    const __nv_bfloat16 h = __float2bfloat16_rn(x), l = __float2bfloat16_rn(x - __bfloat162float(h));
    return (uint32_t)__bfloat16_as_ushort(h) | ((uint32_t)__bfloat16_as_ushort(l) << 16);
}

// Per segment, head and quad of state entries: the state each chunk starts from, over the chunk's U, and the state after
// the last one to the slot.
template <int DECAY>
__global__ void __launch_bounds__(256) decay_carry_kernel(const DecayChunks a) {
    pdl_trigger();
    const int seg = blockIdx.z, h = blockIdx.y;
    const int s0 = a.seg_start[seg], qlen = a.seg_start[seg + 1] - s0;
    const int nc = (qlen + DS_CHUNK - 1) / DS_CHUNK, x0 = s0 / DS_CHUNK + seg;
    const int e4 = a.dv * a.dk / 4, i = blockIdx.x * blockDim.x + threadIdx.x;
    float whole = 0.f, rest = 0.f;
    if (DECAY == PRISM_DS_HEAD) {
        const float* pw = a.pw + (size_t)h * (DS_CHUNK + 1);
        whole = pw[DS_CHUNK];
        rest = pw[qlen - (nc - 1) * DS_CHUNK];
    }
    pdl_wait();
    if (i >= e4) return;
    const float* fac = DECAY == PRISM_DS_TOKEN ? pdl_fresh((const float*)a.fac) + (size_t)x0 * a.H + h : nullptr;
    const float* cum = DECAY == PRISM_DS_CHANNEL ? pdl_fresh((const float*)a.cum) + (size_t)h * a.dk + (4 * i) % a.dk : nullptr;
    float4* st = reinterpret_cast<float4*>(pdl_fresh(a.state)) + ((size_t)a.slots[seg] * a.H + h) * e4 + i;
    float4* u = reinterpret_cast<float4*>(pdl_fresh(a.ws)) + ((size_t)x0 * a.H + h) * e4 + i;
    const size_t stride = (size_t)a.H * e4;
    float4 s = *st;
    constexpr int AHEAD = 8;
    for (int c0 = 0; c0 < nc; c0 += AHEAD) {
        float4 v[AHEAD], w[AHEAD];
#pragma unroll
        for (int j = 0; j < AHEAD; ++j) {
            const int c = min(c0 + j, nc - 1);
            v[j] = u[(size_t)c * stride];
            if (DECAY == PRISM_DS_TOKEN) w[j].x = fac[(size_t)c * a.H];
            if (DECAY == PRISM_DS_CHANNEL)       // the sums at the chunk's last token
                w[j] = *reinterpret_cast<const float4*>(cum + (size_t)(s0 + min((c + 1) * DS_CHUNK, qlen) - 1) * a.H * a.dk);
        }
#pragma unroll
        for (int j = 0; j < AHEAD; ++j) {
            if (c0 + j >= nc) continue;
            *reinterpret_cast<uint4*>(u + (size_t)(c0 + j) * stride) = make_uint4(ds_pack(s.x), ds_pack(s.y), ds_pack(s.z), ds_pack(s.w));
            if (DECAY == PRISM_DS_CHANNEL) {
                w[j] = make_float4(ds_exp2(w[j].x), ds_exp2(w[j].y), ds_exp2(w[j].z), ds_exp2(w[j].w));
            } else {
                const float f = DECAY == PRISM_DS_TOKEN ? w[j].x : (c0 + j + 1 < nc ? whole : rest);
                w[j] = make_float4(f, f, f, f);
            }
            s.x = w[j].x * s.x + v[j].x;
            s.y = w[j].y * s.y + v[j].y;
            s.z = w[j].z * s.z + v[j].z;
            s.w = w[j].w * s.w + v[j].w;
        }
    }
    *st = s;
}

constexpr int DS_OUT_THREADS = 256;

// The outputs of one chunk and head.  Warps w and w + 4 own tokens 16 w .. 16 w + 15 of the chunk and share their work - every
// other k-step against the incoming state, every other sub-chunk of keys - and add up their sums at the end; the operand on
// the other side (64 value channels of the incoming state, the chunk's keys, its values) passes through one shared buffer.  ROT:
// rotated queries and keys, a head norm without weight and a gate behind it.
template <int DVP, int DECAY, bool ROT>
__global__ void __launch_bounds__(DS_OUT_THREADS, DVP <= 128 ? 2 : 1)
decay_chunk_out_kernel(const DecayChunks a) {
    pdl_trigger();
    int t0, n;
    ds_chunk(a, blockIdx.x, t0, n);
    if (n <= 0) return;
    pdl_wait();
    extern __shared__ __align__(16) unsigned char raw[];
    __shared__ float s_b[DS_CHUNK], s_d[DS_CHUNK];       // DS_TOKEN
    const int h = blockIdx.y, dk = a.dk, dv = a.dv, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int dkp = (dk + 15) / 16 * 16, qs = dkp + 8;
    constexpr int VS = DVP + 8;
    constexpr bool CH = DECAY == PRISM_DS_CHANNEL;
    const int bs = qs > VS ? qs : VS;
    // q as two terms, or with a decay per channel q and the sums of the log decays in float32 (every use has factors of its own)
    __nv_bfloat16* qh = reinterpret_cast<__nv_bfloat16*>(raw);
    __nv_bfloat16* ql = qh + DS_CHUNK * qs;
    float* qf = reinterpret_cast<float*>(raw);
    float* bf = qf + DS_CHUNK * qs;
    __nv_bfloat16* bh = CH ? reinterpret_cast<__nv_bfloat16*>(bf + DS_CHUNK * qs) : ql + DS_CHUNK * qs;
    __nv_bfloat16* bl = bh + DS_CHUNK * bs;
    const float* qx = pdl_fresh(a.q) + (size_t)(h / a.rep) * dk;
    const float* kx = pdl_fresh(a.k) + (size_t)(h / a.rep) * dk;
    const float* vx = pdl_fresh(a.v) + (size_t)h * dv;
    const float* pw = DECAY == PRISM_DS_HEAD ? a.pw + (size_t)h * (DS_CHUNK + 1) : nullptr;
    const int kq = dkp / 4, mat = lane >> 3, lr = lane & 7, rw = warp & 3, grp = warp >> 2, row0 = rw * DS_SUB;
    const bool mine = row0 < n;                            // this warp has tokens
    if (DECAY == PRISM_DS_TOKEN) ds_token_sums(a, h, t0, n, s_b, s_d);       // read behind the barriers below
    // q or k rows of the chunk, prepared, as two terms
    auto load_rows = [&](const float* x, float mul, __nv_bfloat16* hi, __nv_bfloat16* lo) {
        ds_batches<ROT ? 2 : 4, DS_OUT_THREADS, typename DsQuad<ROT>::type>(DS_CHUNK, kq, [&](int r, int d) {
            const int t = t0 + min(r, n - 1);
            return ds_quad<ROT>(a, x + (size_t)t * a.xs, t, d < dk ? d : 0);
        }, [&](int r, int d, const typename DsQuad<ROT>::type& q) {
            ds_split4(r < n && d < dk ? ds_turn(a, q, d, mul) : ds_zero4(), hi + r * qs + d, lo + r * qs + d);
        });
    };
    if constexpr (CH) {
        const float* cum = pdl_fresh((const float*)a.cum) + (size_t)h * dk;
        ds_batches<4, DS_OUT_THREADS, float4>(DS_CHUNK, kq, [&](int r, int d) {
            return *reinterpret_cast<const float4*>(qx + (size_t)(t0 + min(r, n - 1)) * a.xs + (d < dk ? d : 0));
        }, [&](int r, int d, const float4& q) {
            *reinterpret_cast<float4*>(qf + r * qs + d) = r < n && d < dk ? ds_turn(a, q, d, a.qmul) : ds_zero4();
        });
        ds_batches<4, DS_OUT_THREADS, float4>(DS_CHUNK, kq, [&](int r, int d) {       // rows beyond n: the last token's
            return *reinterpret_cast<const float4*>(cum + (size_t)(t0 + min(r, n - 1)) * a.H * dk + (d < dk ? d : 0));
        }, [&](int r, int d, const float4& q) { *reinterpret_cast<float4*>(bf + r * qs + d) = d < dk ? q : ds_zero4(); });
    } else {
        load_rows(qx, a.qmul, qh, ql);
    }
    // this warp's query rows at k-step ks as two terms; with a decay per channel times exp(b - ref) (ref null: exp(b))
    auto q_frag = [&](int ks, const float* ref, uint32_t (&ah)[4], uint32_t (&al)[4]) {
        if constexpr (CH) {
#pragma unroll
            for (int u = 0; u < 4; ++u) {
                const int c = ks * 16 + (lane & 3) * 2 + (u >> 1) * 8, at = (row0 + (lane >> 2) + (u & 1) * 8) * qs + c;
                const float2 q = *reinterpret_cast<const float2*>(qf + at), b = *reinterpret_cast<const float2*>(bf + at);
                const float2 e = ref != nullptr ? *reinterpret_cast<const float2*>(ref + c) : make_float2(0.f, 0.f);
                const float x0 = q.x * ds_exp2(b.x - e.x), x1 = q.y * ds_exp2(b.y - e.y);
                const __nv_bfloat162 hh = __floats2bfloat162_rn(x0, x1);
                const float2 hf = __bfloat1622float2(hh);
                ah[u] = *reinterpret_cast<const uint32_t*>(&hh);
                al[u] = pack_bf16(x0 - hf.x, x1 - hf.y);
            }
        } else {
            const int at = (row0 + lr + (mat & 1) * 8) * qs + ks * 16 + (mat >> 1) * 8;
            ldmatrix_x4(ah, qh + at);
            ldmatrix_x4(al, ql + at);
        }
    };
    float o[DVP / 8][4];
#pragma unroll
    for (int i = 0; i < DVP / 8; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;

    // S^T q: the incoming state [c][i], 64 value channels at a time
    const uint32_t* sin = reinterpret_cast<const uint32_t*>(pdl_fresh(a.ws)) + ((size_t)blockIdx.x * a.H + h) * (size_t)dv * dk;
    constexpr int SB = DVP < 64 ? DVP : 64;
#pragma unroll
    for (int n0 = 0; n0 < DVP; n0 += SB) {
        if (n0 < dv) {
            ds_batches<4, DS_OUT_THREADS, uint4>(SB, kq, [&](int r, int d) {
                return *reinterpret_cast<const uint4*>(sin + (size_t)min(n0 + r, dv - 1) * dk + (d < dk ? d : 0));
            }, [&](int r, int d, uint4 v) {
                if (n0 + r >= dv || d >= dk) v = make_uint4(0u, 0u, 0u, 0u);
                *reinterpret_cast<uint2*>(bh + r * qs + d) = make_uint2(__byte_perm(v.x, v.y, 0x5410), __byte_perm(v.z, v.w, 0x5410));
                *reinterpret_cast<uint2*>(bl + r * qs + d) = make_uint2(__byte_perm(v.x, v.y, 0x7632), __byte_perm(v.z, v.w, 0x7632));
            });
            __syncthreads();
            if (mine)
#pragma unroll 1
                for (int ks = grp; ks < dkp / 16; ks += 2) {
                    uint32_t ah[4], al[4];
                    q_frag(ks, nullptr, ah, al);
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
    if (!CH) {
        const float f0 = DECAY == PRISM_DS_HEAD ? pw[r0 + 1] : expf(s_b[r0]), f1 = DECAY == PRISM_DS_HEAD ? pw[r1 + 1] : expf(s_b[r1]);
#pragma unroll
        for (int i = 0; i < DVP / 8; ++i) { o[i][0] *= f0; o[i][1] *= f0; o[i][2] *= f1; o[i][3] *= f1; }
    }
    // scores against the chunk's own keys, decayed by what lies between
    if constexpr (CH) {
        ds_batches<4, DS_OUT_THREADS, float4>(DS_CHUNK, kq, [&](int r, int d) {
            return *reinterpret_cast<const float4*>(kx + (size_t)(t0 + min(r, n - 1)) * a.xs + (d < dk ? d : 0));
        }, [&](int r, int d, const float4& q) {
            float4 v = ds_zero4();
            if (r < n && d < dk) {           // times the decay from there to the end of its sub-chunk
                const float4 b = *reinterpret_cast<const float4*>(bf + r * qs + d);
                const float4 e = *reinterpret_cast<const float4*>(bf + (r | (DS_SUB - 1)) * qs + d);
                v = ds_turn(a, q, d, a.kmul);
                v = make_float4(v.x * ds_exp2(e.x - b.x), v.y * ds_exp2(e.y - b.y), v.z * ds_exp2(e.z - b.z), v.w * ds_exp2(e.w - b.w));
            }
            ds_split4(v, bh + r * qs + d, bl + r * qs + d);
        });
    } else {
        load_rows(kx, a.kmul, bh, bl);
    }
    __syncthreads();
    constexpr int PAIRS = DS_CHUNK / DS_SUB / 2;           // sub-chunks of keys a warp may have: 2 j + grp
    float s[2 * PAIRS][4];
#pragma unroll
    for (int i = 0; i < 2 * PAIRS; ++i) s[i][0] = s[i][1] = s[i][2] = s[i][3] = 0.f;
    if constexpr (CH) {
        float span = 0.f;                                      // how far the log decays go inside this warp's sub-chunk
        for (int d = lane; d < dk; d += 32) span = fmaxf(span, bf[row0 * qs + d] - bf[(row0 + DS_SUB - 1) * qs + d]);
        span = warp_max(span);
        if (mine) {
            const bool by_terms = span > DS_MAX_SPAN;
#pragma unroll
            for (int j = 0; j < PAIRS; ++j) {
                const int np = 2 * j + grp;
                if (np > rw || (np == rw && by_terms)) continue;
                const float* ref = bf + (np * DS_SUB + DS_SUB - 1) * qs;
                for (int ks = 0; ks < dkp / 16; ++ks) {
                    uint32_t ah[4], al[4], xh[4], xl[4];
                    q_frag(ks, ref, ah, al);
                    const int bt = (np * 16 + (mat >> 1) * 8 + lr) * qs + ks * 16 + (mat & 1) * 8;
                    ldmatrix_x4(xh, bh + bt);
                    ldmatrix_x4(xl, bl + bt);
#pragma unroll
                    for (int e = 0; e < 2; ++e) {
                        mma_bf16_16816(s[2 * j + e], ah, xh[2 * e], xh[2 * e + 1]);
                        mma_bf16_16816(s[2 * j + e], ah, xl[2 * e], xl[2 * e + 1]);
                        mma_bf16_16816(s[2 * j + e], al, xh[2 * e], xh[2 * e + 1]);
                    }
                }
            }
            // the warp's own sub-chunk: by terms where it has to be, and only keys up to the query
#pragma unroll
            for (int j = 0; j < PAIRS; ++j) {
                const int np = 2 * j + grp;
                if (np != rw) continue;
                auto key = [&](int i) { return np * DS_SUB + (i >> 2) * 8 + (lane & 3) * 2 + (i & 1); };
                if (by_terms)
#pragma unroll 1
                    for (int i = 0; i < 8; ++i) {
                        const int r = (i & 2) ? r1 : r0, c = min(key(i), n - 1);
                        const float* kr = kx + (size_t)(t0 + c) * a.xs;
                        float sum = 0.f;
#pragma unroll 1
                        for (int d = 0; d < dk; ++d)          // c after r: masked below; the difference may then be large, capped
                            sum += qf[r * qs + d] * ((a.act ? ds_silu(kr[d]) : kr[d]) * a.kmul) * ds_exp2(fminf(bf[r * qs + d] - bf[c * qs + d], 0.f));
#pragma unroll
                        for (int u = 0; u < 8; ++u)
                            if (u == i) s[2 * j + (u >> 2)][u & 3] = sum;
                    }
#pragma unroll
                for (int i = 0; i < 8; ++i)
                    if (key(i) > ((i & 2) ? r1 : r0)) s[2 * j + (i >> 2)][i & 3] = 0.f;
            }
        }
    } else {
        if (mine) {
#pragma unroll 1
            for (int ks = 0; ks < dkp / 16; ++ks) {
                uint32_t ah[4], al[4];
                q_frag(ks, nullptr, ah, al);
#pragma unroll
                for (int j = 0; j < PAIRS; ++j) {
                    const int np = 2 * j + grp;
                    if (np > rw) continue;                     // keys after this warp's last token
                    uint32_t xh[4], xl[4];
                    const int bt = (np * 16 + (mat >> 1) * 8 + lr) * qs + ks * 16 + (mat & 1) * 8;
                    ldmatrix_x4(xh, bh + bt);
                    ldmatrix_x4(xl, bl + bt);
#pragma unroll
                    for (int e = 0; e < 2; ++e) {
                        mma_bf16_16816(s[2 * j + e], ah, xh[2 * e], xh[2 * e + 1]);
                        mma_bf16_16816(s[2 * j + e], ah, xl[2 * e], xl[2 * e + 1]);
                        mma_bf16_16816(s[2 * j + e], al, xh[2 * e], xh[2 * e + 1]);
                    }
                }
            }
        }
    }
    if constexpr (!CH) {
#pragma unroll
        for (int nt = 0; nt < 2 * PAIRS; ++nt)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int r = e < 2 ? r0 : r1, c = (nt & ~1) * 16 + grp * DS_SUB + (nt & 1) * 8 + (lane & 3) * 2 + (e & 1), back = r - c;
                if (DECAY == PRISM_DS_HEAD) s[nt][e] = back >= 0 ? s[nt][e] * pw[back] : 0.f;
                else s[nt][e] = back >= 0 ? s[nt][e] * (expf(s_b[r] - s_b[c]) * s_d[c]) : 0.f;
            }
    }
    __syncthreads();
    ds_batches<4, DS_OUT_THREADS, float4>(DS_CHUNK, DVP / 4, [&](int r, int d) {
        return *reinterpret_cast<const float4*>(vx + (size_t)(t0 + min(r, n - 1)) * a.xs + (d < dv ? d : 0));
    }, [&](int r, int d, float4 v) {
        ds_split4(r < n && d < dv ? (ROT ? v : ds_turn(a, v, d, 1.f)) : ds_zero4(), bh + r * VS + d, bl + r * VS + d);
    });
    __syncthreads();
#pragma unroll
    for (int j2 = 0; j2 < PAIRS; ++j2) {
        const int kk = 2 * j2 + grp;
        if (!mine || kk > rw) continue;
        uint32_t ph[4], pl[4];
#pragma unroll
        for (int u = 0; u < 4; ++u) {
            const float x0 = s[2 * j2 + (u >> 1)][(u & 1) * 2], x1 = s[2 * j2 + (u >> 1)][(u & 1) * 2 + 1];
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
    // the pair's sums come together through the buffer (64 rows of DVP + 8 floats)
    __syncthreads();
    float* sums = reinterpret_cast<float*>(bh);
    if (grp == 1 && mine)
#pragma unroll
        for (int i = 0; i < DVP / 8; ++i) {
            const int d = i * 8 + (lane & 3) * 2;
            *reinterpret_cast<float2*>(sums + r0 * VS + d) = make_float2(o[i][0], o[i][1]);
            *reinterpret_cast<float2*>(sums + r1 * VS + d) = make_float2(o[i][2], o[i][3]);
        }
    __syncthreads();
    if (grp == 1 || !mine) return;
#pragma unroll
    for (int i = 0; i < DVP / 8; ++i) {
        const int d = i * 8 + (lane & 3) * 2;
        const float2 x = *reinterpret_cast<const float2*>(sums + r0 * VS + d), y = *reinterpret_cast<const float2*>(sums + r1 * VS + d);
        o[i][0] += x.x; o[i][1] += x.y; o[i][2] += y.x; o[i][3] += y.y;
    }
    if (!ROT && a.gate == nullptr) {   // the read-out itself, with the skip path where there is one
        const float skip = DECAY == PRISM_DS_TOKEN && a.skip != nullptr ? load_param(a.skip, a.skip_bf16, h) : 0.f;
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            const int r = e ? r1 : r0;
            if (r >= n) continue;
            float* dst = reinterpret_cast<float*>(a.out) + (size_t)(t0 + r) * a.os + (size_t)h * dv;
            const float* vr = vx + (size_t)(t0 + r) * a.xs;
#pragma unroll
            for (int i = 0; i < DVP / 8; ++i) {
                const int d = i * 8 + (lane & 3) * 2;
                if (d >= dv) continue;
                float2 y = make_float2(o[i][2 * e], o[i][2 * e + 1]);
                if (DECAY == PRISM_DS_TOKEN) {
                    const float2 v = *reinterpret_cast<const float2*>(vr + d);
                    y = make_float2(y.x + skip * v.x, y.y + skip * v.y);
                }
                *reinterpret_cast<float2*>(dst + d) = y;
            }
        }
        return;
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
        const float* gate = pdl_fresh(a.gate) + (size_t)(t0 + r) * a.gs + (size_t)h * dv;
        __nv_bfloat16* dst = reinterpret_cast<__nv_bfloat16*>(a.out) + (size_t)(t0 + r) * a.os + (size_t)h * dv;
#pragma unroll
        for (int i = 0; i < DVP / 8; ++i) {
            const int d = i * 8 + (lane & 3) * 2;
            if (d >= dv) continue;
            const float2 gz = *reinterpret_cast<const float2*>(gate + d);
            float2 y = make_float2(o[i][2 * e] * inv * ds_silu(gz.x), o[i][2 * e + 1] * inv * ds_silu(gz.y));
            if (!ROT && a.weight != nullptr) {
                y.x *= load_param(a.weight, a.weight_bf16, d);
                y.y *= load_param(a.weight, a.weight_bf16, d + 1);
            }
            *reinterpret_cast<uint32_t*>(dst + d) = pack_bf16(y.x, y.y);
        }
    }
}

template <int DVP, int DECAY, bool ROT> static int launch_chunk_out(const DecayChunks& a, int chunks, cudaStream_t stream) {
    const int qs = (a.dk + 15) / 16 * 16 + 8, bs = qs > DVP + 8 ? qs : DVP + 8;
    const size_t smem = (size_t)DS_CHUNK * ((DECAY == PRISM_DS_CHANNEL ? 4 : 2) * qs + 2 * bs) * sizeof(__nv_bfloat16);
    auto kern = decay_chunk_out_kernel<DVP, DECAY, ROT>;
    cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    return (int)launch_kernel(kern, dim3(chunks, a.H), dim3(DS_OUT_THREADS), smem, stream, a);
}

template <int DECAY, bool ROT> static int launch_chunks(const DecayChunks& a, int chunks, cudaStream_t stream) {
    const int ks = (a.dk + 63) / 64 * 64 + 8, vs = (a.dv + 31) / 32 * 32 + 8;
    const size_t smem = (size_t)DS_CHUNK * 2 * (ks + vs) * sizeof(__nv_bfloat16);
    auto state = decay_chunk_state_kernel<DECAY, ROT>;
    cudaFuncSetAttribute(state, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    cudaError_t rc = launch_kernel(state, dim3(chunks, a.H), dim3(DS_STATE_THREADS), smem, stream, a);
    if (rc != cudaSuccess) return (int)rc;
    rc = launch_kernel(decay_carry_kernel<DECAY>, dim3((a.dv * a.dk / 4 + 255) / 256, a.H, a.S), dim3(256), 0, stream, a);
    if (rc != cudaSuccess) return (int)rc;
    if (a.dv <= 32) return launch_chunk_out<32, DECAY, ROT>(a, chunks, stream);
    if (a.dv <= 64) return launch_chunk_out<64, DECAY, ROT>(a, chunks, stream);
    if (a.dv <= 128) return launch_chunk_out<128, DECAY, ROT>(a, chunks, stream);
    return launch_chunk_out<256, DECAY, ROT>(a, chunks, stream);
}

}  // namespace prism

// 1 if the one-token kernel takes these sizes.
PRISM_EXPORT int prism_decay_step_supported(int dk, int dv) { return dk >= 4 && dk % 4 == 0 && dk <= 256 && dv >= 1 && 3 * (dk + dv) * 4 <= 48 * 1024; }

// 1 if the chunked kernels take these sizes: whole quads everywhere (rot: entries that turn, pairs or halves of them).
PRISM_EXPORT int prism_decay_chunks_supported(int dk, int dv, int rot, int pairs) {
    return dk >= 8 && dk % 8 == 0 && dk <= 256 && dv >= 8 && dv % 8 == 0 && dv <= 256 && rot % (pairs ? 4 : 8) == 0;
}

// One token per request.  q, k, v: float32 rows with one stride xs (head h: q and k at (h / rep) dk, v at h dv); act 1: all
// three through silu; rotation of q and k by freq [rot / 2] (rot 0: none; pairs: entries (2i, 2i + 1) turn together instead of
// halves; amp: a factor on cosine and sine); qmul, kmul: factors.  kind PRISM_DS_HEAD: decay [H].  PRISM_DS_TOKEN: dt [T, H]
// (row stride dts), dt_bias, a_log, skip [H] (skip may be null).  PRISM_DS_CHANNEL: low [T, R] (row stride ls), a2t [R, H dk]
// float32, a2_bias [H dk] or null, rate.  state [slots, H, dv, dk]; gate [T, H dv] float32 (row stride gs): out = o / rms(o) *
// weight [dv] (null: ones) * silu(gate) in out_dtype; gate null: out = o, float32.
PRISM_EXPORT int prism_decay_step(int kind, const float* q, const float* k, const float* v, long long xs, int T, int H, int rep, int dk,
                                  int dv, int act, const float* freq, int rot, int pairs, float amp, float qmul, float kmul,
                                  const float* decay, const float* dt, long long dts, const void* dt_bias, int dt_bias_dtype,
                                  const void* a_log, int a_log_dtype, const void* skip, int skip_dtype, const float* low, long long ls,
                                  int R, const float* a2t, const void* a2_bias, int a2_bias_dtype, float rate, float* state,
                                  const int* positions, const int* slots, const float* gate, long long gs, const void* weight,
                                  int weight_dtype, float eps, void* out, int out_dtype, long long os, cudaStream_t stream) {
    using namespace prism;
    if (T <= 0) return 0;
    if (!prism_decay_step_supported(dk, dv) || H < 1 || rep < 1 || H % rep || T > 65535 || rot < 0 || rot > dk || rot % 2 ||
        (rot && (freq == nullptr || kind != PRISM_DS_HEAD)) || (uintptr_t)state % 16 || (gate == nullptr && out_dtype == PRISM_DTYPE_BF16))
        return (int)cudaErrorInvalidValue;
    if ((kind == PRISM_DS_HEAD && decay == nullptr) || (kind == PRISM_DS_TOKEN && (dt == nullptr || dt_bias == nullptr || a_log == nullptr || gate)) ||
        (kind == PRISM_DS_CHANNEL && (low == nullptr || a2t == nullptr || R < 1)) || kind < 0 || kind > PRISM_DS_CHANNEL)
        return (int)cudaErrorInvalidValue;
    const size_t smem = (size_t)(3 * dk + 3 * dv) * sizeof(float);
    if (smem > 48 * 1024) return (int)cudaErrorInvalidValue;
    const auto b16 = [](int d) { return d == PRISM_DTYPE_BF16 ? 1 : 0; };
    DecayStep a;
    a.q = q; a.k = k; a.v = v; a.xs = xs; a.H = H; a.rep = rep; a.dk = dk; a.dv = dv; a.act = act;
    a.freq = freq; a.rot = rot; a.pairs = pairs; a.amp = amp; a.qmul = qmul; a.kmul = kmul; a.decay = decay;
    a.dt = dt; a.dts = dts; a.dt_bias = dt_bias; a.dt_bias_bf16 = b16(dt_bias_dtype); a.a_log = a_log; a.a_log_bf16 = b16(a_log_dtype);
    a.skip = skip; a.skip_bf16 = b16(skip_dtype);
    a.low = low; a.ls = ls; a.R = R; a.a2t = a2t; a.a2_bias = a2_bias; a.a2_bias_bf16 = b16(a2_bias_dtype); a.rate = rate;
    a.state = state; a.positions = positions; a.slots = slots; a.gate = gate; a.gs = gs; a.weight = weight;
    a.weight_bf16 = b16(weight_dtype); a.eps = eps; a.out = out; a.os = os;
#define PRISM_DSTEP(TT, L, Q, N, D) \
    return (int)launch_kernel(decay_step_kernel<TT, L, Q, N, D>, dim3(H, T), dim3(DS_STEP_THREADS), smem, stream, a)
#define PRISM_DSTEP_SIZE(TT, D)                       \
    do {                                           \
        if (dk <= 32) PRISM_DSTEP(TT, 8, 1, 4, D);    \
        if (dk <= 64) PRISM_DSTEP(TT, 16, 1, 8, D);   \
        if (dk <= 128 && dv <= 64) PRISM_DSTEP(TT, 32, 1, 8, D); \
        if (dk <= 128) PRISM_DSTEP(TT, 32, 1, 16, D); \
        PRISM_DSTEP(TT, 32, 2, 8, D);                 \
    } while (0)
#define PRISM_DSTEP_KIND(D)                                                     \
    do {                                                                     \
        if (out_dtype == PRISM_DTYPE_BF16) PRISM_DSTEP_SIZE(__nv_bfloat16, D);  \
        PRISM_DSTEP_SIZE(float, D);                                             \
    } while (0)
    if (kind == PRISM_DS_HEAD) PRISM_DSTEP_KIND(PRISM_DS_HEAD);
    if (kind == PRISM_DS_TOKEN) PRISM_DSTEP_SIZE(float, PRISM_DS_TOKEN);
    PRISM_DSTEP_KIND(PRISM_DS_CHANNEL);
#undef PRISM_DSTEP_KIND
#undef PRISM_DSTEP_SIZE
#undef PRISM_DSTEP
}

// As above for segments of any length (q, k, v rows, strides and pointers in whole quads); table [T, rot / 2, 2] float32:
// cosine and sine of position * frequency; pw [H, 65]: powers 0 .. 64 of the heads' decays; cum [T, H dk] float32: scratch of
// PRISM_DS_CHANNEL; ws: (T / 64 + S) * H * dv * dk floats; fac: (T / 64 + S) * H floats.  out bf16 with a gate, else
// float32.
PRISM_EXPORT int prism_decay_chunks(int kind, const float* q, const float* k, const float* v, long long xs, int T, int S, int H, int rep,
                                    int dk, int dv, int act, const float* table, int rot, int pairs, float amp, float qmul, float kmul,
                                    const float* pw, const float* dt, long long dts, const void* dt_bias, int dt_bias_dtype,
                                    const void* a_log, int a_log_dtype, const void* skip, int skip_dtype, const float* low, long long ls,
                                    int R, const float* a2t, const void* a2_bias, int a2_bias_dtype, float rate, float* cum, float* state,
                                    const int* seg_start, const int* slots, const float* gate, long long gs, const void* weight,
                                    int weight_dtype, float eps, float* ws, float* fac, void* out, long long os, cudaStream_t stream) {
    using namespace prism;
    if (T <= 0 || S <= 0) return 0;
    if (!prism_decay_chunks_supported(dk, dv, rot, pairs) || H < 1 || H > 65535 || S > 65535 || rep < 1 || H % rep || rot < 0 || rot > dk ||
        (rot && (table == nullptr || kind != PRISM_DS_HEAD || act || gate == nullptr || weight != nullptr)) || xs % 4 || os % 2 || (uintptr_t)q % 16 || (uintptr_t)k % 16 ||
        (uintptr_t)v % 16 || (uintptr_t)table % 16 || (uintptr_t)state % 16 || (uintptr_t)ws % 16 || (uintptr_t)cum % 16 ||
        (uintptr_t)out % (gate ? 4 : 8) || (gate && (gs % 2 || (uintptr_t)gate % 8)))
        return (int)cudaErrorInvalidValue;
    if ((kind == PRISM_DS_HEAD && pw == nullptr) ||
        (kind == PRISM_DS_TOKEN && (dt == nullptr || dt_bias == nullptr || a_log == nullptr || fac == nullptr || gate != nullptr || act)) ||
        (kind == PRISM_DS_CHANNEL && (cum == nullptr || low == nullptr || a2t == nullptr || R < 1)) || kind < 0 || kind > PRISM_DS_CHANNEL)
        return (int)cudaErrorInvalidValue;
    const auto b16 = [](int d) { return d == PRISM_DTYPE_BF16 ? 1 : 0; };
    DecayChunks a;
    a.q = q; a.k = k; a.v = v; a.xs = xs; a.H = H; a.rep = rep; a.dk = dk; a.dv = dv; a.S = S; a.act = act;
    a.table = reinterpret_cast<const float2*>(table); a.rot = rot; a.pairs = pairs; a.amp = amp; a.qmul = qmul; a.kmul = kmul; a.pw = pw;
    a.dt = dt; a.dts = dts; a.dt_bias = dt_bias; a.dt_bias_bf16 = b16(dt_bias_dtype); a.a_log = a_log; a.a_log_bf16 = b16(a_log_dtype);
    a.low = low; a.ls = ls; a.R = R; a.a2t = a2t; a.a2_bias = a2_bias; a.a2_bias_bf16 = b16(a2_bias_dtype); a.rate = rate;
    a.skip = skip; a.skip_bf16 = b16(skip_dtype); a.cum = cum; a.state = state; a.seg_start = seg_start; a.slots = slots; a.ws = ws;
    a.fac = fac; a.gate = gate; a.gs = gs; a.weight = weight; a.weight_bf16 = b16(weight_dtype); a.eps = eps; a.out = out; a.os = os;
    const int chunks = T / DS_CHUNK + S;
    if (kind == PRISM_DS_TOKEN) return launch_chunks<PRISM_DS_TOKEN, false>(a, chunks, stream);
    if (kind == PRISM_DS_CHANNEL) return launch_chunks<PRISM_DS_CHANNEL, false>(a, chunks, stream);
    return rot ? launch_chunks<PRISM_DS_HEAD, true>(a, chunks, stream) : launch_chunks<PRISM_DS_HEAD, false>(a, chunks, stream);
}
