// What stands around the recurrences of recurrent.cu whose inputs pass an activation or a short convolution first, and their steps of
// single tokens, in which a (request, head) is one CTA that does everything between the input product and the output product.
//
//   short convolution   x_t[c] = silu(sum_{j < taps} w[c, taps-1-j] p_{t-j}[c]), p the projection's rows (fp32), nothing before the
//                       sequence's start.  The last inputs of a request live in its state row as a ring of `taps` rows: the input of
//                       position p is row p % taps.  (One row more than the taps that look back: a token writes its own row while
//                       other CTAs still read the older ones, and the two never meet.)
//   gated delta rule    q and k made unit vectors, x / sqrt(|x|^2 + 1e-6), q times K^-1/2; g = exp(-exp(A) softplus(a + dt)),
//                       beta = sigmoid(b); after the recurrence every head's o is divided by its root mean square, times a weight
//                       that the heads share, times silu of a gate
//   lightning           q, k, v pass silu; one fixed decay per head; the heads of a token are normed together (gated_rows_kernel)
//
// Everything is fp32 until the store of the output product's input.
#include "common.cuh"

namespace {

struct Columns {                      // a [T, n] fp32 matrix that may be a column slice of a wider one
    const float* p;
    int ld;
};

__device__ __forceinline__ float sigmoidf(float x) { return 1.0f / (1.0f + expf(-x)); }
// (a denominator beyond 2^126 gives the 0 that the quotient would round to, or all but)
__device__ __forceinline__ float siluf(float x) { return __fdividef(x, 1.0f + expf(-x)); }
__device__ __forceinline__ float softplusf(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }

// exp(-x) of a small x is a number just below one that hundreds of tokens multiply: 1 + (exp(-x) - 1) is it to the last bit, where an
// error of one unit there would be the same for every token and add up.
__device__ __forceinline__ float decayf(float x) { return 1.0f + expm1f(-x); }

struct ShortConv {
    const float* w;                   // fp32 [taps, channels], row 0 the current token's, row j that of the token j before it
    int taps;
    int channels;                     // numbers in a row of the ring (all tensors that are convolved, side by side)
};

// TP (4 or 8, the kernels' template parameter): taps whose inputs and weights are all asked for before the first is used.

// The convolution of channel c (its column of w and its place in the ring) of token t at position pos; x: the channel's numbers in the
// projection; `first`: the request's first token of the step; ring: the request's ring.  The oldest input is added first, whatever the cut.
template <int TP>
__device__ __forceinline__ float convolve(const ShortConv& cv, const float* __restrict__ x, int ld, int t, int first, int pos, int c,
                                          const float* __restrict__ ring) {
    const int at = pos % cv.taps;
    auto input = [&](int j) {
        if (t - j >= first) return x[(size_t)(t - j) * ld];
        return ring[(size_t)(at >= j ? at - j : at - j + cv.taps) * cv.channels + c];
    };
    float a = 0.f;
    for (int j = cv.taps - 1; j >= TP; --j)
        if (pos >= j) a = fmaf(cv.w[(size_t)j * cv.channels + c], input(j), a);
    float v[TP], w[TP];
#pragma unroll
    for (int j = 0; j < TP; ++j) {
        v[j] = w[j] = 0.f;
        if (j < cv.taps && pos >= j) {
            v[j] = input(j);
            w[j] = cv.w[(size_t)j * cv.channels + c];
        }
    }
#pragma unroll
    for (int j = TP - 1; j >= 0; --j) a = fmaf(w[j], v[j], a);
    return a;
}

struct DeltaPrepare {
    Columns p;                        // the projection: [q | k | v] from its first column, b and a after them
    int b_col, a_col;
    ShortConv cv;
    const float* state;               // request s's ring at state + slots[s] * stride + ring_off
    long long stride, ring_off;
    const int32_t *tok_req, *q_start, *positions, *slots;
    const float *decay_rate, *dt;     // fp32 [N]: exp(A_log), dt_bias
    float* qkv;                       // fp32 [T, 2*M*K + N*V]: q | k | v after convolution and silu, q and k unit vectors, q times K^-1/2
    float* g;                         // fp32 [T, N]
    float* beta;                      // fp32 [T, N]
    int T, N, M, K, V;
};

constexpr int kUnitRegs = 8;          // channels of a q or k head that a lane holds (heads of up to 256)
constexpr int kPrepTokens = 4;        // consecutive tokens that a warp takes at a time, so that most inputs are read once

// kPrepTokens neighbouring tokens of one channel, t0 the first.  inner: all of them and all that they look back on are one request's
// tokens of this step (and n == kPrepTokens, taps <= TP); then a window of inputs is read once and slides over the taps.
template <int TP>
__device__ __forceinline__ void convolve_tile(const DeltaPrepare& d, const float* __restrict__ x, int c, int t0, int n, bool inner, float (&y)[kPrepTokens]) {
    if (inner) {
        float v[TP - 1 + kPrepTokens], w[TP];
#pragma unroll
        for (int i = 0; i < TP - 1 + kPrepTokens; ++i) {               // v[i]: token t0 + i - (TP - 1)
            const int back = TP - 1 - i;
            v[i] = back < d.cv.taps ? __ldg(x + (ptrdiff_t)(t0 - back) * d.p.ld) : 0.f;
        }
#pragma unroll
        for (int j = 0; j < TP; ++j) w[j] = j < d.cv.taps ? __ldg(d.cv.w + (size_t)j * d.cv.channels + c) : 0.f;
#pragma unroll
        for (int k = 0; k < kPrepTokens; ++k) {
            float a = 0.f;
#pragma unroll
            for (int j = TP - 1; j >= 0; --j) a = fmaf(w[j], v[TP - 1 + k - j], a);
            y[k] = siluf(a);
        }
        return;
    }
    for (int k = 0; k < kPrepTokens; ++k) {
        y[k] = 0.f;
        if (k >= n) continue;
        const int t = t0 + k, s = d.tok_req[t];
        y[k] = siluf(convolve<TP>(d.cv, x, d.p.ld, t, d.q_start[s], d.positions[t], c, d.state + (size_t)d.slots[s] * d.stride + d.ring_off));
    }
}

// One tile of one head of q, k or v, by a warp.  NC: the lanes' channels of a q or k head.
template <int NC, int TP>
__device__ __forceinline__ void prepare_tile(const DeltaPrepare& d, int t0, int n, bool inner, int unit, int lane) {
    const int C = 2 * d.M * d.K + d.N * d.V;
    if (unit < 2 * d.M) {
        const int c0 = unit * d.K;
        float x[NC][kPrepTokens], ss[kPrepTokens];
#pragma unroll
        for (int k = 0; k < kPrepTokens; ++k) ss[k] = 0.f;
#pragma unroll
        for (int i = 0; i < NC; ++i) {
            const int c = lane + 32 * i;
            if (32 * i >= d.K) continue;                                  // (the same for the whole warp)
            if (c < d.K) convolve_tile<TP>(d, d.p.p + c0 + c, c0 + c, t0, n, inner, x[i]);
#pragma unroll
            for (int k = 0; k < kPrepTokens; ++k) {
                if (c >= d.K) x[i][k] = 0.f;
                ss[k] = fmaf(x[i][k], x[i][k], ss[k]);
            }
        }
        const float scale = unit < d.M ? 1.0f / sqrtf((float)d.K) : 1.0f;
#pragma unroll
        for (int k = 0; k < kPrepTokens; ++k) {
            const float inv = scale / sqrtf(forge::warp_sum(ss[k]) + 1e-6f);
            if (k >= n) continue;
#pragma unroll
            for (int i = 0; i < NC; ++i) {
                const int c = lane + 32 * i;
                if (c < d.K) d.qkv[(size_t)(t0 + k) * C + c0 + c] = x[i][k] * inv;
            }
        }
        return;
    }
    const int head = unit - 2 * d.M, c0 = 2 * d.M * d.K + head * d.V;
    for (int c = lane; c < d.V; c += 32) {
        float y[kPrepTokens];
        convolve_tile<TP>(d, d.p.p + c0 + c, c0 + c, t0, n, inner, y);
#pragma unroll
        for (int k = 0; k < kPrepTokens; ++k)
            if (k < n) d.qkv[(size_t)(t0 + k) * C + c0 + c] = y[k];
    }
    if (lane < n) {
        const float* row = d.p.p + (size_t)(t0 + lane) * d.p.ld;
        d.beta[(size_t)(t0 + lane) * d.N + head] = sigmoidf(row[d.b_col + head]);
        d.g[(size_t)(t0 + lane) * d.N + head] = decayf(d.decay_rate[head] * softplusf(row[d.a_col + head] + d.dt[head]));
    }
}

// A warp per (`tiles` tiles of kPrepTokens tokens, head of q, k or v).
template <int NC, int TP>
__global__ void __launch_bounds__(128, NC <= 4 ? 8 : 4)
delta_prepare_kernel(const DeltaPrepare d, int tiles) {
    forge::pdl_wait();
    const int first = (blockIdx.x * 4 + (threadIdx.x >> 5)) * kPrepTokens * tiles, lane = threadIdx.x & 31;
    if (first >= d.T) return;
    const int last = min(first + kPrepTokens * tiles, d.T) - 1, s0 = d.tok_req[first], back = d.cv.taps - 1;
    const bool one = d.cv.taps <= TP && d.tok_req[last] == s0 && first - back >= d.q_start[s0];
#pragma unroll 1
    for (int t0 = first; t0 <= last; t0 += kPrepTokens) {
        const int n = min(kPrepTokens, d.T - t0);
        bool inner = one;
        if (!one && d.cv.taps <= TP) {
            const int s = d.tok_req[t0];
            inner = d.tok_req[t0 + n - 1] == s && t0 - back >= d.q_start[s];
        }
        prepare_tile<NC, TP>(d, t0, n, inner && n == kPrepTokens, blockIdx.y, lane);
    }
}

// The ring after a step: the inputs of a request's last `taps` tokens of the step (or of all it brought).
__global__ void __launch_bounds__(256)
conv_keep_kernel(Columns p, ShortConv cv, float* __restrict__ state, long long stride, long long ring_off, const int32_t* __restrict__ q_start,
                 const int32_t* __restrict__ positions, const int32_t* __restrict__ slots) {
    forge::pdl_wait();
    const int s = blockIdx.x, c = blockIdx.y * 256 + threadIdx.x;
    if (c >= cv.channels) return;
    const int hi = q_start[s + 1], lo = max(q_start[s], hi - cv.taps);
    float* ring = state + (size_t)slots[s] * stride + ring_off;
    for (int t = lo; t < hi; ++t) ring[(size_t)(positions[t] % cv.taps) * cv.channels + c] = p.p[(size_t)t * p.ld + c];
}

// x <- silu(x) over n columns of fp32 rows, in place.
__global__ void __launch_bounds__(256)
silu_columns_kernel(float* __restrict__ x, long long ld, int n, int vec) {
    forge::pdl_wait();
    float* row = x + (size_t)blockIdx.x * ld;
    const int first = blockIdx.y * 256 + threadIdx.x, step = gridDim.y * 256;
    if (vec) {
        for (int i = first; i < n / 4; i += step) {
            float4 v = reinterpret_cast<float4*>(row)[i];
            v.x = siluf(v.x); v.y = siluf(v.y); v.z = siluf(v.z); v.w = siluf(v.w);
            reinterpret_cast<float4*>(row)[i] = v;
        }
    } else {
        for (int i = first; i < n; i += step) row[i] = siluf(row[i]);
    }
}

template <int P> struct Pack;
template <> struct Pack<1> { using type = float; };
template <> struct Pack<4> { using type = float4; };
__device__ __forceinline__ float& lane_of(float& v, int) { return v; }
__device__ __forceinline__ float& lane_of(float4& v, int i) { return (&v.x)[i]; }

template <typename TOut> __device__ __forceinline__ void store4(TOut* p, float a, float b, float c, float d);
template <> __device__ __forceinline__ void store4<float>(float* p, float a, float b, float c, float d) {
    *reinterpret_cast<float4*>(p) = make_float4(a, b, c, d);
}
template <> __device__ __forceinline__ void store4<__nv_bfloat16>(__nv_bfloat16* p, float a, float b, float c, float d) {
    const __nv_bfloat162 lo = __floats2bfloat162_rn(a, b), hi = __floats2bfloat162_rn(c, d);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&lo), *reinterpret_cast<const uint32_t*>(&hi));
}

// out = o / rms(o over the whole row) * w * sigmoid(gate).  One CTA per row.
template <typename TA>
__global__ void __launch_bounds__(512)
gated_rows_kernel(const float* __restrict__ o, const float* __restrict__ w, Columns gate, TA* __restrict__ out, long long out_ld, int n, float eps,
                  int vec) {
    __shared__ float red[32];
    forge::pdl_launch_dependents();
    forge::pdl_wait();
    const int t = blockIdx.x;
    const float* row = o + (size_t)t * n;
    const float* g = gate.p + (size_t)t * gate.ld;
    TA* dst = out + (size_t)t * out_ld;
    float ss = 0.f;
    if (vec) {
        for (int i = threadIdx.x; i < n / 4; i += blockDim.x) {
            const float4 v = reinterpret_cast<const float4*>(row)[i];
            ss += (v.x * v.x + v.y * v.y) + (v.z * v.z + v.w * v.w);
        }
    } else {
        for (int i = threadIdx.x; i < n; i += blockDim.x) ss = fmaf(row[i], row[i], ss);
    }
    const float inv = 1.0f / sqrtf(forge::block_sum(ss, red) / (float)n + eps);
    if (vec) {
        for (int i = threadIdx.x; i < n / 4; i += blockDim.x) {
            const float4 v = reinterpret_cast<const float4*>(row)[i], a = reinterpret_cast<const float4*>(w)[i], b = reinterpret_cast<const float4*>(g)[i];
            store4<TA>(dst + 4 * i, v.x * inv * a.x * sigmoidf(b.x), v.y * inv * a.y * sigmoidf(b.y), v.z * inv * a.z * sigmoidf(b.z),
                       v.w * inv * a.w * sigmoidf(b.w));
        }
    } else {
        for (int i = threadIdx.x; i < n; i += blockDim.x) dst[i] = forge::from_float<TA>(row[i] * inv * w[i] * sigmoidf(g[i]));
    }
}

constexpr int kTokenThreads = 512;        // at most
constexpr int kHeld = 16;                 // packs of the state that a thread holds, at most

struct TokenState {
    Columns q, k, v;                  // before convolution and activation
    ShortConv cv;                     // channels of q from 0, of k from M*K, of v from 2*M*K on (DELTA)
    Columns gate, b, a;               // (DELTA)
    const float* decay;               // fp32 [N]: exp(A_log) (DELTA), else the fixed decays
    const float* dt;                  // fp32 [N] (DELTA)
    float* state;
    long long stride, ring_off;
    const int32_t *q_start, *positions, *slots;
    const float* weight;              // fp32 [V] (DELTA)
    float eps;
    int N, M, K, V, CG, RG;
};

// A step in which every request brings one token: a CTA per (request, head).  A row of the state is V / P packs of P value channels;
// thread t holds pack t % CG (CG = V / P) of the rows t / CG, t / CG + RG, ..., the first kHeld of them in registers from the first look
// at the state to the write (longer heads read theirs again).  DELTA: one look gives S^T k and S^T q at once, the RG partial sums are
// added in a fixed order, and with u = beta (v - g S^T k) the output is g S^T q + (k . q) u.  Else S <- decay S + k v^T, o = S^T q.
// out: DELTA: the normed and gated heads in the activation type; else the heads as they are, fp32.
// kMost: the most threads of a launch, kCtas: how many such CTAs an SM should hold.
template <int P, int kHeld, int kMost, int kCtas, int TP, bool DELTA, typename TA>
__global__ void __launch_bounds__(kMost, kCtas)
token_state_kernel(const TokenState d, TA* __restrict__ out, long long out_ld) {
    using S4 = typename Pack<P>::type;
    extern __shared__ __align__(16) float sm[];
    __shared__ float red[32];
    const int K = d.K, V = d.V, CG = d.CG, RG = d.RG;
    float* qs = sm;                    // [K] q, k and v after convolution and silu, side by side
    float* ks = qs + K;                // [K]
    float* vs = ks + K;                // [V]
    float* part = vs + V;              // [RG][V] partial sums of S^T q; DELTA: then [RG][V] of S^T k
    forge::pdl_launch_dependents();
    forge::pdl_wait();
    const int threads = blockDim.x, s = blockIdx.x, head = blockIdx.y, tid = threadIdx.x, lane = tid & 31;
    const int t = d.q_start[s], share = d.N / d.M, hk = head / share;
    float* row_of_slot = d.state + (size_t)d.slots[s] * d.stride;
    float* S = row_of_slot + (size_t)head * K * V;
    const int rg = tid / CG, cp = tid % CG;
    const bool live = rg < RG;
    S4 held[kHeld];
#pragma unroll
    for (int m = 0; m < kHeld; ++m) {
        held[m] = S4{};
        const int row = rg + m * RG;
        if (live && row < K) held[m] = reinterpret_cast<const S4*>(S + (size_t)row * V)[cp];
    }
    float g = 0.f, beta = 0.f, gate[P], weight[P];
    if (DELTA) {
        const float a_in = d.a.p[(size_t)t * d.a.ld + head] + d.dt[head], b_in = d.b.p[(size_t)t * d.b.ld + head], rate = d.decay[head];
        if (rg == 0) {                                     // what the end needs is asked for now
#pragma unroll
            for (int e = 0; e < P; ++e) {
                weight[e] = d.weight[cp * P + e];
                gate[e] = d.gate.p[(size_t)t * d.gate.ld + (size_t)head * V + cp * P + e];
            }
        }
        const int pos = d.positions[t];
        float* ring = row_of_slot + d.ring_off;
        float* now = ring + (size_t)(pos % d.cv.taps) * d.cv.channels;
#pragma unroll 2
        for (int i = tid; i < 2 * K + V; i += threads) {
            // q and k of the shared head, then the head's values: column of the projection's [q | k | v] and of the ring
            const int c = i < K ? hk * K + i : (i < 2 * K ? (d.M - 1 + hk) * K + i : 2 * (d.M - 1) * K + head * V + i);
            sm[i] = siluf(convolve<TP>(d.cv, d.q.p + c, d.q.ld, t, t, pos, c, ring));
            // the token's own row of the ring, which nobody reads in this step
            if (i >= 2 * K || head % share == 0) now[c] = d.q.p[(size_t)t * d.q.ld + c];
        }
        g = decayf(rate * softplusf(a_in));                // (in every thread: one thread's would be waited for)
        beta = sigmoidf(b_in);
    } else {
        g = d.decay[head];
        for (int i = tid; i < K; i += threads) {
            qs[i] = siluf(d.q.p[(size_t)t * d.q.ld + head * K + i]);
            ks[i] = siluf(d.k.p[(size_t)t * d.k.ld + head * K + i]);
        }
        for (int i = tid; i < V; i += threads) vs[i] = siluf(d.v.p[(size_t)t * d.v.ld + head * V + i]);
    }
    __syncthreads();
    float kscale = 1.f;
    if (DELTA) {
        float qq = 0.f, kk = 0.f, qk = 0.f;                // every warp for itself
        for (int i = lane; i < K; i += 32) {
            qq = fmaf(qs[i], qs[i], qq);
            kk = fmaf(ks[i], ks[i], kk);
            qk = fmaf(qs[i], ks[i], qk);
        }
        qq = forge::warp_sum(qq);
        kk = forge::warp_sum(kk);
        qk = forge::warp_sum(qk);
        const float qscale = 1.0f / (sqrtf(qq + 1e-6f) * sqrtf((float)K));
        kscale = 1.0f / sqrtf(kk + 1e-6f);
        qk *= qscale * kscale;
        // the sums over rows take q and k as they are; the unit vectors' factors join where the sums meet
        S4 aq{}, ak{};
        auto look = [&](int row, const S4& x) {
            S4 y = x;
            const float q1 = qs[row], k1 = ks[row];
#pragma unroll
            for (int e = 0; e < P; ++e) {
                lane_of(aq, e) = fmaf(q1, lane_of(y, e), lane_of(aq, e));
                lane_of(ak, e) = fmaf(k1, lane_of(y, e), lane_of(ak, e));
            }
        };
        if (live) {
#pragma unroll
            for (int m = 0; m < kHeld; ++m)
                if (rg + m * RG < K) look(rg + m * RG, held[m]);
#pragma unroll 1
            for (int row = rg + kHeld * RG; row < K; row += RG) look(row, reinterpret_cast<const S4*>(S + (size_t)row * V)[cp]);
            reinterpret_cast<S4*>(part + (size_t)rg * V)[cp] = aq;
            reinterpret_cast<S4*>(part + (size_t)(RG + rg) * V)[cp] = ak;
        }
        __syncthreads();
        float ss = 0.f, o[P];
        if (live) {
            S4 sq{}, sk{}, u{};
            for (int i = 0; i < RG; ++i) {
                S4 x = reinterpret_cast<const S4*>(part + (size_t)i * V)[cp], y = reinterpret_cast<const S4*>(part + (size_t)(RG + i) * V)[cp];
#pragma unroll
                for (int e = 0; e < P; ++e) {
                    lane_of(sq, e) += lane_of(x, e);
                    lane_of(sk, e) += lane_of(y, e);
                }
            }
#pragma unroll
            for (int e = 0; e < P; ++e) {
                const float ue = beta * fmaf(-g, lane_of(sk, e) * kscale, vs[cp * P + e]);
                o[e] = fmaf(g, lane_of(sq, e) * qscale, qk * ue);
                lane_of(u, e) = ue * kscale;
                ss = fmaf(o[e], o[e], ss);
            }
            auto write = [&](int row, S4 x) {
                const float k1 = ks[row];
#pragma unroll
                for (int e = 0; e < P; ++e) lane_of(x, e) = fmaf(g, lane_of(x, e), k1 * lane_of(u, e));
                reinterpret_cast<S4*>(S + (size_t)row * V)[cp] = x;
            };
#pragma unroll
            for (int m = 0; m < kHeld; ++m)
                if (rg + m * RG < K) write(rg + m * RG, held[m]);
#pragma unroll 1
            for (int row = rg + kHeld * RG; row < K; row += RG) write(row, reinterpret_cast<const S4*>(S + (size_t)row * V)[cp]);
        }
        // the head's norm: the first CG threads have every output once
        const float inv = 1.0f / sqrtf(forge::block_sum(rg == 0 ? ss : 0.f, red) / (float)V + d.eps);
        if (rg == 0) {
#pragma unroll
            for (int e = 0; e < P; ++e) {
                const int c = cp * P + e;
                out[(size_t)t * out_ld + (size_t)head * V + c] = forge::from_float<TA>(o[e] * inv * weight[e] * siluf(gate[e]));
            }
        }
    } else {
        if (live) {
            S4 acc{}, vv{};
#pragma unroll
            for (int e = 0; e < P; ++e) lane_of(vv, e) = vs[cp * P + e];
            auto step = [&](int row, S4 x) {
                const float q1 = qs[row], k1 = ks[row];
#pragma unroll
                for (int e = 0; e < P; ++e) {
                    lane_of(x, e) = fmaf(g, lane_of(x, e), k1 * lane_of(vv, e));
                    lane_of(acc, e) = fmaf(q1, lane_of(x, e), lane_of(acc, e));
                }
                reinterpret_cast<S4*>(S + (size_t)row * V)[cp] = x;
            };
#pragma unroll
            for (int m = 0; m < kHeld; ++m)
                if (rg + m * RG < K) step(rg + m * RG, held[m]);
#pragma unroll 1
            for (int row = rg + kHeld * RG; row < K; row += RG) step(row, reinterpret_cast<const S4*>(S + (size_t)row * V)[cp]);
            reinterpret_cast<S4*>(part + (size_t)rg * V)[cp] = acc;
        }
        __syncthreads();
        for (int c = tid; c < V; c += threads) {
            float o = 0.f;
            for (int i = 0; i < RG; ++i) o += part[(size_t)i * V + c];
            out[(size_t)t * out_ld + (size_t)head * V + c] = forge::from_float<TA>(o);
        }
    }
}

struct TokenShape {
    int P, threads, CG, RG;
    size_t smem;
};

// How a head of K x V numbers is dealt to a CTA; threads = 0: it does not fit.
TokenShape token_shape(int K, int V, bool delta, bool vec) {
    TokenShape s{vec ? 4 : 1, 0, 0, 0, 0};
    s.CG = V / s.P;
    if (s.CG > kTokenThreads) return s;
    // the fewest threads with which a head's state stays in registers, whole warps, at least 128
    const long long packs = (long long)K * s.CG;
    int threads = 128;
    while (threads < kTokenThreads && (packs > (long long)threads * kHeld || threads < s.CG)) threads *= 2;
    s.RG = threads / s.CG;
    if (s.RG > K) s.RG = K;
    s.smem = sizeof(float) * ((size_t)2 * K + V + (size_t)(delta ? 2 : 1) * s.RG * V);
    if (s.smem <= 48 * 1024) s.threads = threads;
    return s;
}

bool token_vec(const void* state, long long stride, int K, int V) {
    // (the partial sums' rows lie behind 2 K + V numbers: packs of four need K even, which K * V % 4 alone does not give)
    return V % 4 == 0 && K % 2 == 0 && stride % 4 == 0 && ((uintptr_t)state & 15) == 0;
}

template <int TP, bool DELTA, typename TO>
cudaError_t launch_token(bool vec, const TokenShape& sh, dim3 grid, cudaStream_t stream, const TokenState& d, TO* out, long long out_ld) {
    const bool few = (d.K + sh.RG - 1) / sh.RG <= kHeld / 2;            // rows a thread holds: half the registers where half are enough
    auto kernel = vec ? (few && sh.threads == 128 ? token_state_kernel<4, kHeld / 2, 128, 6, TP, DELTA, TO> : token_state_kernel<4, kHeld, kTokenThreads, 1, TP, DELTA, TO>)
                      : token_state_kernel<1, kHeld, kTokenThreads, 1, TP, DELTA, TO>;
    return forge::launch(kernel, grid, dim3(sh.threads), sh.smem, stream, 1, d, out, out_ld);
}

}  // namespace

// proj fp32 rows of ld numbers: [q: M*K | k: M*K | v: N*V] from their start, then b and a (N each) from columns b_col and a_col.
// conv_w fp32 [taps, 2*M*K + N*V], row j the weights of the token j before.  state fp32 rows of `stride` numbers, row slots[s] holds request s's ring [taps, 2*M*K + N*V] from
// ring_off on.  Leaves qkv fp32 [T, 2*M*K + N*V], g and beta fp32 [T, N], and the rings as they are after the step.
extern "C" int forge_delta_prepare(const float* proj, int ld, int b_col, int a_col, const float* conv_w, int taps, float* state, long long stride,
                                   long long ring_off, const int32_t* tok_req, const int32_t* q_start, const int32_t* positions,
                                   const int32_t* slots, const float* decay_rate, const float* dt, float* qkv, float* g, float* beta, int T, int S,
                                   int N, int M, int K, int V, cudaStream_t stream) {
    const long long C = 2LL * M * K + (long long)N * V;
    if (T < 0 || S < 0 || N <= 0 || M <= 0 || N % M != 0 || K <= 0 || V <= 0 || taps <= 0 || ld < C || b_col < 0 || a_col < 0 || b_col + N > ld || a_col + N > ld)
        return forge::fail(FORGE_ERR_ARG, "delta_prepare: bad sizes T=%d N=%d M=%d K=%d V=%d taps=%d ld=%d", T, N, M, K, V, taps, ld);
    if (K > 32 * kUnitRegs) return forge::fail(FORGE_ERR_UNSUPPORTED, "delta_prepare: heads of %d key channels", K);
    if (ring_off < 0 || stride < ring_off + taps * C) return forge::fail(FORGE_ERR_ARG, "delta_prepare: state rows are too short for the ring");
    if (2 * M + N > 65535) return forge::fail(FORGE_ERR_UNSUPPORTED, "delta_prepare: %d heads", 2 * M + N);
    if (T == 0 || S == 0) return FORGE_OK;
    const ShortConv cv{conv_w, taps, (int)C};
    const DeltaPrepare d{{proj, ld}, b_col, a_col, cv, state, stride, ring_off, tok_req, q_start, positions, slots, decay_rate, dt, qkv, g, beta, T, N, M, K, V};
    // several tiles one after the other in a warp as long as the SMs stay full
    int tiles = 1;
    while (tiles < 4 && (long long)(T / (4 * kPrepTokens * 2 * tiles)) * (2 * M + N) >= 148 * 8) tiles *= 2;
    const int per_cta = 4 * kPrepTokens * tiles;
    auto kernel = taps <= 4 ? (K <= 64 ? delta_prepare_kernel<2, 4> : K <= 128 ? delta_prepare_kernel<4, 4> : delta_prepare_kernel<kUnitRegs, 4>)
                            : (K <= 64 ? delta_prepare_kernel<2, 8> : K <= 128 ? delta_prepare_kernel<4, 8> : delta_prepare_kernel<kUnitRegs, 8>);
    cudaError_t e = forge::launch(kernel, dim3((T + per_cta - 1) / per_cta, 2 * M + N), dim3(128), 0, stream, 1, d, tiles);
    if (e != cudaSuccess) return forge::check_launch("delta_prepare", e);
    e = forge::launch(conv_keep_kernel, dim3(S, (unsigned)((C + 255) / 256)), dim3(256), 0, stream, 1, Columns{proj, ld}, cv, state, stride, ring_off,
                      q_start, positions, slots);
    return forge::check_launch("delta_prepare (ring)", e);
}

extern "C" int forge_silu_columns(float* x, long long ld, int T, int n, cudaStream_t stream) {
    if (T < 0 || n <= 0 || ld < n) return forge::fail(FORGE_ERR_ARG, "silu_columns: bad sizes T=%d n=%d ld=%lld", T, n, ld);
    if (T == 0) return FORGE_OK;
    const int vec = n % 4 == 0 && ld % 4 == 0 && ((uintptr_t)x & 15) == 0 ? 1 : 0;
    const int packs = vec ? n / 4 : n, per_row = (packs + 255) / 256;
    return forge::check_launch("silu_columns", forge::launch(silu_columns_kernel, dim3(T, T >= 592 ? (per_row + 3) / 4 : per_row), dim3(256), 0, stream, 1, x, ld, n, vec));
}

// o fp32 [T, n], w fp32 [n], gate fp32 rows of ld_g; out of type dtype, rows of out_ld with the n values at their start.
extern "C" int forge_gated_rows(const float* o, const float* w, const float* gate, int ld_g, void* out, int dtype, long long out_ld, int T, int n,
                                float eps, cudaStream_t stream) {
    if (T < 0 || n <= 0 || ld_g < n || out_ld < n) return forge::fail(FORGE_ERR_ARG, "gated_rows: bad sizes T=%d n=%d", T, n);
    if (T == 0) return FORGE_OK;
    const int vec = n % 4 == 0 && ld_g % 4 == 0 && out_ld % 4 == 0 && (((uintptr_t)o | (uintptr_t)w | (uintptr_t)gate | (uintptr_t)out) & 15) == 0 ? 1 : 0;
    const int items = vec ? n / 4 : n, most = T <= 148 ? 512 : 128;
    int threads = (items + 31) / 32 * 32;
    threads = threads > most ? most : threads;
    cudaError_t e = cudaSuccess;
    FORGE_DISPATCH_DTYPE(dtype, TT,
        e = forge::launch(gated_rows_kernel<TT>, dim3(T), dim3(threads), 0, stream, 1, o, w, Columns{gate, ld_g}, (TT*)out, out_ld, n, eps, vec));
    return forge::check_launch("gated_rows", e);
}

// 1 if the kernel of single tokens takes heads of these sizes.
extern "C" int forge_token_state_supports(int K, int V, int delta) {
    if (K <= 0 || V <= 0) return 0;
    return token_shape(K, V, delta != 0, false).threads > 0 && (V % 4 != 0 || token_shape(K, V, delta != 0, true).threads > 0) ? 1 : 0;
}

// The gated delta rule where every request brings one token (S tokens, request s's is token q_start[s]): convolutions, gates, the
// state's step, the head's norm (weight fp32 [V], eps) and silu of the gate; proj and state as in forge_delta_prepare, the gate's N*V
// columns from g_col on, request s's N states [K, V] at the start of its row; out of type dtype, rows of out_ld.
extern "C" int forge_gated_delta_token(const float* proj, int ld, int g_col, int b_col, int a_col, const float* conv_w, int taps, float* state,
                                       long long stride, long long ring_off, const int32_t* q_start, const int32_t* positions, const int32_t* slots,
                                       const float* decay_rate, const float* dt, const float* weight, float eps, void* out, int dtype,
                                       long long out_ld, int S, int N, int M, int K, int V, cudaStream_t stream) {
    const long long C = 2LL * M * K + (long long)N * V;
    if (S < 0 || N <= 0 || M <= 0 || N % M != 0 || K <= 0 || V <= 0 || taps <= 0 || ld < C || g_col < 0 || b_col < 0 || a_col < 0 || g_col + N * V > ld ||
        b_col + N > ld || a_col + N > ld || out_ld < (long long)N * V)
        return forge::fail(FORGE_ERR_ARG, "gated_delta_token: bad sizes S=%d N=%d M=%d K=%d V=%d taps=%d ld=%d", S, N, M, K, V, taps, ld);
    if (ring_off < (long long)N * K * V || stride < ring_off + taps * C) return forge::fail(FORGE_ERR_ARG, "gated_delta_token: state rows are too short");
    const bool vec = token_vec(state, stride, K, V);
    const TokenShape sh = token_shape(K, V, true, vec);
    if (sh.threads == 0) return forge::fail(FORGE_ERR_UNSUPPORTED, "gated_delta_token: heads of %d x %d channels", K, V);
    if (S == 0) return FORGE_OK;
    const TokenState d{{proj, ld}, {proj + M * K, ld}, {proj + 2 * M * K, ld}, {conv_w, taps, (int)C}, {proj + g_col, ld}, {proj + b_col, ld}, {proj + a_col, ld},
                       decay_rate, dt, state, stride, ring_off, q_start, positions, slots, weight, eps, N, M, K, V, sh.CG, sh.RG};
    cudaError_t e = cudaSuccess;
    FORGE_DISPATCH_DTYPE(dtype, TO,
        e = taps <= 4 ? launch_token<4, true>(vec, sh, dim3(S, N), stream, d, (TO*)out, out_ld) : launch_token<8, true>(vec, sh, dim3(S, N), stream, d, (TO*)out, out_ld));
    return forge::check_launch("gated_delta_token", e);
}

// Lightning attention where every request brings one token: q, k, v fp32 rows of ld numbers, BEFORE their silu, N heads each from
// columns 0, N*K and 2*N*K of proj; decay fp32 [N]; out fp32 [S, N*V], the heads as the recurrence leaves them.
extern "C" int forge_lightning_token(const float* proj, int ld, const float* decay, float* state, long long stride, const int32_t* q_start,
                                     const int32_t* slots, float* out, int S, int N, int K, int V, cudaStream_t stream) {
    if (S < 0 || N <= 0 || K <= 0 || V <= 0 || ld < N * (2 * K + V)) return forge::fail(FORGE_ERR_ARG, "lightning_token: bad sizes S=%d N=%d K=%d V=%d ld=%d", S, N, K, V, ld);
    if (stride < (long long)N * K * V) return forge::fail(FORGE_ERR_ARG, "lightning_token: state rows are too short");
    const bool vec = token_vec(state, stride, K, V);
    const TokenShape sh = token_shape(K, V, false, vec);
    if (sh.threads == 0) return forge::fail(FORGE_ERR_UNSUPPORTED, "lightning_token: heads of %d x %d channels", K, V);
    if (S == 0) return FORGE_OK;
    const TokenState d{{proj, ld}, {proj + N * K, ld}, {proj + 2 * N * K, ld}, {nullptr, 1, 0}, {nullptr, 0}, {nullptr, 0}, {nullptr, 0},
                       decay, nullptr, state, stride, 0, q_start, nullptr, slots, nullptr, 0.f, N, N, K, V, sh.CG, sh.RG};
    return forge::check_launch("lightning_token", launch_token<4, false>(vec, sh, dim3(S, N), stream, d, out, (long long)N * V));
}
