// The two recurrences whose decay is one number per head and token, eight tokens at a time (fp32 throughout):
//
//     gated delta rule   S <- g_t S;   S <- S + k_t (b_t (v_t - S^T k_t))^T;   o_t = S^T q_t
//     lightning          S <- g S + k_t v_t^T;   o_t = S^T q_t                                        (g fixed per head)
//
// With S the state before a block of tokens 0 .. 7, P_j = g_0 .. g_j and R_ij = g_{i+1} .. g_j, the rule written out over the block is
//     u_j = b_j (v_j - P_j S^T k_j - sum_{i<j} R_ij (k_i . k_j) u_i)            (lightning: u_j = v_j)
//     o_j = P_j S^T q_j + sum_{i<=j} R_ij (k_i . q_j) u_i
//     S  <- P_7 S + sum_i R_i7 k_i u_i^T
// so the sixteen looks at S do not wait for one another, and what does, the eight u_j of a column, is a triangle of 28 multiply-adds.  The
// products k_i . k_j and k_i . q_j are the same for all columns and heads that share q and k: gram_kernel makes them ahead.  Every R is
// the product of its decays (no quotients), so a decay of zero does no harm.
//
// A CTA has 16 columns of one head's S and walks a request's tokens of the step; eight threads share two columns (or one), thread q of
// them holds the rows (4m + e) with m % 8 == q, as pairs of rows that one instruction multiplies and adds (fma.rn.f32x2).  The next
// blocks' vectors are copied into a ring of staging buffers (cp.async) while the present one is worked on.
#include "common.cuh"

namespace {

constexpr int BT = 8, kCols = 16, kGramThreads = 64, kOStride = 12;
typedef unsigned long long u64;

__device__ __forceinline__ u64 fma2(u64 a, u64 b, u64 c) {
    u64 d;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
    return d;
}
__device__ __forceinline__ u64 mul2(u64 a, u64 b) {
    u64 d;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
    return d;
}
__device__ __forceinline__ u64 pack2(float lo, float hi) {
    u64 d;
    asm("mov.b64 %0, {%1, %2};" : "=l"(d) : "f"(lo), "f"(hi));
    return d;
}
__device__ __forceinline__ float2 unpack2(u64 v) {
    float2 d;
    asm("mov.b64 {%0, %1}, %2;" : "=f"(d.x), "=f"(d.y) : "l"(v));
    return d;
}
// 16 or 4 bytes into shared memory; ok == false: zeros
__device__ __forceinline__ void stage(float* dst, const float* src, int bytes, bool ok) {
    const uint32_t d = (uint32_t)__cvta_generic_to_shared(dst);
    if (bytes == 16) asm volatile("cp.async.ca.shared.global [%0], [%1], 16, %2;" ::"r"(d), "l"(src), "r"(ok ? 16 : 0) : "memory");
    else asm volatile("cp.async.ca.shared.global [%0], [%1], 4, %2;" ::"r"(d), "l"(src), "r"(ok ? 4 : 0) : "memory");
}

// The first block of request s in the row of all requests' blocks (a request's n tokens take at most n/8 + 1 of them).
__device__ __forceinline__ int first_block(const int32_t* __restrict__ q_start, int s) { return q_start[s] / BT + s; }

// gram[block][head of q and k][a][b]: k_a . q_b for a <= b, k_a . k_b for a > b.  One CTA per (block, head); rows of zeros for the tokens
// that a request's last block does not have.
__global__ void __launch_bounds__(kGramThreads)
gram_kernel(const float* __restrict__ q, int ld_q, const float* __restrict__ k, int ld_k, const int32_t* __restrict__ q_start, int S, int M, int K,
            int stride, float* __restrict__ gram) {
    extern __shared__ __align__(16) float sm[];          // [k_0 .. k_7 | q_0 .. q_7], rows of `stride` numbers
    forge::pdl_wait();
    const int block = blockIdx.x, head = blockIdx.y, tid = threadIdx.x;
    int lo = 0, hi = S - 1;                               // the last request whose first block is not behind this one
    while (lo < hi) {
        const int mid = (lo + hi + 1) / 2;
        if (first_block(q_start, mid) <= block) lo = mid;
        else hi = mid - 1;
    }
    const int t0 = q_start[lo] + (block - first_block(q_start, lo)) * BT, n = min(BT, q_start[lo + 1] - t0);
    if (n <= 0) return;
    for (int row = 0; row < BT; ++row)
        for (int c = tid; c < stride; c += kGramThreads) {
            const bool ok = row < n && c < K;
            sm[row * stride + c] = ok ? k[(size_t)(t0 + row) * ld_k + head * K + c] : 0.f;
            sm[(BT + row) * stride + c] = ok ? q[(size_t)(t0 + row) * ld_q + head * K + c] : 0.f;
        }
    __syncthreads();
    const int a = tid >> 3, b = tid & 7;
    const float4* x = reinterpret_cast<const float4*>(sm + a * stride);
    const float4* y = reinterpret_cast<const float4*>(sm + ((a <= b ? BT : 0) + b) * stride);
    float d0 = 0.f, d1 = 0.f, d2 = 0.f, d3 = 0.f;
    for (int i = 0; i < (K + 3) / 4; ++i) {
        const float4 u = x[i], v = y[i];
        d0 = fmaf(u.x, v.x, d0);
        d1 = fmaf(u.y, v.y, d1);
        d2 = fmaf(u.z, v.z, d2);
        d3 = fmaf(u.w, v.w, d3);
    }
    gram[((size_t)block * M + head) * (BT * BT) + tid] = (d0 + d1) + (d2 + d3);
}

struct BlockScan {
    const float *q, *k, *v;
    int ld_q, ld_k, ld_v;
    const float* gram;
    const float* g;                   // DELTA: decays [T, N]; else [N]
    const float* beta;                // DELTA: [T, N]
    float* state;
    long long stride;
    const int32_t *q_start, *slots;
    float* out;
    int N, M, K, KV, vec;
};

template <int KMAX, int CT, bool DELTA>
__global__ void __launch_bounds__(8 * kCols / CT)
block_scan_kernel(const BlockScan d) {
    constexpr int kThreads = 8 * kCols / CT;              // CT: columns of S per thread
    constexpr int C4 = KMAX / 32, LD = KMAX + 4;          // float4 pieces of a column per thread; row length of the staged vectors
    constexpr bool kHoldK = KMAX <= 64;                  // the keys stay in registers from the looks at S to its update
    constexpr int kStages = KMAX > 64 && KMAX <= 128 ? 4 : 2;      // blocks on their way (heads of 128: 514 us with two, 424 with four)
    __shared__ __align__(16) float ks[kStages][BT][LD], qs[kStages][BT][LD], vs[kStages][BT][kCols], gs[kStages][BT], bs[kStages][BT], grams[kStages][BT * BT];
    __shared__ __align__(16) float om[BT * kOStride], mm[BT * BT];
    forge::pdl_launch_dependents();
    const int s = blockIdx.x, head = blockIdx.y, tid = threadIdx.x, q = tid & 7, jp = tid >> 3;
    const int K = d.K, KV = d.KV, N = d.N, hk = head / (N / d.M);
    const int col0 = blockIdx.z * kCols, j0 = col0 + CT * jp;
    // channels beyond K stay zero: the copies never touch them
    for (int i = tid; i < kStages * BT * LD; i += kThreads) { (&ks[0][0][0])[i] = 0.f; (&qs[0][0][0])[i] = 0.f; }
    __syncthreads();
    forge::pdl_wait();
    const int t_lo = d.q_start[s], t_hi = d.q_start[s + 1];
    if (t_lo >= t_hi) return;
    float* S_g = d.state + (size_t)d.slots[s] * d.stride + (size_t)head * K * KV;
    auto row_of = [&](int ii) { return ((ii >> 2) * 8 + q) * 4 + (ii & 3); };
    u64 S2[CT][C4 * 2];
#pragma unroll
    for (int c = 0; c < CT; ++c)
#pragma unroll
        for (int ii = 0; ii < C4 * 4; ii += 2) {
            const bool ok = j0 + c < KV;
            const float lo = ok && row_of(ii) < K ? S_g[(size_t)row_of(ii) * KV + j0 + c] : 0.f;
            const float hi = ok && row_of(ii + 1) < K ? S_g[(size_t)row_of(ii + 1) * KV + j0 + c] : 0.f;
            S2[c][ii / 2] = pack2(lo, hi);
        }
    const int piece = d.vec ? 4 : 1, pieces = K / piece, dq = kThreads / pieces, dr = kThreads % pieces, tt0 = tid / pieces, ch0 = tid % pieces;
    const float fixed = DELTA ? 0.f : d.g[head];
    const float* gram_g = d.gram + ((size_t)first_block(d.q_start, s) * d.M + hk) * (BT * BT);
    auto fetch = [&](int buf, int tb) {
        const int n = min(BT, t_hi - tb);
        for (int tt = tt0, ch = ch0; tt < BT;) {
            const size_t t = (size_t)(tt < n ? tb + tt : tb), c = (size_t)hk * K + ch * piece;
            stage(&ks[buf][tt][ch * piece], d.k + t * d.ld_k + c, piece * 4, tt < n);
            stage(&qs[buf][tt][ch * piece], d.q + t * d.ld_q + c, piece * 4, tt < n);
            ch += dr;
            tt += dq;
            if (ch >= pieces) { ch -= pieces; ++tt; }
        }
#pragma unroll
        for (int i = tid; i < BT * kCols; i += kThreads) {
            const int tt = i / kCols, jc = col0 + i % kCols;
            const bool ok = tt < n && jc < KV;
            stage(&vs[buf][tt][i % kCols], ok ? d.v + (size_t)(tb + tt) * d.ld_v + (size_t)head * KV + jc : d.v, 4, ok);
        }
        if (tid < BT * BT / 4) stage(&grams[buf][4 * tid], gram_g + (size_t)((tb - t_lo) / BT) * d.M * (BT * BT) + 4 * tid, 16, true);
        if (DELTA && tid < BT) {
            const size_t at = (size_t)(tid < n ? tb + tid : tb) * N + head;
            if (tid < n) stage(&gs[buf][tid], d.g + at, 4, true);
            else gs[buf][tid] = 1.0f;
            stage(&bs[buf][tid], d.beta + at, 4, tid < n);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
#pragma unroll
    for (int i = 0; i < kStages - 1; ++i) {
        if (t_lo + i * BT < t_hi) fetch(i, t_lo + i * BT);
        else asm volatile("cp.async.commit_group;" ::: "memory");
    }
    int buf = 0;
    for (int tb = t_lo; tb < t_hi; tb += BT, buf = buf + 1 < kStages ? buf + 1 : 0) {
        const int n = min(BT, t_hi - tb);
        asm volatile("cp.async.wait_group %0;" ::"n"(kStages - 2) : "memory");
        __syncthreads();                                  // the block has landed for every thread, and the one before is done with
        if (tb + (kStages - 1) * BT < t_hi) fetch(buf > 0 ? buf - 1 : kStages - 1, tb + (kStages - 1) * BT);
        else asm volatile("cp.async.commit_group;" ::: "memory");
        float g[BT];
        if (DELTA) {
            *reinterpret_cast<float4*>(&g[0]) = *reinterpret_cast<const float4*>(&gs[buf][0]);
            *reinterpret_cast<float4*>(&g[4]) = *reinterpret_cast<const float4*>(&gs[buf][4]);
        } else {
#pragma unroll
            for (int l = 0; l < BT; ++l) g[l] = l < n ? fixed : 1.0f;
        }
        // the triangles with their decays: thread (a, b) = (tid / 8, tid % 8) does entry (a, b)
        if (kThreads == BT * BT || tid < BT * BT) {
            const int a = tid >> 3, b = tid & 7, lo = min(a, b), hi = max(a, b);
            float r = grams[buf][tid];
#pragma unroll
            for (int l = 0; l < BT; ++l) r *= l > lo && l <= hi ? g[l] : 1.0f;
            om[b * kOStride + a] = a <= b ? r : 0.f;      // token b's output takes R_ab (k_a . q_b) u_a
            if (DELTA && a > b) mm[a * BT + b] = r;       // token a's write takes R_ba (k_b . k_a) u_b
        }
        // the looks at S: partial sums of S^T k_t and S^T q_t over this thread's rows, pairs of rows side by side
        u64 A[DELTA ? BT : 1][CT], B[BT][CT], kh[kHoldK ? BT : 1][C4 * 2];
#pragma unroll
        for (int tt = 0; tt < BT; ++tt) {
            const ulonglong2* k4 = reinterpret_cast<const ulonglong2*>(&ks[buf][tt][0]) + q;
            const ulonglong2* q4 = reinterpret_cast<const ulonglong2*>(&qs[buf][tt][0]) + q;
#pragma unroll
            for (int c4 = 0; c4 < C4; ++c4) {
                const ulonglong2 qq = q4[c4 * 8];
                ulonglong2 kk{};
                if (DELTA || kHoldK) kk = k4[c4 * 8];
                if (kHoldK) { kh[kHoldK ? tt : 0][2 * c4] = kk.x; kh[kHoldK ? tt : 0][2 * c4 + 1] = kk.y; }
#pragma unroll
                for (int c = 0; c < CT; ++c) {
                    B[tt][c] = c4 == 0 ? mul2(S2[c][0], qq.x) : fma2(S2[c][2 * c4], qq.x, B[tt][c]);
                    B[tt][c] = fma2(S2[c][2 * c4 + 1], qq.y, B[tt][c]);
                    if (DELTA) {
                        u64& x = A[DELTA ? tt : 0][c];
                        x = c4 == 0 ? mul2(S2[c][0], kk.x) : fma2(S2[c][2 * c4], kk.x, x);
                        x = fma2(S2[c][2 * c4 + 1], kk.y, x);
                    }
                }
            }
        }
        // the eight threads' sums meet so that thread q ends with token q's
        float a1[CT], b1[CT];
#pragma unroll
        for (int c = 0; c < CT; ++c) {
            float x[BT], y[BT];
#pragma unroll
            for (int tt = 0; tt < BT; ++tt) {
                const float2 p = unpack2(B[tt][c]);
                y[tt] = p.x + p.y;
                if (DELTA) {
                    const float2 r = unpack2(A[DELTA ? tt : 0][c]);
                    x[tt] = r.x + r.y;
                }
            }
#pragma unroll
            for (int w = 4; w >= 1; w >>= 1) {
                const bool up = q & w;
#pragma unroll
                for (int tt = 0; tt < w; ++tt) {
                    const float sy = up ? y[tt] : y[tt + w], ky = up ? y[tt + w] : y[tt];
                    y[tt] = ky + __shfl_xor_sync(0xffffffffu, sy, w);
                    if (DELTA) {
                        const float sx = up ? x[tt] : x[tt + w], kx = up ? x[tt + w] : x[tt];
                        x[tt] = kx + __shfl_xor_sync(0xffffffffu, sx, w);
                    }
                }
            }
            b1[c] = y[0];
            a1[c] = DELTA ? x[0] : 0.f;
        }
        float p_q = 1.f;                                  // P of token q
#pragma unroll
        for (int l = 0; l < BT; ++l) p_q *= l <= q ? g[l] : 1.0f;
        __syncthreads();                                  // the triangles stand
        // the writes u of both columns, all eight tokens, in every thread
        float u[BT][CT];
        if (DELTA) {
            float mine[CT];
#pragma unroll
            for (int c = 0; c < CT; ++c) mine[c] = fmaf(-p_q, a1[c], vs[buf][q][CT * jp + c]);
#pragma unroll
            for (int j = 0; j < BT; ++j) {
#pragma unroll
                for (int c = 0; c < CT; ++c) u[j][c] = __shfl_sync(0xffffffffu, mine[c], j, 8);
            }
            float bt[BT];
            *reinterpret_cast<float4*>(&bt[0]) = *reinterpret_cast<const float4*>(&bs[buf][0]);
            *reinterpret_cast<float4*>(&bt[4]) = *reinterpret_cast<const float4*>(&bs[buf][4]);
#pragma unroll
            for (int j = 0; j < BT; ++j) {
                float m[BT];
                *reinterpret_cast<float4*>(&m[0]) = *reinterpret_cast<const float4*>(&mm[j * BT]);
                if (j > 4) *reinterpret_cast<float4*>(&m[4]) = *reinterpret_cast<const float4*>(&mm[j * BT + 4]);
#pragma unroll
                for (int c = 0; c < CT; ++c) {
#pragma unroll
                    for (int i = 0; i < j; ++i) u[j][c] = fmaf(-m[i], u[i][c], u[j][c]);
                    u[j][c] *= bt[j];
                }
            }
        } else {
#pragma unroll
            for (int j = 0; j < BT; ++j) {
#pragma unroll
                for (int c = 0; c < CT; ++c) u[j][c] = vs[buf][j][CT * jp + c];
            }
        }
        // token q's output
        {
            float om8[BT];
            *reinterpret_cast<float4*>(&om8[0]) = *reinterpret_cast<const float4*>(&om[q * kOStride]);
            *reinterpret_cast<float4*>(&om8[4]) = *reinterpret_cast<const float4*>(&om[q * kOStride + 4]);
#pragma unroll
            for (int c = 0; c < CT; ++c) {
                float o = p_q * b1[c];
#pragma unroll
                for (int i = 0; i < BT; ++i) o = fmaf(om8[i], u[i][c], o);
                if (q < n && j0 + c < KV) d.out[(size_t)(tb + q) * N * KV + (size_t)head * KV + j0 + c] = o;
            }
        }
        // the state after the block
        float w = 1.f;
        u64 uw[BT][CT];
#pragma unroll
        for (int i = BT - 1; i >= 0; --i) {
#pragma unroll
            for (int c = 0; c < CT; ++c) uw[i][c] = pack2(w * u[i][c], w * u[i][c]);
            w *= g[i];
        }
        const u64 w2 = pack2(w, w);
#pragma unroll
        for (int c = 0; c < CT; ++c)
#pragma unroll
            for (int ii = 0; ii < C4 * 2; ++ii) S2[c][ii] = mul2(S2[c][ii], w2);
#pragma unroll
        for (int tt = 0; tt < BT; ++tt) {
            const ulonglong2* k4 = reinterpret_cast<const ulonglong2*>(&ks[buf][tt][0]) + q;
#pragma unroll
            for (int c4 = 0; c4 < C4; ++c4) {
                ulonglong2 kk;
                if (kHoldK) { kk.x = kh[kHoldK ? tt : 0][2 * c4]; kk.y = kh[kHoldK ? tt : 0][2 * c4 + 1]; }
                else kk = k4[c4 * 8];
#pragma unroll
                for (int c = 0; c < CT; ++c) {
                    S2[c][2 * c4] = fma2(kk.x, uw[tt][c], S2[c][2 * c4]);
                    S2[c][2 * c4 + 1] = fma2(kk.y, uw[tt][c], S2[c][2 * c4 + 1]);
                }
            }
        }
    }
#pragma unroll
    for (int c = 0; c < CT; ++c)
#pragma unroll
        for (int ii = 0; ii < C4 * 4; ii += 2) {
            const float2 p = unpack2(S2[c][ii / 2]);
            if (j0 + c < KV && row_of(ii) < K) S_g[(size_t)row_of(ii) * KV + j0 + c] = p.x;
            if (j0 + c < KV && row_of(ii + 1) < K) S_g[(size_t)row_of(ii + 1) * KV + j0 + c] = p.y;
        }
}

template <bool DELTA>
int run(BlockScan d, float* gram, int T, int S, cudaStream_t stream) {
    const int stride = (d.K + 3) / 4 * 4 + 4, blocks = T / BT + S;
    cudaError_t e = forge::launch(gram_kernel, dim3(blocks, d.M), dim3(kGramThreads), sizeof(float) * 2 * BT * stride, stream, 1, d.q, d.ld_q, d.k, d.ld_k,
                                  d.q_start, S, d.M, d.K, stride, gram);
    if (e != cudaSuccess) return forge::check_launch("block_scan (products)", e);
    auto aligned = [](const float* p, int ld) { return ((uintptr_t)p & 15) == 0 && ld % 4 == 0; };
    d.gram = gram;
    d.vec = d.K % 4 == 0 && aligned(d.q, d.ld_q) && aligned(d.k, d.ld_k) ? 1 : 0;
    const dim3 grid(S, d.N, (d.KV + kCols - 1) / kCols);
    const int kmax = (d.K + 31) / 32 * 32;
    // a column per thread where the CTAs do not even fill the SMs (one request, 32 heads of 64 x 64: 245 us for 2,048 tokens, with two
    // columns 290), else two (64 heads: 304 us, with one column 336)
    const bool few = (long long)S * d.N * grid.z <= 148;
#define FORGE_BLOCK_CASE(KM, CT) \
    if (kmax <= KM) return forge::check_launch("block_scan", forge::launch(block_scan_kernel<KM, CT, DELTA>, grid, dim3(8 * kCols / CT), 0, stream, 1, d));
    if (few) {
        FORGE_BLOCK_CASE(32, 1) FORGE_BLOCK_CASE(64, 1)
    }
    FORGE_BLOCK_CASE(32, 2) FORGE_BLOCK_CASE(64, 2) FORGE_BLOCK_CASE(96, 2) FORGE_BLOCK_CASE(128, 2) FORGE_BLOCK_CASE(192, 2) FORGE_BLOCK_CASE(256, 2)
#undef FORGE_BLOCK_CASE
    return forge::fail(FORGE_ERR_UNSUPPORTED, "block_scan: heads of %d key channels (at most 256)", d.K);
}

int check(const char* what, int T, int S, int N, int M, int K, int KV, long long stride) {
    if (T < 0 || S < 0 || N <= 0 || M <= 0 || N % M != 0 || K <= 0 || KV <= 0) return forge::fail(FORGE_ERR_ARG, "%s: bad sizes S=%d N=%d M=%d K=%d V=%d", what, S, N, M, K, KV);
    if (K > 256) return forge::fail(FORGE_ERR_UNSUPPORTED, "%s: heads of %d key channels (at most 256)", what, K);
    if (N > 65535 || (KV + kCols - 1) / kCols > 65535) return forge::fail(FORGE_ERR_UNSUPPORTED, "%s: %d heads of %d value channels", what, N, KV);
    if (stride < (long long)N * K * KV) return forge::fail(FORGE_ERR_ARG, "%s: state rows are too short", what);
    return FORGE_OK;
}

}  // namespace

extern "C" int forge_silu_columns(float* x, long long ld, int T, int n, cudaStream_t stream);       // recurrent_token.cu

// Gated delta rule over the step's tokens: per head n, with q and k of head n / (N / M).  q, k fp32 (row t at p + t * ld, M heads of K
// channels), v fp32 (N heads of KV channels), g and beta fp32 [T, N]; gram: fp32 scratch, 64 * M * (T / 8 + S) numbers; out fp32 [T, N*KV]; a
// head's state is [K, KV], row slots[s] of `state` (rows of state_stride numbers) holds request s's N of them from its start.
extern "C" int forge_gated_delta_scan(const float* q, int ld_q, const float* k, int ld_k, const float* v, int ld_v, const float* g,
                                      const float* beta, float* gram, float* state, long long state_stride, const int32_t* q_start,
                                      const int32_t* slots, float* out, int T, int S, int N, int M, int K, int KV, cudaStream_t stream) {
    const int rc = check("gated_delta_scan", T, S, N, M, K, KV, state_stride);
    if (rc != FORGE_OK || S == 0 || T == 0) return rc;
    return run<true>(BlockScan{q, k, v, ld_q, ld_k, ld_v, nullptr, g, beta, state, state_stride, q_start, slots, out, N, M, K, KV, 0}, gram, T, S, stream);
}

// Lightning attention over the step's tokens: fp32 rows of ld numbers [q: N*K | k: N*K | v: N*KV] from proj on pass silu IN PLACE, then the
// recurrence with decay fp32 [N]; gram: fp32 scratch, 64 * N * (T / 8 + S) numbers; out fp32 [T, N*KV]; the state as above.
extern "C" int forge_lightning_scan(float* proj, int ld, const float* decay, float* gram, float* state, long long state_stride,
                                    const int32_t* q_start, const int32_t* slots, float* out, int T, int S, int N, int K, int KV, cudaStream_t stream) {
    int rc = check("lightning_scan", T, S, N, N, K, KV, state_stride);
    if (rc == FORGE_OK && ld < N * (2 * K + KV)) rc = forge::fail(FORGE_ERR_ARG, "lightning_scan: rows of %d are too short", ld);
    if (rc != FORGE_OK || S == 0 || T == 0) return rc;
    rc = forge_silu_columns(proj, ld, T, N * (2 * K + KV), stream);
    if (rc != FORGE_OK) return rc;
    return run<false>(BlockScan{proj, proj + N * K, proj + 2 * N * K, ld, ld, ld, nullptr, decay, nullptr, state, state_stride, q_start, slots, out, N, N, K, KV, 0},
                      gram, T, S, stream);
}
