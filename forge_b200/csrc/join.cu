// Several sublayers' outputs join the residual stream at once, some of them normed first, and the next layer's input norm follows:
//
//     x <- x + sum_i scale_i * n_i(y_i),    n_i(y) = y / sqrt(mean(y^2) + eps) * w_i   (or y itself, where a term has no w)
//     h  = x / sqrt(mean(x^2) + next_eps) * next_w                                      (if asked for)
//
// x, y_i, w_i fp32, h in the activation type.  The terms' sum is taken in their order before x is added to it.  Every mean runs in the
// fixed tree of block_sum, so a token's numbers do not depend on what else the step brings.
#include "common.cuh"

namespace {

constexpr int kMaxTerms = 4, kMaxThreads = 512;

struct Term {
    const float* y;
    const float* w;                    // or null
    float scale;
};

struct Join {
    Term term[kMaxTerms];
    int n;
    float eps;
    float* x;
    const float* next_w;               // or null
    float next_eps;
    int W;
};

template <int V> struct Pack;
template <> struct Pack<1> { using type = float; };
template <> struct Pack<4> { using type = float4; };
__device__ __forceinline__ float& lane_of(float& v, int) { return v; }
__device__ __forceinline__ float& lane_of(float4& v, int i) { return (&v.x)[i]; }

template <typename TOut, int V>
__device__ __forceinline__ void store_pack(TOut* p, const typename Pack<V>::type& v);
template <> __device__ __forceinline__ void store_pack<float, 1>(float* p, const float& v) { *p = v; }
template <> __device__ __forceinline__ void store_pack<__nv_bfloat16, 1>(__nv_bfloat16* p, const float& v) { *p = __float2bfloat16_rn(v); }
template <> __device__ __forceinline__ void store_pack<float, 4>(float* p, const float4& v) { *reinterpret_cast<float4*>(p) = v; }
template <> __device__ __forceinline__ void store_pack<__nv_bfloat16, 4>(__nv_bfloat16* p, const float4& v) {
    const __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&lo), *reinterpret_cast<const uint32_t*>(&hi));
}

// One CTA per row; thread i takes the packs i, i + blockDim, ... of V channels in every walk, so what it keeps in shared memory (the
// normed terms, W floats each, if they fit: `keep`; and the new x) it reads back itself.
template <typename TOut, int V>
__global__ void __launch_bounds__(kMaxThreads)
join_kernel(const Join d, TOut* __restrict__ h, int keep) {
    using P = typename Pack<V>::type;
    extern __shared__ __align__(16) float u[];
    __shared__ float red[32];
    forge::pdl_launch_dependents();
    forge::pdl_wait();
    const int W = d.W, packs = W / V;
    const size_t row = (size_t)blockIdx.x * W;
    float factor[kMaxTerms], part[kMaxTerms];
#pragma unroll
    for (int k = 0; k < kMaxTerms; ++k) part[k] = 0.f;
    float* kept = u + W;               // [term][W]
#pragma unroll 2
    for (int i = threadIdx.x; i < packs; i += blockDim.x) {
#pragma unroll
        for (int k = 0; k < kMaxTerms; ++k) {
            if (k >= d.n || !d.term[k].w) continue;
            P y = __ldg(reinterpret_cast<const P*>(d.term[k].y + row) + i);
            if (keep) *reinterpret_cast<P*>(kept + (size_t)k * W + (size_t)i * V) = y;
#pragma unroll
            for (int e = 0; e < V; ++e) part[k] = fmaf(lane_of(y, e), lane_of(y, e), part[k]);
        }
    }
#pragma unroll
    for (int k = 0; k < kMaxTerms; ++k) {
        factor[k] = 0.f;
        if (k >= d.n) continue;
        factor[k] = d.term[k].scale;
        if (d.term[k].w) factor[k] *= 1.0f / sqrtf(forge::block_sum(part[k], red) / (float)W + d.eps);
    }
    float ss = 0.f;
    for (int i = threadIdx.x; i < packs; i += blockDim.x) {
        P x = reinterpret_cast<const P*>(d.x + row)[i], s{};
#pragma unroll
        for (int k = 0; k < kMaxTerms; ++k) {
            if (k >= d.n) continue;
            P y = keep && d.term[k].w ? *reinterpret_cast<const P*>(kept + (size_t)k * W + (size_t)i * V)
                                      : __ldg(reinterpret_cast<const P*>(d.term[k].y + row) + i);
            if (d.term[k].w) {
                P w = __ldg(reinterpret_cast<const P*>(d.term[k].w) + i);
#pragma unroll
                for (int e = 0; e < V; ++e) lane_of(y, e) *= lane_of(w, e);
            }
#pragma unroll
            for (int e = 0; e < V; ++e) lane_of(s, e) = fmaf(factor[k], lane_of(y, e), lane_of(s, e));
        }
#pragma unroll
        for (int e = 0; e < V; ++e) {
            lane_of(x, e) += lane_of(s, e);
            ss = fmaf(lane_of(x, e), lane_of(x, e), ss);
        }
        reinterpret_cast<P*>(d.x + row)[i] = x;
        if (d.next_w) *reinterpret_cast<P*>(u + (size_t)i * V) = x;
    }
    if (d.next_w == nullptr) return;
    const float inv = 1.0f / sqrtf(forge::block_sum(ss, red) / (float)W + d.next_eps);
    for (int i = threadIdx.x; i < packs; i += blockDim.x) {
        P x = *reinterpret_cast<const P*>(u + (size_t)i * V), w = __ldg(reinterpret_cast<const P*>(d.next_w) + i);
#pragma unroll
        for (int e = 0; e < V; ++e) lane_of(x, e) *= inv * lane_of(w, e);
        store_pack<TOut, V>(h + row + (size_t)i * V, x);
    }
}

constexpr int kSmemLimit = 200 * 1024;
forge::PerDeviceFlag g_attr[2][2];

template <typename TOut, int V>
cudaError_t run(const Join& d, void* h, int T, cudaStream_t stream) {
    bool& done = g_attr[sizeof(TOut) == 2][V == 4].current();
    if (!done) {
        cudaError_t e = cudaFuncSetAttribute(join_kernel<TOut, V>, cudaFuncAttributeMaxDynamicSharedMemorySize, kSmemLimit);
        if (e != cudaSuccess) return e;
        done = true;
    }
    // few rows: as many threads as the row has packs, so that a walk is one trip to memory; many rows: two packs a thread
    int threads = (d.W / V + 31) / 32 * 32;
    if (T > 148) threads = (threads / 2 + 31) / 32 * 32;
    threads = threads < 32 ? 32 : (threads > kMaxThreads ? kMaxThreads : threads);
    int last = 0;                       // terms up to the last normed one have room in shared memory
    for (int k = 0; k < d.n; ++k)
        if (d.term[k].w) last = k + 1;
    size_t smem = sizeof(float) * (size_t)d.W * (1 + last);
    const int keep = last > 0 && smem <= 64 * 1024 ? 1 : 0;
    if (!keep) smem = sizeof(float) * (size_t)d.W;
    return forge::launch(join_kernel<TOut, V>, dim3(T), dim3(threads), d.next_w || keep ? smem : 0, stream, 1, d, (TOut*)h, keep);
}

}  // namespace

// y0 .. y3 fp32 [T, W] (the first n are used), w0 .. w3 fp32 [W] or null, s0 .. s3 their factors; x fp32 [T, W]; next_w fp32 [W] and h
// [T, W] of out_dtype, or both null.
extern "C" int forge_join(float* x, int n, const float* y0, const float* w0, float s0, const float* y1, const float* w1, float s1, const float* y2,
                          const float* w2, float s2, const float* y3, const float* w3, float s3, float eps, const float* next_w, float next_eps,
                          void* h, int out_dtype, int T, int W, cudaStream_t stream) {
    if (T < 0 || W <= 0 || n < 1 || n > kMaxTerms) return forge::fail(FORGE_ERR_ARG, "join: bad sizes T=%d W=%d n=%d", T, W, n);
    const Join d{{{y0, w0, s0}, {y1, w1, s1}, {y2, w2, s2}, {y3, w3, s3}}, n, eps, x, next_w, next_eps, W};
    uintptr_t ptrs = (uintptr_t)x | (uintptr_t)next_w | (uintptr_t)h;
    for (int k = 0; k < n; ++k) {
        if (!d.term[k].y) return forge::fail(FORGE_ERR_ARG, "join: term %d of %d is missing", k, n);
        ptrs |= (uintptr_t)d.term[k].y | (uintptr_t)d.term[k].w;
    }
    if ((next_w == nullptr) != (h == nullptr)) return forge::fail(FORGE_ERR_ARG, "join: the next norm needs its weight and its output");
    if (next_w && sizeof(float) * (size_t)W > (size_t)kSmemLimit) return forge::fail(FORGE_ERR_UNSUPPORTED, "join: rows of %d channels", W);
    if (T == 0) return FORGE_OK;
    const bool vec = W % 4 == 0 && (ptrs & 15) == 0;
    cudaError_t e = cudaSuccess;
    FORGE_DISPATCH_DTYPE(out_dtype, TO, e = vec ? run<TO, 4>(d, h, T, stream) : run<TO, 1>(d, h, T, stream));
    return forge::check_launch("join", e);
}
