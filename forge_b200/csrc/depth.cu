// What a layer does to the residual stream when its sublayers' outputs are gated and the stream is averaged over the depth.
//
// The stream's history is kept as planes of fp32 rows [T, W]: plane j holds X_j (j = 0: the embedding output, j = i + 1: what
// layer i left).  With x the layer's input, y1 and y2 its sublayers' outputs and z1, z2 their gates before the sigmoid,
//
//     X_new = x + (y1 * sigmoid(z1) + y2 * sigmoid(z2))                   (no z: no gate; no y2: one sublayer)
//     s     = sum_j c[j] X_j + c[n-1] X_new        over the n - 1 planes before it   (no c: s = X_new)
//
// s is the next layer's x, and the pass that makes it also leaves that layer's normed input: a layer norm
// (s - mean) / sqrt(var + eps) * w (+ b), or an RMS norm.  Everything is fp32; the planes are added in the order j = 0, 1, ...,
// and the norm's sums run in the fixed tree of block_sum, so a token's numbers do not depend on what else the step brings.
#include "common.cuh"

namespace {

constexpr int kMaxThreads = 512;

struct DepthStep {
    float* planes;                 // plane j at planes + j * plane
    long long plane;
    int n;                         // numbers in c (planes 0 .. n-2 are read); 0: no average
    int x_plane, new_plane, s_plane;      // where x lies; where X_new and s go (-1: nowhere)
    const float* c;
    const float* y1;
    const float* y2;               // or null
    const float* z;                // gates, rows of ld_z numbers: z1 from column z1, z2 from column z2; null: none
    int ld_z, z1, z2;
    const float* w;                // the next norm's weight (null: no norm follows) and bias (or null)
    const float* b;
    int center;                    // 1: layer norm, 0: RMS norm
    float eps;
    const int32_t* rows;           // the tokens to work on, or null: all
    int W;
};

template <int V> struct Pack;
template <> struct Pack<1> { using type = float; };
template <> struct Pack<4> { using type = float4; };
__device__ __forceinline__ float& lane_of(float& v, int) { return v; }
__device__ __forceinline__ float& lane_of(float4& v, int i) { return (&v.x)[i]; }
__device__ __forceinline__ float sigmoidf(float x) { return 1.0f / (1.0f + expf(-x)); }

template <typename TOut, int V>
__device__ __forceinline__ void store_pack(TOut* p, const typename Pack<V>::type& v);
template <> __device__ __forceinline__ void store_pack<float, 1>(float* p, const float& v) { *p = v; }
template <> __device__ __forceinline__ void store_pack<__nv_bfloat16, 1>(__nv_bfloat16* p, const float& v) { *p = __float2bfloat16_rn(v); }
template <> __device__ __forceinline__ void store_pack<float, 4>(float* p, const float4& v) { *reinterpret_cast<float4*>(p) = v; }
template <> __device__ __forceinline__ void store_pack<__nv_bfloat16, 4>(__nv_bfloat16* p, const float4& v) {
    const __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&lo), *reinterpret_cast<const uint32_t*>(&hi));
}

// One CTA per row; thread i takes the packs i, i + blockDim, ... of V channels in every walk, so what it keeps of s in shared
// memory (u, W floats) it reads back itself.
template <typename TOut, int V>
__global__ void __launch_bounds__(kMaxThreads)
depth_step_kernel(const DepthStep d, TOut* __restrict__ normed) {
    using P = typename Pack<V>::type;
    extern __shared__ __align__(16) float u[];
    __shared__ float red[32];
    forge::pdl_launch_dependents();
    forge::pdl_wait();
    const int t = d.rows ? d.rows[blockIdx.x] : blockIdx.x, W = d.W;
    const size_t row = (size_t)t * W;
    const float* zr = d.z ? d.z + (size_t)t * d.ld_z : nullptr;
    const P* xp = reinterpret_cast<const P*>(d.planes + (size_t)d.x_plane * d.plane + row);
    const P* y1 = reinterpret_cast<const P*>(d.y1 + row);
    const P* y2 = d.y2 ? reinterpret_cast<const P*>(d.y2 + row) : nullptr;
    const P* z1 = zr ? reinterpret_cast<const P*>(zr + d.z1) : nullptr;
    const P* z2 = zr && y2 ? reinterpret_cast<const P*>(zr + d.z2) : nullptr;
    const float* base = d.planes + row;
    const int packs = W / V;
    float sum = 0.f;
    for (int i = threadIdx.x; i < packs; i += blockDim.x) {
        // all loads ahead of the first store.  The planes that are summed are not written here (x's own may be, by this thread)
        P x = xp[i], a = __ldg(y1 + i), b{}, ga{}, gb{}, s{};
        if (y2) b = __ldg(y2 + i);
        if (z1) ga = __ldg(z1 + i);
        if (z2) gb = __ldg(z2 + i);
#pragma unroll 2
        for (int j = 0; j < d.n - 1; ++j) {
            P h = __ldg(reinterpret_cast<const P*>(base + (size_t)j * d.plane) + i);
            const float cj = d.c[j];
#pragma unroll
            for (int e = 0; e < V; ++e) lane_of(s, e) = fmaf(cj, lane_of(h, e), lane_of(s, e));
        }
#pragma unroll
        for (int e = 0; e < V; ++e) {
            if (z1) lane_of(a, e) *= sigmoidf(lane_of(ga, e));
            if (z2) lane_of(b, e) *= sigmoidf(lane_of(gb, e));
            lane_of(x, e) += y2 ? lane_of(a, e) + lane_of(b, e) : lane_of(a, e);              // X_new
        }
        if (d.new_plane >= 0) *reinterpret_cast<P*>(d.planes + (size_t)d.new_plane * d.plane + row + (size_t)i * V) = x;
        if (d.n > 0) {
            const float cn = d.c[d.n - 1];
#pragma unroll
            for (int e = 0; e < V; ++e) lane_of(s, e) = fmaf(cn, lane_of(x, e), lane_of(s, e));
        } else {
            s = x;
        }
        if (d.s_plane >= 0) *reinterpret_cast<P*>(d.planes + (size_t)d.s_plane * d.plane + row + (size_t)i * V) = s;
        if (d.w) {
            *reinterpret_cast<P*>(u + (size_t)i * V) = s;
#pragma unroll
            for (int e = 0; e < V; ++e) sum += d.center ? lane_of(s, e) : lane_of(s, e) * lane_of(s, e);
        }
    }
    if (d.w == nullptr) return;
    float mean = 0.f;
    sum = forge::block_sum(sum, red) / (float)W;
    if (d.center) {
        mean = sum;
        float ss = 0.f;
        for (int i = threadIdx.x; i < packs; i += blockDim.x) {
            P s = *reinterpret_cast<const P*>(u + (size_t)i * V);
#pragma unroll
            for (int e = 0; e < V; ++e) {
                const float v = lane_of(s, e) - mean;
                ss = fmaf(v, v, ss);
            }
        }
        sum = forge::block_sum(ss, red) / (float)W;
    }
    const float inv = 1.0f / sqrtf(sum + d.eps);
    TOut* o = normed + (size_t)blockIdx.x * W;
    for (int i = threadIdx.x; i < packs; i += blockDim.x) {
        P s = *reinterpret_cast<const P*>(u + (size_t)i * V), w = reinterpret_cast<const P*>(d.w)[i], b{};
        if (d.b) b = reinterpret_cast<const P*>(d.b)[i];
#pragma unroll
        for (int e = 0; e < V; ++e) lane_of(s, e) = fmaf((lane_of(s, e) - mean) * inv, lane_of(w, e), lane_of(b, e));
        store_pack<TOut, V>(o + (size_t)i * V, s);
    }
}

constexpr int kSmemLimit = 200 * 1024;
forge::PerDeviceFlag g_attr[2][2];

template <typename TOut, int V>
cudaError_t run(const DepthStep& d, void* normed, int R, cudaStream_t stream) {
    const size_t smem = d.w ? sizeof(float) * (size_t)d.W : 0;
    bool& done = g_attr[sizeof(TOut) == 2][V == 4].current();
    if (!done) {
        cudaError_t e = cudaFuncSetAttribute(depth_step_kernel<TOut, V>, cudaFuncAttributeMaxDynamicSharedMemorySize, kSmemLimit);
        if (e != cudaSuccess) return e;
        done = true;
    }
    // few rows: as many threads as the row has packs, so that a row is one trip to memory; many rows: 128 (5.3 to 5.6 TB/s at rows of
    // 2,048 and 4,096 channels; 256 threads 4.5 to 5.4, 64 threads 3.4 to 5.6, fewer registers per thread slower at every size)
    int threads = (d.W / V + 31) / 32 * 32;
    const int most = R <= 148 ? kMaxThreads : 128;
    threads = threads < 32 ? 32 : (threads > most ? most : threads);
    return forge::launch(depth_step_kernel<TOut, V>, dim3(R), dim3(threads), smem, stream, 1, d, (TOut*)normed);
}

}  // namespace

// planes fp32 (plane j at planes + j * plane_stride, rows of W); y1, y2 (or null) fp32 [T, W]; z fp32 rows of ld_z (or null), the
// gates' columns from z1 and z2; c fp32 [n] (or null with n = 0); w (b optional) fp32 [W]: the norm that follows (null: none), its
// result in normed [R, W] of out_dtype; rows int32 [R] (or null: the tokens 0 .. R-1).  Plane indices of -1: not stored.
extern "C" int forge_depth_step(float* planes, long long plane_stride, int n, int x_plane, int new_plane, int s_plane, const float* c,
                                const float* y1, const float* y2, const float* z, int ld_z, int z1, int z2, const float* w, const float* b,
                                int center, float eps, void* normed, int out_dtype, const int32_t* rows, int R, int W, cudaStream_t stream) {
    if (R < 0 || W <= 0 || n < 0 || (n > 0) != (c != nullptr) || x_plane < 0 || !planes || !y1)
        return forge::fail(FORGE_ERR_ARG, "depth_step: bad sizes R=%d W=%d n=%d", R, W, n);
    if (z && (z1 < 0 || z2 < 0 || z1 + W > ld_z || (y2 && z2 + W > ld_z)))
        return forge::fail(FORGE_ERR_ARG, "depth_step: gates of %d channels from columns %d and %d do not fit rows of %d", W, z1, z2, ld_z);
    if ((w == nullptr) != (normed == nullptr)) return forge::fail(FORGE_ERR_ARG, "depth_step: the next norm needs its weight and its output");
    if (w && sizeof(float) * (size_t)W > (size_t)kSmemLimit) return forge::fail(FORGE_ERR_UNSUPPORTED, "depth_step: rows of %d channels", W);
    if (R == 0) return FORGE_OK;
    const DepthStep d{planes, plane_stride, n, x_plane, new_plane, s_plane, c, y1, y2, z, ld_z, z1, z2, w, b, center, eps, rows, W};
    const uintptr_t ptrs = (uintptr_t)planes | (uintptr_t)y1 | (uintptr_t)y2 | (uintptr_t)z | (uintptr_t)w | (uintptr_t)b | (uintptr_t)normed;
    const bool vec = W % 4 == 0 && plane_stride % 4 == 0 && (ptrs & 15) == 0 && (!z || (ld_z % 4 == 0 && z1 % 4 == 0 && (!y2 || z2 % 4 == 0)));
    cudaError_t e = cudaSuccess;
    FORGE_DISPATCH_DTYPE(out_dtype, TO, e = vec ? run<TO, 4>(d, normed, R, stream) : run<TO, 1>(d, normed, R, stream));
    return forge::check_launch("depth_step", e);
}
