// twm_dense_moe.cuh — routed feed-forwards: the choice of experts, the rows grouped by expert, and plain
// tiles of the grouped product (the tcgen05 one is twm_dense_tc.cuh's, with its tiles dealt by expert; the
// decode one is twm_dense_decode.cuh's, with its rows looked up by expert).
#pragma once

#include "twm_dense_simt.cuh"

namespace twm {
namespace dense {

constexpr int MOE_MAX_EXPERTS = 1024, MOE_MAX_TOP = 32;

struct RouterArgs { int experts, top, groups, keep; };

// (value, index) of the largest value over the warp; the smaller index wins a tie
__device__ __forceinline__ void warp_argmax(float& v, int& i) {
#pragma unroll
    for (int d = 16; d > 0; d >>= 1) {
        const float ov = __shfl_xor_sync(0xffffffffu, v, d);
        const int oi = __shfl_xor_sync(0xffffffffu, i, d);
        if (ov > v || (ov == v && oi < i)) { v = ov; i = oi; }
    }
}

// One warp routes one token: softmax over all experts in FP32, the `keep` groups of neighbours with the largest single
// score, the `top` largest scores among their experts; the weights are the scores.  s: [experts] and gs: [groups] floats
// of shared memory.  Lane k < top returns choice k.
__device__ __forceinline__ void route_warp(const float* logits, const RouterArgs& r, float* s, float* gs, int lane, int& id, float& weight)
{
    float m = -INFINITY;
    for (int e = lane; e < r.experts; e += 32) { const float v = logits[e]; s[e] = v; m = fmaxf(m, v); }
    m = ops::warp_max(m);
    float sum = 0.0f;
    for (int e = lane; e < r.experts; e += 32) { const float v = expf(s[e] - m); s[e] = v; sum += v; }
    sum = ops::warp_sum(sum);
    for (int e = lane; e < r.experts; e += 32) s[e] /= sum;
    __syncwarp();
    const int per = r.experts / r.groups;
    const bool limited = r.keep < r.groups;
    if (limited) {
        for (int g = lane; g < r.groups; g += 32) {
            float best = -1.0f;
            for (int e = 0; e < per; ++e) best = fmaxf(best, s[g * per + e]);
            gs[g] = best;
        }
        __syncwarp();
        for (int k = 0; k < r.keep; ++k) {                  // a kept group's score becomes -1
            float v = -2.0f;
            int g = 0;
            for (int i = lane; i < r.groups; i += 32)
                if (gs[i] > v) { v = gs[i]; g = i; }
            warp_argmax(v, g);
            if (lane == 0) gs[g] = -1.0f;
            __syncwarp();
        }
    }
    id = 0;
    weight = 0.0f;
    for (int k = 0; k < r.top; ++k) {                       // a chosen expert's score becomes -1
        float v = -2.0f;
        int e = 0;
        for (int i = lane; i < r.experts; i += 32)
            if (s[i] > v && (!limited || gs[i / per] == -1.0f)) { v = s[i]; e = i; }
        warp_argmax(v, e);
        if (lane == k) { id = e; weight = v; }
        __syncwarp();
        if (lane == 0) s[e] = -1.0f;
        __syncwarp();
    }
}

// A warp per token: choices and weights [rows][top], and each choice's place among its expert's rows (in no
// particular order: the rows of a product do not depend on one another).
constexpr int RT_WARPS = 4;
__global__ void __launch_bounds__(RT_WARPS * 32)
route_kernel(const float* __restrict__ logits, int ld, const RouterArgs r, int rows, int* __restrict__ ids, float* __restrict__ weights,
             int* __restrict__ place, int* __restrict__ counts)
{
    extern __shared__ float route_smem[];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    float* s = route_smem + warp * (r.experts + r.groups);
    const int t = blockIdx.x * RT_WARPS + warp;
    pdl_wait_prior_grids();
    pdl_launch_dependents();
    if (t >= rows) return;
    int id;
    float weight;
    route_warp(logits + (size_t)t * ld, r, s, s + r.experts, lane, id, weight);
    if (lane < r.top) {
        ids[t * r.top + lane] = id;
        weights[t * r.top + lane] = weight;
        if (counts != nullptr) place[t * r.top + lane] = atomicAdd(counts + id, 1);
    }
}

// One warp: out[0 .. n] = running sums of f(0) ... f(n - 1)
template <typename F>
__device__ __forceinline__ void warp_prefix(F f, int n, int* out, int lane) {
    int base = 0;
    for (int i0 = 0; i0 < n; i0 += 32) {
        const int own = i0 + lane < n ? f(i0 + lane) : 0;
        int sum = own;
#pragma unroll
        for (int d = 1; d < 32; d <<= 1) {
            const int o = __shfl_up_sync(0xffffffffu, sum, d);
            if (lane >= d) sum += o;
        }
        if (i0 + lane < n) out[i0 + lane] = base + sum - own;
        base += __shfl_sync(0xffffffffu, sum, 31);
    }
    if (lane == 0) out[n] = base;
}
// largest e with pre[e] <= t, for t < pre[n]
__device__ __forceinline__ int prefix_find(const int* pre, int n, int t) {
    int lo = 0, hi = n - 1;
    while (lo < hi) {
        const int mid = (lo + hi + 1) >> 1;
        if (pre[mid] <= t) lo = mid; else hi = mid - 1;
    }
    return lo;
}

// Copies every token's row to its places, grouped by expert.  row[t][k] = where choice k of token t went;
// offsets[experts + 1] = where each expert's rows start.
constexpr int MG_THREADS = 256;
template <typename T>
__global__ void __launch_bounds__(MG_THREADS)
group_rows_kernel(const T* __restrict__ a, int wp, const RouterArgs r, int rows, const int* __restrict__ ids, const int* __restrict__ place,
                  const int* __restrict__ counts, int* __restrict__ row, int* __restrict__ offsets, T* __restrict__ grouped)
{
    __shared__ int off[MOE_MAX_EXPERTS + 1];
    pdl_wait_prior_grids();
    pdl_launch_dependents();
    if (threadIdx.x < 32) warp_prefix([&](int e) { return counts[e]; }, r.experts, off, threadIdx.x);
    __syncthreads();
    if (blockIdx.x == 0)
        for (int e = threadIdx.x; e <= r.experts; e += MG_THREADS) offsets[e] = off[e];
    const int nvec = wp * (int)sizeof(T) / 16;
    for (int t = blockIdx.x; t < rows; t += gridDim.x) {
        const uint4* src = reinterpret_cast<const uint4*>(a + (size_t)t * wp);
        if (threadIdx.x < r.top) row[t * r.top + threadIdx.x] = off[ids[t * r.top + threadIdx.x]] + place[t * r.top + threadIdx.x];
        for (int i = threadIdx.x; i < nvec; i += MG_THREADS) {
            const uint4 v = src[i];
            for (int k = 0; k < r.top; ++k) {
                const int dst = off[__ldg(ids + t * r.top + k)] + __ldg(place + t * r.top + k);
                reinterpret_cast<uint4*>(grouped + (size_t)dst * wp)[i] = v;
            }
        }
    }
}

// C[row][N] = epi(A[row][K] . W[e][N][K]^T) for the rows [offsets[e], offsets[e + 1]) of every expert e, 64 x 64 tiles
// (grid y: at least as many as there can be row tiles).
template <typename T, int EPI>
__global__ void __launch_bounds__(256)
moe_gemm_simt_kernel(const T* __restrict__ a, int lda, const T* __restrict__ w, int ldw, void* __restrict__ c, int ldc,
                     const int* __restrict__ offsets, int experts, int N, int K)
{
    __shared__ int pre[MOE_MAX_EXPERTS + 1];
    __shared__ __align__(16) float as[SK][ST + 4];
    __shared__ __align__(16) float bs[SK][ST + 4];
    pdl_wait_prior_grids();
    pdl_launch_dependents();
    if (threadIdx.x < 32) warp_prefix([&](int e) { return (offsets[e + 1] - offsets[e] + ST - 1) / ST; }, experts, pre, threadIdx.x);
    __syncthreads();
    if ((int)blockIdx.y >= pre[experts]) return;
    const int e = prefix_find(pre, experts, blockIdx.y);
    const int m0 = offsets[e] + ((int)blockIdx.y - pre[e]) * ST, M = offsets[e + 1], n0 = blockIdx.x * ST;
    const T* we = w + (size_t)e * N * ldw;
    const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
    float acc[4][4] = {};
    for (int k0 = 0; k0 < K; k0 += SK) {
        const int row = threadIdx.x >> 2, kk = (threadIdx.x & 3) * 4;
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int k = k0 + kk + j;
            as[kk + j][row] = (m0 + row < M && k < K) ? to_f32(a[(size_t)(m0 + row) * lda + k]) : 0.0f;
            bs[kk + j][row] = (n0 + row < N && k < K) ? to_f32(we[(size_t)(n0 + row) * ldw + k]) : 0.0f;
        }
        __syncthreads();
#pragma unroll
        for (int k = 0; k < SK; ++k) {
            const float4 av = *reinterpret_cast<const float4*>(&as[k][ty * 4]);
            const float4 bv = *reinterpret_cast<const float4*>(&bs[k][tx * 4]);
            const float am[4] = {av.x, av.y, av.z, av.w}, bn[4] = {bv.x, bv.y, bv.z, bv.w};
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(am[i], bn[j], acc[i][j]);
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int m = m0 + ty * 4 + i;
        if (m >= M) continue;
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int n = n0 + tx * 4 + j;
            if (n >= N) continue;
            const float v = epilogue_value<EPI>(acc[i][j]);
            if (EPI == TWM_EPI_STORE_F32) reinterpret_cast<float*>(c)[(size_t)m * ldc + n] = v;
            else reinterpret_cast<T*>(c)[(size_t)m * ldc + n] = from_f32<T>(v);
        }
    }
}

}  // namespace dense
}  // namespace twm
