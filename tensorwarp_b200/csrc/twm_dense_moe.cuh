// twm_dense_moe.cuh — routed feed-forwards: the choice of experts, the rows grouped by expert, and plain
// tiles of the grouped product (the tcgen05 one is twm_dense_tc.cuh's, with its tiles dealt by expert; the
// decode one is twm_dense_decode.cuh's, with its rows looked up by expert).
#pragma once

#include "twm_dense_rows.cuh"
#include "twm_dense_simt.cuh"

namespace twm {
namespace dense {

constexpr int MOE_MAX_EXPERTS = 1024, MOE_MAX_TOP = MAX_TOP;

struct RouterArgs { int experts, top, groups, keep; };

// The largest of the lanes' N values each (value j of a lane stands for index lane + 32 j; negative = not there): its index,
// the smallest on a tie, and in `best` its value; its owner's copy becomes negative.
template <int N>
__device__ __forceinline__ int warp_take_largest(float (&v)[N], int lane, float& best) {
    unsigned top = 0;
    int at = 0;
#pragma unroll
    for (int j = 0; j < N; ++j) {
        const unsigned key = v[j] < 0.0f ? 0u : __float_as_uint(v[j]) + 1u;      // scores are not negative: their bits sort as they do
        if (key > top) { top = key; at = lane + 32 * j; }
    }
    const unsigned all = __reduce_max_sync(0xffffffffu, top);
    const int index = (int)__reduce_min_sync(0xffffffffu, top == all ? (unsigned)at : 0x7fffffffu);
#pragma unroll
    for (int j = 0; j < N; ++j)
        if (index == lane + 32 * j) v[j] = -1.0f;
    best = __uint_as_float(all - 1u);
    return index;
}

template <int N>
__device__ __forceinline__ void route_values(const float* logits, const RouterArgs& r, float* s, float* gs, int lane, int& id, float& weight)
{
    float v[N], m = -INFINITY, sum = 0.0f;
#pragma unroll
    for (int j = 0; j < N; ++j) {
        const int e = lane + 32 * j;
        v[j] = e < r.experts ? logits[e] : -INFINITY;
        m = fmaxf(m, v[j]);
    }
    m = ops::warp_max(m);
#pragma unroll
    for (int j = 0; j < N; ++j) {
        v[j] = expf(v[j] - m);
        sum += v[j];
    }
    sum = ops::warp_sum(sum);
#pragma unroll
    for (int j = 0; j < N; ++j) v[j] = lane + 32 * j < r.experts ? v[j] / sum : -1.0f;
    if (r.keep < r.groups) {
        const int per = r.experts / r.groups;
#pragma unroll
        for (int j = 0; j < N; ++j)
            if (lane + 32 * j < r.experts) s[lane + 32 * j] = v[j];
        __syncwarp();
        float best[N];
#pragma unroll
        for (int j = 0; j < N; ++j) {
            const int g = lane + 32 * j;
            best[j] = -1.0f;
            if (g < r.groups) {
                for (int e = 0; e < per; ++e) best[j] = fmaxf(best[j], s[g * per + e]);
                gs[g] = 0.0f;
            }
        }
        __syncwarp();
        for (int k = 0; k < r.keep; ++k) {
            float unused;
            const int g = warp_take_largest<N>(best, lane, unused);
            if (lane == 0) gs[g] = 1.0f;
        }
        __syncwarp();
#pragma unroll
        for (int j = 0; j < N; ++j)
            if (lane + 32 * j < r.experts && gs[(lane + 32 * j) / per] == 0.0f) v[j] = -1.0f;
    }
    id = 0;
    weight = 0.0f;
    for (int k = 0; k < r.top; ++k) {
        float best;
        const int e = warp_take_largest<N>(v, lane, best);
        if (lane == k) { id = e < r.experts ? e : 0; weight = best; }           // an index past the end: scores that are not numbers
    }
}

// One warp routes one token: softmax over all experts in FP32, the `keep` groups of neighbours with the largest single
// score, the `top` largest scores among their experts; the weights are the scores.  s: [experts] and gs: [groups] floats
// of shared memory.  Lane k < top returns choice k.
__device__ __forceinline__ void route_warp(const float* logits, const RouterArgs& r, float* s, float* gs, int lane, int& id, float& weight)
{
    if (r.experts <= 64) route_values<2>(logits, r, s, gs, lane, id, weight);
    else if (r.experts <= 256) route_values<8>(logits, r, s, gs, lane, id, weight);
    else route_values<MOE_MAX_EXPERTS / 32>(logits, r, s, gs, lane, id, weight);
}

// A warp per token: choices and weights [rows][top], and each choice's place among its expert's rows (in no
// particular order: the rows of a product do not depend on one another).  A CTA counts its tokens' choices itself and
// asks for its places once per expert.
constexpr int RT_WARPS = 16;
__host__ __device__ inline size_t route_smem_bytes(const RouterArgs& r) { return sizeof(float) * (RT_WARPS * (size_t)(r.experts + r.groups) + 2 * (size_t)r.experts); }
__global__ void __launch_bounds__(RT_WARPS * 32)
route_kernel(const float* __restrict__ logits, int ld, const RouterArgs r, int rows, int* __restrict__ ids, float* __restrict__ weights,
             int* __restrict__ place, int* __restrict__ counts)
{
    extern __shared__ float route_smem[];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    float* s = route_smem + warp * (r.experts + r.groups);
    int* own = reinterpret_cast<int*>(route_smem + RT_WARPS * (r.experts + r.groups));      // [experts] this CTA's choices
    int* base = own + r.experts;
    for (int e = threadIdx.x; e < r.experts; e += RT_WARPS * 32) own[e] = 0;
    pdl_wait_prior_grids();
    pdl_launch_dependents();
    __syncthreads();
    const int t = blockIdx.x * RT_WARPS + warp;
    int id = 0, rank = 0;
    const bool valid = t < rows && lane < r.top;
    if (t < rows) {
        float weight;
        route_warp(logits + (size_t)t * ld, r, s, s + r.experts, lane, id, weight);
        if (valid) {
            ids[t * r.top + lane] = id;
            weights[t * r.top + lane] = weight;
            rank = atomicAdd(own + id, 1);
        }
    }
    if (counts == nullptr) return;
    __syncthreads();
    for (int e = threadIdx.x; e < r.experts; e += RT_WARPS * 32) base[e] = own[e] > 0 ? atomicAdd(counts + e, own[e]) : 0;
    __syncthreads();
    if (valid) place[t * r.top + lane] = base[id] + rank;
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
