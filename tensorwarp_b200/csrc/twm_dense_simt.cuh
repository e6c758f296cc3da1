// twm_dense_simt.cuh — FP32-arithmetic tiles for any size and either element type: the matrix
// product and the windowed sigmoid attention.  The 32-bit models run on these (true FP32, no reduced
// matrix mode); the 16-bit ones where the tensor-core kernels' size rules do not hold.
#pragma once

#include "twm_dense_common.cuh"

namespace twm {
namespace dense {

// C[M][N] = A[M][K] . W[N][K]^T, 64 x 64 tile, 16 K at a time, 4 x 4 outputs per thread.  EPI = TWM_EPI_GELU_GLU:
// W holds N gate rows and then N up rows; both products of a tile stay in registers.
constexpr int ST = 64, SK = 16;
template <typename T, int EPI>
__global__ void __launch_bounds__(256)
gemm_simt_kernel(const T* __restrict__ a, int lda, const T* __restrict__ w, int ldw, void* __restrict__ c, int ldc, int M, int N,
                 int K)
{
    constexpr int NB = EPI == TWM_EPI_GELU_GLU ? 2 : 1;
    pdl_launch_dependents();
    __shared__ __align__(16) float as[SK][ST + 4];
    __shared__ __align__(16) float bs[NB][SK][ST + 4];
    pdl_wait_prior_grids();
    const int m0 = blockIdx.y * ST, n0 = blockIdx.x * ST;
    const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
    float acc[NB][4][4] = {};
    for (int k0 = 0; k0 < K; k0 += SK) {
        // 64 rows x 16 K of each operand: four elements per thread
        const int row = threadIdx.x >> 2, kk = (threadIdx.x & 3) * 4;
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int k = k0 + kk + j;
            as[kk + j][row] = (m0 + row < M && k < K) ? to_f32(a[(size_t)(m0 + row) * lda + k]) : 0.0f;
#pragma unroll
            for (int b = 0; b < NB; ++b)
                bs[b][kk + j][row] = (n0 + row < N && k < K) ? to_f32(w[(size_t)(b * N + n0 + row) * ldw + k]) : 0.0f;
        }
        __syncthreads();
#pragma unroll
        for (int k = 0; k < SK; ++k) {
            const float4 av = *reinterpret_cast<const float4*>(&as[k][ty * 4]);
            const float am[4] = {av.x, av.y, av.z, av.w};
#pragma unroll
            for (int b = 0; b < NB; ++b) {
                const float4 bv = *reinterpret_cast<const float4*>(&bs[b][k][tx * 4]);
                const float bn[4] = {bv.x, bv.y, bv.z, bv.w};
#pragma unroll
                for (int i = 0; i < 4; ++i)
#pragma unroll
                    for (int j = 0; j < 4; ++j) acc[b][i][j] = fmaf(am[i], bn[j], acc[b][i][j]);
            }
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
            const float v = EPI == TWM_EPI_GELU_GLU ? gelu_tanh(acc[0][i][j]) * acc[NB - 1][i][j] : acc[0][i][j];
            if (EPI == TWM_EPI_STORE_F32) reinterpret_cast<float*>(c)[(size_t)m * ldc + n] = v;
            else reinterpret_cast<T*>(c)[(size_t)m * ldc + n] = from_f32<T>(v);
        }
    }
}

// What an attention launch reads of its layer.
template <typename T>
struct AttnArgs {
    const T* proj;              // [rows][ld]: q (normalised) | k | v | gate
    T* out;                     // [rows][heads * vdim_pad]
    const T* k_cache;           // [slots][capacity][kv_heads * dim_pad]
    const T* v_cache;
    const float* bias_table;    // [heads][bias_len] or null
    const int* meta;
    int ld, gate_off;           // gate_off < 0: no output gate
    int heads, kv_heads, dim_pad, vdim_pad, window, keep_first, capacity, bias_len, rows;
    float scale;
};

// One query of one head per CTA: scores one key per thread, 128 keys at a time, then P.V with threads along vdim
// (grid z: blocks of 512 value columns).
constexpr int AS_THREADS = 128, AS_VPT = 4;
template <typename T>
__global__ void __launch_bounds__(AS_THREADS)
attn_simt_kernel(const AttnArgs<T> g)
{
    using V = Vec<T>;
    pdl_launch_dependents();
    extern __shared__ __align__(16) float attn_smem[];
    float* qs = attn_smem;                      // [dim_pad]
    float* ws = qs + g.dim_pad;                 // [AS_THREADS]
    pdl_wait_prior_grids();
    const int r = blockIdx.x, h = blockIdx.y, kvh = h / (g.heads / g.kv_heads);
    const int p = g.meta[0] + r;
    const int kd = g.kv_heads * g.dim_pad, vd = g.kv_heads * g.vdim_pad;
    const T* kc = g.k_cache + (size_t)g.meta[1] * g.capacity * kd + kvh * g.dim_pad;
    const T* vc = g.v_cache + (size_t)g.meta[1] * g.capacity * vd + kvh * g.vdim_pad;
    const float* bias = g.bias_table != nullptr ? g.bias_table + (size_t)h * g.bias_len : nullptr;
    for (int d = threadIdx.x; d < g.dim_pad; d += AS_THREADS) qs[d] = to_f32(g.proj[(size_t)r * g.ld + h * g.dim_pad + d]);
    int sinks, lo;
    visible_range(p, g.window, g.keep_first, sinks, lo);
    const int total = sinks + (p - lo + 1);
    const int c0 = blockIdx.z * AS_VPT * AS_THREADS + threadIdx.x;
    float acc[AS_VPT] = {};
    for (int t0 = 0; t0 < total; t0 += AS_THREADS) {
        __syncthreads();                        // qs written / the previous chunk's weights read
        const int t = t0 + threadIdx.x;
        float wgt = 0.0f;
        if (t < total) {
            const int j = t < sinks ? t : lo + (t - sinks);
            const uint4* kr = reinterpret_cast<const uint4*>(kc + (size_t)j * kd);
            float s = 0.0f;
            for (int d = 0; d < g.dim_pad / V::N; ++d) {
                float f[V::N];
                V::unpack(kr[d], f);
#pragma unroll
                for (int e = 0; e < V::N; ++e) s = fmaf(f[e], qs[d * V::N + e], s);
            }
            wgt = sigmoid_f32(fmaf(s, g.scale, bias != nullptr ? bias[p - j] : 0.0f));
        }
        ws[threadIdx.x] = wgt;
        __syncthreads();
        const int n = min(AS_THREADS, total - t0);
        for (int tt = 0; tt < n; ++tt) {
            const int j = (t0 + tt) < sinks ? (t0 + tt) : lo + (t0 + tt - sinks);
            const float pw = ws[tt];
#pragma unroll
            for (int i = 0; i < AS_VPT; ++i) {
                const int d = c0 + i * AS_THREADS;
                if (d < g.vdim_pad) acc[i] = fmaf(pw, to_f32(vc[(size_t)j * vd + d]), acc[i]);
            }
        }
    }
#pragma unroll
    for (int i = 0; i < AS_VPT; ++i) {
        const int d = c0 + i * AS_THREADS;
        if (d < g.vdim_pad) {
            float o = acc[i];
            if (g.gate_off >= 0) o *= sigmoid_f32(to_f32(g.proj[(size_t)r * g.ld + g.gate_off + h * g.vdim_pad + d]));
            g.out[(size_t)r * g.heads * g.vdim_pad + h * g.vdim_pad + d] = from_f32<T>(o);
        }
    }
}

}  // namespace dense
}  // namespace twm
