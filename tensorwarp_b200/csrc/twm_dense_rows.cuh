// twm_dense_rows.cuh — the row-wise kernels of a dense decoder's step over several tokens: the
// residual stream with the norm of the sublayer output that joins it, the token shift, the q/k norm
// with the cache append, and the rows that go to the head.  All of them compute in FP32.
#pragma once

#include "twm_dense_common.cuh"

namespace twm {
namespace dense {

constexpr int ROW_THREADS = 256;

// One row's residual value, x_in + y * inv_rms(y) * y_norm (or the embedding), element by element.
template <typename T>
struct ResidualSource {
    const int* tokens;          // embedding rows instead of x_in when not null
    const T* embed;             // [vocab][wp]
    const T* pos_embed;         // [positions][wp] or null
    const float* x_in;          // [rows][wp]
    const float* y;             // [rows][wp] or null
    const float* y_norm;        // [wp] or null (y joins as it is)
    float eps;
    int width, wp;

    // four consecutive elements of row r; ir = inverse RMS of y's row
    __device__ __forceinline__ float4 at(int r, int p, int token, int i4, float ir) const {
        float4 v;
        if (tokens != nullptr) {
            const T* e = embed + (size_t)token * wp + i4 * 4;
            v = make_float4(to_f32(e[0]), to_f32(e[1]), to_f32(e[2]), to_f32(e[3]));
            if (pos_embed != nullptr) {
                const T* pe = pos_embed + (size_t)p * wp + i4 * 4;
                v.x += to_f32(pe[0]); v.y += to_f32(pe[1]); v.z += to_f32(pe[2]); v.w += to_f32(pe[3]);
            }
        } else {
            v = reinterpret_cast<const float4*>(x_in + (size_t)r * wp)[i4];
        }
        if (y != nullptr) {
            const float4 t = reinterpret_cast<const float4*>(y + (size_t)r * wp)[i4];
            float4 g = make_float4(1.f, 1.f, 1.f, 1.f);
            if (y_norm != nullptr) g = __ldg(reinterpret_cast<const float4*>(y_norm) + i4);
            v.x += t.x * ir * g.x; v.y += t.y * ir * g.y; v.z += t.z * ir * g.z; v.w += t.w * ir * g.w;
        }
        return v;
    }
    // inverse RMS of y's row (1 without a norm); all `threads` threads of the barrier take part
    __device__ __forceinline__ float row_inv_rms(int r, float* red, int threads, int bar) const {
        if (y == nullptr || y_norm == nullptr) return 1.0f;
        float ss = 0.0f;
        const float4* yr = reinterpret_cast<const float4*>(y + (size_t)r * wp);
        for (int i = threadIdx.x; i < (wp >> 2); i += threads) ss += ops::sumsq4(yr[i]);
        return inv_rms(group_sum(ss, red, threads, bar), width, eps);
    }
};

template <typename T>
__device__ __forceinline__ void store4(T* dst, const float4 v);
template <>
__device__ __forceinline__ void store4<float>(float* dst, const float4 v) { *reinterpret_cast<float4*>(dst) = v; }
template <>
__device__ __forceinline__ void store4<bf16>(bf16* dst, const float4 v) {
    const __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
    uint2 o;
    o.x = *reinterpret_cast<const uint32_t*>(&lo);
    o.y = *reinterpret_cast<const uint32_t*>(&hi);
    *reinterpret_cast<uint2*>(dst) = o;
}

// four consecutive elements as floats
__device__ __forceinline__ float4 load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 load4(const bf16* p) {
    const uint2 v = *reinterpret_cast<const uint2*>(p);
    return make_float4(__uint_as_float(v.x << 16), __uint_as_float(v.x & 0xffff0000u), __uint_as_float(v.y << 16),
                       __uint_as_float(v.y & 0xffff0000u));
}

// x + (before - x) * mix
__device__ __forceinline__ float4 shift4(const float4 x, const float4 before, const float4 mix) {
    return make_float4(fmaf(before.x - x.x, mix.x, x.x), fmaf(before.y - x.y, mix.y, x.y), fmaf(before.z - x.z, mix.z, x.z),
                       fmaf(before.w - x.w, mix.w, x.w));
}

// x_out = residual row; a = T(x_out), or T(token shift of x_out).  A CTA walks `rows_per_cta` consecutive rows and
// keeps the row before in shared memory; its first row's predecessor is computed again (or comes from the state).
template <typename T>
__global__ void __launch_bounds__(ROW_THREADS)
residual_rows_kernel(ResidualSource<T> src, float* __restrict__ x_out, T* __restrict__ a, const float* __restrict__ shift,
                     const float* __restrict__ shift_state, const int* __restrict__ meta, int rows, int rows_per_cta)
{
    pdl_launch_dependents();
    extern __shared__ __align__(16) float row_smem[];       // [wp]: the residual row before
    __shared__ float red[32];
    pdl_wait_prior_grids();
    const int wp = src.wp, nvec = wp >> 2;
    const int r0 = blockIdx.x * rows_per_cta, r1 = min(rows, r0 + rows_per_cta);
    const int pos0 = meta[0];
    if (shift != nullptr) {
        if (r0 == 0) {
            const float* st = shift_state + ((size_t)meta[1] * 2 + ((pos0 - 1) & 1)) * wp;
            for (int i = threadIdx.x; i < nvec; i += ROW_THREADS)
                reinterpret_cast<float4*>(row_smem)[i] =
                    pos0 > 0 ? reinterpret_cast<const float4*>(st)[i] : make_float4(0.f, 0.f, 0.f, 0.f);
        } else {
            const int r = r0 - 1;
            const int tok = src.tokens != nullptr ? src.tokens[r] : 0;
            const float ir = src.row_inv_rms(r, red, ROW_THREADS, 1);
            for (int i = threadIdx.x; i < nvec; i += ROW_THREADS)
                reinterpret_cast<float4*>(row_smem)[i] = src.at(r, pos0 + r, tok, i, ir);
        }
    }
    for (int r = r0; r < r1; ++r) {
        const int tok = src.tokens != nullptr ? src.tokens[r] : 0;
        const float ir = src.row_inv_rms(r, red, ROW_THREADS, 1);
        // every thread reads and replaces its own elements of row_smem: no barrier needed between rows
        for (int i = threadIdx.x; i < nvec; i += ROW_THREADS) {
            const float4 x = src.at(r, pos0 + r, tok, i, ir);
            reinterpret_cast<float4*>(x_out + (size_t)r * wp)[i] = x;
            float4 h = x;
            if (shift != nullptr) {
                float4* before = reinterpret_cast<float4*>(row_smem) + i;
                h = shift4(x, *before, __ldg(reinterpret_cast<const float4*>(shift) + i));
                *before = x;
            }
            if (a != nullptr) store4<T>(a + (size_t)r * wp + i * 4, h);
        }
    }
}

// a[w] = T(rms_norm(residual row want[w]) * final_norm): the rows whose logits are wanted.
template <typename T>
__global__ void __launch_bounds__(ROW_THREADS)
final_rows_kernel(ResidualSource<T> src, T* __restrict__ a, const float* __restrict__ final_norm, const int* __restrict__ want,
                  const int* __restrict__ meta)
{
    pdl_launch_dependents();
    extern __shared__ __align__(16) float row_smem[];
    __shared__ float red[32];
    pdl_wait_prior_grids();
    const int wp = src.wp, nvec = wp >> 2;
    const int r = want[blockIdx.x];
    const int tok = src.tokens != nullptr ? src.tokens[r] : 0;
    const float ir = src.row_inv_rms(r, red, ROW_THREADS, 1);
    float ss = 0.0f;
    for (int i = threadIdx.x; i < nvec; i += ROW_THREADS) {
        const float4 x = src.at(r, meta[0] + r, tok, i, ir);
        reinterpret_cast<float4*>(row_smem)[i] = x;
        ss += ops::sumsq4(x);
    }
    const float fr = inv_rms(group_sum(ss, red, ROW_THREADS, 1), src.width, src.eps);
    for (int i = threadIdx.x; i < nvec; i += ROW_THREADS) {
        const float4 x = reinterpret_cast<const float4*>(row_smem)[i];
        const float4 g = __ldg(reinterpret_cast<const float4*>(final_norm) + i);
        store4<T>(a + (size_t)blockIdx.x * wp + i * 4, make_float4(x.x * fr * g.x, x.y * fr * g.y, x.z * fr * g.z, x.w * fr * g.w));
    }
}

// One CTA per token: RMS norm of the whole q row (in place) and of the whole k row (into the cache), v into the cache.
// The CTA of the last token also stores that token's mixer input for the next step's token shift.
template <typename T>
__global__ void __launch_bounds__(ROW_THREADS)
qk_norm_append_kernel(T* __restrict__ proj, int ld, const float* __restrict__ q_norm, const float* __restrict__ k_norm,
                      T* __restrict__ k_cache, T* __restrict__ v_cache, int q_n, int k_n, int v_n, int q_true, int k_true,
                      float eps, int capacity, const float* __restrict__ x, int wp, float* __restrict__ shift_state,
                      const int* __restrict__ meta)
{
    pdl_launch_dependents();
    __shared__ float red[32];
    pdl_wait_prior_grids();
    using V = Vec<T>;
    const int r = blockIdx.x, p = meta[0] + r, slot = meta[1];
    T* row = proj + (size_t)r * ld;
    auto sum_sq = [&](const T* base, int n) {
        float ss = 0.0f;
        for (int i = threadIdx.x; i < n / V::N; i += ROW_THREADS) {
            float f[V::N];
            V::unpack(reinterpret_cast<const uint4*>(base)[i], f);
#pragma unroll
            for (int j = 0; j < V::N; ++j) ss = fmaf(f[j], f[j], ss);
        }
        return ss;
    };
    auto scale_row = [&](const T* base, T* dst, int n, float ir, const float* g) {
        for (int i = threadIdx.x; i < n / V::N; i += ROW_THREADS) {
            uint4 raw = reinterpret_cast<const uint4*>(base)[i];
            if (g != nullptr) {
                float f[V::N];
                V::unpack(raw, f);
#pragma unroll
                for (int j = 0; j < V::N; ++j) f[j] *= ir * __ldg(g + i * V::N + j);
                raw = V::pack(f);
            }
            reinterpret_cast<uint4*>(dst)[i] = raw;
        }
    };
    if (q_norm != nullptr) {
        const float ir = inv_rms(group_sum(sum_sq(row, q_n), red, ROW_THREADS, 1), q_true, eps);
        scale_row(row, row, q_n, ir, q_norm);
    }
    if (p < capacity) {
        const size_t at = (size_t)slot * capacity + p;
        float ir = 1.0f;
        if (k_norm != nullptr) ir = inv_rms(group_sum(sum_sq(row + q_n, k_n), red, ROW_THREADS, 1), k_true, eps);
        scale_row(row + q_n, k_cache + at * k_n, k_n, ir, k_norm);
        scale_row(row + q_n + k_n, v_cache + at * v_n, v_n, 1.0f, nullptr);
    }
    if (shift_state != nullptr && r == gridDim.x - 1) {
        float* st = shift_state + ((size_t)slot * 2 + (p & 1)) * wp;
        for (int i = threadIdx.x; i < (wp >> 2); i += ROW_THREADS)
            reinterpret_cast<float4*>(st)[i] = reinterpret_cast<const float4*>(x + (size_t)r * wp)[i];
    }
}

__global__ void set_step_kernel(int* __restrict__ meta, int* __restrict__ tokens, int first_pos, int slot, int token)
{
    pdl_launch_dependents();
    pdl_wait_prior_grids();
    meta[0] = first_pos;
    meta[1] = slot;
    meta[2] = first_pos + 1;
    if (token >= 0) tokens[0] = token;
}

}  // namespace dense
}  // namespace twm
