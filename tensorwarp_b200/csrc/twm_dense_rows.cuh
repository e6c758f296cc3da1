// twm_dense_rows.cuh — the row-wise kernels of a dense decoder's step over several tokens: the
// residual stream with the norm of the sublayer output that joins it, the token shift, the q/k norm
// with the cache append, and the rows that go to the head.  All of them compute in FP32.
#pragma once

#include "twm_dense_common.cuh"

namespace twm {
namespace dense {

constexpr int ROW_THREADS = 256;
constexpr int MAX_TOP = 32;                             // experts a token uses, at most

// Outputs of the chosen experts: a token's sublayer output is the sum over its `top` slots of weight * row.
template <typename T>
struct RoutedOutput {
    const T* rows;              // [tokens * top][wp], grouped by expert; null = the sublayer was not routed
    const int* row;             // [tokens][top]: a slot's row
    const float* weight;        // [tokens][top]
    int top;
};

// four consecutive elements as floats
__device__ __forceinline__ float4 load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 load4(const bf16* p) {
    const uint2 v = *reinterpret_cast<const uint2*>(p);
    return make_float4(__uint_as_float(v.x << 16), __uint_as_float(v.x & 0xffff0000u), __uint_as_float(v.y << 16),
                       __uint_as_float(v.y & 0xffff0000u));
}

// One row's residual value, x_in + y * inv_rms(y) * y_norm (or the embedding), element by element.
template <typename T>
struct ResidualSource {
    const int* tokens;          // embedding rows instead of x_in when not null
    const T* embed;             // [vocab][wp]
    const T* pos_embed;         // [positions][wp] or null
    const float* x_in;          // [rows][wp]
    const float* y;             // [rows][wp] or null
    const float* y_norm;        // [wp] or null (y joins as it is)
    const float* step;          // [wp]: added to every row, or null
    RoutedOutput<T> routed;     // instead of y
    float eps, embed_scale;
    int width, wp;

    __device__ __forceinline__ bool has_y() const { return y != nullptr || routed.rows != nullptr; }
    // four consecutive elements of what joins row r
    __device__ __forceinline__ float4 y_at(int r, int i4) const {
        if (y != nullptr) return reinterpret_cast<const float4*>(y + (size_t)r * wp)[i4];
        float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
        const int* at = routed.row + (size_t)r * routed.top;
        const float* w = routed.weight + (size_t)r * routed.top;
#pragma unroll 8
        for (int s = 0; s < routed.top; ++s) {
            const float4 t = load4(routed.rows + (size_t)at[s] * wp + i4 * 4);
            const float ws = w[s];
            v.x = fmaf(t.x, ws, v.x); v.y = fmaf(t.y, ws, v.y); v.z = fmaf(t.z, ws, v.z); v.w = fmaf(t.w, ws, v.w);
        }
        return v;
    }

    // four consecutive elements of row r; ir = inverse RMS of y's row
    __device__ __forceinline__ float4 at(int r, int p, int token, int i4, float ir) const {
        float4 v;
        if (tokens != nullptr) {
            const T* e = embed + (size_t)token * wp + i4 * 4;
            v = make_float4(to_f32(e[0]) * embed_scale, to_f32(e[1]) * embed_scale, to_f32(e[2]) * embed_scale, to_f32(e[3]) * embed_scale);
            if (pos_embed != nullptr) {
                const T* pe = pos_embed + (size_t)p * wp + i4 * 4;
                v.x += to_f32(pe[0]); v.y += to_f32(pe[1]); v.z += to_f32(pe[2]); v.w += to_f32(pe[3]);
            }
        } else {
            v = reinterpret_cast<const float4*>(x_in + (size_t)r * wp)[i4];
        }
        if (has_y()) {
            const float4 t = y_at(r, i4);
            float4 g = make_float4(1.f, 1.f, 1.f, 1.f);
            if (y_norm != nullptr) g = __ldg(reinterpret_cast<const float4*>(y_norm) + i4);
            v.x += t.x * ir * g.x; v.y += t.y * ir * g.y; v.z += t.z * ir * g.z; v.w += t.w * ir * g.w;
        }
        if (step != nullptr) {
            const float4 t = __ldg(reinterpret_cast<const float4*>(step) + i4);
            v.x += t.x; v.y += t.y; v.z += t.z; v.w += t.w;
        }
        return v;
    }
    // inverse RMS of y's row (1 without a norm); all `threads` threads of the barrier take part
    __device__ __forceinline__ float row_inv_rms(int r, float* red, int threads, int bar) const {
        if (!has_y() || y_norm == nullptr) return 1.0f;
        float ss = 0.0f;
        for (int i = threadIdx.x; i < (wp >> 2); i += threads) ss += ops::sumsq4(y_at(r, i));
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

// x + (before - x) * mix
__device__ __forceinline__ float4 shift4(const float4 x, const float4 before, const float4 mix) {
    return make_float4(fmaf(before.x - x.x, mix.x, x.x), fmaf(before.y - x.y, mix.y, x.y), fmaf(before.z - x.z, mix.z, x.z),
                       fmaf(before.w - x.w, mix.w, x.w));
}

__device__ __forceinline__ float4 scale4(const float4 x, float s, const float4 g) {
    return make_float4(x.x * s * g.x, x.y * s * g.y, x.z * s * g.z, x.w * s * g.w);
}

// x_out = residual row; a = T(x_out), or T(token shift of x_out), or T(rms_norm(x_out) * pre_norm).  clear: words set to
// zero on the way (the expert counts of the routing that follows).  A CTA walks `rows_per_cta` consecutive rows and
// keeps the row before; its first row's predecessor is computed again (or comes from the state).  PER > 0: a
// thread's share of a row is PER vectors, held in registers, every load issued before the first use; PER = 0: rows
// of any length, in shared memory.  FULL = false: without pre_norm, step, routed outputs and clear.
template <typename T, int PER, bool FULL>
__global__ void __launch_bounds__(ROW_THREADS)
residual_rows_kernel(ResidualSource<T> src, float* __restrict__ x_out, T* __restrict__ a, const float* __restrict__ shift,
                     const float* __restrict__ shift_state, const float* __restrict__ pre_norm, const int* __restrict__ meta, int rows,
                     int rows_per_cta, int* __restrict__ clear, int n_clear)
{
    pdl_launch_dependents();
    extern __shared__ __align__(16) float row_smem[];       // PER = 0: [wp], the residual row before
    __shared__ float red[32];
    pdl_wait_prior_grids();
    const int wp = src.wp, nvec = wp >> 2;
    const int r0 = blockIdx.x * rows_per_cta, r1 = min(rows, r0 + rows_per_cta);
    const int pos0 = meta[0];
    if (FULL && blockIdx.x == 0)
        for (int i = threadIdx.x; i < n_clear; i += ROW_THREADS) clear[i] = 0;
    const float* st = shift != nullptr && r0 == 0 && pos0 > 0
                          ? shift_state + ((size_t)meta[1] * 2 + ((pos0 - 1) & 1)) * wp : nullptr;
    const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
    if constexpr (PER > 0) {
        __shared__ int slot_row[FULL ? MAX_TOP : 1];
        __shared__ float slot_weight[FULL ? MAX_TOP : 1];
        float4 before[PER];
#pragma unroll
        for (int j = 0; j < PER; ++j) {
            const int i = threadIdx.x + j * ROW_THREADS;
            before[j] = st != nullptr && i < nvec ? reinterpret_cast<const float4*>(st)[i] : zero;
        }
        for (int r = (shift != nullptr && r0 > 0) ? r0 - 1 : r0; r < r1; ++r) {
            float4 x[PER], y[PER];
            if (FULL && src.routed.rows != nullptr) {       // the row's slots, known before the first of their loads
                __syncthreads();
                if (threadIdx.x < src.routed.top) {
                    slot_row[threadIdx.x] = src.routed.row[(size_t)r * src.routed.top + threadIdx.x];
                    slot_weight[threadIdx.x] = src.routed.weight[(size_t)r * src.routed.top + threadIdx.x];
                }
                __syncthreads();
            }
            const int tok = src.tokens != nullptr ? src.tokens[r] : 0;
            ResidualSource<T> plain = src;                  // the row without what joins it
            plain.y = nullptr;
            plain.routed.rows = nullptr;
            if (!FULL) plain.step = nullptr;
#pragma unroll
            for (int j = 0; j < PER; ++j) {
                const int i = threadIdx.x + j * ROW_THREADS;
                y[j] = src.y != nullptr && i < nvec ? src.y_at(r, i) : zero;
                x[j] = i < nvec ? plain.at(r, pos0 + r, tok, i, 1.0f) : zero;
            }
            if (FULL && src.routed.rows != nullptr) {
#pragma unroll 4
                for (int s = 0; s < src.routed.top; ++s) {
                    const T* row = src.routed.rows + (size_t)slot_row[s] * wp;
                    const float ws = slot_weight[s];
#pragma unroll
                    for (int j = 0; j < PER; ++j) {
                        const int i = threadIdx.x + j * ROW_THREADS;
                        if (i >= nvec) continue;
                        const float4 t = load4(row + i * 4);
                        y[j].x = fmaf(t.x, ws, y[j].x); y[j].y = fmaf(t.y, ws, y[j].y); y[j].z = fmaf(t.z, ws, y[j].z); y[j].w = fmaf(t.w, ws, y[j].w);
                    }
                }
            }
            float ir = 1.0f;
            if ((src.y != nullptr || (FULL && src.routed.rows != nullptr)) && src.y_norm != nullptr) {
                float ss = 0.0f;
#pragma unroll
                for (int j = 0; j < PER; ++j) ss += ops::sumsq4(y[j]);
                ir = inv_rms(group_sum(ss, red, ROW_THREADS, 1), src.width, src.eps);
            }
            float xs = 0.0f, pr = 1.0f;
#pragma unroll
            for (int j = 0; j < PER; ++j) {
                const int i = threadIdx.x + j * ROW_THREADS;
                if (i >= nvec) continue;
                float4 n = make_float4(1.f, 1.f, 1.f, 1.f);
                if (src.y_norm != nullptr) n = __ldg(reinterpret_cast<const float4*>(src.y_norm) + i);
                x[j].x += y[j].x * ir * n.x; x[j].y += y[j].y * ir * n.y; x[j].z += y[j].z * ir * n.z; x[j].w += y[j].w * ir * n.w;
                if (FULL) xs += ops::sumsq4(x[j]);
            }
            if (FULL && pre_norm != nullptr) pr = inv_rms(group_sum(xs, red, ROW_THREADS, 1), src.width, src.eps);
#pragma unroll
            for (int j = 0; j < PER; ++j) {
                const int i = threadIdx.x + j * ROW_THREADS;
                if (i >= nvec) continue;
                if (r >= r0) {
                    reinterpret_cast<float4*>(x_out + (size_t)r * wp)[i] = x[j];
                    float4 h = x[j];
                    if (shift != nullptr) h = shift4(x[j], before[j], __ldg(reinterpret_cast<const float4*>(shift) + i));
                    if (FULL && pre_norm != nullptr) h = scale4(x[j], pr, __ldg(reinterpret_cast<const float4*>(pre_norm) + i));
                    if (a != nullptr) store4<T>(a + (size_t)r * wp + i * 4, h);
                }
                before[j] = x[j];
            }
        }
    } else {
        if (shift != nullptr) {
            if (r0 == 0) {
                for (int i = threadIdx.x; i < nvec; i += ROW_THREADS)
                    reinterpret_cast<float4*>(row_smem)[i] = st != nullptr ? reinterpret_cast<const float4*>(st)[i] : zero;
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
            float pr = 1.0f;
            if (FULL && pre_norm != nullptr) {
                float xs = 0.0f;
                for (int i = threadIdx.x; i < nvec; i += ROW_THREADS) xs += ops::sumsq4(src.at(r, pos0 + r, tok, i, ir));
                pr = inv_rms(group_sum(xs, red, ROW_THREADS, 1), src.width, src.eps);
            }
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
                if (FULL && pre_norm != nullptr) h = scale4(x, pr, __ldg(reinterpret_cast<const float4*>(pre_norm) + i));
                if (a != nullptr) store4<T>(a + (size_t)r * wp + i * 4, h);
            }
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
    const bool cached = p < capacity;
    T* k_dst = k_cache + ((size_t)slot * capacity + p) * k_n;
    T* v_dst = v_cache + ((size_t)slot * capacity + p) * v_n;
    auto sum_sq = [&](const uint4& raw) {
        float f[V::N], ss = 0.0f;
        V::unpack(raw, f);
#pragma unroll
        for (int j = 0; j < V::N; ++j) ss = fmaf(f[j], f[j], ss);
        return ss;
    };
    auto scaled = [&](const uint4& raw, float ir, const float* g, int i) {
        float f[V::N];
        V::unpack(raw, f);
#pragma unroll
        for (int j = 0; j < V::N; j += 4) {
            const float4 n = __ldg(reinterpret_cast<const float4*>(g + i * V::N + j));
            f[j] *= ir * n.x; f[j + 1] *= ir * n.y; f[j + 2] *= ir * n.z; f[j + 3] *= ir * n.w;
        }
        return V::pack(f);
    };
    const uint4* q_row = reinterpret_cast<const uint4*>(row);
    const uint4* k_row = reinterpret_cast<const uint4*>(row + q_n);
    const uint4* v_row = reinterpret_cast<const uint4*>(row + q_n + k_n);
    // a thread's first pieces stay in registers between the sum and the scaling; longer rows read the rest again
    constexpr int QP = 4, KP = 2;
    uint4 q[QP], k[KP];
    float qs = 0.0f, ks = 0.0f;
#pragma unroll
    for (int j = 0; j < QP; ++j) {
        const int i = threadIdx.x + j * ROW_THREADS;
        q[j] = q_norm != nullptr && i < q_n / V::N ? q_row[i] : make_uint4(0, 0, 0, 0);
    }
#pragma unroll
    for (int j = 0; j < KP; ++j) {
        const int i = threadIdx.x + j * ROW_THREADS;
        k[j] = i < k_n / V::N ? k_row[i] : make_uint4(0, 0, 0, 0);
    }
    if (cached)
        for (int i = threadIdx.x; i < v_n / V::N; i += ROW_THREADS) reinterpret_cast<uint4*>(v_dst)[i] = v_row[i];
    if (q_norm != nullptr) {
#pragma unroll
        for (int j = 0; j < QP; ++j) qs += sum_sq(q[j]);
        for (int i = threadIdx.x + QP * ROW_THREADS; i < q_n / V::N; i += ROW_THREADS) qs += sum_sq(q_row[i]);
        const float ir = inv_rms(group_sum(qs, red, ROW_THREADS, 1), q_true, eps);
#pragma unroll
        for (int j = 0; j < QP; ++j) {
            const int i = threadIdx.x + j * ROW_THREADS;
            if (i < q_n / V::N) reinterpret_cast<uint4*>(row)[i] = scaled(q[j], ir, q_norm, i);
        }
        for (int i = threadIdx.x + QP * ROW_THREADS; i < q_n / V::N; i += ROW_THREADS)
            reinterpret_cast<uint4*>(row)[i] = scaled(q_row[i], ir, q_norm, i);
    }
    float kir = 1.0f;
    if (k_norm != nullptr) {
#pragma unroll
        for (int j = 0; j < KP; ++j) ks += sum_sq(k[j]);
        for (int i = threadIdx.x + KP * ROW_THREADS; i < k_n / V::N; i += ROW_THREADS) ks += sum_sq(k_row[i]);
        kir = inv_rms(group_sum(ks, red, ROW_THREADS, 1), k_true, eps);
    }
    if (cached) {
#pragma unroll
        for (int j = 0; j < KP; ++j) {
            const int i = threadIdx.x + j * ROW_THREADS;
            if (i < k_n / V::N) reinterpret_cast<uint4*>(k_dst)[i] = k_norm != nullptr ? scaled(k[j], kir, k_norm, i) : k[j];
        }
        for (int i = threadIdx.x + KP * ROW_THREADS; i < k_n / V::N; i += ROW_THREADS)
            reinterpret_cast<uint4*>(k_dst)[i] = k_norm != nullptr ? scaled(k_row[i], kir, k_norm, i) : k_row[i];
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
