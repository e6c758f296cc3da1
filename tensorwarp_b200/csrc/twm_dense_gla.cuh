// twm_dense_gla.cuh — gated linear attention: per head a matrix state S [dim][vdim] in FP32 with one decay per key
// channel, S_t = diag(alpha_t) S_{t-1} + k_t v_t^T, o_t = S_t^T q_t; each head's o is RMS-normed, weighted and
// multiplied by silu(gate).
//
// Prompt steps, bfloat16: chunks of 64 tokens.  With b_t the running sum of log alpha inside a chunk,
//   o_t = (q_t e^{b_t})^T S_chunk + sum_{s <= t} (sum_d q_td k_sd e^{b_td - b_sd}) v_s.
//   gla_chunk_state_kernel  b, from the low-rank projection, and what each chunk adds to the state, all chunks at once
//   gla_scan_kernel         the state ahead of every chunk, chunk by chunk, element by element
//   gla_chunk_out_kernel    o, norm and gate, all chunks at once
// Every factor with a decay is computed in FP32 and enters a warp-level MMA as a bf16 pair hi + lo.  The scores inside a
// chunk are one product, with the exponents taken against the chunk's middle token: safe while neither half of the
// chunk decays by more than e^60; a chunk that does is scored token pair by token pair.
// Everything else (FP32, wide heads): gla_decay_kernel makes log alpha, gla_rows_kernel walks the tokens one by one,
// gla_gate_kernel norms and gates.
// Decoding: gla_decode_kernel.
#pragma once

#include "twm_dense_attn.cuh"
#include "twm_dense_rows.cuh"

namespace twm {
namespace dense {

constexpr int GLA_CHUNK = 64, GLA_MIDDLE = 31;
constexpr float GLA_HALF_LIMIT = 60.0f;         // largest decay (its logarithm) of half a chunk that goes through one product

template <typename T>
struct GlaArgs {
    const T* proj;              // [rows][ld]: q | k | v | gate | low-rank
    float* decay;               // [rows][heads * dim_pad]: log alpha, or (chunks) its running sums inside a chunk
    float* chunk_state;         // [chunks][heads][dim_pad][vdim_pad]
    float* mix;                 // [rows][heads * vdim_pad], token by token only
    T* out;                     // [rows][heads * vdim_pad]
    float* state;               // [slots][heads][dim_pad][vdim_pad]
    const T* w_decay;           // [heads * dim_pad][rank_pad]
    const float* decay_bias;    // [heads * dim_pad]
    const float* head_norm;     // [vdim_pad]
    const int* meta;
    int ld, heads, dim_pad, vdim, vdim_pad, rank_pad, rows;
    float inv_tau, q_scale, eps;
    __device__ __forceinline__ int k_off() const { return heads * dim_pad; }
    __device__ __forceinline__ int v_off() const { return 2 * heads * dim_pad; }
    __device__ __forceinline__ int gate_off() const { return 2 * heads * dim_pad + heads * vdim_pad; }
    __device__ __forceinline__ int low_off() const { return 2 * heads * (dim_pad + vdim_pad); }
    __device__ __forceinline__ float* slot_state(int h) const { return state + ((size_t)meta[1] * heads + h) * dim_pad * vdim_pad; }
};

// log(sigmoid(z)) to about 2^-22 of itself or 2e-7, whichever is larger
__device__ __forceinline__ float log_sigmoid_fast(float z) {
    const float e = ex2_approx(-1.4426950408889634f * fabsf(z));
    const float near_one = e * fmaf(-e, fmaf(-e, fmaf(-e, 0.25f, 1.0f / 3.0f), 0.5f), 1.0f);      // log(1 + e) for small e
    return fminf(z, 0.0f) - (e < 0.0078125f ? near_one : __logf(1.0f + e));
}

// A thread per key channel and run of rows: log alpha = log(sigmoid(z)) / tau.
constexpr int GD_THREADS = 128, GD_ROWS = 16, GD_RANK = 32;
template <typename T>
__global__ void __launch_bounds__(GD_THREADS)
gla_decay_kernel(const GlaArgs<T> g)
{
    using V = Vec<T>;
    __shared__ __align__(16) float low[GD_ROWS][GD_RANK];
    const int col = blockIdx.x * GD_THREADS + threadIdx.x, r0 = blockIdx.y * GD_ROWS, n = min(GD_ROWS, g.rows - r0);
    const int cols = g.heads * g.dim_pad;
    const float bias = col < cols ? __ldg(g.decay_bias + col) : 0.0f;
    pdl_wait_prior_grids();
    pdl_launch_dependents();
    float z[GD_ROWS];
#pragma unroll
    for (int r = 0; r < GD_ROWS; ++r) z[r] = bias;
    for (int k0 = 0; k0 < g.rank_pad; k0 += GD_RANK) {
        const int kn = min(GD_RANK, g.rank_pad - k0);
        __syncthreads();
        for (int i = threadIdx.x; i < GD_ROWS * kn; i += GD_THREADS) {
            const int r = i / kn, k = i - r * kn;
            low[r][k] = r < n ? to_f32(g.proj[(size_t)(r0 + r) * g.ld + g.low_off() + k0 + k]) : 0.0f;
        }
        __syncthreads();
        if (col < cols) {
            for (int k = 0; k < kn; k += V::N) {
                float w[V::N];
                V::unpack(__ldg(reinterpret_cast<const uint4*>(g.w_decay + (size_t)col * g.rank_pad + k0 + k)), w);
#pragma unroll
                for (int r = 0; r < GD_ROWS; ++r)
#pragma unroll
                    for (int e = 0; e < V::N; e += 4) {
                        const float4 a = *reinterpret_cast<const float4*>(&low[r][k + e]);
                        z[r] = fmaf(w[e], a.x, fmaf(w[e + 1], a.y, fmaf(w[e + 2], a.z, fmaf(w[e + 3], a.w, z[r]))));
                    }
            }
        }
    }
    if (col >= cols) return;
#pragma unroll
    for (int r = 0; r < GD_ROWS; ++r)
        if (r < n) g.decay[(size_t)(r0 + r) * cols + col] = log_sigmoid_f32(z[r]) * g.inv_tau;
}

// Token by token: CTA = 32 value columns of a head, thread = a column and every eighth key channel.
constexpr int GR_THREADS = 256, GR_COLS = 32, GR_TOKENS = 8;
__host__ inline size_t gla_rows_smem_bytes(int dim_pad) { return sizeof(float) * (size_t)(dim_pad * GR_COLS + 3 * GR_TOKENS * dim_pad); }
template <typename T>
__global__ void __launch_bounds__(GR_THREADS)
gla_rows_kernel(const GlaArgs<T> g)
{
    extern __shared__ __align__(16) float gr_smem[];
    __shared__ float part[GR_TOKENS][8][GR_COLS];
    float* s = gr_smem;                                    // [dim_pad][32]
    float* qs = s + g.dim_pad * GR_COLS;                   // [tokens][dim_pad]
    float* ks = qs + GR_TOKENS * g.dim_pad;
    float* as = ks + GR_TOKENS * g.dim_pad;
    pdl_wait_prior_grids();
    pdl_launch_dependents();
    const int h = blockIdx.y, c = threadIdx.x & 31, grp = threadIdx.x >> 5, col = blockIdx.x * GR_COLS + c;
    const bool in = col < g.vdim_pad;
    float* st = g.slot_state(h);
    const bool fresh = g.meta[0] == 0;                     // the state ahead of a sequence's first token is zero
    for (int d = grp; d < g.dim_pad; d += 8) s[d * GR_COLS + c] = in && !fresh ? st[(size_t)d * g.vdim_pad + col] : 0.0f;
    for (int t0 = 0; t0 < g.rows; t0 += GR_TOKENS) {
        const int n = min(GR_TOKENS, g.rows - t0);
        __syncthreads();
        for (int i = threadIdx.x; i < n * g.dim_pad; i += GR_THREADS) {
            const int t = i / g.dim_pad, d = i - t * g.dim_pad;
            const T* row = g.proj + (size_t)(t0 + t) * g.ld + h * g.dim_pad + d;
            qs[i] = to_f32(row[0]) * g.q_scale;
            ks[i] = to_f32(row[g.k_off()]);
            as[i] = expf(g.decay[(size_t)(t0 + t) * g.heads * g.dim_pad + h * g.dim_pad + d]);
        }
        __syncthreads();
        for (int t = 0; t < n; ++t) {
            const float v = in ? to_f32(g.proj[(size_t)(t0 + t) * g.ld + g.v_off() + h * g.vdim_pad + col]) : 0.0f;
            float o = 0.0f;
            for (int d = grp; d < g.dim_pad; d += 8) {
                const float x = fmaf(s[d * GR_COLS + c], as[t * g.dim_pad + d], ks[t * g.dim_pad + d] * v);
                s[d * GR_COLS + c] = x;
                o = fmaf(x, qs[t * g.dim_pad + d], o);
            }
            part[t][grp][c] = o;
        }
        __syncthreads();
        for (int i = threadIdx.x; i < n * GR_COLS; i += GR_THREADS) {
            const int t = i / GR_COLS, k = i - t * GR_COLS;
            float o = 0.0f;
            for (int w = 0; w < 8; ++w) o += part[t][w][k];
            if (blockIdx.x * GR_COLS + k < g.vdim_pad)
                g.mix[(size_t)(t0 + t) * g.heads * g.vdim_pad + h * g.vdim_pad + blockIdx.x * GR_COLS + k] = o;
        }
    }
    if (in)
        for (int d = grp; d < g.dim_pad; d += 8) st[(size_t)d * g.vdim_pad + col] = s[d * GR_COLS + c];
}

// One warp per (row, head): norm over the head's value columns, weight, silu(gate).
template <typename T>
__global__ void __launch_bounds__(ROW_THREADS)
gla_gate_kernel(const GlaArgs<T> g)
{
    pdl_wait_prior_grids();
    pdl_launch_dependents();
    const int lane = threadIdx.x & 31, r = blockIdx.x;
    for (int h = threadIdx.x >> 5; h < g.heads; h += ROW_THREADS / 32) {
        const float* o = g.mix + ((size_t)r * g.heads + h) * g.vdim_pad;
        float ss = 0.0f;
        for (int i = lane; i < g.vdim_pad; i += 32) ss = fmaf(o[i], o[i], ss);
        const float ir = inv_rms(ops::warp_sum(ss), g.vdim, g.eps);
        const T* gate = g.proj + (size_t)r * g.ld + g.gate_off() + h * g.vdim_pad;
        for (int i = lane; i < g.vdim_pad; i += 32)
            g.out[((size_t)r * g.heads + h) * g.vdim_pad + i] = from_f32<T>(o[i] * ir * __ldg(g.head_norm + i) * silu_f32(to_f32(gate[i])));
    }
}

// ------------------------------------------------------------------ chunks --
constexpr int GC_THREADS = 256;
constexpr float GLA_LOG2E = 1.4426950408889634f;

// eight values times 2^(e - f), as bf16 pairs hi + lo
__device__ __forceinline__ void decayed8(const uint4& x, const float4& e0, const float4& e1, const float4& f0, const float4& f1, float factor,
                                         uint4& hi, uint4& lo)
{
    float v[8];
    Vec<bf16>::unpack(x, v);
    const float e[8] = {e0.x, e0.y, e0.z, e0.w, e1.x, e1.y, e1.z, e1.w}, f[8] = {f0.x, f0.y, f0.z, f0.w, f1.x, f1.y, f1.z, f1.w};
#pragma unroll
    for (int i = 0; i < 8; ++i) v[i] *= factor * ex2_approx((e[i] - f[i]) * GLA_LOG2E);
    split_bf16(v[0], v[1], hi.x, lo.x);
    split_bf16(v[2], v[3], hi.y, lo.y);
    split_bf16(v[4], v[5], hi.z, lo.z);
    split_bf16(v[6], v[7], hi.w, lo.w);
}

// The chunk kernels take 64 key channels at a time: rows of 64 bf16, padded so that eight rows of a fragment hit distinct banks.
constexpr int GC_DIMS = 64, GC_ROW = GC_DIMS * 2 + 16, GC_BROW = GC_DIMS + 4;

// CTA = chunk, head and 64 key channels: the running sums b of log alpha, and dS[d][v] = sum_t k_td e^{b_last,d - b_td} v_tv.
// DK, DV: padded head sizes (0: read from the arguments).
__host__ inline size_t gla_chunk_state_smem_bytes(int vdim_pad) {
    return (size_t)GLA_CHUNK * (2 * GC_ROW + vdim_pad * 2 + 16 + GC_BROW * sizeof(float)) + 4 * GC_DIMS * sizeof(float);
}
template <int DK, int DV>
__global__ void __launch_bounds__(GC_THREADS)
gla_chunk_state_kernel(const GlaArgs<bf16> g)
{
    extern __shared__ __align__(16) uint8_t gc_smem[];
    const int dim_pad = DK > 0 ? DK : g.dim_pad, vdim_pad = DV > 0 ? DV : g.vdim_pad;
    const int vrow = vdim_pad * 2 + 16;
    uint8_t* khi = gc_smem;                                // [64][64]
    uint8_t* klo = khi + GLA_CHUNK * GC_ROW;
    uint8_t* vs = klo + GLA_CHUNK * GC_ROW;                // [64][vdim_pad]
    float* bs = reinterpret_cast<float*>(vs + GLA_CHUNK * vrow);          // [64][64]
    float* quarter_sum = bs + GLA_CHUNK * GC_BROW;         // [4][64]
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int h = blockIdx.y, r0 = blockIdx.x * GLA_CHUNK, n = min(GLA_CHUNK, g.rows - r0);
    const int d0 = blockIdx.z * GC_DIMS, dims = min(GC_DIMS, dim_pad - d0);
    const int cols = g.heads * dim_pad;
    pdl_wait_prior_grids();
    pdl_launch_dependents();
    const bf16* row0 = g.proj + (size_t)r0 * g.ld;
    const int vp = vdim_pad / 8;
    for (int i = tid; i < GLA_CHUNK * vp; i += GC_THREADS) {
        const int t = i / vp, c = i - t * vp;
        ops::att_cp_async16(smem_u32(vs + t * vrow + c * 16), row0 + (size_t)(t < n ? t : 0) * g.ld + g.v_off() + h * vdim_pad + c * 8, t < n ? 16 : 0);
    }
    ops::att_cp_async_commit();
    // keys on their way; their decays are made meanwhile.  Vector i: token i / 8, channels 8 (i % 8) on
    constexpr int KV = GLA_CHUNK * GC_DIMS / 8 / GC_THREADS;
    uint4 kv[KV];
#pragma unroll
    for (int j = 0; j < KV; ++j) {
        const int i = tid + j * GC_THREADS, t = i >> 3, d = (i & 7) * 8;
        kv[j] = t < n && d < dims ? *reinterpret_cast<const uint4*>(row0 + (size_t)t * g.ld + g.k_off() + h * dim_pad + d0 + d) : make_uint4(0, 0, 0, 0);
    }
    // z = low-rank row times the decay's weights: a warp's unit is 16 tokens x 8 channels
#pragma unroll
    for (int j = 0; j < 4; ++j) {
        const int u = warp + j * (GC_THREADS / 32), t0 = (u & 3) * 16, c0 = (u >> 2) * 8;
        if (c0 >= dims) break;
        const int ta = min(t0 + (lane >> 2), n - 1), tb = min(t0 + (lane >> 2) + 8, n - 1), k = (lane & 3) * 2;
        const bf16 *la = row0 + (size_t)ta * g.ld + g.low_off() + k, *lb = row0 + (size_t)tb * g.ld + g.low_off() + k;
        const bf16* w = g.w_decay + (size_t)(h * dim_pad + d0 + c0 + (lane >> 2)) * g.rank_pad + k;
        float z[4] = {0.0f, 0.0f, 0.0f, 0.0f};
        for (int k0 = 0; k0 < g.rank_pad; k0 += 16) {
            const uint32_t a[4] = {*reinterpret_cast<const uint32_t*>(la + k0), *reinterpret_cast<const uint32_t*>(lb + k0),
                                   *reinterpret_cast<const uint32_t*>(la + k0 + 8), *reinterpret_cast<const uint32_t*>(lb + k0 + 8)};
            mma_bf16(z, a, __ldg(reinterpret_cast<const uint32_t*>(w + k0)), __ldg(reinterpret_cast<const uint32_t*>(w + k0 + 8)));
        }
        const float2 bias = __ldg(reinterpret_cast<const float2*>(g.decay_bias + h * dim_pad + d0 + c0 + k));
#pragma unroll
        for (int i = 0; i < 2; ++i)
            *reinterpret_cast<float2*>(bs + (t0 + (lane >> 2) + i * 8) * GC_BROW + c0 + k) =
                make_float2(log_sigmoid_fast(z[2 * i] + bias.x) * g.inv_tau, log_sigmoid_fast(z[2 * i + 1] + bias.y) * g.inv_tau);
    }
    __syncthreads();
    {   // running sums, kept for the kernels that follow: a thread sums 16 tokens of a channel
        const int d = tid & 63, q = tid >> 6;
        float sum[16];
#pragma unroll
        for (int t = 0; t < 16; ++t) sum[t] = bs[(q * 16 + t) * GC_BROW + d] + (t > 0 ? sum[t - 1] : 0.0f);
        quarter_sum[q * GC_DIMS + d] = sum[15];
        __syncthreads();
        float before = 0.0f;
        for (int k = 0; k < q; ++k) before += quarter_sum[k * GC_DIMS + d];
        float* to = g.decay + (size_t)r0 * cols + h * dim_pad + d0 + d;
#pragma unroll
        for (int t = 0; t < 16; ++t) {
            const float b = before + sum[t];
            bs[(q * 16 + t) * GC_BROW + d] = b;
            if (q * 16 + t < n && d < dims) to[(size_t)(q * 16 + t) * cols] = b;
        }
    }
    __syncthreads();
#pragma unroll
    for (int j = 0; j < KV; ++j) {
        const int i = tid + j * GC_THREADS, t = i >> 3, d = (i & 7) * 8;
        uint4 hi = make_uint4(0, 0, 0, 0), lo = hi;
        if (t < n && d < dims) {
            const float *b = bs + t * GC_BROW + d, *last = bs + (n - 1) * GC_BROW + d;
            decayed8(kv[j], load4(last), load4(last + 4), load4(b), load4(b + 4), 1.0f, hi, lo);
        }
        *reinterpret_cast<uint4*>(khi + t * GC_ROW + d * 2) = hi;
        *reinterpret_cast<uint4*>(klo + t * GC_ROW + d * 2) = lo;
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    float* out = g.chunk_state + (((size_t)blockIdx.x * g.heads + h) * dim_pad + d0) * vdim_pad;
    // a warp's unit: 16 key channels x 64 value columns
    const int nb = (vdim_pad + 63) / 64;
    for (int u = warp; u < 4 * nb; u += GC_THREADS / 32) {
        const int m0 = (u & 3) * 16, v0 = (u >> 2) * 64;
        if (m0 >= dims) continue;
        float acc[8][4];
#pragma unroll
        for (int j = 0; j < 8; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) acc[j][e] = 0.0f;
#pragma unroll
        for (int kk = 0; kk < GLA_CHUNK / 16; ++kk) {
            // A = K'^T (channels x tokens) out of rows of tokens: transposing loads
            const uint32_t at = (uint32_t)((kk * 16 + (lane & 7) + (lane >> 4) * 8) * GC_ROW + (m0 + ((lane >> 3) & 1) * 8) * 2);
            uint32_t ahi[4], alo[4];
            ops::att_ldmatrix_x4_trans(ahi, smem_u32(khi) + at);
            ops::att_ldmatrix_x4_trans(alo, smem_u32(klo) + at);
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                if (v0 + j * 16 >= vdim_pad) continue;
                uint32_t b[4];
                ops::att_ldmatrix_x4_trans(b, smem_u32(vs) + (kk * 16 + (lane & 15)) * vrow + (v0 + j * 16 + (lane >> 4) * 8) * 2);
                mma_bf16(acc[2 * j], ahi, b[0], b[1]);
                mma_bf16(acc[2 * j + 1], ahi, b[2], b[3]);
                mma_bf16(acc[2 * j], alo, b[0], b[1]);
                mma_bf16(acc[2 * j + 1], alo, b[2], b[3]);
            }
        }
#pragma unroll
        for (int j = 0; j < 8; ++j) {
            const int v = v0 + j * 8 + (lane & 3) * 2, d = m0 + (lane >> 2);
            if (v0 + j * 8 >= vdim_pad) continue;
            *reinterpret_cast<float2*>(out + (size_t)d * vdim_pad + v) = make_float2(acc[j][0], acc[j][1]);
            *reinterpret_cast<float2*>(out + (size_t)(d + 8) * vdim_pad + v) = make_float2(acc[j][2], acc[j][3]);
        }
    }
}

// chunk_state[n] becomes the state ahead of chunk n; the slot's state moves on to the end.  A thread per four columns.
constexpr int GS_THREADS = 128, GS_AHEAD = 8;
template <typename T>
__global__ void __launch_bounds__(GS_THREADS)
gla_scan_kernel(const GlaArgs<T> g)
{
    pdl_wait_prior_grids();
    pdl_launch_dependents();
    const int per_head = g.dim_pad * g.vdim_pad / 4, i = blockIdx.x * GS_THREADS + threadIdx.x;
    if (i >= g.heads * per_head) return;
    const int h = i / per_head, e = i - h * per_head, d = e * 4 / g.vdim_pad;
    const int chunks = (g.rows + GLA_CHUNK - 1) / GLA_CHUNK, cols = g.heads * g.dim_pad;
    float4* st = reinterpret_cast<float4*>(g.slot_state(h)) + e;
    float4 s = g.meta[0] == 0 ? make_float4(0.f, 0.f, 0.f, 0.f) : *st;
    float4* cs = reinterpret_cast<float4*>(g.chunk_state) + (size_t)h * per_head + e;
    const size_t step = (size_t)g.heads * per_head;
    const float* b = g.decay + h * g.dim_pad + d;
    float4 add[GS_AHEAD];
    float a[GS_AHEAD];
    auto fetch = [&](int j, int n) {
        if (n >= chunks) return;
        add[j] = cs[n * step];
        a[j] = b[(size_t)(min(g.rows, (n + 1) * GLA_CHUNK) - 1) * cols];
    };
#pragma unroll
    for (int j = 0; j < GS_AHEAD; ++j) fetch(j, j);
    for (int n0 = 0; n0 < chunks; n0 += GS_AHEAD) {
#pragma unroll
        for (int j = 0; j < GS_AHEAD; ++j) {
            const int n = n0 + j;
            if (n >= chunks) break;
            cs[n * step] = s;
            const float f = expf(a[j]);
            s = make_float4(fmaf(s.x, f, add[j].x), fmaf(s.y, f, add[j].y), fmaf(s.z, f, add[j].z), fmaf(s.w, f, add[j].w));
            fetch(j, n + GS_AHEAD);                        // eight chunks ahead of its use
        }
    }
    *st = s;
}

// CTA = chunk and head; four warps = 16 of its tokens.  For 64 key channels at a time: the scores' share and the state's,
// (q 2^(b - ref)) (2^ref S); then scores V.  DK, DV: padded head sizes (DK = 0: read from the arguments, vdim_pad <= DV).
__host__ inline size_t gla_chunk_out_smem_bytes(int dim_pad, int vdim_pad) {
    return (size_t)GLA_CHUNK * (4 * GC_ROW + 2 * (vdim_pad * 2 + 16)) + sizeof(float) * (size_t)(dim_pad + 4 * GLA_CHUNK);
}
constexpr int GO_THREADS = 512;
template <int DK, int DV>
__global__ void __launch_bounds__(GO_THREADS, 2)
gla_chunk_out_kernel(const GlaArgs<bf16> g)
{
    extern __shared__ __align__(16) uint8_t gc_smem[];
    const int dim_pad = DK > 0 ? DK : g.dim_pad, vdim_pad = DK > 0 ? DV : g.vdim_pad;
    const int vrow = vdim_pad * 2 + 16;
    uint8_t* qhi = gc_smem;                                // [64][64] q 2^(b_t - ref); at the end the scores
    uint8_t* qlo = qhi + GLA_CHUNK * GC_ROW;
    uint8_t* khi = qlo + GLA_CHUNK * GC_ROW;               // [64][64] k 2^(ref - b_t)
    uint8_t* klo = khi + GLA_CHUNK * GC_ROW;
    uint8_t* shi = klo + GLA_CHUNK * GC_ROW;               // [64][vdim_pad] rows of the state; at the end the values
    uint8_t* slo = shi + GLA_CHUNK * vrow;
    float* refs = reinterpret_cast<float*>(slo + GLA_CHUNK * vrow);       // [dim_pad]
    float* sums = refs + dim_pad;                          // [4][64]
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int h = blockIdx.y, r0 = blockIdx.x * GLA_CHUNK, n = min(GLA_CHUNK, g.rows - r0);
    const int cols = g.heads * dim_pad, middle = min(GLA_MIDDLE, n - 1);
    pdl_wait_prior_grids();
    pdl_launch_dependents();
    const bf16* row0 = g.proj + (size_t)r0 * g.ld;
    const float* b0 = g.decay + (size_t)r0 * cols + h * dim_pad;
    const float* st = g.chunk_state + ((size_t)blockIdx.x * g.heads + h) * dim_pad * vdim_pad;
    constexpr int QV = GLA_CHUNK * GC_DIMS / 8 / GO_THREADS, SV = DV / 32;
    uint4 qv[QV], kv[QV];
    float4 bv[QV][2];
    auto load_rows = [&](int d0) {                         // vector i: token i / 8, channels 8 (i % 8) on
#pragma unroll
        for (int j = 0; j < QV; ++j) {
            const int i = tid + j * GO_THREADS, t = i >> 3, d = d0 + (i & 7) * 8;
            if (t >= n || d >= dim_pad) continue;
            const bf16* row = row0 + (size_t)t * g.ld + h * dim_pad + d;
            qv[j] = *reinterpret_cast<const uint4*>(row);
            kv[j] = *reinterpret_cast<const uint4*>(row + g.k_off());
            bv[j][0] = load4(b0 + (size_t)t * cols + d);
            bv[j][1] = load4(b0 + (size_t)t * cols + d + 4);
        }
    };
    load_rows(0);
    bool steep = false;
    for (int d = tid; d < dim_pad; d += GO_THREADS) {
        const float first = b0[d], mid = b0[(size_t)middle * cols + d], last = b0[(size_t)(n - 1) * cols + d];
        steep = steep || first - mid > GLA_HALF_LIMIT || mid - last > GLA_HALF_LIMIT;
        refs[d] = mid;
    }
    steep = __syncthreads_or(steep);
    const float4 zero4 = make_float4(0.f, 0.f, 0.f, 0.f);
    const int block = warp >> 2, quarter = warp & 3;       // this warp's 16 tokens; which 16 tokens they are scored against, which columns
    const uint32_t q_at = (uint32_t)((block * 16 + (lane & 15)) * GC_ROW + (lane >> 4) * 16);
    const bool scoring = !steep && quarter <= block;
    float a[2][4], o[DV / 32][4];
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) a[j][e] = 0.0f;
#pragma unroll
    for (int j = 0; j < DV / 32; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) o[j][e] = 0.0f;

    for (int d0 = 0; d0 < dim_pad; d0 += GC_DIMS) {
        const int dims = min(GC_DIMS, dim_pad - d0);
        if (d0 > 0) load_rows(d0);
        float4 sv[SV];
        const int vq = vdim_pad / 4, count = dims * vq;
#pragma unroll
        for (int j = 0; j < SV; ++j) {
            const int i = tid + j * GO_THREADS;
            if (i < count) sv[j] = load4(st + (size_t)d0 * vdim_pad + i * 4);
        }
#pragma unroll
        for (int j = 0; j < QV; ++j) {
            const int i = tid + j * GO_THREADS, t = i >> 3, d = (i & 7) * 8;
            uint4 qh = make_uint4(0, 0, 0, 0), ql = qh, kh = qh, kl = qh;
            if (t < n && d < dims) {
                const float4 f0 = steep ? zero4 : load4(refs + d0 + d), f1 = steep ? zero4 : load4(refs + d0 + d + 4);
                decayed8(qv[j], bv[j][0], bv[j][1], f0, f1, g.q_scale, qh, ql);
                if (!steep) decayed8(kv[j], f0, f1, bv[j][0], bv[j][1], 1.0f, kh, kl);
            }
            *reinterpret_cast<uint4*>(qhi + t * GC_ROW + d * 2) = qh;
            *reinterpret_cast<uint4*>(qlo + t * GC_ROW + d * 2) = ql;
            *reinterpret_cast<uint4*>(khi + t * GC_ROW + d * 2) = kh;
            *reinterpret_cast<uint4*>(klo + t * GC_ROW + d * 2) = kl;
        }
#pragma unroll
        for (int j = 0; j < SV; ++j) {
            const int i = tid + j * GO_THREADS;
            if (i >= count) continue;
            const int d = i / vq, v = (i - d * vq) * 4;
            const float f = steep ? 1.0f : ex2_approx(refs[d0 + d] * GLA_LOG2E);
            uint2 hi, lo;
            split_bf16(sv[j].x * f, sv[j].y * f, hi.x, lo.x);
            split_bf16(sv[j].z * f, sv[j].w * f, hi.y, lo.y);
            *reinterpret_cast<uint2*>(shi + d * vrow + v * 2) = hi;
            *reinterpret_cast<uint2*>(slo + d * vrow + v * 2) = lo;
        }
        __syncthreads();
        const uint32_t k_at = (uint32_t)((quarter * 16 + (lane & 7) + (lane >> 4) * 8) * GC_ROW + ((lane >> 3) & 1) * 16);
        for (int c = 0; c < dims / 16; ++c) {
            uint32_t qh[4], ql[4];
            ldmatrix_x4(qh, smem_u32(qhi) + q_at + c * 32);
            ldmatrix_x4(ql, smem_u32(qlo) + q_at + c * 32);
            if (scoring) {
                uint32_t kh[4], kl[4];
                ldmatrix_x4(kh, smem_u32(khi) + k_at + c * 32);
                ldmatrix_x4(kl, smem_u32(klo) + k_at + c * 32);
#pragma unroll
                for (int i = 0; i < 2; ++i) {
                    mma_bf16(a[i], qh, kh[2 * i], kh[2 * i + 1]);
                    mma_bf16(a[i], ql, kh[2 * i], kh[2 * i + 1]);
                    mma_bf16(a[i], qh, kl[2 * i], kl[2 * i + 1]);
                }
            }
#pragma unroll
            for (int j = 0; j < DV / 64; ++j) {            // the warp takes every fourth 16 value columns
                const int v0 = (4 * j + quarter) * 16;
                if (v0 >= vdim_pad) continue;
                const uint32_t at = (uint32_t)((c * 16 + (lane & 15)) * vrow + (v0 + (lane >> 4) * 8) * 2);
                uint32_t bh[4], bl[4];
                ops::att_ldmatrix_x4_trans(bh, smem_u32(shi) + at);
                ops::att_ldmatrix_x4_trans(bl, smem_u32(slo) + at);
#pragma unroll
                for (int i = 0; i < 2; ++i) {
                    mma_bf16(o[2 * j + i], qh, bh[2 * i], bh[2 * i + 1]);
                    mma_bf16(o[2 * j + i], ql, bh[2 * i], bh[2 * i + 1]);
                    mma_bf16(o[2 * j + i], qh, bl[2 * i], bl[2 * i + 1]);
                }
            }
        }
        __syncthreads();                                   // this part has been used
    }
    // ---- the values over the state's rows, the scores over the queries ----
    uint8_t *vs = shi, *ahi = qhi, *alo = qlo;
    const int vp = vdim_pad / 8;
    for (int i = tid; i < GLA_CHUNK * vp; i += GO_THREADS) {
        const int t = i / vp, c = i - t * vp;
        ops::att_cp_async16(smem_u32(vs + t * vrow + c * 16), row0 + (size_t)(t < n ? t : 0) * g.ld + g.v_off() + h * vdim_pad + c * 8, t < n ? 16 : 0);
    }
    ops::att_cp_async_commit();
    if (scoring) {
#pragma unroll
        for (int j = 0; j < 2; ++j)
#pragma unroll
            for (int i = 0; i < 2; ++i) {
                const int t = block * 16 + (lane >> 2) + i * 8, s = quarter * 16 + j * 8 + (lane & 3) * 2;
                uint32_t hi, lo;
                split_bf16(s <= t ? a[j][2 * i] : 0.0f, s + 1 <= t ? a[j][2 * i + 1] : 0.0f, hi, lo);
                *reinterpret_cast<uint32_t*>(ahi + t * GC_ROW + s * 2) = hi;
                *reinterpret_cast<uint32_t*>(alo + t * GC_ROW + s * 2) = lo;
            }
    }
    if (steep) {                                           // a warp per token pair
        for (int u = warp; u < GLA_CHUNK * GLA_CHUNK; u += GO_THREADS / 32) {
            const int t = u / GLA_CHUNK, s = u - t * GLA_CHUNK;
            float sum = 0.0f;
            if (s <= t && t < n)
                for (int d = lane; d < dim_pad; d += 32)
                    sum = fmaf(to_f32(row0[(size_t)t * g.ld + h * dim_pad + d]) * g.q_scale * to_f32(row0[(size_t)s * g.ld + g.k_off() + h * dim_pad + d]),
                               ex2_approx((b0[(size_t)t * cols + d] - b0[(size_t)s * cols + d]) * GLA_LOG2E), sum);
            sum = ops::warp_sum(sum);
            const bf16 hi = __float2bfloat16_rn(sum);
            if (lane == 0) {
                reinterpret_cast<bf16*>(ahi + t * GC_ROW)[s] = hi;
                reinterpret_cast<bf16*>(alo + t * GC_ROW)[s] = __float2bfloat16_rn(sum - to_f32(hi));
            }
        }
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    for (int kk = 0; kk <= block; ++kk) {
        uint32_t xh[4], xl[4];
        ldmatrix_x4(xh, smem_u32(ahi) + q_at + kk * 32);
        ldmatrix_x4(xl, smem_u32(alo) + q_at + kk * 32);
#pragma unroll
        for (int j = 0; j < DV / 64; ++j) {
            const int v0 = (4 * j + quarter) * 16;
            if (v0 >= vdim_pad) continue;
            uint32_t b[4];
            ops::att_ldmatrix_x4_trans(b, smem_u32(vs) + (kk * 16 + (lane & 15)) * vrow + (v0 + (lane >> 4) * 8) * 2);
            mma_bf16(o[2 * j], xh, b[0], b[1]);
            mma_bf16(o[2 * j + 1], xh, b[2], b[3]);
            mma_bf16(o[2 * j], xl, b[0], b[1]);
            mma_bf16(o[2 * j + 1], xl, b[2], b[3]);
        }
    }
    // ---- norm over the head's columns, gate, store ----
#pragma unroll
    for (int i = 0; i < 2; ++i) {
        float ss = 0.0f;
#pragma unroll
        for (int j = 0; j < DV / 32; ++j) ss = fmaf(o[j][2 * i], o[j][2 * i], fmaf(o[j][2 * i + 1], o[j][2 * i + 1], ss));
        ss += __shfl_xor_sync(0xffffffffu, ss, 1);
        ss += __shfl_xor_sync(0xffffffffu, ss, 2);
        if ((lane & 3) == 0) sums[quarter * GLA_CHUNK + block * 16 + (lane >> 2) + i * 8] = ss;
    }
    __syncthreads();
#pragma unroll
    for (int i = 0; i < 2; ++i) {
        const int t = block * 16 + (lane >> 2) + i * 8;
        if (t >= n) continue;
        const float ir = inv_rms((sums[t] + sums[GLA_CHUNK + t]) + (sums[2 * GLA_CHUNK + t] + sums[3 * GLA_CHUNK + t]), g.vdim, g.eps);
        const bf16* gate = row0 + (size_t)t * g.ld + g.gate_off() + h * vdim_pad;
        bf16* out = g.out + ((size_t)(r0 + t) * g.heads + h) * vdim_pad;
#pragma unroll
        for (int j = 0; j < DV / 32; ++j) {
            const int v = (4 * (j >> 1) + quarter) * 16 + (j & 1) * 8 + (lane & 3) * 2;
            if (v >= vdim_pad) continue;
            const float2 w = *reinterpret_cast<const float2*>(g.head_norm + v);
            const uint32_t z = *reinterpret_cast<const uint32_t*>(gate + v);
            const float z0 = __uint_as_float(z << 16), z1 = __uint_as_float(z & 0xffff0000u);
            *reinterpret_cast<__nv_bfloat162*>(out + v) =
                __floats2bfloat162_rn(o[j][2 * i] * ir * w.x * z0 * rcp_approx(1.0f + ex2_approx(-GLA_LOG2E * z0)),
                                      o[j][2 * i + 1] * ir * w.y * z1 * rcp_approx(1.0f + ex2_approx(-GLA_LOG2E * z1)));
        }
    }
}

// ------------------------------------------------------------------ decode --
// One token.  A cluster of CTAs per head, each with a share of the value columns: decays, the state's share moved on in
// place, the share of o; the sums of squares of the cluster make the norm.
constexpr int GX_THREADS = 256, GX_MAX_SPLITS = 8;
template <typename T>
struct GlaDecodeArgs {
    const float* proj;          // f32: q | k | v | gate | low-rank
    float* out;                 // f32 [heads * vdim_pad]
    float* state;
    const T* w_decay;
    const float* decay_bias;
    const float* head_norm;
    const int* meta;
    int heads, dim_pad, vdim, vdim_pad, rank_pad;
    float inv_tau, q_scale, eps;
};
__host__ __device__ inline int gla_decode_share(int vdim_pad, int splits) { return ((vdim_pad / 4 + splits - 1) / splits) * 4; }
__host__ inline size_t gla_decode_smem_bytes(int dim_pad, int vdim_pad, int splits) {
    const int quads = gla_decode_share(vdim_pad, splits) / 4;
    const int groups = GX_THREADS / quads < 1 ? 1 : GX_THREADS / quads;
    return sizeof(float) * ((size_t)3 * dim_pad + (size_t)groups * quads * 4);
}
template <typename T>
__global__ void __launch_bounds__(GX_THREADS)
gla_decode_kernel(const GlaDecodeArgs<T> g)
{
    using V = Vec<T>;
    pdl_launch_dependents();
    extern __shared__ __align__(16) float gx_smem[];
    __shared__ float red[32];
    __shared__ float recv[GX_MAX_SPLITS];
    const int splits = gridDim.x, rank = blockIdx.x, h = blockIdx.y, tid = threadIdx.x;
    const int share = gla_decode_share(g.vdim_pad, splits), quads = share / 4;
    const int groups = GX_THREADS / quads < 1 ? 1 : GX_THREADS / quads;
    float* qs = gx_smem;                                   // [dim_pad]
    float* ks = qs + g.dim_pad;
    float* as = ks + g.dim_pad;
    float* part = as + g.dim_pad;                          // [groups][share]
    const int kd = g.heads * g.dim_pad, vd = g.heads * g.vdim_pad;
    asm volatile("barrier.cluster.arrive.relaxed.aligned;" ::: "memory");
    // weights do not depend on the kernel before
    constexpr int WV = 2;                                  // vectors of the decay's weights held ahead
    uint4 wv[WV];
    const float bias = tid < g.dim_pad ? __ldg(g.decay_bias + h * g.dim_pad + tid) : 0.0f;
#pragma unroll
    for (int i = 0; i < WV; ++i)
        wv[i] = tid < g.dim_pad && i * V::N < g.rank_pad ? __ldg(reinterpret_cast<const uint4*>(g.w_decay + (size_t)(h * g.dim_pad + tid) * g.rank_pad) + i)
                                                         : make_uint4(0, 0, 0, 0);
    {   // the state's share into L2; the slot as it is now (a stale one prefetches another sequence's)
        const float* st_now = g.state + ((size_t)*(volatile const int*)(g.meta + 1) * g.heads + h) * g.dim_pad * g.vdim_pad + rank * share;
        if (rank * share < g.vdim_pad)
            for (int d = tid; d < g.dim_pad; d += GX_THREADS)
                for (int c = 0; c < share; c += 32) l2_prefetch(st_now + (size_t)d * g.vdim_pad + c);
    }
    pdl_wait_prior_grids();
    const float* low = g.proj + 2 * kd + 2 * vd;
    for (int d = tid; d < g.dim_pad; d += GX_THREADS) {
        qs[d] = g.proj[h * g.dim_pad + d] * g.q_scale;
        ks[d] = g.proj[kd + h * g.dim_pad + d];
        float z = d == tid ? bias : __ldg(g.decay_bias + h * g.dim_pad + d);
        for (int i = 0; i * V::N < g.rank_pad; ++i) {
            float w[V::N];
            V::unpack(d == tid && i == 0 ? wv[0] : d == tid && i == 1 ? wv[1]
                          : __ldg(reinterpret_cast<const uint4*>(g.w_decay + (size_t)(h * g.dim_pad + d) * g.rank_pad) + i), w);
#pragma unroll
            for (int e = 0; e < V::N; e += 4) {
                const float4 a = *reinterpret_cast<const float4*>(low + i * V::N + e);
                z = fmaf(w[e], a.x, fmaf(w[e + 1], a.y, fmaf(w[e + 2], a.z, fmaf(w[e + 3], a.w, z))));
            }
        }
        as[d] = expf(log_sigmoid_f32(z) * g.inv_tau);
    }
    const bool fresh = g.meta[0] == 0;
    float* st = g.state + ((size_t)g.meta[1] * g.heads + h) * g.dim_pad * g.vdim_pad;
    __syncthreads();
    const int c0 = rank * share, grp = tid / quads;
    for (int qi = tid % quads; qi < quads; qi += GX_THREADS) {            // one round unless a share has more quads than threads
        const int c = c0 + qi * 4;
        float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
        if (c < g.vdim_pad && grp < groups) {
            const float4 v = *reinterpret_cast<const float4*>(g.proj + 2 * kd + h * g.vdim_pad + c);
#pragma unroll 4
            for (int d = grp; d < g.dim_pad; d += groups) {
                float4* at = reinterpret_cast<float4*>(st + (size_t)d * g.vdim_pad + c);
                const float4 s = fresh ? make_float4(0.f, 0.f, 0.f, 0.f) : *at;
                const float a = as[d], k = ks[d], q = qs[d];
                const float4 x = make_float4(fmaf(s.x, a, k * v.x), fmaf(s.y, a, k * v.y), fmaf(s.z, a, k * v.z), fmaf(s.w, a, k * v.w));
                *at = x;
                o.x = fmaf(x.x, q, o.x); o.y = fmaf(x.y, q, o.y); o.z = fmaf(x.z, q, o.z); o.w = fmaf(x.w, q, o.w);
            }
        }
        if (grp < groups) *reinterpret_cast<float4*>(part + (size_t)grp * share + qi * 4) = o;
    }
    __syncthreads();
    float ss = 0.0f;
    for (int i = tid; i < share; i += GX_THREADS) {
        float o = 0.0f;
        for (int k = 0; k < groups; ++k) o += part[(size_t)k * share + i];
        part[i] = o;                                       // column i is this thread's alone
        if (c0 + i < g.vdim_pad) ss = fmaf(o, o, ss);
    }
    ss = group_sum(ss, red, GX_THREADS, 1);
    asm volatile("barrier.cluster.wait.aligned;" ::: "memory");
    if (tid < splits) st_cluster_f32(mapa_shared(smem_u32(recv + rank), tid), ss);
    cluster_sync_all();
    float all = 0.0f;
    for (int s = 0; s < splits; ++s) all += recv[s];
    const float ir = inv_rms(all, g.vdim, g.eps);
    for (int i = tid; i < share; i += GX_THREADS) {
        const int c = c0 + i;
        if (c >= g.vdim_pad) continue;
        g.out[h * g.vdim_pad + c] = part[i] * ir * __ldg(g.head_norm + c) * silu_f32(g.proj[2 * kd + vd + h * g.vdim_pad + c]);
    }
}

}  // namespace dense
}  // namespace twm
