// twm_dense_attn.cuh — windowed sigmoid attention of a portion of a prompt, bfloat16, on warp-level MMAs.
//
// CTA = 64 queries of one head (four warps of 16) and a block of DV value columns; it walks the 64-key
// tiles that hold a visible key: the tiles of the kept first keys, then the window's.  K and V tiles
// arrive by cp.async, one tile ahead.  S = Q K^T in FP32; the weights sigmoid(scale * s + table[distance])
// are computed in FP32 (one FMA, one ex2, one reciprocal: the per-head table already holds the distance
// bias and the head's offset) and enter P V as a bf16 pair hi + lo, two MMAs, so that no more than
// 2^-17 of a weight is lost.  Nothing is normalised over keys, so tiles simply add up.  The output gate
// is applied to the accumulator before it is stored.
#pragma once

#include "twm_dense_simt.cuh"

namespace twm {
namespace dense {

constexpr int AM_Q = 64, AM_K = 64, AM_THREADS = 128;

__device__ __forceinline__ void ldmatrix_x4(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void mma_bf16(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ float ex2_approx(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
__device__ __forceinline__ float rcp_approx(float x) {
    float y;
    asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
// two floats as a bf16 pair, and what the rounding left over as another
__device__ __forceinline__ void split_bf16(float a, float b, uint32_t& hi, uint32_t& lo) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
    hi = *reinterpret_cast<const uint32_t*>(&h);
    const __nv_bfloat162 l = __floats2bfloat162_rn(a - __uint_as_float(hi << 16), b - __uint_as_float(hi & 0xffff0000u));
    lo = *reinterpret_cast<const uint32_t*>(&l);
}

template <int DV>
__host__ inline size_t attn_mma_smem_bytes(int dim_pad) {
    return (size_t)(AM_Q + 2 * AM_K) * (dim_pad * 2 + 16) + (size_t)2 * AM_K * (DV * 2 + 16) + 2 * 128 * sizeof(float);
}

// DK = padded key size (0: read from the arguments)
template <int DK, int DV>
__global__ void __launch_bounds__(AM_THREADS)
attn_mma_kernel(const AttnArgs<bf16> g)
{
    pdl_launch_dependents();
    extern __shared__ __align__(16) uint8_t am_smem[];
    const int dim_pad = DK > 0 ? DK : g.dim_pad;
    const int krow = dim_pad * 2 + 16;                    // padded: the eight rows of a fragment hit distinct banks
    constexpr int vrow = DV * 2 + 16;
    uint8_t* qs = am_smem;
    uint8_t* ks = qs + AM_Q * krow;
    uint8_t* vs = ks + 2 * AM_K * krow;
    float* bs = reinterpret_cast<float*>(vs + 2 * AM_K * vrow);      // [2][128]: the table over a tile's distances
    constexpr float LOG2E = 1.4426950408889634f;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    pdl_wait_prior_grids();

    const int h = blockIdx.y, kvh = h / (g.heads / g.kv_heads), vc0 = blockIdx.z * DV;
    const int r0 = blockIdx.x * AM_Q;
    const int pos0 = g.meta[0], end = pos0 + g.rows;        // keys at `end` and later do not exist yet
    const int p0 = pos0 + r0, p1 = min(end, p0 + AM_Q) - 1; // positions of the CTA's first and last query
    const int kd = g.kv_heads * dim_pad, vd = g.kv_heads * g.vdim_pad;
    const bf16* kc = g.k_cache + (size_t)g.meta[1] * g.capacity * kd + kvh * dim_pad;
    const bf16* vc = g.v_cache + (size_t)g.meta[1] * g.capacity * vd + kvh * g.vdim_pad + vc0;
    const float* table = g.bias_table != nullptr ? g.bias_table + (size_t)h * g.bias_len : nullptr;
    int sinks, lo;
    visible_range(p0, g.window, g.keep_first, sinks, lo);
    const int w_first = lo / AM_K;                          // first tile of the window
    const int n_sink = min((g.keep_first + AM_K - 1) / AM_K, w_first);
    const int n_tiles = n_sink + p1 / AM_K - w_first + 1;
    auto tile_key = [&](int t) { return (t < n_sink ? t : w_first + t - n_sink) * AM_K; };

    const int kpieces = dim_pad / 8;                      // 16-byte pieces of a row
    constexpr int vpieces = DV / 8;
    const int vvalid = min(vpieces, (g.vdim_pad - vc0) / 8);
    auto load_tile = [&](int t, int buf) {
        const int k0 = tile_key(t);
        for (int i = tid; i < AM_K * kpieces; i += AM_THREADS) {
            const int r = i / kpieces, c = i - r * kpieces;
            const bool in = k0 + r < end;
            ops::att_cp_async16(smem_u32(ks + (size_t)buf * AM_K * krow + r * krow + c * 16), kc + (size_t)(in ? k0 + r : 0) * kd + c * 8,
                                in ? 16 : 0);
        }
        for (int i = tid; i < AM_K * vpieces; i += AM_THREADS) {
            const int r = i / vpieces, c = i - r * vpieces;
            const bool in = k0 + r < end && c < vvalid;
            ops::att_cp_async16(smem_u32(vs + (size_t)buf * AM_K * vrow + r * vrow + c * 16), vc + (size_t)(in ? k0 + r : 0) * vd + (in ? c * 8 : 0),
                                in ? 16 : 0);
        }
        // entry x: distance x - 63 + (first query - first key)
        const int d = p0 - k0 - (AM_K - 1) + tid;
        if (table != nullptr)
            asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(smem_u32(bs + buf * 128 + tid)),
                         "l"(table + min(max(d, 0), g.bias_len - 1)) : "memory");
        ops::att_cp_async_commit();
    };
    for (int i = tid; i < AM_Q * kpieces; i += AM_THREADS) {
        const int r = i / kpieces, c = i - r * kpieces;
        const bool in = r0 + r < g.rows;
        ops::att_cp_async16(smem_u32(qs + r * krow + c * 16), g.proj + (size_t)(in ? r0 + r : 0) * g.ld + h * dim_pad + c * 8, in ? 16 : 0);
    }
    if (table == nullptr) { bs[tid] = 0.0f; bs[128 + tid] = 0.0f; }
    load_tile(0, 0);

    float o[DV / 8][4];
#pragma unroll
    for (int n = 0; n < DV / 8; ++n)
#pragma unroll
        for (int j = 0; j < 4; ++j) o[n][j] = 0.0f;
    const int rw = warp * 16 + (lane >> 2);                 // this thread's rows: rw and rw + 8
    const uint32_t q_at = smem_u32(qs + (warp * 16 + (lane & 15)) * krow + (lane >> 4) * 16);

    for (int t = 0; t < n_tiles; ++t) {
        const int buf = t & 1;
        if (t + 1 < n_tiles) {
            load_tile(t + 1, buf ^ 1);
            ops::att_cp_async_wait_all_but_one();
        } else {
            asm volatile("cp.async.wait_group 0;" ::: "memory");
        }
        __syncthreads();
        const int k0 = tile_key(t);
        // ---- S = Q K^T: 16 queries x 64 keys per warp ----
        float s[AM_K / 8][4];
#pragma unroll
        for (int n = 0; n < AM_K / 8; ++n)
#pragma unroll
            for (int j = 0; j < 4; ++j) s[n][j] = 0.0f;
        const uint32_t k_at = smem_u32(ks + (size_t)buf * AM_K * krow + ((lane & 7) + (lane >> 4) * 8) * krow + ((lane >> 3) & 1) * 16);
#pragma unroll 4
        for (int c = 0; c < dim_pad / 16; ++c) {
            uint32_t a[4];
            ldmatrix_x4(a, q_at + c * 32);
#pragma unroll
            for (int n = 0; n < AM_K / 16; ++n) {
                uint32_t b[4];
                ldmatrix_x4(b, k_at + n * 16 * krow + c * 32);
                mma_bf16(s[2 * n], a, b[0], b[1]);
                mma_bf16(s[2 * n + 1], a, b[2], b[3]);
            }
        }
        // ---- weights ----
        const bool all_seen = k0 + AM_K - 1 <= p0 && (p1 - k0 < g.window || k0 + AM_K <= g.keep_first);
        const float* bt = bs + buf * 128 + (AM_K - 1) + rw;
#pragma unroll
        for (int n = 0; n < AM_K / 8; ++n) {
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                const int c = n * 8 + (lane & 3) * 2 + (j & 1), rr = (j >> 1) * 8;
                const float e = ex2_approx(-LOG2E * fmaf(s[n][j], g.scale, bt[rr - c]));
                float w = rcp_approx(1.0f + e);
                if (!all_seen) {
                    const int p = p0 + rw + rr, key = k0 + c;
                    if (!(key <= p && (p - key < g.window || key < g.keep_first))) w = 0.0f;
                }
                s[n][j] = w;
            }
        }
        // ---- O += P V ----
        const uint32_t v_at = smem_u32(vs + (size_t)buf * AM_K * vrow + (lane & 15) * vrow + (lane >> 4) * 16);
#pragma unroll
        for (int kk = 0; kk < AM_K / 16; ++kk) {
            uint32_t hi[4], lw[4];
            split_bf16(s[2 * kk][0], s[2 * kk][1], hi[0], lw[0]);
            split_bf16(s[2 * kk][2], s[2 * kk][3], hi[1], lw[1]);
            split_bf16(s[2 * kk + 1][0], s[2 * kk + 1][1], hi[2], lw[2]);
            split_bf16(s[2 * kk + 1][2], s[2 * kk + 1][3], hi[3], lw[3]);
#pragma unroll
            for (int n = 0; n < DV / 16; ++n) {
                uint32_t b[4];
                ops::att_ldmatrix_x4_trans(b, v_at + kk * 16 * vrow + n * 32);
                mma_bf16(o[2 * n], hi, b[0], b[1]);
                mma_bf16(o[2 * n + 1], hi, b[2], b[3]);
                mma_bf16(o[2 * n], lw, b[0], b[1]);
                mma_bf16(o[2 * n + 1], lw, b[2], b[3]);
            }
        }
        __syncthreads();                                    // the next-but-one tile overwrites this buffer
    }
    // ---- gate and store ----
#pragma unroll
    for (int i = 0; i < 2; ++i) {
        const int r = r0 + rw + i * 8;
        if (r >= g.rows) continue;
        bf16* out = g.out + (size_t)r * g.heads * g.vdim_pad + h * g.vdim_pad + vc0;
        const bf16* gate = g.gate_off >= 0 ? g.proj + (size_t)r * g.ld + g.gate_off + h * g.vdim_pad + vc0 : nullptr;
#pragma unroll
        for (int n = 0; n < DV / 8; ++n) {
            const int c = n * 8 + (lane & 3) * 2;
            if (vc0 + c >= g.vdim_pad) continue;
            float a = o[n][2 * i], b = o[n][2 * i + 1];
            if (gate != nullptr) {
                const uint32_t gv = *reinterpret_cast<const uint32_t*>(gate + c);
                a *= sigmoid_f32(__uint_as_float(gv << 16));
                b *= sigmoid_f32(__uint_as_float(gv & 0xffff0000u));
            }
            const __nv_bfloat162 pair = __floats2bfloat162_rn(a, b);
            *reinterpret_cast<__nv_bfloat162*>(out + c) = pair;
        }
    }
}

}  // namespace dense
}  // namespace twm
