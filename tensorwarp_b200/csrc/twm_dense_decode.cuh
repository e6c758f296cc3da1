// twm_dense_decode.cuh — one decoded token of a dense model: the streaming matrix-vector product and
// the split-key attention.
//
// gemv_kernel: y = W a for one token, HBM-bound.  A CTA owns a run of W's rows.  One warp streams them
// with 1-D bulk copies into a shared-memory ring, eight row pieces of 2 KB a stage, and starts
// before the preceding kernel has finished (weights are constants); eight warps multiply: warps 0-3 the
// stage's rows 0-3, a quarter of the piece each, warps 4-7 the rows 4-7.  The steps between two products
// are its prologue: every CTA makes the product's input row itself, from the residual stream and the
// sublayer output that joins it (norm, add, token shift or final norm), in FP32, and rounds it once.
// The epilogue of the gate/up product applies the gated activation, so no launch stands between products
// but the attention.
#pragma once

#include "twm_dense_rows.cuh"
#include "twm_dense_simt.cuh"
#include "twm_gemm_tc.cuh"

namespace twm {
namespace dense {

enum { PRO_VEC = 0, PRO_RESIDUAL = 1, PRO_SHIFT = 2, PRO_FINAL = 3 };

constexpr int GV_CONSUMERS = 256;
constexpr int GV_THREADS = GV_CONSUMERS + 32;
constexpr int GV_ROWS = 8;                  // rows per stage
constexpr int GV_PIECE = 2048;              // bytes of a row per stage
constexpr int GV_STAGE = GV_ROWS * GV_PIECE;
constexpr int GV_MAX_STAGES = 8;
constexpr int GV_FLUSH = 16;                // row groups between two cross-warp sums

template <typename T>
struct GemvArgs {
    const T* w;                 // [N (gated: N gate rows, then N up rows)][ldw]
    int N, ldw;                 // ldw = K: padded, a multiple of 16 bytes
    float* out;                 // [N]
    int rows_per_cta, stages;
    const float* vec;           // PRO_VEC: the input row, f32 [ldw]
    ResidualSource<T> src;      // otherwise: row 0 of the residual stream
    float* x_out;               // the residual row after the add, written by CTA 0
    const float* shift;
    float* shift_state;
    const float* final_norm;
    const int* meta;
};

template <typename T>
__host__ __device__ inline size_t gemv_smem_bytes(int ldw, int stages) {
    return (size_t)stages * GV_STAGE + (((size_t)ldw * sizeof(T) + 127) & ~(size_t)127);
}

template <typename T, int PRO, bool GATED>
__global__ void __launch_bounds__(GV_THREADS, 1)
gemv_kernel(const GemvArgs<T> g)
{
    using V = Vec<T>;
    extern __shared__ __align__(128) uint8_t gemv_smem[];
    uint8_t* ring = gemv_smem;
    T* as = reinterpret_cast<T*>(gemv_smem + (size_t)g.stages * GV_STAGE);
    __shared__ __align__(8) uint64_t full[GV_MAX_STAGES], empty[GV_MAX_STAGES];
    __shared__ float part[2][GV_FLUSH][8][4];
    __shared__ float red[32];
    __shared__ int abort_s;
    volatile int* abort_flag = &abort_s;

    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    constexpr int OUT_ROWS = GATED ? GV_ROWS / 2 : GV_ROWS;         // outputs per row group
    const int n_begin = blockIdx.x * g.rows_per_cta, n_end = min(g.N, n_begin + g.rows_per_cta);
    const int groups = (n_end - n_begin + OUT_ROWS - 1) / OUT_ROWS;
    const int row_bytes = g.ldw * (int)sizeof(T);
    const int chunks = (row_bytes + GV_PIECE - 1) / GV_PIECE;
    const int iters = groups * chunks;

    if (tid == 0) {
        for (int s = 0; s < g.stages; ++s) { mbar_init(&full[s], 1); mbar_init(&empty[s], GV_CONSUMERS / 32); }
        abort_s = 0;
        mbar_fence_init();
    }
    __syncthreads();
    pdl_launch_dependents();

    if (warp == GV_CONSUMERS / 32) {
        // ------------------------------------------------------------ producer --
        int slot = 0, c = 0, gi = 0;
        uint32_t phase = 1;                                          // a fresh barrier passes a wait for the phase before
        for (int it = 0; it < iters; ++it) {
            if (it >= g.stages && !mbar_wait_bounded(&empty[slot], phase, abort_flag)) break;
            const int bytes = min(GV_PIECE, row_bytes - c * GV_PIECE);
            const int o0 = n_begin + gi * OUT_ROWS;
            const int valid = min(OUT_ROWS, n_end - o0);             // outputs of this group
            if (lane == 0) mbar_arrive_expect_tx(&full[slot], (uint32_t)bytes * (uint32_t)(GATED ? 2 * valid : valid));
            __syncwarp();
            if (lane < GV_ROWS && (GATED ? (lane & 3) : lane) < valid) {
                const int row = GATED ? (lane < 4 ? o0 + lane : g.N + o0 + lane - 4) : o0 + lane;
                bulk_g2s(ring + (size_t)slot * GV_STAGE + lane * GV_PIECE,
                         reinterpret_cast<const uint8_t*>(g.w) + (size_t)row * row_bytes + (size_t)c * GV_PIECE, (uint32_t)bytes,
                         &full[slot]);
            }
            if (++c == chunks) { c = 0; ++gi; }
            if (++slot == g.stages) { slot = 0; if (it >= g.stages) phase ^= 1u; else phase = 0; }
        }
        return;
    }

    // ------------------------------------------------------- prologue (256 threads) --
    pdl_wait_prior_grids();
    if (PRO == PRO_VEC) {
        for (int i = tid; i < (g.ldw >> 2); i += GV_CONSUMERS) store4<T>(as + i * 4, reinterpret_cast<const float4*>(g.vec)[i]);
    } else {
        const int pos = g.meta[0];
        const int tok = g.src.tokens != nullptr ? g.src.tokens[0] : 0;
        const float ir = g.src.row_inv_rms(0, red, GV_CONSUMERS, 1);
        const int wp = g.src.wp, nvec = wp >> 2;
        float fr = 1.0f;
        if (PRO == PRO_FINAL) {
            float ss = 0.0f;
            for (int i = tid; i < nvec; i += GV_CONSUMERS) ss += ops::sumsq4(g.src.at(0, pos, tok, i, ir));
            fr = inv_rms(group_sum(ss, red, GV_CONSUMERS, 1), g.src.width, g.src.eps);
        }
        const bool writer = blockIdx.x == 0;
        float* st = PRO == PRO_SHIFT ? g.shift_state + (size_t)g.meta[1] * 2 * wp : nullptr;
        for (int i = tid; i < nvec; i += GV_CONSUMERS) {
            const float4 x = g.src.at(0, pos, tok, i, ir);
            float4 h = x;
            if (PRO == PRO_SHIFT) {
                const float4 before = pos > 0 ? reinterpret_cast<const float4*>(st + (size_t)((pos - 1) & 1) * wp)[i]
                                              : make_float4(0.f, 0.f, 0.f, 0.f);
                h = shift4(x, before, __ldg(reinterpret_cast<const float4*>(g.shift) + i));
                if (writer) reinterpret_cast<float4*>(st + (size_t)(pos & 1) * wp)[i] = x;      // the other half of the pair
            }
            if (PRO == PRO_FINAL) {
                const float4 n = __ldg(reinterpret_cast<const float4*>(g.final_norm) + i);
                h = make_float4(x.x * fr * n.x, x.y * fr * n.y, x.z * fr * n.z, x.w * fr * n.w);
            }
            if (writer && g.x_out != nullptr) reinterpret_cast<float4*>(g.x_out)[i] = x;
            store4<T>(as + i * 4, h);
        }
    }
    named_bar_sync(1, GV_CONSUMERS);

    // -------------------------------------------------------------- multiply --
    const int half = warp >> 2;                                      // which four rows of a stage
    const int off = (warp & 3) * (GV_PIECE / 4) + lane * 16;         // this lane's 16 bytes of a row piece
    int slot = 0;
    uint32_t phase = 0;
    bool ok = true;
    for (int gi = 0; gi < groups; ++gi) {
        float acc[4] = {0.f, 0.f, 0.f, 0.f};
        for (int c = 0; c < chunks; ++c) {
            ok = tc::wait_uniform(&full[slot], phase, abort_flag) && ok;
            if (ok && c * GV_PIECE + off < row_bytes) {
                float af[V::N];
                V::unpack(lds128(reinterpret_cast<const uint8_t*>(as) + (size_t)c * GV_PIECE + off), af);
                const uint8_t* st = ring + (size_t)slot * GV_STAGE + half * 4 * GV_PIECE + off;
                uint4 wv[4];
#pragma unroll
                for (int r = 0; r < 4; ++r) wv[r] = lds128(st + r * GV_PIECE);
#pragma unroll
                for (int r = 0; r < 4; ++r) {
                    float wf[V::N];
                    V::unpack(wv[r], wf);
#pragma unroll
                    for (int j = 0; j < V::N; ++j) acc[r] = fmaf(wf[j], af[j], acc[r]);
                }
            }
            __syncwarp();
            if (lane == 0) mbar_arrive(&empty[slot]);
            if (++slot == g.stages) { slot = 0; phase ^= 1u; }
        }
        // four sums over 32 lanes: halves exchange until lanes 0-7 hold row 0, 8-15 row 1, ...
        const bool hi = (lane & 16) != 0, mid = (lane & 8) != 0;
        float k0 = (hi ? acc[2] : acc[0]) + __shfl_xor_sync(0xffffffffu, hi ? acc[0] : acc[2], 16);
        float k1 = (hi ? acc[3] : acc[1]) + __shfl_xor_sync(0xffffffffu, hi ? acc[1] : acc[3], 16);
        float v = (mid ? k1 : k0) + __shfl_xor_sync(0xffffffffu, mid ? k0 : k1, 8);
        v += __shfl_xor_sync(0xffffffffu, v, 4);
        v += __shfl_xor_sync(0xffffffffu, v, 2);
        v += __shfl_xor_sync(0xffffffffu, v, 1);
        const int buf = (gi / GV_FLUSH) & 1, at = gi % GV_FLUSH;
        if ((lane & 7) == 0) part[buf][at][warp][lane >> 3] = v;
        if (at == GV_FLUSH - 1 || gi == groups - 1) {
            named_bar_sync(1, GV_CONSUMERS);
            const int o = tid;                                       // output within this flush
            const int first = n_begin + (gi - at) * OUT_ROWS;
            if (o < (at + 1) * OUT_ROWS && first + o < n_end && *abort_flag == 0) {
                const int grp = o / OUT_ROWS, row = o % OUT_ROWS;
                auto sum = [&](int stage_row) {
                    const float(*p)[4] = &part[buf][grp][(stage_row >> 2) * 4];
                    const int r = stage_row & 3;
                    return ((p[0][r] + p[1][r]) + (p[2][r] + p[3][r]));
                };
                g.out[first + o] = GATED ? gelu_tanh(sum(row)) * sum(row + 4) : sum(row);
            }
        }
    }
}

// One query of every head over the slot's cache.  CTA = (share of the visible keys, key/value head); the CTAs of a head
// are one cluster and add their partial outputs through distributed shared memory (the weights are not
// normalised, so a partial is a plain sum).  Takes the projection row as the product leaves it: the RMS norms of
// the whole q and k rows are taken here, the CTA with the newest key appends it and its value.
constexpr int AD_THREADS = 256, AD_CHUNK = 256, AD_HB = 4;       // keys per pass, query heads per pass

template <typename T>
struct AttnDecodeArgs {
    const float* proj;          // f32 [q | k | v | gate], q and k not normalised
    float* out;                 // f32 [heads * vdim_pad]
    const float* q_norm;
    const float* k_norm;
    T* k_cache;
    T* v_cache;
    const float* bias_table;
    const int* meta;
    int heads, kv_heads, dim, dim_pad, vdim_pad, window, keep_first, capacity, bias_len, gated;
    float scale, eps;
};

template <typename T>
__host__ inline size_t attn_decode_smem_bytes(int group, int dim_pad, int vdim_pad) {
    return sizeof(float) * ((size_t)group * dim_pad + AD_HB * AD_CHUNK + (size_t)group * vdim_pad +
                            (size_t)AD_THREADS * AD_HB * Vec<T>::N);
}

__device__ __forceinline__ float ld_cluster_f32(uint32_t addr) {
    float v;
    asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(v) : "r"(addr) : "memory");
    return v;
}

template <typename T>
__global__ void __launch_bounds__(AD_THREADS)
attn_decode_kernel(const AttnDecodeArgs<T> g)
{
    using V = Vec<T>;
    pdl_launch_dependents();
    extern __shared__ __align__(16) float ad_smem[];
    __shared__ float red[32];
    const int group = g.heads / g.kv_heads;
    float* qs = ad_smem;                                   // [group][dim_pad], normalised and scaled
    float* ws = qs + group * g.dim_pad;                    // [AD_HB][AD_CHUNK]
    float* os = ws + AD_HB * AD_CHUNK;                     // [group][vdim_pad]: this CTA's share of the output
    float* sums = os + group * g.vdim_pad;                 // [key group][AD_HB][vdim_pad]
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int kvh = blockIdx.y, splits = gridDim.x, rank = blockIdx.x;
    const int kd = g.kv_heads * g.dim_pad, vd = g.kv_heads * g.vdim_pad, q_n = g.heads * g.dim_pad;
    pdl_wait_prior_grids();
    const int p = g.meta[0];
    T* kc = g.k_cache + (size_t)g.meta[1] * g.capacity * kd + kvh * g.dim_pad;
    T* vc = g.v_cache + (size_t)g.meta[1] * g.capacity * vd + kvh * g.vdim_pad;
    int sinks, lo;
    visible_range(p, g.window, g.keep_first, sinks, lo);
    const int total = sinks + (p - lo + 1);
    const int per = (total + splits - 1) / splits;
    const int t_begin = min(total, rank * per), t_end = min(total, t_begin + per);

    // norms of the whole rows
    float qr = 1.0f, kr = 1.0f;
    auto row_sq = [&](const float* v, int n) {
        float ss = 0.0f;
        for (int i = tid; i < (n >> 2); i += AD_THREADS) ss += ops::sumsq4(reinterpret_cast<const float4*>(v)[i]);
        return group_sum(ss, red, AD_THREADS, 1);
    };
    if (g.q_norm != nullptr) qr = inv_rms(row_sq(g.proj, q_n), g.heads * g.dim, g.eps);
    const bool newest = t_begin < t_end && t_end == total && p < g.capacity;      // this CTA's share ends with key p
    if (newest) {
        if (g.k_norm != nullptr) kr = inv_rms(row_sq(g.proj + q_n, kd), g.kv_heads * g.dim, g.eps);
        for (int d = tid; d < g.dim_pad; d += AD_THREADS) {
            float k = g.proj[q_n + kvh * g.dim_pad + d];
            if (g.k_norm != nullptr) k *= kr * g.k_norm[kvh * g.dim_pad + d];
            kc[(size_t)p * kd + d] = from_f32<T>(k);
        }
        for (int d = tid; d < g.vdim_pad; d += AD_THREADS)
            vc[(size_t)p * vd + d] = from_f32<T>(g.proj[q_n + kd + kvh * g.vdim_pad + d]);
    }
    for (int i = tid; i < group * g.dim_pad; i += AD_THREADS) {
        const int e = kvh * group * g.dim_pad + i;
        float q = g.proj[e];
        if (g.q_norm != nullptr) q *= qr * g.q_norm[e];
        qs[i] = q * g.scale;
    }
    __syncthreads();

    const int kp = g.dim_pad / V::N, vp = g.vdim_pad / V::N;       // 16-byte pieces of a key and of a value row
    const int kgroups = AD_THREADS / vp, piece = tid % vp, kg = tid / vp;
    auto key_of = [&](int t) { return t < sinks ? t : lo + (t - sinks); };
    for (int h0 = 0; h0 < group; h0 += AD_HB) {
        const int nh = min(AD_HB, group - h0);
        float acc[AD_HB][V::N];
#pragma unroll
        for (int h = 0; h < AD_HB; ++h)
#pragma unroll
            for (int e = 0; e < V::N; ++e) acc[h][e] = 0.0f;
        for (int t0 = t_begin; t0 < t_end; t0 += AD_CHUNK) {
            const int n = min(AD_CHUNK, t_end - t0);
            // scores: eight lanes per key, 32 keys per pass of the CTA
            const int sub = lane & 7;
            for (int k0 = 0; k0 < n; k0 += 32) {
                const int tt = k0 + warp * 4 + (lane >> 3);
                const bool in = tt < n;
                const int j = key_of(t0 + (in ? tt : 0));
                float s[AD_HB] = {0.f, 0.f, 0.f, 0.f};
                for (int c = sub; c < kp; c += 8) {
                    float kf[V::N];
                    V::unpack(*reinterpret_cast<const uint4*>(kc + (size_t)j * kd + c * V::N), kf);
#pragma unroll
                    for (int h = 0; h < AD_HB; ++h) {
                        if (h < nh) {
                            const float* q = qs + (h0 + h) * g.dim_pad + c * V::N;
#pragma unroll
                            for (int e = 0; e < V::N; ++e) s[h] = fmaf(kf[e], q[e], s[h]);
                        }
                    }
                }
#pragma unroll
                for (int h = 0; h < AD_HB; ++h) {
                    s[h] += __shfl_xor_sync(0xffffffffu, s[h], 4);
                    s[h] += __shfl_xor_sync(0xffffffffu, s[h], 2);
                    s[h] += __shfl_xor_sync(0xffffffffu, s[h], 1);
                }
                if (in && sub < nh) {
                    float sc = s[0];
                    if (sub == 1) sc = s[1];
                    if (sub == 2) sc = s[2];
                    if (sub == 3) sc = s[3];
                    if (g.bias_table != nullptr) sc += g.bias_table[(size_t)(kvh * group + h0 + sub) * g.bias_len + (p - j)];
                    ws[sub * AD_CHUNK + tt] = sigmoid_f32(sc);
                }
            }
            __syncthreads();
            if (kg < kgroups) {
#pragma unroll 2
                for (int tt = kg; tt < n; tt += kgroups) {
                    float vf[V::N];
                    V::unpack(*reinterpret_cast<const uint4*>(vc + (size_t)key_of(t0 + tt) * vd + piece * V::N), vf);
#pragma unroll
                    for (int h = 0; h < AD_HB; ++h) {
                        const float w = h < nh ? ws[h * AD_CHUNK + tt] : 0.0f;
#pragma unroll
                        for (int e = 0; e < V::N; ++e) acc[h][e] = fmaf(w, vf[e], acc[h][e]);
                    }
                }
            }
            __syncthreads();                                        // ws is written again
        }
        if (kg < kgroups) {
#pragma unroll
            for (int h = 0; h < AD_HB; ++h)
#pragma unroll
                for (int e = 0; e < V::N; ++e) sums[(kg * AD_HB + h) * g.vdim_pad + piece * V::N + e] = acc[h][e];
        }
        __syncthreads();
        for (int i = tid; i < nh * g.vdim_pad; i += AD_THREADS) {
            float o = 0.0f;
            for (int k = 0; k < kgroups; ++k) o += sums[k * AD_HB * g.vdim_pad + i];
            os[h0 * g.vdim_pad + i] = o;
        }
        __syncthreads();
    }
    cluster_sync_all();
    for (int i = rank * AD_THREADS + tid; i < group * g.vdim_pad; i += splits * AD_THREADS) {
        float o = 0.0f;
        const uint32_t at = smem_u32(os + i);
        for (int s = 0; s < splits; ++s) o += ld_cluster_f32(mapa_shared(at, s));
        const int e = kvh * group * g.vdim_pad + i;
        if (g.gated) o *= sigmoid_f32(g.proj[q_n + kd + vd + e]);
        g.out[e] = o;
    }
    cluster_sync_all();                                             // nobody leaves while its shared memory may be read
}

}  // namespace dense
}  // namespace twm
