// twm_dense_softmax_tc.cuh — windowed softmax attention of a portion of a prompt on the 5th-generation tensor cores,
// bfloat16: keys of a part per head (up to 128 columns) and a part all heads share (up to 64; both together at most
// four 64-column boxes), value heads of up to 128 columns.
//
// CTA = 128 queries of one head, 64 keys at a time, two CTAs per SM where their shared memory allows.
//   warp 4   TMA: Q once, then a K and a V tile at a time (128-byte swizzled boxes of 64 columns; the shared key part
//            is a box of its own; columns past a head and keys past the end arrive as zeros).
//   warp 5   one thread issues tcgen05.mma: the scores of tile t + 1 go to the other score buffer while tile t is
//            being weighted; then P V of tile t (P from tensor memory).
//   warps 0-3  thread = query row: maximum, weights, sum.  The reference of the exponents moves only when a row's maximum
//            has grown by more than 2^8; then the row's output is scaled in tensor memory, before the tile's P V.
//            Weights and sums are FP32; a weight enters P V as a bf16 pair hi + lo, two MMAs, so that no more than
//            2^-17 of it is lost; the pair overwrites the scores in place.
// Tensor memory: two score buffers of 64 columns and 128 columns of output.
#pragma once

#include "twm_dense_attn_tc.cuh"
#include "twm_dense_latent.cuh"

namespace twm {
namespace dense {

constexpr int SX_Q = 128, SX_K = 64, SX_THREADS = 192, SX_MAX_KBOXES = 4;
constexpr int SX_QBOX = SX_Q * 128, SX_KBOX = SX_K * 128;       // bytes of a box of 64 columns

struct SoftmaxTcArgs {
    SoftmaxArgs<bf16> a;
    alignas(64) CUtensorMap q_map;      // [rows][heads][dim_pad]
    alignas(64) CUtensorMap qr_map;     // [rows][heads][rot_pad]
    alignas(64) CUtensorMap k_map;      // [keys][heads][dim_pad]
    alignas(64) CUtensorMap kr_map;     // [keys][rot_pad]
    alignas(64) CUtensorMap v_map;      // [keys][heads][vdim_pad]
};
struct SoftmaxTcSync {
    alignas(8) uint64_t q_full, k_full, k_empty, v_full, v_empty, p_full, o_done, s_full[2];
    uint32_t tmem_base;
    int abort_flag;
};
__host__ __device__ inline int softmax_tc_kboxes(int dim_pad, int rot_pad) { return (dim_pad + 63) / 64 + (rot_pad + 63) / 64; }
__host__ inline size_t softmax_tc_smem_bytes(int dim_pad, int rot_pad, int vdim_pad) {
    return (size_t)softmax_tc_kboxes(dim_pad, rot_pad) * (SX_QBOX + SX_KBOX) + (size_t)((vdim_pad + 63) / 64) * SX_KBOX + 1024;
}
__device__ __forceinline__ uint64_t sx_value_desc(uint32_t addr) {      // columns contiguous, the next 64 in the next box
    return (uint64_t)((addr & 0x3FFFF) >> 4) | ((uint64_t)(SX_KBOX >> 4) << 16) | ((uint64_t)(1024 >> 4) << 32) | ((uint64_t)1 << 46) |
           ((uint64_t)2 << 61);
}

__global__ void __launch_bounds__(SX_THREADS, 2)
attn_softmax_tc_kernel(const __grid_constant__ SoftmaxTcArgs args)
{
    extern __shared__ uint8_t sx_smem_raw[];
    __shared__ SoftmaxTcSync sm;
    const SoftmaxArgs<bf16>& g = args.a;
    const int d_boxes = (g.dim_pad + 63) / 64, k_boxes = softmax_tc_kboxes(g.dim_pad, g.rot_pad), v_boxes = (g.vdim_pad + 63) / 64;
    uint8_t* qs = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(sx_smem_raw) + 1023) & ~(uintptr_t)1023);
    uint8_t* ks = qs + k_boxes * SX_QBOX;
    uint8_t* vs = ks + k_boxes * SX_KBOX;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;

    if (tid == 0) {
        prefetch_map(&args.q_map);
        prefetch_map(&args.k_map);
        prefetch_map(&args.v_map);
        for (uint64_t* bar : {&sm.q_full, &sm.k_full, &sm.k_empty, &sm.v_full, &sm.v_empty, &sm.o_done, &sm.s_full[0], &sm.s_full[1]}) mbar_init(bar, 1);
        mbar_init(&sm.p_full, SX_Q / 32);
        sm.abort_flag = 0;
        mbar_fence_init();
    }
    // Tensor memory is asked for once the kernel before is over (its CTAs and pairs of CTAs have given theirs back), and
    // the next kernel may come once this CTA has it: an allocation waits without a limit.
    pdl_wait_prior_grids();
    if (warp == 5) {
        tc::tmem_alloc(&sm.tmem_base, 256);
        tc::tc_fence_before();
    }
    __syncthreads();
    tc::tc_fence_after();
    pdl_launch_dependents();
    volatile int* abort_flag = &sm.abort_flag;
    const uint32_t tmem = sm.tmem_base, tmem_o = tmem + 2 * SX_K;

    const int h = blockIdx.y, r0 = blockIdx.x * SX_Q;
    const int p0 = g.first_pos + r0, p1 = g.first_pos + min(g.rows, r0 + SX_Q) - 1;      // positions of the CTA's first and last query
    const int lo = g.window > p0 ? 0 : p0 - g.window + 1;
    const int t_first = (lo - g.first_key) / SX_K;
    const int n_tiles = (p1 - g.first_key) / SX_K - t_first + 1;

    if (warp == 4) {
        // ------------------------------------------------------------- loads --
        if (elect_one()) {
            mbar_arrive_expect_tx(&sm.q_full, (uint32_t)(k_boxes * SX_QBOX));
            for (int b = 0; b < d_boxes; ++b) tma_load_3d(qs + b * SX_QBOX, &args.q_map, b * 64, h, r0, &sm.q_full);
            for (int b = d_boxes; b < k_boxes; ++b) tma_load_3d(qs + b * SX_QBOX, &args.qr_map, (b - d_boxes) * 64, h, r0, &sm.q_full);
            for (int t = 0; t < n_tiles; ++t) {
                const int k0 = (t_first + t) * SX_K;
                const uint32_t parity = (uint32_t)(t - 1) & 1u;
                if (t > 0 && !mbar_wait_bounded(&sm.k_empty, parity, abort_flag)) break;
                mbar_arrive_expect_tx(&sm.k_full, (uint32_t)(k_boxes * SX_KBOX));
                for (int b = 0; b < d_boxes; ++b) tma_load_3d(ks + b * SX_KBOX, &args.k_map, b * 64, h, k0, &sm.k_full);
                for (int b = d_boxes; b < k_boxes; ++b) tma_load_2d(ks + b * SX_KBOX, &args.kr_map, (b - d_boxes) * 64, k0, &sm.k_full);
                if (t > 0 && !mbar_wait_bounded(&sm.v_empty, parity, abort_flag)) break;
                mbar_arrive_expect_tx(&sm.v_full, (uint32_t)(v_boxes * SX_KBOX));
                for (int b = 0; b < v_boxes; ++b) tma_load_3d(vs + b * SX_KBOX, &args.v_map, b * 64, h, k0, &sm.v_full);
            }
        }
        __syncwarp();
    } else if (warp == 5) {
        // -------------------------------------------------------------- MMAs --
        if (elect_one()) {
            constexpr uint32_t types = (1u << 4) | (1u << 7) | (1u << 10);              // D f32, A and B bf16
            constexpr uint32_t idesc_s = types | ((uint32_t)(SX_K >> 3) << 17) | ((uint32_t)(SX_Q >> 4) << 24);
            const uint32_t idesc_o = types | (1u << 16) | ((uint32_t)(v_boxes * 64 >> 3) << 17) | ((uint32_t)(SX_Q >> 4) << 24);
            bool ok = mbar_wait_bounded(&sm.q_full, 0, abort_flag);
            // the buffer held the weights of t - 2, whose MMAs were issued before: they run in order
            auto scores = [&](int t) {
                if (!mbar_wait_bounded(&sm.k_full, (uint32_t)t & 1u, abort_flag)) return false;
                tc::tc_fence_after();
                bool first = true;
                for (int b = 0; b < k_boxes; ++b) {
                    const int cols = b < d_boxes ? min(64, g.dim_pad - b * 64) : min(64, g.rot_pad - (b - d_boxes) * 64);
                    for (int c = 0; c < cols / 16; ++c) {
                        tcw::mma_ss(tmem + (t & 1) * SX_K, sw128_desc(smem_u32(qs) + b * SX_QBOX + c * 32), sw128_desc(smem_u32(ks) + b * SX_KBOX + c * 32),
                                    idesc_s, first ? 0u : 1u);
                        first = false;
                    }
                }
                tc::tc_commit(&sm.k_empty);
                tc::tc_commit(&sm.s_full[t & 1]);
                return true;
            };
            ok = ok && scores(0);
            for (int t = 0; t < n_tiles && ok; ++t) {
                const uint32_t parity = (uint32_t)t & 1u;
                if (t + 1 < n_tiles && !scores(t + 1)) break;
                if (!mbar_wait_bounded(&sm.v_full, parity, abort_flag) || !mbar_wait_bounded(&sm.p_full, parity, abort_flag)) break;
                tc::tc_fence_after();
                for (int c = 0; c < SX_K / 16; ++c) {                                     // 16 keys: 8 columns of hi, 8 of lo
                    const uint64_t vd = sx_value_desc(smem_u32(vs) + c * 2048);
                    const uint32_t a = tmem + (t & 1) * SX_K + (c >> 1) * 32 + (c & 1) * 8;
                    tc::tc_mma_ts(tmem_o, a, vd, idesc_o, (t == 0 && c == 0) ? 0u : 1u);
                    tc::tc_mma_ts(tmem_o, a + 16, vd, idesc_o, 1u);
                }
                tc::tc_commit(&sm.v_empty);
                tc::tc_commit(&sm.o_done);
            }
        }
        __syncwarp();
    } else {
        // ----------------------------------------------------------- weights --
        const int row = warp * 32 + lane, p = p0 + row, r = r0 + row;
        const uint32_t lane_tmem = tmem + ((uint32_t)(warp * 32) << 16), lane_o = lane_tmem + 2 * SX_K;
        const float factor = 1.4426950408889634f * g.scale;
        const float gate = g.gate_off >= 0 && r < g.rows ? to_f32(g.proj[(size_t)r * g.ld + g.gate_off + h]) : 0.0f;
        float m = -INFINITY, l = 0.0f;
        bool ok = true;
        for (int t = 0; t < n_tiles; ++t) {
            const uint32_t at = lane_tmem + (t & 1) * SX_K;
            ok = tc::wait_uniform(&sm.s_full[t & 1], (t >> 1) & 1, abort_flag) && ok;
            tc::tc_fence_after();
            const int k0 = g.first_key + (t_first + t) * SX_K;                              // position of the tile's first key
            uint32_t s[4][16];
#pragma unroll
            for (int c = 0; c < 4; ++c) tc::tmem_ld<16>(at + c * 16, s[c]);
            tc::tmem_wait_ld();
            const bool all_seen = k0 + SX_K - 1 <= p0 && p1 - k0 < g.window;
            if (!all_seen) {
#pragma unroll
                for (int c = 0; c < 4; ++c)
#pragma unroll
                    for (int j = 0; j < 16; ++j) {
                        const int key = k0 + c * 16 + j;
                        if (!(key <= p && p - key < g.window)) s[c][j] = __float_as_uint(-INFINITY);
                    }
            }
            float mx[4];
#pragma unroll
            for (int c = 0; c < 4; ++c) {
                mx[c] = __uint_as_float(s[c][0]);
#pragma unroll
                for (int j = 1; j < 16; ++j) mx[c] = fmaxf(mx[c], __uint_as_float(s[c][j]));
            }
            const float tile_max = fmaxf(fmaxf(mx[0], mx[1]), fmaxf(mx[2], mx[3])) * factor;      // the scale is positive
            float before = 1.0f;
            const bool moved = tile_max > m + 8.0f;
            if (moved) {
                before = ex2_approx(m - tile_max);                                          // 0 at the first visible tile
                m = tile_max;
                l *= before;
            }
            const float ref = m == -INFINITY ? 0.0f : m;
            float sum[4] = {0.0f, 0.0f, 0.0f, 0.0f};
#pragma unroll
            for (int c = 0; c < 2; ++c) {                                                   // 32 keys: 16 columns of hi, 16 of lo
                uint32_t hi[16], lw[16];
#pragma unroll
                for (int j = 0; j < 16; ++j) {
                    const int k = 2 * j;
                    const float a = ex2_approx(fmaf(__uint_as_float(s[2 * c + (k >> 4)][k & 15]), factor, -ref));
                    const float b = ex2_approx(fmaf(__uint_as_float(s[2 * c + (k >> 4)][(k & 15) + 1]), factor, -ref));
                    sum[j & 3] += a + b;
                    split_bf16(a, b, hi[j], lw[j]);
                }
                tc::tmem_st16(at + c * 32, hi);
                tc::tmem_st16(at + c * 32 + 16, lw);
            }
            l += (sum[0] + sum[1]) + (sum[2] + sum[3]);
            if (t > 0) {
                ok = tc::wait_uniform(&sm.o_done, (uint32_t)(t - 1) & 1u, abort_flag) && ok;
                if (__any_sync(0xffffffffu, moved)) {
                    tc::tc_fence_after();
                    for (int c = 0; c < v_boxes * 64; c += 16) {
                        uint32_t o[16];
                        tc::tmem_ld<16>(lane_o + c, o);
                        tc::tmem_wait_ld();
#pragma unroll
                        for (int j = 0; j < 16; ++j) o[j] = __float_as_uint(__uint_as_float(o[j]) * before);
                        tc::tmem_st16(lane_o + c, o);
                    }
                }
            }
            tc::tmem_wait_st();
            tc::tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(&sm.p_full);
        }
        // ---- divide, gate and store this thread's row ----
        ok = tc::wait_uniform(&sm.o_done, (uint32_t)(n_tiles - 1) & 1u, abort_flag) && ok;
        tc::tc_fence_after();
        const float f = (g.gate_off >= 0 ? sigmoid_f32(gate) : 1.0f) / l;
        bf16* out = g.out + (size_t)r * g.heads * g.vdim_pad + h * g.vdim_pad;
        for (int c = 0; c < g.vdim_pad; c += 16) {
            uint32_t d[16];
            tc::tmem_ld<16>(lane_o + c, d);
            tc::tmem_wait_ld();
            if (!ok || r >= g.rows) continue;
#pragma unroll
            for (int j = 0; j < 16; j += 8) {
                float v[8];
#pragma unroll
                for (int e = 0; e < 8; ++e) v[e] = __uint_as_float(d[j + e]) * f;
                *reinterpret_cast<uint4*>(out + c + j) = Vec<bf16>::pack(v);
            }
        }
    }
    tc::tc_fence_before();
    __syncthreads();
    if (warp == 5) {
        tc::tc_fence_after();
        tc::tmem_dealloc(tmem, 256);
    }
}

}  // namespace dense
}  // namespace twm
