// twm_dense_attn_tc.cuh — windowed sigmoid attention of a portion of a prompt on the 5th-generation tensor
// cores, bfloat16, heads of up to 128 columns.
//
// CTA = 128 queries of one head.  It walks the 128-key tiles that hold a visible key: those of the kept
// first keys, then the window's.  Since the weights are not normalised over keys there is no running
// maximum and nothing is ever rescaled: S = Q K^T goes to tensor memory, eight warps turn it into weights,
// and O += P V accumulates in tensor memory over all tiles.
//   warp 8   TMA: Q once, then a K and a V tile at a time (128-byte swizzled boxes of 64 columns; keys that do
//            not exist yet and columns past the head arrive as zeros).  K of tile t + 1 is on its way as soon
//            as the scores of tile t are done.
//   warp 9   one thread issues tcgen05.mma: S (128 x 128 x 16, both operands K-major), then, when its weights
//            are there, P V (P from tensor memory, V as it lies: its columns are contiguous, "MN-major").
//   warps 0-7  thread = query row; warps 0-3 take a tile's first 64 keys, warps 4-7 the others.  A weight is
//            sigmoid(scale * s + table[distance]) in FP32; the per-head table already holds the distance
//            bias and the head's offset.  Two weights share one reciprocal (1/ab times b and a).  A weight
//            enters P V as a bf16 pair hi + lo, two MMAs, so that no more than 2^-17 of it is lost; the
//            pair overwrites the scores in place (32 keys' scores = 16 columns hi + 16 columns lo).
// Tensor memory: scores and output, 128 columns each: two CTAs share an SM, and the MMAs, loads, start and end of one
// run beside the weights of the other.
#pragma once

#include <type_traits>

#include "twm_dense_attn.cuh"
#include "twm_dense_tc.cuh"

namespace twm {
namespace dense {

constexpr int AT_Q = 128, AT_K = 128;
constexpr int AT_BOX_BYTES = 128 * 128;                 // 128 rows of 64 columns
constexpr int AT_SOFT = 256, AT_THREADS = AT_SOFT + 64;

struct AttnTcArgs {
    AttnArgs<bf16> a;
    alignas(64) CUtensorMap q_map;      // [rows][heads][dim_pad]
    alignas(64) CUtensorMap k_map;      // [slots][keys so far][kv_heads][dim_pad]
    alignas(64) CUtensorMap v_map;
};

struct AttnTcSmem {
    uint8_t q[2 * AT_BOX_BYTES];
    uint8_t k[2 * AT_BOX_BYTES];
    uint8_t v[2 * AT_BOX_BYTES];
    float bias[2][256];                 // -log2(e) * table over a tile's distances
    alignas(8) uint64_t q_full, k_full, k_empty, v_full, v_empty, s_full, p_full, o_full;
    uint32_t tmem_base;
    int abort_flag;
};

__device__ __forceinline__ void tma_load_4d(void* smem_dst, const CUtensorMap* map, int x, int y, int z, int w, uint64_t* bar) {
    asm volatile(
        "cp.async.bulk.tensor.4d.shared::cluster.global.tile.mbarrier::complete_tx::bytes [%0], [%1, {%2, %3, %4, %5}], [%6];"
        ::"r"(smem_u32(smem_dst)), "l"(reinterpret_cast<uint64_t>(map)), "r"(x), "r"(y), "r"(z), "r"(w), "r"(smem_u32(bar))
        : "memory");
}
// Matrix descriptor of an operand whose M/N columns are contiguous, in 128-byte swizzled boxes of 64 columns: eight K rows
// are 1024 bytes, the next 64 columns are the next box.
__device__ __forceinline__ uint64_t sw128_mn_desc(uint32_t addr) {
    return (uint64_t)((addr & 0x3FFFF) >> 4) | ((uint64_t)(AT_BOX_BYTES >> 4) << 16) | ((uint64_t)(1024 >> 4) << 32) |
           ((uint64_t)1 << 46) | ((uint64_t)2 << 61);
}

__global__ void __launch_bounds__(AT_THREADS, 2)
attn_tc_kernel(const __grid_constant__ AttnTcArgs args)
{
    pdl_launch_dependents();
    extern __shared__ uint8_t at_smem_raw[];
    AttnTcSmem& sm = *reinterpret_cast<AttnTcSmem*>((reinterpret_cast<uintptr_t>(at_smem_raw) + 1023) & ~(uintptr_t)1023);
    const AttnArgs<bf16>& g = args.a;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    constexpr float LOG2E = 1.4426950408889634f;

    if (tid == 0) {
        prefetch_map(&args.q_map);
        prefetch_map(&args.k_map);
        prefetch_map(&args.v_map);
        for (uint64_t* bar : {&sm.q_full, &sm.k_full, &sm.k_empty, &sm.v_full, &sm.v_empty, &sm.s_full, &sm.o_full}) mbar_init(bar, 1);
        mbar_init(&sm.p_full, AT_SOFT / 32);
        sm.abort_flag = 0;
        mbar_fence_init();
    }
    if (warp == 9) {
        tc::tmem_alloc(&sm.tmem_base, 256);
        tc::tc_fence_before();
    }
    __syncthreads();
    tc::tc_fence_after();
    volatile int* abort_flag = &sm.abort_flag;
    const uint32_t tmem = sm.tmem_base, tmem_o = tmem + AT_K;
    pdl_wait_prior_grids();

    const int h = blockIdx.y, kvh = h / (g.heads / g.kv_heads);
    const int r0 = blockIdx.x * AT_Q;
    const int pos0 = g.meta[0], slot = g.meta[1];
    const int p0 = pos0 + r0, p1 = min(pos0 + g.rows, p0 + AT_Q) - 1;     // positions of the CTA's first and last query
    int sinks, lo;
    visible_range(p0, g.window, g.keep_first, sinks, lo);
    const int w_first = lo / AT_K;
    const int n_sink = min((g.keep_first + AT_K - 1) / AT_K, w_first);
    const int n_tiles = n_sink + p1 / AT_K - w_first + 1;
    auto tile_key = [&](int t) { return (t < n_sink ? t : w_first + t - n_sink) * AT_K; };
    const int k_boxes = (g.dim_pad + 63) / 64, v_boxes = (g.vdim_pad + 63) / 64;

    if (warp == 8) {
        // ------------------------------------------------------------- loads --
        if (elect_one()) {
            mbar_arrive_expect_tx(&sm.q_full, (uint32_t)(k_boxes * AT_BOX_BYTES));
            for (int b = 0; b < k_boxes; ++b) tma_load_3d(sm.q + b * AT_BOX_BYTES, &args.q_map, b * 64, h, r0, &sm.q_full);
            for (int t = 0; t < n_tiles; ++t) {
                const int k0 = tile_key(t);
                const uint32_t parity = (uint32_t)(t - 1) & 1u;
                if (t > 0 && !mbar_wait_bounded(&sm.k_empty, parity, abort_flag)) break;
                mbar_arrive_expect_tx(&sm.k_full, (uint32_t)(k_boxes * AT_BOX_BYTES));
                for (int b = 0; b < k_boxes; ++b) tma_load_4d(sm.k + b * AT_BOX_BYTES, &args.k_map, b * 64, kvh, k0, slot, &sm.k_full);
                if (t > 0 && !mbar_wait_bounded(&sm.v_empty, parity, abort_flag)) break;
                mbar_arrive_expect_tx(&sm.v_full, (uint32_t)(v_boxes * AT_BOX_BYTES));
                for (int b = 0; b < v_boxes; ++b) tma_load_4d(sm.v + b * AT_BOX_BYTES, &args.v_map, b * 64, kvh, k0, slot, &sm.v_full);
            }
        }
        __syncwarp();
    } else if (warp == 9) {
        // -------------------------------------------------------------- MMAs --
        if (elect_one()) {
            constexpr uint32_t types = (1u << 4) | (1u << 7) | (1u << 10);              // D f32, A and B bf16
            const uint32_t idesc_s = types | ((uint32_t)(AT_K >> 3) << 17) | ((uint32_t)(AT_Q >> 4) << 24);
            const uint32_t idesc_o = types | (1u << 16) | ((uint32_t)(v_boxes * 64 >> 3) << 17) | ((uint32_t)(AT_Q >> 4) << 24);
            const int k_steps = (g.dim_pad + 15) / 16;
            bool ok = mbar_wait_bounded(&sm.q_full, 0, abort_flag);
            for (int t = 0; t < n_tiles && ok; ++t) {
                const uint32_t parity = (uint32_t)t & 1u;
                if (!mbar_wait_bounded(&sm.k_full, parity, abort_flag)) { ok = false; break; }
                tc::tc_fence_after();
                // the columns held the weights of t - 1, whose MMAs were issued before: they run in order
                for (int c = 0; c < k_steps; ++c) {
                    const uint32_t at = (c >> 2) * AT_BOX_BYTES + (c & 3) * 32;
                    tcw::mma_ss(tmem, sw128_desc(smem_u32(sm.q) + at), sw128_desc(smem_u32(sm.k) + at), idesc_s, c == 0 ? 0u : 1u);
                }
                tc::tc_commit(&sm.k_empty);
                tc::tc_commit(&sm.s_full);
                if (!mbar_wait_bounded(&sm.v_full, parity, abort_flag) || !mbar_wait_bounded(&sm.p_full, parity, abort_flag)) {
                    ok = false;
                    break;
                }
                tc::tc_fence_after();
                for (int c = 0; c < AT_K / 16; ++c) {                                     // 16 keys: 8 columns of hi, 8 of lo
                    const uint64_t vd = sw128_mn_desc(smem_u32(sm.v) + c * 2048);
                    const uint32_t a = tmem + (c >> 1) * 32 + (c & 1) * 8;
                    tc::tc_mma_ts(tmem_o, a, vd, idesc_o, (t == 0 && c == 0) ? 0u : 1u);
                    tc::tc_mma_ts(tmem_o, a + 16, vd, idesc_o, 1u);
                }
                tc::tc_commit(&sm.v_empty);
            }
            if (ok) tc::tc_commit(&sm.o_full);
        }
        __syncwarp();
    } else {
        // ----------------------------------------------------------- weights --
        const int quarter = warp & 3, half = warp >> 2;
        const int row = quarter * 32 + lane;
        const uint32_t lane_tmem = tmem + ((uint32_t)(quarter * 32) << 16);
        const float* table = g.bias_table != nullptr ? g.bias_table + (size_t)h * g.bias_len : nullptr;
        const float factor = -LOG2E * g.scale;
        // entry x of a tile's slice: distance x - 127 + (first query - first key)
        auto table_at = [&](int t) {
            const int d = p0 - tile_key(t) - (AT_K - 1) + tid;
            return table != nullptr ? -LOG2E * __ldg(table + min(max(d, 0), g.bias_len - 1)) : 0.0f;
        };
        float next = table_at(0);
        bool ok = true;
        for (int t = 0; t < n_tiles; ++t) {
            sm.bias[t & 1][tid] = next;
            named_bar_sync(1, AT_SOFT);                     // also: everybody is done with the slice of t - 1
            if (t + 1 < n_tiles) next = table_at(t + 1);
            ok = tc::wait_uniform(&sm.s_full, t & 1, abort_flag) && ok;
            tc::tc_fence_after();
            const int k0 = tile_key(t);
            const bool all_seen = k0 + AT_K - 1 <= p0 && (p1 - k0 < g.window || k0 + AT_K <= g.keep_first);
            const float* bt = &sm.bias[t & 1][(AT_K - 1) + row];
            const int p = p0 + row;
            // one body for tiles with a mask and one without: a test per pair would keep the pairs from overlapping
            auto weights = [&](auto masked) {
                constexpr bool MASKED = decltype(masked)::value;
#pragma unroll
                for (int c = 0; c < 2; ++c) {                   // 32 keys at a time
                    const int col = half * 64 + c * 32;
                    const uint32_t at = lane_tmem + col;
                    uint32_t s0[16], s1[16];
                    tc::tmem_ld<16>(at, s0);
                    tc::tmem_ld<16>(at + 16, s1);
                    tc::tmem_wait_ld();
                    uint32_t hi[16], lw[16];
#pragma unroll
                    for (int j = 0; j < 16; ++j) {
                        const int k = 2 * j;                    // keys col + k and col + k + 1
                        const float sa = __uint_as_float(k < 16 ? s0[k & 15] : s1[k & 15]);
                        const float sb = __uint_as_float(k < 16 ? s0[(k + 1) & 15] : s1[(k + 1) & 15]);
                        // below -41 in its argument a sigmoid is under 1e-18: the clamp keeps the product finite
                        const float a = 1.0f + ex2_approx(fminf(fmaf(sa, factor, bt[-(col + k)]), 60.0f));
                        const float b = 1.0f + ex2_approx(fminf(fmaf(sb, factor, bt[-(col + k + 1)]), 60.0f));
                        const float r = rcp_approx(a * b);
                        float wa = r * b, wb = r * a;
                        if (MASKED) {
                            const int key = k0 + col + k;
                            if (!(key <= p && (p - key < g.window || key < g.keep_first))) wa = 0.0f;
                            if (!(key + 1 <= p && (p - key - 1 < g.window || key + 1 < g.keep_first))) wb = 0.0f;
                        }
                        split_bf16(wa, wb, hi[j], lw[j]);
                    }
                    tc::tmem_st16(at, hi);
                    tc::tmem_st16(at + 16, lw);
                }
            };
            if (all_seen) weights(std::false_type()); else weights(std::true_type());
            tc::tmem_wait_st();
            tc::tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(&sm.p_full);
        }
        // ---- gate and store: this thread's row, a half of the value columns ----
        const int r = r0 + row;
        const int cols = v_boxes * 32, c_first = half * cols;
        bf16* out = g.out + (size_t)r * g.heads * g.vdim_pad + h * g.vdim_pad;
        const bf16* gate = g.gate_off >= 0 ? g.proj + (size_t)r * g.ld + g.gate_off + h * g.vdim_pad : nullptr;
        uint4 gates[8];                                     // on their way while the last product runs
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            const int c = c_first + i * 8;
            gates[i] = gate != nullptr && r < g.rows && i * 8 < cols && c < g.vdim_pad ? *reinterpret_cast<const uint4*>(gate + c)
                                                                                      : make_uint4(0, 0, 0, 0);
        }
        ok = tc::wait_uniform(&sm.o_full, 0, abort_flag) && ok;
        tc::tc_fence_after();
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const int c = c_first + i * 16;
            if (i * 16 >= cols) break;                      // CTA-uniform
            uint32_t d[16];
            tc::tmem_ld<16>(lane_tmem + AT_K + c, d);
            tc::tmem_wait_ld();
            if (!ok || r >= g.rows || c >= g.vdim_pad) continue;
#pragma unroll
            for (int j = 0; j < 16; j += 8) {
                float f[8], gf[8];
                Vec<bf16>::unpack(gates[i * 2 + j / 8], gf);
#pragma unroll
                for (int e = 0; e < 8; ++e) {
                    f[e] = __uint_as_float(d[j + e]);
                    if (gate != nullptr) f[e] *= rcp_approx(1.0f + ex2_approx(-LOG2E * gf[e]));
                }
                *reinterpret_cast<uint4*>(out + c + j) = Vec<bf16>::pack(f);
            }
        }
    }
    tc::tc_fence_before();
    __syncthreads();
    if (warp == 9) {
        tc::tc_fence_after();
        tc::tmem_dealloc(tmem, 256);
    }
}

}  // namespace dense
}  // namespace twm
