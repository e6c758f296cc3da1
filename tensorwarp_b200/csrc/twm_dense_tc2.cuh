// twm_dense_tc2.cuh — the product of twm_dense_tc.cuh with two SMs on one tile, for many rows.
//
// One SM's 128 x 256 tile is bound by its shared memory: 48 KB come in and go out again per 512 clocks of
// MMA.  Here a pair of CTAs (one cluster) computes 256 x 256: each loads its own 128 activation rows and
// HALF of the weight rows (32 KB a stage, six stages), the tensor cores of the pair share the halves
// (tcgen05.mma.cta_group::2, M = 256), and each CTA ends up with its 128 rows of the result in its own
// tensor memory.  The leader's MMA thread issues for both; both CTAs' loads count on the leader's barriers;
// a commit tells both when a stage is free and when an accumulator is complete.  A gated product takes
// its gate rows through the leader and its up rows through the other CTA.  No load is multicast.
#pragma once

#include "twm_dense_tc.cuh"

namespace twm {
namespace dense {

constexpr int T2_BN = 256, T2_STAGES = 6, T2_STAGE_BYTES = 2 * TC_A_BYTES;      // per CTA: 128 activation rows, 128 weight rows
constexpr int T2_SMEM_BYTES = T2_STAGES * T2_STAGE_BYTES + 1024;

__device__ __forceinline__ void tma_load_2d_pair(void* smem_dst, const CUtensorMap* map, int x, int y, uint32_t cluster_bar) {
    asm volatile(
        "cp.async.bulk.tensor.2d.cta_group::2.shared::cluster.global.tile.mbarrier::complete_tx::bytes [%0], [%1, {%2, %3}], [%4];"
        ::"r"(smem_u32(smem_dst)), "l"(reinterpret_cast<uint64_t>(map)), "r"(x), "r"(y), "r"(cluster_bar)
        : "memory");
}
__device__ __forceinline__ void mma_pair(uint32_t d_tmem, uint64_t a_desc, uint64_t b_desc, uint32_t idesc, uint32_t accumulate) {
    asm volatile(
        "{\n\t.reg .pred p;\n\tsetp.ne.b32 p, %4, 0;\n\t"
        "tcgen05.mma.cta_group::2.kind::f16 [%0], %1, %2, %3, p;\n\t}"
        ::"r"(d_tmem), "l"(a_desc), "l"(b_desc), "r"(idesc), "r"(accumulate) : "memory");
}
// arrives on the barrier at this offset in both CTAs of the pair once the MMAs issued so far are complete
__device__ __forceinline__ void commit_pair(uint64_t* bar) {
    asm volatile("tcgen05.commit.cta_group::2.mbarrier::arrive::one.shared::cluster.multicast::cluster.b64 [%0], %1;"
                 ::"r"(smem_u32(bar)), "h"((uint16_t)3) : "memory");
}
__device__ __forceinline__ void mbar_arrive_cluster(uint32_t cluster_bar) {
    asm volatile("mbarrier.arrive.release.cluster.shared::cluster.b64 _, [%0];" ::"r"(cluster_bar) : "memory");
}

template <int EPI>
__global__ void __launch_bounds__(TC_THREADS, 1)
gemm_tc2_kernel(const __grid_constant__ TcArgs g)
{
    constexpr bool GATED = EPI == TWM_EPI_GELU_GLU;
    constexpr int OUT = GATED ? T2_BN / 2 : T2_BN;           // output columns per tile
    extern __shared__ uint8_t tc_smem_raw[];
    uint8_t* ring = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(tc_smem_raw) + 1023) & ~(uintptr_t)1023);
    __shared__ __align__(8) uint64_t full[T2_STAGES], empty[T2_STAGES], acc_full[2], acc_empty[2];
    __shared__ uint32_t tmem_s;
    __shared__ int abort_s;
    volatile int* abort_flag = &abort_s;

    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int rank = (int)cluster_ctarank();                 // 0 = leader
    const int pair = blockIdx.x >> 1, pairs = gridDim.x >> 1;
    const int tiles = g.m_tiles * g.n_tiles;
    const int k_steps = (g.K + TC_BK - 1) / TC_BK;

    if (tid == 0) {
        prefetch_map(&g.a_map);
        prefetch_map(&g.w_map);
        for (int s = 0; s < T2_STAGES; ++s) { mbar_init(&full[s], 1); mbar_init(&empty[s], 1); }
        for (int i = 0; i < 2; ++i) { mbar_init(&acc_full[i], 1); mbar_init(&acc_empty[i], 8); }
        abort_s = 0;
        mbar_fence_init();
    }
    if (warp == TC_WARP_MMA) {
        asm volatile("tcgen05.alloc.cta_group::2.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(&tmem_s)), "r"(2u * T2_BN) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::2.sync.aligned;" ::: "memory");
        tc::tc_fence_before();
    }
    __syncthreads();
    cluster_sync_all();                                      // the other CTA's barriers are ready as well
    tc::tc_fence_after();
    pdl_launch_dependents();
    const uint32_t tmem = tmem_s;

    if (warp == TC_WARP_TMA) {
        if (elect_one()) {
            // the leader announces both CTAs' bytes on its barrier; a load of the other CTA that is faster only runs the count ahead
            auto load_w = [&](int slot, int n, int kk) {
                if (rank == 0) mbar_arrive_expect_tx(&full[slot], 2u * T2_STAGE_BYTES);
                const int row = GATED ? (rank == 0 ? n * OUT : g.N + n * OUT) : n * OUT + rank * 128;
                tma_load_2d_pair(ring + (size_t)slot * T2_STAGE_BYTES + TC_A_BYTES, &g.w_map, kk * TC_BK, row,
                                 mapa_shared(smem_u32(&full[slot]), 0));
            };
            auto load_a = [&](int slot, int m, int kk) {
                tma_load_2d_pair(ring + (size_t)slot * T2_STAGE_BYTES, &g.a_map, kk * TC_BK, m * 2 * TC_BM + rank * TC_BM,
                                 mapa_shared(smem_u32(&full[slot]), 0));
            };
            int m, n, it = 0;
            bool ok = true;
            const int early = min(T2_STAGES, k_steps);
            tc_tile(pair, g.m_tiles, g.n_tiles, m, n);       // the host launches no more pairs than tiles
            for (int kk = 0; kk < early; ++kk) load_w(kk, n, kk);
            pdl_wait_prior_grids();
            for (int kk = 0; kk < early; ++kk) load_a(kk, m, kk);
            for (int t = pair; t < tiles && ok; t += pairs) {
                tc_tile(t, g.m_tiles, g.n_tiles, m, n);
                for (int kk = 0; kk < k_steps; ++kk, ++it) {
                    if (it < early) continue;
                    const int slot = it % T2_STAGES;
                    if (it >= T2_STAGES && !mbar_wait_bounded(&empty[slot], ((it / T2_STAGES) - 1) & 1, abort_flag)) { ok = false; break; }
                    load_w(slot, n, kk);
                    load_a(slot, m, kk);
                }
            }
        }
        __syncwarp();
    } else if (warp == TC_WARP_MMA) {
        if (rank == 0 && elect_one()) {
            // D f32, A and B bf16, both K-major, 256 x 256 over the pair
            constexpr uint32_t idesc = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(T2_BN >> 3) << 17) | ((uint32_t)(2 * TC_BM >> 4) << 24);
            int it = 0, nt = 0;
            bool ok = true;
            for (int t = pair; t < tiles && ok; t += pairs, ++nt) {
                const int acc = nt & 1;
                if (nt >= 2 && !mbar_wait_bounded(&acc_empty[acc], ((nt >> 1) - 1) & 1, abort_flag)) { ok = false; break; }
                tc::tc_fence_after();
                for (int kk = 0; kk < k_steps; ++kk, ++it) {
                    const int slot = it % T2_STAGES;
                    if (!mbar_wait_bounded(&full[slot], (it / T2_STAGES) & 1, abort_flag)) { ok = false; break; }
                    tc::tc_fence_after();
                    const uint32_t base = smem_u32(ring + (size_t)slot * T2_STAGE_BYTES);
                    uint64_t ad = sw128_desc(base), bd = sw128_desc(base + TC_A_BYTES);
#pragma unroll
                    for (int h = 0; h < TC_BK / 16; ++h) {
                        mma_pair(tmem + acc * T2_BN, ad, bd, idesc, (kk == 0 && h == 0) ? 0u : 1u);
                        ad += 2;
                        bd += 2;
                    }
                    commit_pair(&empty[slot]);
                }
                if (ok) commit_pair(&acc_full[acc]);
            }
        }
        __syncwarp();
    } else {
        // read-back: thread = row (its TMEM lane) of this CTA's half, 16 columns at a time
        int nt = 0;
        for (int t = pair; t < tiles; t += pairs, ++nt) {
            int m, n;
            tc_tile(t, g.m_tiles, g.n_tiles, m, n);
            const int acc = nt & 1;
            if (!tc::wait_uniform(&acc_full[acc], (nt >> 1) & 1, abort_flag)) break;
            tc::tc_fence_after();
            const int row = m * 2 * TC_BM + rank * TC_BM + warp * 32 + lane;
            const size_t row_off = (size_t)row * g.ldc;
            const uint32_t at = tmem + ((uint32_t)(warp * 32) << 16) + acc * T2_BN;
#pragma unroll 1
            for (int c0 = 0; c0 < OUT; c0 += 16) {
                uint32_t d[16];
                float v[16];
                tc::tmem_ld<16>(at + c0, d);
                if (GATED) {
                    uint32_t u[16];
                    tc::tmem_ld<16>(at + OUT + c0, u);
                    tc::tmem_wait_ld();
#pragma unroll
                    for (int j = 0; j < 16; ++j) v[j] = gelu_tanh(__uint_as_float(d[j])) * __uint_as_float(u[j]);
                } else {
                    tc::tmem_wait_ld();
#pragma unroll
                    for (int j = 0; j < 16; ++j) v[j] = __uint_as_float(d[j]);
                }
                if (row < g.M && n * OUT + c0 < g.N) tc_store16<EPI>(g.c, row_off, n * OUT + c0, g.N, v);
            }
            tc::tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive_cluster(mapa_shared(smem_u32(&acc_empty[acc]), 0));
        }
    }
    tc::tc_fence_before();
    __syncthreads();
    cluster_sync_all();                                      // nobody leaves while the pair's MMAs or arrivals may touch its memory
    if (warp == TC_WARP_MMA) {
        tc::tc_fence_after();
        asm volatile("tcgen05.dealloc.cta_group::2.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(2u * T2_BN) : "memory");
    }
}

}  // namespace dense
}  // namespace twm
