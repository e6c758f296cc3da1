// twm_dense_tc.cuh — C[M][N] = A[M][K] . W[N][K]^T in bfloat16 on the 5th-generation tensor cores, for
// steps of several tokens.
//
// Tile 128 rows x BN columns, 64 K per stage.  Both operands are K-major rows in global memory and land in
// shared memory as 128-byte swizzled rows (one tiled TMA load each; a gated product takes the gate and
// the up rows of the weight as two boxes).  Persistent CTAs, one per SM: warp 4 loads, one thread of
// warp 5 issues tcgen05.mma (128 x BN x 16), warps 0-3 read a finished accumulator back and store it
// while the next tile accumulates into the other one.  Weights are constants: the first ring-full of
// them is on its way before the preceding kernel has finished; the activations follow after it.
//
// GROUPED: the rows are grouped by expert (offsets[e] .. offsets[e + 1], known on the device only) and each group has a
// weight matrix of its own.  A tile belongs to one expert; it may load rows of the next one, which are not stored.
#pragma once

#include "twm_dense_moe.cuh"
#include "twm_gemm_tc.cuh"
#include "twm_gemm_tcw.cuh"

namespace twm {
namespace dense {

constexpr int TC_BM = 128, TC_BK = 64;
constexpr int TC_A_BYTES = TC_BM * TC_BK * 2;
constexpr int TC_WARP_TMA = 4, TC_WARP_MMA = 5, TC_THREADS = 192;

template <int BN>
struct TcCfg {
    static constexpr int B_BYTES = BN * TC_BK * 2;
    static constexpr int STAGE_BYTES = TC_A_BYTES + B_BYTES;
    static constexpr int STAGES = BN == 256 ? 4 : (BN == 128 ? 6 : 8);
    static constexpr int TMEM_COLS = 2 * BN < 32 ? 32 : 2 * BN;
    static constexpr int SMEM_BYTES = STAGES * STAGE_BYTES + 1024;      // + alignment of the first stage
};

struct TcArgs {
    void* c;
    int ldc, M, N, K;               // gated: N output columns, 2 N weight rows
    int m_tiles, n_tiles;
    const int* offsets;             // grouped: [experts + 1]
    int experts;
    alignas(64) CUtensorMap a_map;  // bf16 [M][K], box 64 x 128
    alignas(64) CUtensorMap w_map;  // bf16 [rows][K], box 64 x BN (gated: 64 x BN/2)
};

// Shared-memory matrix descriptor of a K-major operand in 128-byte swizzled rows: eight rows are 1024 bytes.
__device__ __forceinline__ uint64_t sw128_desc(uint32_t addr) {
    return (uint64_t)((addr & 0x3FFFF) >> 4) | ((uint64_t)1 << 16) | ((uint64_t)(1024 >> 4) << 32) | ((uint64_t)1 << 46) |
           ((uint64_t)2 << 61);
}

// tiles in groups of 16 row blocks: the CTAs of a wave share weight columns and activation rows in L2
__device__ __forceinline__ void tc_tile(int t, int m_tiles, int n_tiles, int& m, int& n) {
    constexpr int G = 16;
    const int per = G * n_tiles, grp = t / per, rest = t - grp * per;
    const int rows = min(G, m_tiles - grp * G);
    m = grp * G + rest % rows;
    n = rest / rows;
}

template <int EPI>
__device__ __forceinline__ void tc_store16(void* c, size_t row_off, int n, int N, const float (&v)[16]) {
    if (EPI == TWM_EPI_STORE_F32) {
        float* p = reinterpret_cast<float*>(c) + row_off + n;
        if (n + 16 <= N && (reinterpret_cast<uintptr_t>(p) & 15) == 0) {
#pragma unroll
            for (int j = 0; j < 16; j += 4) *reinterpret_cast<float4*>(p + j) = make_float4(v[j], v[j + 1], v[j + 2], v[j + 3]);
        } else {
#pragma unroll
            for (int j = 0; j < 16; ++j) if (n + j < N) p[j] = v[j];
        }
    } else {
        bf16* p = reinterpret_cast<bf16*>(c) + row_off + n;
        if (n + 16 <= N && (reinterpret_cast<uintptr_t>(p) & 15) == 0) {
#pragma unroll
            for (int j = 0; j < 16; j += 8) {
                const float f[8] = {v[j], v[j + 1], v[j + 2], v[j + 3], v[j + 4], v[j + 5], v[j + 6], v[j + 7]};
                *reinterpret_cast<uint4*>(p + j) = Vec<bf16>::pack(f);
            }
        } else {
#pragma unroll
            for (int j = 0; j < 16; ++j) if (n + j < N) p[j] = __float2bfloat16_rn(v[j]);
        }
    }
}

template <int BN, int EPI, bool GROUPED>
__global__ void __launch_bounds__(TC_THREADS, 1)
gemm_tc_kernel(const __grid_constant__ TcArgs g)
{
    using C = TcCfg<BN>;
    constexpr bool GATED = EPI == TWM_EPI_GELU_GLU;
    constexpr int OUT = GATED ? BN / 2 : BN;                 // output columns per tile
    constexpr int STAGES = C::STAGES;
    extern __shared__ uint8_t tc_smem_raw[];
    uint8_t* ring = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(tc_smem_raw) + 1023) & ~(uintptr_t)1023);
    __shared__ __align__(8) uint64_t full[STAGES], empty[STAGES], acc_full[2], acc_empty[2];
    __shared__ uint32_t tmem_s;
    __shared__ int abort_s;
    volatile int* abort_flag = &abort_s;

    __shared__ int pre[GROUPED ? MOE_MAX_EXPERTS + 1 : 1];       // grouped: the tiles ahead of each expert's

    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int k_steps = (g.K + TC_BK - 1) / TC_BK;

    if (tid == 0) {
        prefetch_map(&g.a_map);
        prefetch_map(&g.w_map);
        for (int s = 0; s < STAGES; ++s) { mbar_init(&full[s], 1); mbar_init(&empty[s], 1); }
        for (int i = 0; i < 2; ++i) { mbar_init(&acc_full[i], 1); mbar_init(&acc_empty[i], 4); }
        abort_s = 0;
        mbar_fence_init();
    }
    if (warp == TC_WARP_MMA) {
        tc::tmem_alloc(&tmem_s, C::TMEM_COLS);
        tc::tc_fence_before();
    }
    if (GROUPED && warp == 0) {
        pdl_wait_prior_grids();
        warp_prefix([&](int e) { return (g.offsets[e + 1] - g.offsets[e] + TC_BM - 1) / TC_BM * g.n_tiles; }, g.experts, pre, lane);
    }
    __syncthreads();
    tc::tc_fence_after();
    pdl_launch_dependents();
    const uint32_t tmem = tmem_s;
    const int tiles = GROUPED ? pre[g.experts] : g.m_tiles * g.n_tiles;
    // tile t: its first row, the end of its rows, its column tile and the first row of its weight matrix
    struct Tile { int row, end, n, w0; };
    auto tile_at = [&](int t) {
        Tile x;
        if (GROUPED) {
            const int e = prefix_find(pre, g.experts, t), mt = (pre[e + 1] - pre[e]) / g.n_tiles, i = t - pre[e];
            x.n = i / mt;
            x.row = g.offsets[e] + (i - x.n * mt) * TC_BM;
            x.end = g.offsets[e + 1];
            x.w0 = e * g.N;
        } else {
            int m;
            tc_tile(t, g.m_tiles, g.n_tiles, m, x.n);
            x.row = m * TC_BM;
            x.end = g.M;
            x.w0 = 0;
        }
        return x;
    };

    if (warp == TC_WARP_TMA) {
        if (elect_one()) {
            auto load_w = [&](int slot, const Tile& x, int kk) {
                uint8_t* dst = ring + (size_t)slot * C::STAGE_BYTES + TC_A_BYTES;
                mbar_arrive_expect_tx(&full[slot], (uint32_t)C::STAGE_BYTES);
                tma_load_2d(dst, &g.w_map, kk * TC_BK, x.w0 + x.n * OUT, &full[slot]);
                if (GATED) tma_load_2d(dst + C::B_BYTES / 2, &g.w_map, kk * TC_BK, g.N + x.n * OUT, &full[slot]);
            };
            auto load_a = [&](int slot, const Tile& x, int kk) {
                tma_load_2d(ring + (size_t)slot * C::STAGE_BYTES, &g.a_map, kk * TC_BK, x.row, &full[slot]);
            };
            int it = 0;
            bool ok = true;
            // the first tile's first stages: weights before the wait for the preceding kernel, activations after it
            const int early = min(STAGES, k_steps);
            if ((int)blockIdx.x < tiles) {
                const Tile x = tile_at(blockIdx.x);
                for (int kk = 0; kk < early; ++kk) load_w(kk, x, kk);
                pdl_wait_prior_grids();
                for (int kk = 0; kk < early; ++kk) load_a(kk, x, kk);
            } else {
                pdl_wait_prior_grids();
            }
            for (int t = blockIdx.x; t < tiles && ok; t += gridDim.x) {
                const Tile x = tile_at(t);
                for (int kk = 0; kk < k_steps; ++kk, ++it) {
                    if (it < early) continue;
                    const int slot = it % STAGES;
                    if (it >= STAGES && !mbar_wait_bounded(&empty[slot], ((it / STAGES) - 1) & 1, abort_flag)) { ok = false; break; }
                    load_w(slot, x, kk);
                    load_a(slot, x, kk);
                }
            }
        }
        __syncwarp();
    } else if (warp == TC_WARP_MMA) {
        if (elect_one()) {
            // D f32, A and B bf16, both K-major
            const uint32_t idesc = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(BN >> 3) << 17) | ((uint32_t)(TC_BM >> 4) << 24);
            int it = 0, nt = 0;
            bool ok = true;
            for (int t = blockIdx.x; t < tiles && ok; t += gridDim.x, ++nt) {
                const int acc = nt & 1;
                if (nt >= 2 && !mbar_wait_bounded(&acc_empty[acc], ((nt >> 1) - 1) & 1, abort_flag)) { ok = false; break; }
                tc::tc_fence_after();
                for (int kk = 0; kk < k_steps; ++kk, ++it) {
                    const int slot = it % STAGES;
                    if (!mbar_wait_bounded(&full[slot], (it / STAGES) & 1, abort_flag)) { ok = false; break; }
                    tc::tc_fence_after();
                    const uint32_t base = smem_u32(ring + (size_t)slot * C::STAGE_BYTES);
                    uint64_t ad = sw128_desc(base), bd = sw128_desc(base + TC_A_BYTES);
#pragma unroll
                    for (int h = 0; h < TC_BK / 16; ++h) {               // 16 K = 32 bytes further along the swizzled rows
                        tcw::mma_ss(tmem + acc * BN, ad, bd, idesc, (kk == 0 && h == 0) ? 0u : 1u);
                        ad += 2;
                        bd += 2;
                    }
                    tc::tc_commit(&empty[slot]);
                }
                if (ok) tc::tc_commit(&acc_full[acc]);
            }
        }
        __syncwarp();
    } else {
        // read-back: thread = row (its TMEM lane), 16 columns at a time
        int nt = 0;
        for (int t = blockIdx.x; t < tiles; t += gridDim.x, ++nt) {
            const Tile x = tile_at(t);
            const int acc = nt & 1;
            if (!tc::wait_uniform(&acc_full[acc], (nt >> 1) & 1, abort_flag)) break;
            tc::tc_fence_after();
            const int row = x.row + warp * 32 + lane;
            const size_t row_off = (size_t)row * g.ldc;
            const uint32_t at = tmem + ((uint32_t)(warp * 32) << 16) + acc * BN;
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
                    for (int j = 0; j < 16; ++j) v[j] = epilogue_value<EPI>(__uint_as_float(d[j]));
                }
                if (row < x.end && x.n * OUT + c0 < g.N) tc_store16<EPI>(g.c, row_off, x.n * OUT + c0, g.N, v);
            }
            tc::tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(&acc_empty[acc]);
        }
    }
    tc::tc_fence_before();
    __syncthreads();
    if (warp == TC_WARP_MMA) {
        tc::tc_fence_after();
        tc::tmem_dealloc(tmem, C::TMEM_COLS);
    }
}

}  // namespace dense
}  // namespace twm
