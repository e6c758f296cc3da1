// twm_dense_decode.cuh — one decoded token of a dense model: the streaming matrix-vector product and
// the split-key attention.
//
// gemv_kernel: y = W a for one token, HBM-bound.  W is read as two streams of rows (gate and up rows of a
// gated product, otherwise its two halves).  The CTAs (one per SM) take four rows of each at a time in
// turn, so that together they read two contiguous windows; what is left after the last full round is
// shared out evenly.  One thread streams them into a shared-memory ring,
// eight row pieces of 2 KB a stage: two tiled TMA loads (a copy per row piece would keep that thread busier
// than the memory), and one bulk copy per row for the first ring-full, which need not wait for the tensor
// map, and in the last, partial round.  It starts before the preceding
// kernel has finished (weights are constants);
// eight warps multiply: warps 0-3 the stage's rows 0-3, a quarter of the piece each, warps 4-7 the rows 4-7.
// A CTA asks for more than half an SM's shared memory: with two to an SM, those of the next launch would
// gather on the SMs that happen to be free.  The steps between two products
// are its prologue: every CTA makes the product's input row itself, from the residual stream and the
// sublayer output that joins it (norm, add, token shift or final norm), in FP32, and rounds it once.
// The epilogue of the gate/up product applies the gated activation, so no launch stands between products
// but the attention.
//
// Routed products (experts) differ in where a row comes from.  ROUTE_ROWS (up): the `top` chosen experts' rows, one
// expert after the other, are one long list of rows.  ROUTE_COLUMNS (down): a row is the chosen experts' rows side by
// side, and the input is their activations side by side, each times its expert's weight; so the sum over experts is
// part of the product.  The choice is made by router_decode_kernel, two launches ahead of the down product: the up
// product lets that one start only after its own wait for the router, so the down product takes the choice as soon
// as it starts and streams its weights while the up product still runs.
#pragma once

#include "twm_dense_moe.cuh"
#include "twm_dense_rows.cuh"
#include "twm_dense_simt.cuh"
#include "twm_gemm_tc.cuh"

namespace twm {
namespace dense {

enum { PRO_VEC = 0, PRO_RESIDUAL = 1, PRO_SHIFT = 2, PRO_NORM = 3 };
enum { ROUTE_NONE = 0, ROUTE_ROWS = 1, ROUTE_COLUMNS = 2 };

constexpr int GV_CONSUMERS = 256;
constexpr int GV_THREADS = GV_CONSUMERS + 32;
constexpr int GV_ROWS = 8;                  // rows per stage
constexpr int GV_PIECE = 2048;              // bytes of a row per stage
constexpr int GV_STAGE = GV_ROWS * GV_PIECE;
constexpr int GV_MAX_STAGES = 9;
constexpr int GV_FLUSH = 16;                // row groups between two cross-warp sums

template <typename T>
struct GemvArgs {
    const T* w;                 // [N (gated: N gate rows, then N up rows)][ldw]
    int N, ldw;                 // ldw = K: padded, a multiple of 16 bytes
    float* out;                 // [N]
    int rounds, last_rows;      // full rounds of row groups over the grid, then rows per CTA of what is left (0 = none)
    int stages;
    const float* vec;           // PRO_VEC: the input row, f32 [ldw]
    ResidualSource<T> src;      // otherwise: row 0 of the residual stream
    float* x_out;               // the residual row after the add, written by CTA 0
    const float* shift;
    float* shift_state;
    const float* pre_norm;      // PRO_NORM: the input row is rms_norm(residual row) * pre_norm
    const int* meta;
    // routed: W is [experts][expert_rows][ldw].  ROUTE_ROWS: N = top * expert_rows.  ROUTE_COLUMNS: N = expert_rows, vec is
    // [top][ldw].
    RouterArgs router;
    int expert_rows;
    const int* ids;
    const float* weights;
    alignas(64) CUtensorMap w_map;      // W's rows as 64-bit words, boxes of 256 words x 4 rows
};

// row pieces of one expert's row: each expert's input starts on a piece of its own
__host__ __device__ inline int gemv_pieces(size_t row_bytes) { return (int)((row_bytes + GV_PIECE - 1) / GV_PIECE); }
__host__ __device__ inline size_t gemv_smem_bytes(size_t row_bytes, int parts, int stages) {
    return (size_t)stages * GV_STAGE + (parts > 1 ? (size_t)parts * gemv_pieces(row_bytes) * GV_PIECE : ((row_bytes + 127) & ~(size_t)127));
}

template <typename T, int PRO, int EPI, int ROUTE>
__global__ void __launch_bounds__(GV_THREADS, 1)
gemv_kernel(const __grid_constant__ GemvArgs<T> g)
{
    using V = Vec<T>;
    constexpr bool GATED = EPI == TWM_EPI_GELU_GLU;
    extern __shared__ __align__(128) uint8_t gemv_smem[];
    __shared__ int ids_s[ROUTE != ROUTE_NONE ? MOE_MAX_TOP : 1];
    uint8_t* ring = gemv_smem;
    T* as = reinterpret_cast<T*>(gemv_smem + (size_t)g.stages * GV_STAGE);
    __shared__ __align__(8) uint64_t full[GV_MAX_STAGES], empty[GV_MAX_STAGES];
    __shared__ float part[2][GV_FLUSH][8][4];
    __shared__ float red[32];
    __shared__ int abort_s;
    volatile int* abort_flag = &abort_s;

    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    constexpr int OUT_ROWS = GV_ROWS / 2;                            // rows of each stream per row group
    const int stream = GATED ? g.N : (g.N + 1) / 2;                  // rows of a stream; the second one may be a row shorter
    const int last_first = g.rounds * (int)gridDim.x * OUT_ROWS + (int)blockIdx.x * g.last_rows;
    const int last_valid = max(0, min(g.last_rows, stream - last_first));
    const int groups = g.rounds + (last_valid > 0 ? 1 : 0);
    auto group_first = [&](int gi) { return gi < g.rounds ? (gi * (int)gridDim.x + (int)blockIdx.x) * OUT_ROWS : last_first; };
    auto group_rows = [&](int gi) { return gi < g.rounds ? OUT_ROWS : last_valid; };
    auto second_rows = [&](int gi) { return GATED ? group_rows(gi) : min(group_rows(gi), g.N - stream - group_first(gi)); };
    const int row_bytes = g.ldw * (int)sizeof(T);
    const int pieces = (row_bytes + GV_PIECE - 1) / GV_PIECE;        // of one row as it lies in memory
    const int chunks = ROUTE == ROUTE_COLUMNS ? pieces * g.router.top : pieces;
    // where row o of the list lies (ROUTE_COLUMNS: in an expert's matrix)
    auto physical = [&](int o) {
        if (ROUTE != ROUTE_ROWS) return o;
        const int slot = o / g.expert_rows;
        return ids_s[slot] * g.expert_rows + o - slot * g.expert_rows;
    };
    const int iters = groups * chunks;

    if (tid == 0) {
        prefetch_map(&g.w_map);
        for (int s = 0; s < g.stages; ++s) { mbar_init(&full[s], 1); mbar_init(&empty[s], GV_CONSUMERS / 32); }
        abort_s = 0;
        mbar_fence_init();
    }
    __syncthreads();
    if (ROUTE != ROUTE_ROWS) pdl_launch_dependents();

    if (warp == GV_CONSUMERS / 32) {
        // ------------------------------------------------------------ producer --
        if (ROUTE == ROUTE_ROWS) {
            pdl_wait_prior_grids();                                  // for the router's choice ...
            pdl_launch_dependents();                                 // ... which the next launch relies on from its start
        }
        if (ROUTE != ROUTE_NONE) {
            if (lane < g.router.top) ids_s[lane] = ld_cg_s32(g.ids + lane);
            __syncwarp();
        }
        if (elect_one()) {
            int slot = 0, c = 0, gi = 0, piece = 0, part = 0, first = 0, second_first = 0;
            uint32_t phase = 0;
            for (int it = 0; it < iters; ++it) {
                if (it >= g.stages && !mbar_wait_bounded(&empty[slot], phase, abort_flag)) break;
                uint8_t* dst = ring + (size_t)slot * GV_STAGE;
                const int o0 = group_first(gi);
                if (ROUTE == ROUTE_NONE) {
                    piece = c; first = o0; second_first = stream + o0;
                } else if (c == 0) {
                    first = physical(o0); second_first = physical(stream + o0);
                }
                const int matrix = ROUTE == ROUTE_COLUMNS ? ids_s[part] * g.expert_rows : 0;
                // a full group's four rows lie together: an expert's rows are a multiple of 16.  Routed products have nothing to gain
                // from row copies: by the time the choice is known the map has been fetched.
                if (gi < g.rounds && (it >= g.stages || ROUTE != ROUTE_NONE)) {
                    mbar_arrive_expect_tx(&full[slot], GV_STAGE);
                    tma_load_2d(dst, &g.w_map, piece * (GV_PIECE / 8), matrix + first, &full[slot]);
                    tma_load_2d(dst + OUT_ROWS * GV_PIECE, &g.w_map, piece * (GV_PIECE / 8), matrix + second_first, &full[slot]);
                } else {
                    const int bytes = min(GV_PIECE, row_bytes - piece * GV_PIECE), valid = group_rows(gi), second = second_rows(gi);
                    mbar_arrive_expect_tx(&full[slot], (uint32_t)bytes * (uint32_t)(valid + second));
                    const uint8_t* src = reinterpret_cast<const uint8_t*>(g.w) + (size_t)piece * GV_PIECE;
                    for (int r = 0; r < valid; ++r)
                        bulk_g2s(dst + r * GV_PIECE, src + (size_t)(matrix + physical(o0 + r)) * row_bytes, (uint32_t)bytes, &full[slot]);
                    for (int r = 0; r < second; ++r)
                        bulk_g2s(dst + (r + OUT_ROWS) * GV_PIECE, src + (size_t)(matrix + physical(stream + o0 + r)) * row_bytes, (uint32_t)bytes,
                                 &full[slot]);
                }
                if (ROUTE != ROUTE_NONE && ++piece == pieces) { piece = 0; ++part; }
                if (++c == chunks) { c = 0; part = 0; ++gi; }
                if (++slot == g.stages) { slot = 0; if (it >= g.stages) phase ^= 1u; }
            }
        }
        return;
    }

    // ------------------------------------------------------- prologue (256 threads) --
    pdl_wait_prior_grids();
    if (ROUTE == ROUTE_ROWS) pdl_launch_dependents();
    if (ROUTE == ROUTE_COLUMNS) {
        for (int i = tid; i < (g.ldw >> 2); i += GV_CONSUMERS) {
#pragma unroll 8
            for (int s = 0; s < g.router.top; ++s) {
                const float ws = g.weights[s];
                const float4 v = reinterpret_cast<const float4*>(g.vec + (size_t)s * g.ldw)[i];
                store4<T>(as + (size_t)s * pieces * (GV_PIECE / sizeof(T)) + i * 4, make_float4(v.x * ws, v.y * ws, v.z * ws, v.w * ws));
            }
        }
    } else if (PRO == PRO_VEC) {
        for (int i = tid; i < (g.ldw >> 2); i += GV_CONSUMERS) store4<T>(as + i * 4, reinterpret_cast<const float4*>(g.vec)[i]);
    } else {
        const int pos = g.meta[0];
        const int tok = g.src.tokens != nullptr ? g.src.tokens[0] : 0;
        const int wp = g.src.wp, nvec = wp >> 2;
        const bool writer = blockIdx.x == 0;
        float* st = PRO == PRO_SHIFT ? g.shift_state + (size_t)g.meta[1] * 2 * wp : nullptr;
        const float* st_before = PRO == PRO_SHIFT && pos > 0 ? st + (size_t)((pos - 1) & 1) * wp : nullptr;
        float fr = 1.0f;
        // element i of the residual row x; before = the state's, for the token shift
        auto finish = [&](int i, const float4 x, const float4 before) {
            float4 h = x;
            if (PRO == PRO_SHIFT) {
                h = shift4(x, before, __ldg(reinterpret_cast<const float4*>(g.shift) + i));
                if (writer) reinterpret_cast<float4*>(st + (size_t)(pos & 1) * wp)[i] = x;      // the other half of the pair
            }
            if (PRO == PRO_NORM) h = scale4(x, fr, __ldg(reinterpret_cast<const float4*>(g.pre_norm) + i));
            if (writer && g.x_out != nullptr) reinterpret_cast<float4*>(g.x_out)[i] = x;
            store4<T>(as + i * 4, h);
        };
        auto state_at = [&](int i) {
            return st_before != nullptr ? reinterpret_cast<const float4*>(st_before)[i] : make_float4(0.f, 0.f, 0.f, 0.f);
        };
        constexpr int PER = 4;
        // without a norm of its own the input is taken this way only where nothing but a normed sublayer output joins
        const bool plain = g.src.y != nullptr && g.src.y_norm != nullptr && g.src.step == nullptr;
        if (nvec <= PER * GV_CONSUMERS && g.src.tokens == nullptr && (PRO == PRO_NORM || plain)) {
            // rows of up to 4096: everything is requested before the first use
            const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
            float4 x[PER], y[PER], before[PER];
#pragma unroll
            for (int j = 0; j < PER; ++j) {
                const int i = tid + j * GV_CONSUMERS;
                const bool in = i < nvec;
                y[j] = in && (PRO != PRO_NORM || g.src.y != nullptr) ? reinterpret_cast<const float4*>(g.src.y)[i] : zero;
                x[j] = in ? reinterpret_cast<const float4*>(g.src.x_in)[i] : zero;
                before[j] = PRO == PRO_SHIFT && in ? state_at(i) : zero;
            }
            float ss = 0.0f, ir = 1.0f;
            const bool normed = PRO != PRO_NORM || (g.src.y != nullptr && g.src.y_norm != nullptr);
            if (normed) {
#pragma unroll
                for (int j = 0; j < PER; ++j) ss += ops::sumsq4(y[j]);
                ir = inv_rms(group_sum(ss, red, GV_CONSUMERS, 1), g.src.width, g.src.eps);
            }
            ss = 0.0f;
#pragma unroll
            for (int j = 0; j < PER; ++j) {
                const int i = tid + j * GV_CONSUMERS;
                if (i < nvec) {
                    float4 n = make_float4(1.f, 1.f, 1.f, 1.f);
                    if (normed) n = __ldg(reinterpret_cast<const float4*>(g.src.y_norm) + i);
                    x[j].x += y[j].x * ir * n.x; x[j].y += y[j].y * ir * n.y; x[j].z += y[j].z * ir * n.z; x[j].w += y[j].w * ir * n.w;
                    if (PRO == PRO_NORM && g.src.step != nullptr) {
                        const float4 t = __ldg(reinterpret_cast<const float4*>(g.src.step) + i);
                        x[j].x += t.x; x[j].y += t.y; x[j].z += t.z; x[j].w += t.w;
                    }
                }
                ss += ops::sumsq4(x[j]);
            }
            if (PRO == PRO_NORM) fr = inv_rms(group_sum(ss, red, GV_CONSUMERS, 1), g.src.width, g.src.eps);
#pragma unroll
            for (int j = 0; j < PER; ++j)
                if (tid + j * GV_CONSUMERS < nvec) finish(tid + j * GV_CONSUMERS, x[j], before[j]);
        } else {
            const float ir = g.src.row_inv_rms(0, red, GV_CONSUMERS, 1);
            if (PRO == PRO_NORM) {
                float ss = 0.0f;
                for (int i = tid; i < nvec; i += GV_CONSUMERS) ss += ops::sumsq4(g.src.at(0, pos, tok, i, ir));
                fr = inv_rms(group_sum(ss, red, GV_CONSUMERS, 1), g.src.width, g.src.eps);
            }
            for (int i = tid; i < nvec; i += GV_CONSUMERS) finish(i, g.src.at(0, pos, tok, i, ir), state_at(i));
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
        int piece = 0;
        for (int c = 0; c < chunks; ++c) {
            ok = tc::wait_uniform(&full[slot], phase, abort_flag) && ok;
            const bool in = (ROUTE == ROUTE_COLUMNS ? piece : c) * GV_PIECE + off < row_bytes;
            if (ROUTE == ROUTE_COLUMNS && ++piece == pieces) piece = 0;
            if (ok && in) {
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
            const int grp = tid / GV_ROWS, row = tid % OUT_ROWS, which = (tid / OUT_ROWS) & 1;     // one row of one stream per thread
            const int gg = gi - at + grp;
            if (grp <= at && (GATED ? which == 0 && row < group_rows(gg) : row < (which ? second_rows(gg) : group_rows(gg))) &&
                *abort_flag == 0) {
                auto sum = [&](int stage_row) {
                    const float(*p)[4] = &part[buf][grp][(stage_row >> 2) * 4];
                    const int r = stage_row & 3;
                    return ((p[0][r] + p[1][r]) + (p[2][r] + p[3][r]));
                };
                g.out[group_first(gg) + row + (GATED ? 0 : which * stream)] = GATED ? gelu_tanh(sum(row)) * sum(row + 4)
                                                                                  : epilogue_value<EPI>(sum(row + 4 * which));
            }
        }
    }
}

// One token's router: one cluster of CTAs.  Every CTA makes the feed-forward's input row (the residual stream brought up to
// date, normed) for itself, a warp takes the logits of every (8 * CTAs)-th expert, and the first CTA's first warp chooses.
// Leaves the residual row, the input row in FP32, and the choice.
constexpr int RD_THREADS = 256, RD_CTAS = 8;
template <typename T>
struct RouterDecodeArgs {
    ResidualSource<T> src;
    float* x_out;               // [wp]
    float* h_out;               // [wp]
    const float* pre_norm;      // [wp] or null
    const T* w;                 // [experts][wp]
    const int* meta;
    RouterArgs router;
    int* ids;
    float* weights;
};
template <typename T>
__host__ inline size_t router_decode_smem_bytes(int wp) { return sizeof(float) * 2 * (size_t)wp; }
template <typename T>
__global__ void __launch_bounds__(RD_THREADS)
router_decode_kernel(const RouterDecodeArgs<T> g)
{
    using V = Vec<T>;
    pdl_launch_dependents();
    asm volatile("barrier.cluster.arrive.relaxed.aligned;" ::: "memory");      // waited for before the first push
    extern __shared__ __align__(16) float rd_smem[];
    __shared__ float logits[MOE_MAX_EXPERTS], scores[MOE_MAX_EXPERTS], group_scores[MOE_MAX_EXPERTS], red[32];
    const int wp = g.src.wp, nvec = wp >> 2, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int first = blockIdx.x * (RD_THREADS / 32) + warp, stride = gridDim.x * (RD_THREADS / 32);
    float4* hs = reinterpret_cast<float4*>(rd_smem);       // [wp]
    float4* ys = hs + nvec;
    for (int e = first; e < g.router.experts; e += stride)
        if (lane == 0) l2_prefetch_bulk(g.w + (size_t)e * wp, (uint32_t)(wp * sizeof(T)));
    pdl_wait_prior_grids();
    const bool writer = blockIdx.x == 0, joined = g.src.y != nullptr, normed = joined && g.src.y_norm != nullptr;
    const int tok = g.src.tokens != nullptr ? g.src.tokens[0] : 0, pos = g.meta[0];
    ResidualSource<T> plain = g.src;                       // the row without what joins it
    plain.y = nullptr;
    float ss = 0.0f;
    for (int i = tid; i < nvec; i += RD_THREADS) {         // every thread keeps to its own elements
        const float4 y = joined ? reinterpret_cast<const float4*>(g.src.y)[i] : make_float4(0.f, 0.f, 0.f, 0.f);
        hs[i] = plain.at(0, pos, tok, i, 1.0f);
        ys[i] = y;
        ss += ops::sumsq4(y);
    }
    const float ir = normed ? inv_rms(group_sum(ss, red, RD_THREADS, 1), g.src.width, g.src.eps) : 1.0f;
    ss = 0.0f;
    for (int i = tid; i < nvec; i += RD_THREADS) {
        float4 x = hs[i], n = make_float4(1.f, 1.f, 1.f, 1.f);
        if (normed) n = __ldg(reinterpret_cast<const float4*>(g.src.y_norm) + i);
        const float4 y = scale4(ys[i], ir, n);
        x.x += y.x; x.y += y.y; x.z += y.z; x.w += y.w;
        hs[i] = x;
        if (writer) reinterpret_cast<float4*>(g.x_out)[i] = x;
        ss += ops::sumsq4(x);
    }
    const float fr = g.pre_norm != nullptr ? inv_rms(group_sum(ss, red, RD_THREADS, 1), g.src.width, g.src.eps) : 1.0f;
    for (int i = tid; i < nvec; i += RD_THREADS) {
        if (g.pre_norm != nullptr) hs[i] = scale4(hs[i], fr, __ldg(reinterpret_cast<const float4*>(g.pre_norm) + i));
        if (writer) reinterpret_cast<float4*>(g.h_out)[i] = hs[i];
    }
    __syncthreads();
    asm volatile("barrier.cluster.wait.aligned;" ::: "memory");    // every CTA of the cluster has started
    for (int e = first; e < g.router.experts; e += stride) {
        const uint4* w = reinterpret_cast<const uint4*>(g.w + (size_t)e * wp);
        float s = 0.0f;
#pragma unroll 4
        for (int c = lane; c < wp / V::N; c += 32) {
            float f[V::N];
            V::unpack(__ldg(w + c), f);
#pragma unroll
            for (int k = 0; k < V::N; k += 4) {
                const float4 h = hs[c * (V::N / 4) + k / 4];
                s = fmaf(f[k], h.x, fmaf(f[k + 1], h.y, fmaf(f[k + 2], h.z, fmaf(f[k + 3], h.w, s))));
            }
        }
        s = ops::warp_sum(s);
        if (lane == 0) st_cluster_f32(mapa_shared(smem_u32(logits + e), 0), s);
    }
    cluster_sync_all();
    if (writer && warp == 0) {
        int id;
        float weight;
        route_warp(logits, g.router, scores, group_scores, lane, id, weight);
        if (lane < g.router.top) { g.ids[lane] = id; g.weights[lane] = weight; }
    }
}

// One query of every head over the slot's cache.  CTA = (share of the visible keys, key/value head); the CTAs of a head
// are one cluster: each pushes its partial output, which is a plain sum because the weights are not normalised,
// into the shared memory of the CTA that owns the columns, and after one cluster barrier the owners add up in rank
// order, apply the gate and store.  Takes the projection row as the product leaves it: the RMS norms of the whole q
// and k rows are taken here, the CTA with the newest key appends it and its value.  A share of keys and values is on
// its way into shared memory (cp.async) while the norms are taken; then a thread takes one (key, query head) score at
// a time, and four value columns of one query head over a part of the share's keys.
constexpr int AD_THREADS = 512, AD_MAX_CHUNK = 128;   // keys in shared memory at a time, at most

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
    int chunk;                  // keys in shared memory at a time, a multiple of 8
    int parts;                  // threads that share the keys of one output column quad
    float scale, eps;
};

// threads per column quad: as many as the CTA has, up to four
__host__ inline int attn_decode_parts(int group, int vdim_pad) {
    const int n = AD_THREADS / (group * (vdim_pad / 4));
    return n < 1 ? 1 : n > 4 ? 4 : n;
}
template <typename T>
__host__ inline size_t attn_decode_smem_bytes(int group, int dim_pad, int vdim_pad, int chunk, int splits) {
    const int slice = (group * vdim_pad + splits - 1) / splits;
    return sizeof(float) * ((size_t)group * dim_pad + (size_t)group * chunk +
                            (size_t)group * vdim_pad * attn_decode_parts(group, vdim_pad) + (((size_t)slice * splits + 3) & ~(size_t)3)) +
           (size_t)chunk * (dim_pad * sizeof(T) + 16 + vdim_pad * sizeof(T));
}

template <typename T>
__global__ void __launch_bounds__(AD_THREADS)
attn_decode_kernel(const AttnDecodeArgs<T> g)
{
    using V = Vec<T>;
    pdl_launch_dependents();
    asm volatile("barrier.cluster.arrive.relaxed.aligned;" ::: "memory");      // waited for before the first push
    extern __shared__ __align__(16) float ad_smem[];
    __shared__ float red[32];
    const int group = g.heads / g.kv_heads, splits = gridDim.x, rank = blockIdx.x;
    const int columns = group * g.vdim_pad, slice = (columns + splits - 1) / splits;       // a CTA owns `slice` output columns
    float* qs = ad_smem;                                   // [group][dim_pad], normalised and scaled
    float* ws = qs + group * g.dim_pad;                    // [group][chunk]
    float* os = ws + group * g.chunk;                      // [parts][group][vdim_pad]: this CTA's share of the output
    float* recv = os + g.parts * columns;                  // [splits][slice]: what the cluster pushed here
    const int krow = g.dim_pad * (int)sizeof(T) + 16, vrow = g.vdim_pad * (int)sizeof(T);
    uint8_t* ks = reinterpret_cast<uint8_t*>(recv + ((slice * splits + 3) & ~3));       // rows padded: a lane per key reads distinct banks
    uint8_t* vs = ks + g.chunk * krow;
    const int tid = threadIdx.x;
    const int kvh = blockIdx.y;
    const int kd = g.kv_heads * g.dim_pad, vd = g.kv_heads * g.vdim_pad, q_n = g.heads * g.dim_pad;
    const int kp = g.dim_pad / V::N, vp = g.vdim_pad / V::N;       // 16-byte pieces of a key and of a value row
    const int krow0 = tid / kp, kcol0 = tid - krow0 * kp, vrow0 = tid / vp, vcol0 = tid - vrow0 * vp;
    const int kstep = AD_THREADS / kp, kwrap = AD_THREADS - kstep * kp, vstep = AD_THREADS / vp, vwrap = AD_THREADS - vstep * vp;
    constexpr int QV = 2;                                  // a thread's first q elements and norm weights, ahead of the sum
    float nq[QV];
#pragma unroll
    for (int j = 0; j < QV; ++j) {
        const int i = tid + j * AD_THREADS;
        nq[j] = g.q_norm != nullptr && i < group * g.dim_pad ? __ldg(g.q_norm + kvh * group * g.dim_pad + i) : 1.0f;
    }
    pdl_wait_prior_grids();
    const int p = g.meta[0], slot = g.meta[1];
    float q[QV];
#pragma unroll
    for (int j = 0; j < QV; ++j) {
        const int i = tid + j * AD_THREADS;
        q[j] = i < group * g.dim_pad ? g.proj[kvh * group * g.dim_pad + i] : 0.0f;
    }
    const int own = min(slice, columns - rank * slice);    // may be <= 0
    const float gate = g.gated && tid < own ? g.proj[q_n + kd + vd + kvh * columns + rank * slice + tid] : 0.0f;
    float qss = 0.0f;
    if (g.q_norm != nullptr) {
#pragma unroll 4
        for (int i = tid; i < (q_n >> 2); i += AD_THREADS) qss += ops::sumsq4(reinterpret_cast<const float4*>(g.proj)[i]);
    }
    T* kc = g.k_cache + (size_t)slot * g.capacity * kd + kvh * g.dim_pad;
    T* vc = g.v_cache + (size_t)slot * g.capacity * vd + kvh * g.vdim_pad;
    int sinks, lo;
    visible_range(p, g.window, g.keep_first, sinks, lo);
    const int total = sinks + (p - lo + 1);
    const int per = (total + splits - 1) / splits;
    const int t_begin = min(total, rank * per), t_end = min(total, t_begin + per);

    auto key_of = [&](int t) { return t < sinks ? t : lo + (t - sinks); };
    const bool newest = t_begin < t_end && t_end == total && p < g.capacity;      // this CTA's share ends with key p
    // the share's rows, all but the newest one, which is not in the cache yet
    auto load_share = [&](int t0, int n) {
        for (int r = krow0, c = kcol0; r < n;) {
            const int j = key_of(t0 + r);
            if (j < p) ops::att_cp_async16(smem_u32(ks + r * krow + c * 16), kc + (size_t)j * kd + c * V::N, 16);
            r += kstep; c += kwrap;
            if (c >= kp) { c -= kp; ++r; }
        }
        for (int r = vrow0, c = vcol0; r < n;) {
            const int j = key_of(t0 + r);
            if (j < p) ops::att_cp_async16(smem_u32(vs + r * vrow + c * 16), vc + (size_t)j * vd + c * V::N, 16);
            r += vstep; c += vwrap;
            if (c >= vp) { c -= vp; ++r; }
        }
        ops::att_cp_async_commit();
    };
    load_share(t_begin, min(g.chunk, t_end - t_begin));

    // norms of the whole rows
    float kr = 1.0f;
    const float qr = g.q_norm != nullptr ? inv_rms(group_sum(qss, red, AD_THREADS, 1), g.heads * g.dim, g.eps) : 1.0f;
    if (newest && g.k_norm != nullptr) {
        float kss = 0.0f;
        for (int i = tid; i < (kd >> 2); i += AD_THREADS) kss += ops::sumsq4(reinterpret_cast<const float4*>(g.proj + q_n)[i]);
        kr = inv_rms(group_sum(kss, red, AD_THREADS, 1), g.kv_heads * g.dim, g.eps);
    }
#pragma unroll
    for (int j = 0; j < QV; ++j) {
        const int i = tid + j * AD_THREADS;
        if (i < group * g.dim_pad) qs[i] = q[j] * (g.q_norm != nullptr ? qr * nq[j] : 1.0f) * g.scale;
    }
    for (int i = tid + QV * AD_THREADS; i < group * g.dim_pad; i += AD_THREADS) {
        const int e = kvh * group * g.dim_pad + i;
        qs[i] = g.proj[e] * (g.q_norm != nullptr ? qr * g.q_norm[e] : 1.0f) * g.scale;
    }
    for (int i = tid; i < g.parts * columns; i += AD_THREADS) os[i] = 0.0f;

    for (int t0 = t_begin; t0 < t_end; t0 += g.chunk) {
        const int n = min(g.chunk, t_end - t0);
        if (t0 > t_begin) {
            __syncthreads();                                       // the chunk before has been used
            load_share(t0, n);
        }
        if (newest && t0 + n == t_end) {                           // the new row: into the cache and beside the others
            for (int d = tid; d < g.dim_pad; d += AD_THREADS) {
                float k = g.proj[q_n + kvh * g.dim_pad + d];
                if (g.k_norm != nullptr) k *= kr * g.k_norm[kvh * g.dim_pad + d];
                const T kt = from_f32<T>(k);
                kc[(size_t)p * kd + d] = kt;
                reinterpret_cast<T*>(ks + (n - 1) * krow)[d] = kt;
            }
            for (int d = tid; d < g.vdim_pad; d += AD_THREADS) {
                const T vt = from_f32<T>(g.proj[q_n + kd + kvh * g.vdim_pad + d]);
                vc[(size_t)p * vd + d] = vt;
                reinterpret_cast<T*>(vs + (n - 1) * vrow)[d] = vt;
            }
        }
        const int nr = (n + 31) & ~31;
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();
        for (int i = tid; i < group * nr; i += AD_THREADS) {
            const int h = i / nr, tt = i - h * nr;                 // a warp's lanes: consecutive keys of one head
            if (tt >= n) continue;
            float bias = 0.0f;
            if (g.bias_table != nullptr) bias = __ldg(g.bias_table + (size_t)(kvh * group + h) * g.bias_len + (p - key_of(t0 + tt)));
            const uint8_t* kr_s = ks + tt * krow;
            const float* qh = qs + h * g.dim_pad;
            float s0 = 0.0f, s1 = 0.0f;
#pragma unroll 4
            for (int c = 0; c < kp; ++c) {
                float kf[V::N];
                V::unpack(lds128(kr_s + c * 16), kf);
#pragma unroll
                for (int e = 0; e < V::N; e += 4) {
                    const float4 qv = *reinterpret_cast<const float4*>(qh + c * V::N + e);
                    s0 = fmaf(kf[e], qv.x, fmaf(kf[e + 1], qv.y, s0));
                    s1 = fmaf(kf[e + 2], qv.z, fmaf(kf[e + 3], qv.w, s1));
                }
            }
            ws[h * g.chunk + tt] = sigmoid_f32(s0 + s1 + bias);
        }
        __syncthreads();
        const int quads = g.vdim_pad / 4, items = group * quads;
        for (int i = tid; i < items * g.parts; i += AD_THREADS) {
            const int part = i / items, item = i - part * items;
            const int h = item / quads, c = (item - h * quads) * 4;
            float o0 = 0.f, o1 = 0.f, o2 = 0.f, o3 = 0.f;
            const float* w = ws + h * g.chunk;
            const uint8_t* v0 = vs + c * sizeof(T);
#pragma unroll 8
            for (int tt = part; tt < n; tt += g.parts) {
                const float4 vf = load4(reinterpret_cast<const T*>(v0 + (size_t)tt * vrow));
                const float wt = w[tt];
                o0 = fmaf(wt, vf.x, o0); o1 = fmaf(wt, vf.y, o1); o2 = fmaf(wt, vf.z, o2); o3 = fmaf(wt, vf.w, o3);
            }
            float4* o = reinterpret_cast<float4*>(os + part * columns + h * g.vdim_pad + c);     // this thread's own columns
            const float4 before = *o;
            *o = make_float4(before.x + o0, before.y + o1, before.z + o2, before.w + o3);
        }
    }
    asm volatile("barrier.cluster.wait.aligned;" ::: "memory");    // every CTA of the cluster has started
    __syncthreads();
    for (int i = tid; i < columns; i += AD_THREADS) {
        float o = os[i];
        for (int part = 1; part < g.parts; ++part) o += os[part * columns + i];
        const int owner = i / slice;
        st_cluster_f32(mapa_shared(smem_u32(recv + rank * slice + i - owner * slice), owner), o);
    }
    cluster_sync_all();
    for (int i = tid; i < own; i += AD_THREADS) {
        float o = 0.0f;
#pragma unroll 8
        for (int s = 0; s < splits; ++s) o += recv[s * slice + i];
        const int e = kvh * columns + rank * slice + i;
        if (g.gated) o *= sigmoid_f32(i < AD_THREADS ? gate : g.proj[q_n + kd + vd + e]);
        g.out[e] = o;
    }
}

}  // namespace dense
}  // namespace twm
