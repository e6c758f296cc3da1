// twm_dense.cu — host side and C ABI of the dense-weight decoder models (include/twm_dense.h).  A library of
// its own (libtwmdense.so): a model with 16-bit weights needs none of the 4-bit kernels.
#include <algorithm>
#include <cstdio>
#include <mutex>
#include <type_traits>
#include <unordered_map>

#include "twm_dense_attn.cuh"
#include "twm_dense_attn_tc.cuh"
#include "twm_dense_common.cuh"
#include "twm_dense_decode.cuh"
#include "twm_dense_gla.cuh"
#include "twm_dense_latent.cuh"
#include "twm_dense_moe.cuh"
#include "twm_dense_rows.cuh"
#include "twm_dense_simt.cuh"
#include "twm_dense_softmax_tc.cuh"
#include "twm_dense_tc.cuh"
#include "twm_dense_tc2.cuh"

namespace {

using namespace twm;
using namespace twm::dense;

thread_local char t_last_error[256] = "";
thread_local int t_launches = 0;

twm_status fail(const char* where, cudaError_t e)
{
    snprintf(t_last_error, sizeof(t_last_error), "%s: %s", where, cudaGetErrorString(e));
    return TWM_ELAUNCH;
}
twm_status invalid(const char* what)
{
    snprintf(t_last_error, sizeof(t_last_error), "%s", what);
    return TWM_EINVAL;
}
#define TRY(expr) do { const twm_status st_ = (expr); if (st_ != TWM_OK) return st_; } while (0)

constexpr int kArgmaxParts = 148;
constexpr size_t kSmemLimit = 227 * 1024;

struct DeviceState { bool ready = false; twm_status status = TWM_OK; int sms = 148; };
DeviceState g_dev[64];
std::mutex g_mutex;

twm_status device(int* sms)
{
    int dev = 0;
    cudaError_t e = cudaGetDevice(&dev);
    if (e != cudaSuccess) return fail("cudaGetDevice", e);
    if (dev < 0 || dev >= 64) return invalid("device index");
    std::lock_guard<std::mutex> lock(g_mutex);
    DeviceState& st = g_dev[dev];
    if (!st.ready) {
        int major = 0;
        cudaDeviceGetAttribute(&major, cudaDevAttrComputeCapabilityMajor, dev);
        cudaDeviceGetAttribute(&st.sms, cudaDevAttrMultiProcessorCount, dev);
        if (major != 10) {
            snprintf(t_last_error, sizeof(t_last_error), "device %d is sm_%d*, libtwmdense holds sm_100a code only", dev, major);
            st.status = TWM_EARCH;
        }
        st.ready = true;
    }
    if (sms) *sms = st.sms;
    return st.status;
}

// One launch: raises the kernel's dynamic shared memory limit when needed, asks for programmatic dependent launch
// when the caller allows it, and a cluster of `cluster` CTAs along x when > 0.
template <typename... KArgs, typename... Args>
twm_status launch(const char* what, void (*kernel)(KArgs...), dim3 grid, int threads, size_t smem, int flags, void* stream,
                  int cluster, Args&&... args)
{
    if (smem > kSmemLimit) return invalid("a row does not fit shared memory");
    if (smem > 32 * 1024) {                              // 48 KB without asking, static shared memory included
        const cudaError_t r = cudaFuncSetAttribute((const void*)kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (r != cudaSuccess) return fail(what, r);
    }
    if (cluster > 8) {
        const cudaError_t r = cudaFuncSetAttribute((const void*)kernel, cudaFuncAttributeNonPortableClusterSizeAllowed, 1);
        if (r != cudaSuccess) return fail(what, r);
    }
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = grid;
    cfg.blockDim = dim3(threads);
    cfg.dynamicSmemBytes = smem;
    cfg.stream = (cudaStream_t)stream;
    cudaLaunchAttribute attr[2];
    int n = 0;
    if (flags & TWM_FLAG_PDL) {
        attr[n].id = cudaLaunchAttributeProgrammaticStreamSerialization;
        attr[n++].val.programmaticStreamSerializationAllowed = 1;
    }
    if (cluster > 0) {
        attr[n].id = cudaLaunchAttributeClusterDimension;
        attr[n].val.clusterDim.x = cluster;
        attr[n].val.clusterDim.y = 1;
        attr[n++].val.clusterDim.z = 1;
    }
    cfg.attrs = attr;
    cfg.numAttrs = n;
    const cudaError_t e = cudaLaunchKernelEx(&cfg, kernel, static_cast<KArgs>(args)...);
    if (e != cudaSuccess) return fail(what, e);
    ++t_launches;
    return TWM_OK;
}

// Columns of the fused projection (k: keys, or the latent and the shared key part; low: GLA's low-rank part), and of the
// mixer's output.
struct Sizes { int q, k, v, g, low, in, out; };
Sizes sizes_of(const twm_dense_layer& l)
{
    Sizes s = {};
    s.out = l.heads * l.vdim_pad;
    if (l.mixer == TWM_MIX_LATENT) {
        s.q = l.heads * (l.dim_pad + l.rot_pad);
        s.k = l.rank_pad + l.rot_pad;
        s.g = (l.heads + 15) / 16 * 16;
    } else {
        const int kv_heads = l.mixer == TWM_MIX_GLA ? l.heads : l.kv_heads;
        s.q = l.heads * l.dim_pad;
        s.k = kv_heads * l.dim_pad;
        s.v = kv_heads * l.vdim_pad;
        s.g = s.out;
        if (l.mixer == TWM_MIX_GLA) s.low = l.rank_pad;
    }
    s.in = s.q + s.k + s.v + s.g + s.low;
    return s;
}
// columns of the feed-forward's activations, over all chosen experts
int act_columns(const twm_dense_layer& l) { return l.experts > 0 ? l.top * l.ff_pad : l.ff_pad; }

twm_status check_model(const twm_dense_model* m, const twm_dense_buffers* b)
{
    if (!m || !b || !m->layers) return invalid("null model or buffers");
    if (m->dtype != TWM_DENSE_F32 && m->dtype != TWM_DENSE_BF16) return invalid("dtype");
    if (m->width < 1 || m->width_pad < m->width || m->width_pad % 16 || m->vocab < 1 || m->n_layers < 0 || m->capacity < 1 || m->slots < 1)
        return invalid("model sizes");
    if (!m->embed || !m->head || !m->final_norm) return invalid("embedding, head or final norm missing");
    if (!b->meta || !b->tokens || !b->want || !b->x0 || !b->x1 || !b->y || !b->a || !b->proj || !b->att || !b->act || !b->vec ||
        !b->logits || b->max_rows < 1 || b->max_want < 1)
        return invalid("buffers");
    for (int i = 0; i < m->n_layers; ++i) {
        const twm_dense_layer& l = m->layers[i];
        if (l.heads < 1) return invalid("heads");
        if (l.pre1 && l.shift) return invalid("a mixer's input is shifted or normed, not both");
        if (l.dim < 1 || l.vdim < 1 || l.dim_pad < l.dim || l.vdim_pad < l.vdim || l.dim_pad % 16 || l.vdim_pad % 16 || l.ff_pad % 16)
            return invalid("head or feed-forward sizes");
        if (l.vdim_pad > 1024) return invalid("value heads of more than 1024 columns");
        if (!l.w_in || !l.w_out || (l.shift && !l.shift_state)) return invalid("layer pointers");
        if (l.ff_pad > 0 && (!l.w_gate_up || !l.w_down)) return invalid("feed-forward pointers");
        switch (l.mixer) {
            case TWM_MIX_SIGMOID:
                if (l.kv_heads < 1 || l.heads % l.kv_heads) return invalid("heads must be a multiple of kv_heads");
                if (l.window < 1 || l.keep_first < 0) return invalid("window");
                if (l.bias_table && m->bias_len < m->capacity) return invalid("bias table shorter than the cache");
                if (!l.k_cache || !l.v_cache) return invalid("layer pointers");
                break;
            case TWM_MIX_LATENT:
                if (l.window < 1) return invalid("window");
                if (l.rank < 1 || l.rank_pad < l.rank || l.rank_pad % 16 || l.rot_pad < 16 || l.rot_pad % 16) return invalid("latent sizes");
                if (!l.w_expand || !l.latent_norm || !l.rot_table || !l.latent_cache || !b->lat || !b->kv) return invalid("latent pointers");
                break;
            case TWM_MIX_GLA:
                if (l.rank_pad < 16 || l.rank_pad % 16) return invalid("low-rank size");
                if (!l.w_decay || !l.decay_bias || !l.head_norm || !l.gla_state || !b->decay || !b->chunk_state || !b->mix)
                    return invalid("gated linear attention pointers");
                break;
            default: return invalid("mixer");
        }
        if (l.experts != 0) {
            if (l.experts < 0 || l.experts > MOE_MAX_EXPERTS || l.top < 1 || l.top > MOE_MAX_TOP || l.groups < 1 || l.experts % l.groups ||
                l.keep < 1 || l.keep > l.groups || l.top > l.keep * (l.experts / l.groups) || l.ff_pad < 16)
                return invalid("router sizes");
            if (!l.w_router || !b->router_logits || !b->route || !b->route_weight || !b->grouped || !b->expert_out || b->max_slots < l.top * b->max_rows)
                return invalid("router pointers");
        }
    }
    return TWM_OK;
}

// ------------------------------------------------------------ tensor maps --
typedef CUresult (*EncodeTiledFn)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*, const cuuint64_t*,
                                  const cuuint32_t*, const cuuint32_t*, CUtensorMapInterleave, CUtensorMapSwizzle,
                                  CUtensorMapL2promotion, CUtensorMapFloatOOBfill);
EncodeTiledFn encode_tiled()
{
    static EncodeTiledFn fn = []() -> EncodeTiledFn {
        void* ptr = nullptr;
        cudaDriverEntryPointQueryResult q;
        if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &ptr, cudaEnableDefault, &q) != cudaSuccess ||
            q != cudaDriverEntryPointSuccess)
            return nullptr;
        return reinterpret_cast<EncodeTiledFn>(ptr);
    }();
    return fn;
}

// A tensor of up to four dimensions (innermost first; strides in elements), zeros outside.  A map is a pure description
// of memory, so maps are kept by what they describe.
enum MapKind { MAP_BF16_SWIZZLED = 0, MAP_WORDS = 1 };      // bfloat16 in 128-byte swizzled boxes; 64-bit words as they are
struct MapKey {
    MapKind kind;
    const void* ptr;
    int rank;
    long dim[4], stride[4], box[4];
    bool operator==(const MapKey& o) const {
        return kind == o.kind && ptr == o.ptr && rank == o.rank && std::equal(dim, dim + 4, o.dim) && std::equal(stride, stride + 4, o.stride) &&
               std::equal(box, box + 4, o.box);
    }
};
struct MapHash {
    size_t operator()(const MapKey& k) const {
        size_t h = (size_t)k.ptr + (size_t)k.rank + 16 * (size_t)k.kind;
        for (int i = 0; i < 4; ++i)
            for (long v : {k.dim[i], k.stride[i], k.box[i]}) h = h * 1000003u ^ (size_t)v;
        return h;
    }
};
bool tensor_map(CUtensorMap* map, const MapKey& key)
{
    static std::unordered_map<MapKey, CUtensorMap, MapHash> cache;
    static std::mutex mutex;
    std::lock_guard<std::mutex> lock(mutex);
    auto it = cache.find(key);
    if (it != cache.end()) { *map = it->second; return true; }
    EncodeTiledFn enc = encode_tiled();
    if (!enc) return false;
    cuuint64_t gdim[4], gstride[3];
    cuuint32_t box[4], estride[4] = {1, 1, 1, 1};
    for (int i = 0; i < key.rank; ++i) {
        gdim[i] = (cuuint64_t)key.dim[i];
        box[i] = (cuuint32_t)key.box[i];
        if (i > 0) gstride[i - 1] = (cuuint64_t)key.stride[i] * (key.kind == MAP_WORDS ? 8 : 2);
    }
    const bool words = key.kind == MAP_WORDS;
    if (enc(map, words ? CU_TENSOR_MAP_DATA_TYPE_UINT64 : CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, (cuuint32_t)key.rank, const_cast<void*>(key.ptr), gdim, gstride, box, estride,
            CU_TENSOR_MAP_INTERLEAVE_NONE, words ? CU_TENSOR_MAP_SWIZZLE_NONE : CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
            CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) != CUDA_SUCCESS)
        return false;
    if (cache.size() > 8192) cache.clear();
    cache.emplace(key, *map);
    return true;
}
// [rows][cols] with row stride ld, boxes of 64 columns x box_rows
bool rows_map(CUtensorMap* map, const void* ptr, long rows, long cols, long ld, int box_rows)
{
    return tensor_map(map, MapKey{MAP_BF16_SWIZZLED, ptr, 2, {cols, rows, 0, 0}, {1, ld, 0, 0}, {TC_BK, box_rows, 0, 0}});
}

// [rows][words] of 64-bit words, boxes of box_words x box_rows
bool word_rows_map(CUtensorMap* map, const void* ptr, long rows, long words, int box_words, int box_rows)
{
    return tensor_map(map, MapKey{MAP_WORDS, ptr, 2, {words, rows, 0, 0}, {1, words, 0, 0}, {box_words, box_rows, 0, 0}});
}

// ------------------------------------------------------------- operations --
// The tcgen05 product takes rows that start on 16-byte boundaries.
bool tc_fits(const void* a, int lda, const void* w, int ldw)
{
    return lda % 8 == 0 && ldw % 8 == 0 && ((uintptr_t)a & 15) == 0 && ((uintptr_t)w & 15) == 0;
}

template <int BN, int EPI>
twm_status gemm_tc_launch(const bf16* a, int lda, const bf16* w, int ldw, void* c, int ldc, int M, int N, int K, int sms, int flags,
                          void* stream)
{
    constexpr bool gated = EPI == TWM_EPI_GELU_GLU;
    constexpr int out = gated ? BN / 2 : BN;
    TcArgs g;
    g.c = c; g.ldc = ldc; g.M = M; g.N = N; g.K = K;
    g.m_tiles = (M + TC_BM - 1) / TC_BM;
    g.n_tiles = (N + out - 1) / out;
    if (!rows_map(&g.a_map, a, M, K, lda, TC_BM) || !rows_map(&g.w_map, w, gated ? 2L * N : N, K, ldw, out))
        return invalid("cuTensorMapEncodeTiled refused a map of the tcgen05 product");
    g.offsets = nullptr; g.experts = 0;
    return launch("gemm_tc", gemm_tc_kernel<BN, EPI, false>, dim3(std::min(sms, g.m_tiles * g.n_tiles)), TC_THREADS, TcCfg<BN>::SMEM_BYTES,
                  flags, stream, 0, g);
}

// the same with a weight matrix per group of rows; the tiles are counted on the device
template <int BN, int EPI>
twm_status grouped_gemm_tc_launch(const bf16* a, int lda, const bf16* w, int ldw, void* c, int ldc, const int* offsets, int experts, int rows,
                                  int N, int K, int sms, int flags, void* stream)
{
    TcArgs g;
    g.c = c; g.ldc = ldc; g.M = rows; g.N = N; g.K = K;
    g.n_tiles = (N + BN - 1) / BN;
    g.m_tiles = std::min(rows, rows / TC_BM + experts);                // at most
    g.offsets = offsets; g.experts = experts;
    if (!rows_map(&g.a_map, a, rows, K, lda, TC_BM) || !rows_map(&g.w_map, w, (long)experts * N, K, ldw, BN))
        return invalid("cuTensorMapEncodeTiled refused a map of the grouped tcgen05 product");
    return launch("gemm_tc(grouped)", gemm_tc_kernel<BN, EPI, true>, dim3((int)std::min<long>(sms, (long)g.m_tiles * g.n_tiles)), TC_THREADS,
                  TcCfg<BN>::SMEM_BYTES, flags, stream, 0, g);
}

template <int EPI>
twm_status gemm_tc2_launch(const bf16* a, int lda, const bf16* w, int ldw, void* c, int ldc, int M, int N, int K, int sms, int flags,
                           void* stream)
{
    constexpr bool gated = EPI == TWM_EPI_GELU_GLU;
    constexpr int out = gated ? T2_BN / 2 : T2_BN;
    TcArgs g;
    g.c = c; g.ldc = ldc; g.M = M; g.N = N; g.K = K;
    g.m_tiles = (M + 2 * TC_BM - 1) / (2 * TC_BM);
    g.n_tiles = (N + out - 1) / out;
    if (!rows_map(&g.a_map, a, M, K, lda, TC_BM) || !rows_map(&g.w_map, w, gated ? 2L * N : N, K, ldw, TC_BM))
        return invalid("cuTensorMapEncodeTiled refused a map of the paired tcgen05 product");
    return launch("gemm_tc2", gemm_tc2_kernel<EPI>, dim3(2 * std::min(sms / 2, g.m_tiles * g.n_tiles)), TC_THREADS, T2_SMEM_BYTES, flags,
                  stream, 2, g);
}

// Tile: the one whose waves cost least.  Measured time of one 64-K stage of a wave: 0.42, 0.25 and 0.20 us for tiles of
// 128 rows x 256, 128 and 64 columns; 0.33 us for 256 x 256 on a pair of SMs (returned as 512).
int tc_tile_choice(int M, int N, bool gated, int sms)
{
    int best = 256;
    long best_cost = -1;
    auto consider = [&](int choice, int rows, int bn, long units, int cost) {
        const int out = gated ? bn / 2 : bn;
        const long tiles = (long)((M + rows - 1) / rows) * ((N + out - 1) / out);
        const long c = ((tiles + units - 1) / units) * cost;
        if (best_cost < 0 || c < best_cost) { best = choice; best_cost = c; }
    };
    consider(512, 256, 256, sms / 2, 33);
    consider(256, 128, 256, sms, 42);
    consider(128, 128, 128, sms, 25);
    consider(64, 128, 64, sms, 20);
    return best;
}

template <int EPI>
twm_status gemm_tc(const bf16* a, int lda, const bf16* w, int ldw, void* c, int ldc, int M, int N, int K, int width, int flags,
                   void* stream)
{
    int sms = 148;
    TRY(device(&sms));
    if (width == 0) width = tc_tile_choice(M, N, EPI == TWM_EPI_GELU_GLU, sms);
    switch (width) {
        case 512: return gemm_tc2_launch<EPI>(a, lda, w, ldw, c, ldc, M, N, K, sms, flags, stream);
        case 256: return gemm_tc_launch<256, EPI>(a, lda, w, ldw, c, ldc, M, N, K, sms, flags, stream);
        case 128: return gemm_tc_launch<128, EPI>(a, lda, w, ldw, c, ldc, M, N, K, sms, flags, stream);
        default: return gemm_tc_launch<64, EPI>(a, lda, w, ldw, c, ldc, M, N, K, sms, flags, stream);
    }
}
twm_status gemm_tc_any(const float*, int, const float*, int, void*, int, int, int, int, int, int, int, void*)
{
    return invalid("the tcgen05 product takes bfloat16");
}
twm_status gemm_tc_any(const bf16* a, int lda, const bf16* w, int ldw, void* c, int ldc, int M, int N, int K, int epi, int width,
                       int flags, void* stream)
{
    switch (epi) {
        case TWM_EPI_STORE: return gemm_tc<TWM_EPI_STORE>(a, lda, w, ldw, c, ldc, M, N, K, width, flags, stream);
        case TWM_EPI_STORE_F32: return gemm_tc<TWM_EPI_STORE_F32>(a, lda, w, ldw, c, ldc, M, N, K, width, flags, stream);
        case TWM_EPI_GELU_GLU: return gemm_tc<TWM_EPI_GELU_GLU>(a, lda, w, ldw, c, ldc, M, N, K, width, flags, stream);
    }
    return invalid("epilogue");
}

template <typename T>
twm_status gemm(const T* a, int lda, const T* w, int ldw, void* c, int ldc, int M, int N, int K, int epi, int kernel, int flags,
                void* stream)
{
    const bool fits = std::is_same<T, bf16>::value && tc_fits(a, lda, w, ldw);
    if (kernel != 0 && kernel != 1 && kernel != 2 && kernel != 64 && kernel != 128 && kernel != 256 && kernel != 512) return invalid("kernel");
    if (kernel >= 2 && !fits) return invalid("the tcgen05 product takes bfloat16 rows on 16-byte boundaries");
    if (kernel >= 2 || (kernel == 0 && fits))
        return gemm_tc_any(a, lda, w, ldw, c, ldc, M, N, K, epi, kernel > 2 ? kernel : 0, flags, stream);
    const dim3 grid((N + ST - 1) / ST, (M + ST - 1) / ST);
    switch (epi) {
        case TWM_EPI_STORE:
            return launch("gemm_simt", gemm_simt_kernel<T, TWM_EPI_STORE>, grid, 256, 0, flags, stream, 0, a, lda, w, ldw, c, ldc, M, N, K);
        case TWM_EPI_STORE_F32:
            return launch("gemm_simt", gemm_simt_kernel<T, TWM_EPI_STORE_F32>, grid, 256, 0, flags, stream, 0, a, lda, w, ldw, c, ldc, M, N, K);
        case TWM_EPI_GELU_GLU:
            return launch("gemm_simt", gemm_simt_kernel<T, TWM_EPI_GELU_GLU>, grid, 256, 0, flags, stream, 0, a, lda, w, ldw, c, ldc, M, N, K);
    }
    return invalid("epilogue");
}

// columns of a grouped product's tiles: as for a plain one, with the rows spread evenly over the experts
int grouped_tile_choice(int rows, int experts, int N, int sms)
{
    const long groups = std::min(rows, experts), m_tiles = groups * ((rows / groups + TC_BM - 1) / TC_BM);
    int best = 256;
    long best_cost = -1;
    for (const auto [bn, cost] : {std::pair<int, int>{256, 42}, {128, 25}, {64, 20}}) {
        const long tiles = m_tiles * ((N + bn - 1) / bn), c = ((tiles + sms - 1) / sms) * cost;
        if (best_cost < 0 || c < best_cost) { best = bn; best_cost = c; }
    }
    return best;
}
template <int EPI>
twm_status grouped_gemm_tc(const bf16* a, int lda, const bf16* w, int ldw, void* c, int ldc, const int* offsets, int experts, int rows, int N,
                           int K, int width, int flags, void* stream)
{
    int sms = 148;
    TRY(device(&sms));
    if (width == 0) width = grouped_tile_choice(rows, experts, N, sms);
    switch (width) {
        case 256: return grouped_gemm_tc_launch<256, EPI>(a, lda, w, ldw, c, ldc, offsets, experts, rows, N, K, sms, flags, stream);
        case 128: return grouped_gemm_tc_launch<128, EPI>(a, lda, w, ldw, c, ldc, offsets, experts, rows, N, K, sms, flags, stream);
        default: return grouped_gemm_tc_launch<64, EPI>(a, lda, w, ldw, c, ldc, offsets, experts, rows, N, K, sms, flags, stream);
    }
}
template <int EPI>
twm_status grouped_gemm_tc(const float*, int, const float*, int, void*, int, const int*, int, int, int, int, int, int, void*)
{
    return invalid("the tcgen05 product takes bfloat16");
}
template <typename T, int EPI>
twm_status grouped_gemm_epi(const T* a, int lda, const T* w, int ldw, void* c, int ldc, const int* offsets, int experts, int rows, int N, int K,
                            int kernel, int flags, void* stream)
{
    const bool fits = std::is_same<T, bf16>::value && tc_fits(a, lda, w, ldw);
    if (kernel != 0 && kernel != 1 && kernel != 2 && kernel != 64 && kernel != 128 && kernel != 256) return invalid("kernel");
    if (kernel >= 2 && !fits) return invalid("the tcgen05 product takes bfloat16 rows on 16-byte boundaries");
    if (kernel >= 2 || (kernel == 0 && fits))
        return grouped_gemm_tc<EPI>(a, lda, w, ldw, c, ldc, offsets, experts, rows, N, K, kernel > 2 ? kernel : 0, flags, stream);
    return launch("moe_gemm_simt", moe_gemm_simt_kernel<T, EPI>, dim3((N + ST - 1) / ST, std::min(rows, rows / ST + experts)), 256, 0, flags,
                  stream, 0, a, lda, w, ldw, c, ldc, offsets, experts, N, K);
}
template <typename T>
twm_status grouped_gemm(const T* a, int lda, const T* w, int ldw, void* c, int ldc, const int* offsets, int experts, int rows, int N, int K,
                        int epi, int kernel, int flags, void* stream)
{
    switch (epi) {
        case TWM_EPI_STORE:
            return grouped_gemm_epi<T, TWM_EPI_STORE>(a, lda, w, ldw, c, ldc, offsets, experts, rows, N, K, kernel, flags, stream);
        case TWM_EPI_STORE_F32:
            return grouped_gemm_epi<T, TWM_EPI_STORE_F32>(a, lda, w, ldw, c, ldc, offsets, experts, rows, N, K, kernel, flags, stream);
        case TWM_EPI_RELU2:
            return grouped_gemm_epi<T, TWM_EPI_RELU2>(a, lda, w, ldw, c, ldc, offsets, experts, rows, N, K, kernel, flags, stream);
    }
    return invalid("epilogue");
}

twm_status route(const float* logits, const RouterArgs& r, int rows, int* ids, float* weights, int* place, int* counts, int flags, void* stream)
{
    return launch("route", route_kernel, dim3((rows + RT_WARPS - 1) / RT_WARPS), RT_WARPS * 32, route_smem_bytes(r), flags, stream, 0, logits, r.experts, r, rows, ids, weights, place, counts);
}

template <typename T>
AttnArgs<T> attn_args(const twm_dense_model* m, const twm_dense_layer& l, const twm_dense_buffers* b, int rows)
{
    const Sizes s = sizes_of(l);
    AttnArgs<T> g;
    g.proj = (const T*)b->proj;
    g.out = (T*)b->att;
    g.k_cache = (const T*)l.k_cache;
    g.v_cache = (const T*)l.v_cache;
    g.bias_table = l.bias_table;
    g.meta = b->meta;
    g.ld = s.in;
    g.gate_off = s.q + s.k + s.v;
    g.heads = l.heads; g.kv_heads = l.kv_heads; g.dim_pad = l.dim_pad; g.vdim_pad = l.vdim_pad;
    g.window = l.window; g.keep_first = l.keep_first; g.capacity = m->capacity; g.bias_len = m->bias_len; g.rows = rows;
    g.scale = l.scale;
    return g;
}

template <int DV>
twm_status attention_mma(const AttnArgs<bf16>& g, int flags, void* stream)
{
    auto kernel = g.dim_pad == 128 ? attn_mma_kernel<128, DV> : g.dim_pad == 64 ? attn_mma_kernel<64, DV> : attn_mma_kernel<0, DV>;
    return launch("attn_mma", kernel, dim3((g.rows + AM_Q - 1) / AM_Q, g.heads, (g.vdim_pad + DV - 1) / DV), AM_THREADS,
                  attn_mma_smem_bytes<DV>(g.dim_pad), flags, stream, 0, g);
}
bool attention_tiles_fit(const AttnArgs<bf16>& g) { return attn_mma_smem_bytes<128>(g.dim_pad) <= kSmemLimit; }
bool attention_tiles_fit(const AttnArgs<float>&) { return false; }
twm_status attention_tiles(const AttnArgs<bf16>& g, int flags, void* stream)
{
    return g.vdim_pad <= 64 ? attention_mma<64>(g, flags, stream) : attention_mma<128>(g, flags, stream);
}
twm_status attention_tiles(const AttnArgs<float>&, int, void*) { return invalid("the tensor-core attention takes bfloat16"); }

// The tcgen05 attention: heads of up to 128 columns.
bool attention_tc_fits(const AttnArgs<bf16>& g)
{
    return g.dim_pad <= 128 && g.vdim_pad <= 128 && ((uintptr_t)g.proj & 15) == 0 && ((uintptr_t)g.k_cache & 15) == 0 &&
           ((uintptr_t)g.v_cache & 15) == 0;
}
bool attention_tc_fits(const AttnArgs<float>&) { return false; }
twm_status attention_tc(const AttnArgs<bf16>& g, int end, int slots, int flags, void* stream)
{
    AttnTcArgs t;
    t.a = g;
    auto cache_map = [&](CUtensorMap* map, const bf16* base, int pad) {
        const long row = (long)g.kv_heads * pad;
        return tensor_map(map, MapKey{MAP_BF16_SWIZZLED, base, 4, {pad, g.kv_heads, end, slots}, {1, pad, row, row * g.capacity}, {64, 1, AT_K, 1}});
    };
    if (!tensor_map(&t.q_map, MapKey{MAP_BF16_SWIZZLED, g.proj, 3, {g.dim_pad, g.heads, g.rows, 0}, {1, g.dim_pad, g.ld, 0}, {64, 1, AT_Q, 0}}) ||
        !cache_map(&t.k_map, g.k_cache, g.dim_pad) || !cache_map(&t.v_map, g.v_cache, g.vdim_pad))
        return invalid("cuTensorMapEncodeTiled refused a map of the tcgen05 attention");
    return launch("attn_tc", attn_tc_kernel, dim3((g.rows + AT_Q - 1) / AT_Q, g.heads), AT_THREADS, sizeof(AttnTcSmem) + 1024, flags,
                  stream, 0, t);
}
twm_status attention_tc(const AttnArgs<float>&, int, int, int, void*) { return invalid("the tcgen05 attention takes bfloat16"); }

template <typename T>
twm_status attention(const twm_dense_model* m, const twm_dense_layer& l, const twm_dense_buffers* b, int rows, int first_pos,
                     int kernel, int flags, void* stream)
{
    const AttnArgs<T> g = attn_args<T>(m, l, b, rows);
    if (kernel < 0 || kernel > 3) return invalid("kernel");
    if (kernel == 3 && !attention_tc_fits(g)) return invalid("the tcgen05 attention takes bfloat16 heads of up to 128 columns");
    if (kernel == 3 || (kernel == 0 && attention_tc_fits(g))) return attention_tc(g, first_pos + rows, m->slots, flags, stream);
    if (kernel == 2 && !attention_tiles_fit(g)) return invalid("the tensor-core attention takes bfloat16 heads that fit shared memory");
    if (kernel == 2 || (kernel == 0 && attention_tiles_fit(g))) return attention_tiles(g, flags, stream);
    const int vblock = AS_VPT * AS_THREADS;
    return launch("attn_simt", attn_simt_kernel<T>, dim3(rows, l.heads, (l.vdim_pad + vblock - 1) / vblock), AS_THREADS,
                  sizeof(float) * (size_t)(l.dim_pad + AS_THREADS), flags, stream, 0, g);
}

// ------------------------------------------------------------------ latent --
bool softmax_tc_fits(const SoftmaxArgs<float>&) { return false; }
bool softmax_tc_fits(const SoftmaxArgs<bf16>& g)
{
    return g.vdim_pad <= 128 && softmax_tc_kboxes(g.dim_pad, g.rot_pad) <= SX_MAX_KBOXES && g.scale > 0.0f && ((uintptr_t)g.proj & 15) == 0 &&
           ((uintptr_t)g.kv & 15) == 0 && ((uintptr_t)g.shared & 15) == 0;
}
twm_status softmax_tc(const SoftmaxArgs<float>&, int, void*) { return invalid("the tcgen05 attention takes bfloat16"); }
twm_status softmax_tc(const SoftmaxArgs<bf16>& g, int flags, void* stream)
{
    SoftmaxTcArgs t;
    t.a = g;
    const long qw = g.dim_pad + g.rot_pad, kv_ld = (long)g.heads * (g.dim_pad + g.vdim_pad), keys = g.first_pos - g.first_key + g.rows;
    auto heads_map = [&](CUtensorMap* map, const bf16* base, int cols, long per_head, long rows, long ld, int box_rows) {
        return tensor_map(map, MapKey{MAP_BF16_SWIZZLED, base, 3, {cols, g.heads, rows, 0}, {1, per_head, ld, 0}, {64, 1, box_rows, 0}});
    };
    if (!heads_map(&t.q_map, g.proj, g.dim_pad, qw, g.rows, g.ld, SX_Q) || !heads_map(&t.qr_map, g.proj + g.dim_pad, g.rot_pad, qw, g.rows, g.ld, SX_Q) ||
        !heads_map(&t.k_map, g.kv, g.dim_pad, g.dim_pad, keys, kv_ld, SX_K) || !rows_map(&t.kr_map, g.shared, keys, g.rot_pad, g.shared_ld, SX_K) ||
        !heads_map(&t.v_map, g.kv + (long)g.heads * g.dim_pad, g.vdim_pad, g.vdim_pad, keys, kv_ld, SX_K))
        return invalid("cuTensorMapEncodeTiled refused a map of the tcgen05 softmax attention");
    return launch("attn_softmax_tc", attn_softmax_tc_kernel, dim3((g.rows + SX_Q - 1) / SX_Q, g.heads), SX_THREADS,
                  softmax_tc_smem_bytes(g.dim_pad, g.rot_pad, g.vdim_pad), flags, stream, 0, t);
}
template <typename T>
twm_status softmax_attention(const SoftmaxArgs<T>& g, int kernel, int flags, void* stream)
{
    if (kernel != 0 && kernel != 1 && kernel != 3) return invalid("kernel");
    if (kernel == 3 && !softmax_tc_fits(g)) return invalid("the tcgen05 softmax attention takes bfloat16 heads of up to 128 columns");
    if (kernel == 3 || (kernel == 0 && softmax_tc_fits(g))) return softmax_tc(g, flags, stream);
    const int vblock = AS_VPT * AS_THREADS;
    return launch("attn_softmax_simt", attn_softmax_simt_kernel<T>, dim3(g.rows, g.heads, (g.vdim_pad + vblock - 1) / vblock), AS_THREADS,
                  sizeof(float) * (size_t)(g.dim_pad + g.rot_pad + AS_THREADS), flags, stream, 0, g);
}

// From the fused projection to the gated head outputs: norms, rotations and cache, the visible tokens' keys and values,
// attention.
template <typename T>
twm_status latent_mixer(const twm_dense_model* m, const twm_dense_layer& l, const twm_dense_buffers* b, int rows, int first_pos, int kernel,
                        int flags, void* stream)
{
    const Sizes s = sizes_of(l);
    const int first_key = std::max(0, first_pos - l.window + 1), older = first_pos - first_key, keys = older + rows;
    const int width = l.rank_pad + l.rot_pad, n = l.heads * (l.dim_pad + l.vdim_pad);
    if (keys > b->max_keys) return invalid("more visible tokens than the buffers take");
    LatentRowsArgs<T> r;
    r.proj = (T*)b->proj; r.cache = (T*)l.latent_cache; r.lat = (T*)b->lat; r.norm = l.latent_norm; r.rot_table = (const float2*)l.rot_table;
    r.meta = b->meta; r.ld = s.in; r.heads = l.heads; r.dim_pad = l.dim_pad; r.rot_pad = l.rot_pad; r.rank = l.rank; r.rank_pad = l.rank_pad;
    r.capacity = m->capacity; r.rows = rows; r.older = older; r.eps = m->eps;
    TRY(launch("latent_rows", latent_rows_kernel<T>, dim3(keys), ROW_THREADS, 0, flags, stream, 0, r));
    TRY(gemm<T>((const T*)b->lat, width, (const T*)l.w_expand, l.rank_pad, b->kv, n, keys, n, l.rank_pad, TWM_EPI_STORE, 0, flags, stream));
    SoftmaxArgs<T> g;
    g.proj = (const T*)b->proj; g.kv = (const T*)b->kv; g.shared = (const T*)b->lat + l.rank_pad; g.out = (T*)b->att;
    g.ld = s.in; g.gate_off = s.q + s.k; g.shared_ld = width; g.heads = l.heads; g.dim_pad = l.dim_pad; g.rot_pad = l.rot_pad;
    g.vdim_pad = l.vdim_pad; g.window = l.window; g.rows = rows; g.first_pos = first_pos; g.first_key = first_key; g.scale = l.scale;
    return softmax_attention<T>(g, kernel, flags, stream);
}

// --------------------------------------------------- gated linear attention --
template <typename T>
GlaArgs<T> gla_args(const twm_dense_model* m, const twm_dense_layer& l, const twm_dense_buffers* b, int rows)
{
    GlaArgs<T> g;
    g.proj = (const T*)b->proj; g.decay = b->decay; g.chunk_state = b->chunk_state; g.mix = b->mix; g.out = (T*)b->att; g.state = l.gla_state;
    g.w_decay = (const T*)l.w_decay; g.decay_bias = l.decay_bias; g.head_norm = l.head_norm; g.meta = b->meta;
    g.ld = sizes_of(l).in; g.heads = l.heads; g.dim_pad = l.dim_pad; g.vdim = l.vdim; g.vdim_pad = l.vdim_pad; g.rank_pad = l.rank_pad;
    g.rows = rows; g.inv_tau = l.inv_tau; g.q_scale = l.scale; g.eps = m->eps;
    return g;
}
bool gla_chunks_fit(const GlaArgs<float>&) { return false; }
bool gla_chunks_fit(const GlaArgs<bf16>& g)
{
    return g.vdim_pad <= 128 && gla_chunk_out_smem_bytes(g.dim_pad, g.vdim_pad) <= kSmemLimit &&
           gla_chunk_state_smem_bytes(g.vdim_pad) <= kSmemLimit;
}
twm_status gla_chunks(const GlaArgs<float>&, int, void*) { return invalid("the chunked linear attention takes bfloat16"); }
twm_status gla_chunks(const GlaArgs<bf16>& g, int flags, void* stream)
{
    const int chunks = (g.rows + GLA_CHUNK - 1) / GLA_CHUNK, quads = g.heads * g.dim_pad * g.vdim_pad / 4;
    const bool d128 = g.dim_pad == 128 && g.vdim_pad == 128, d64 = g.dim_pad == 64 && g.vdim_pad == 64;
    auto state = d128 ? gla_chunk_state_kernel<128, 128> : d64 ? gla_chunk_state_kernel<64, 64> : gla_chunk_state_kernel<0, 0>;
    auto out = d128 ? gla_chunk_out_kernel<128, 128> : d64 ? gla_chunk_out_kernel<64, 64> : g.vdim_pad <= 64 ? gla_chunk_out_kernel<0, 64>
                                                                                                     : gla_chunk_out_kernel<0, 128>;
    TRY(launch("gla_chunk_state", state, dim3(chunks, g.heads, (g.dim_pad + GC_DIMS - 1) / GC_DIMS), GC_THREADS,
               gla_chunk_state_smem_bytes(g.vdim_pad), flags, stream, 0, g));
    TRY(launch("gla_scan", gla_scan_kernel<bf16>, dim3((quads + GS_THREADS - 1) / GS_THREADS), GS_THREADS, 0, flags, stream, 0, g));
    return launch("gla_chunk_out", out, dim3(chunks, g.heads), GO_THREADS, gla_chunk_out_smem_bytes(g.dim_pad, g.vdim_pad), flags, stream, 0, g);
}
template <typename T>
twm_status gla_mixer(const twm_dense_model* m, const twm_dense_layer& l, const twm_dense_buffers* b, int rows, int kernel, int flags, void* stream)
{
    const GlaArgs<T> g = gla_args<T>(m, l, b, rows);
    if (kernel < 0 || kernel > 2) return invalid("kernel");
    if (kernel == 2 && !gla_chunks_fit(g)) return invalid("the chunked linear attention takes bfloat16 heads that fit shared memory");
    if (kernel == 2 || (kernel == 0 && gla_chunks_fit(g))) return gla_chunks(g, flags, stream);
    const int cols = g.heads * g.dim_pad;
    TRY(launch("gla_decay", gla_decay_kernel<T>, dim3((cols + GD_THREADS - 1) / GD_THREADS, (rows + GD_ROWS - 1) / GD_ROWS), GD_THREADS, 0, flags,
               stream, 0, g));
    TRY(launch("gla_rows", gla_rows_kernel<T>, dim3((g.vdim_pad + GR_COLS - 1) / GR_COLS, g.heads), GR_THREADS, gla_rows_smem_bytes(g.dim_pad), flags,
               stream, 0, g));
    return launch("gla_gate", gla_gate_kernel<T>, dim3(rows), ROW_THREADS, 0, flags, stream, 0, g);
}

// ------------------------------------------------------------------ routed --
struct RouteBuffers { int *ids, *place, *row, *counts, *offsets; };
RouteBuffers route_buffers(const twm_dense_buffers* b, int experts)
{
    RouteBuffers r;
    r.ids = b->route; r.place = r.ids + b->max_slots; r.row = r.place + b->max_slots; r.counts = r.row + b->max_slots; r.offsets = r.counts + experts;
    return r;
}
// The chosen experts' outputs of `rows` tokens (buffers->a), grouped by expert, to buffers->expert_out.  The counts are
// zero at the start.
template <typename T>
twm_status routed_ff(const twm_dense_model* m, const twm_dense_layer& l, const twm_dense_buffers* b, int rows, int flags, void* stream)
{
    const int wp = m->width_pad, slots = rows * l.top;
    const RouterArgs r = {l.experts, l.top, l.groups, l.keep};
    const RouteBuffers rb = route_buffers(b, l.experts);
    TRY(gemm<T>((const T*)b->a, wp, (const T*)l.w_router, wp, b->router_logits, l.experts, rows, l.experts, wp, TWM_EPI_STORE_F32, 0, flags, stream));
    TRY(route(b->router_logits, r, rows, rb.ids, b->route_weight, rb.place, rb.counts, flags, stream));
    TRY(launch("group_rows", group_rows_kernel<T>, dim3(rows), MG_THREADS, 0, flags, stream, 0, (const T*)b->a, wp, r, rows, (const int*)rb.ids,
               (const int*)rb.place, (const int*)rb.counts, rb.row, rb.offsets, (T*)b->grouped));
    TRY(grouped_gemm<T>((const T*)b->grouped, wp, (const T*)l.w_gate_up, wp, b->act, l.ff_pad, rb.offsets, l.experts, slots, l.ff_pad, wp,
                        TWM_EPI_RELU2, 0, flags, stream));
    return grouped_gemm<T>((const T*)b->act, l.ff_pad, (const T*)l.w_down, l.ff_pad, b->expert_out, wp, rb.offsets, l.experts, slots, m->width,
                           l.ff_pad, TWM_EPI_STORE, 0, flags, stream);
}

template <typename T>
twm_status prefill(const twm_dense_model* m, const twm_dense_buffers* b, int rows, int first_pos, int n_want, float* layer_trace,
                   int flags, void* stream)
{
    // With early launches, prompt steps of routed, latent and linear layers have stopped for good at 2048 tokens (never without
    // them, and never in chains of sigmoid attention and gated feed-forwards alone); the cause is not known.
    for (int i = 0; i < m->n_layers; ++i)
        if (m->layers[i].mixer != TWM_MIX_SIGMOID || m->layers[i].experts > 0) flags &= ~TWM_FLAG_PDL;
    const int wp = m->width_pad;
    float *x = b->x0, *x_next = b->x1;
    const float* y = nullptr;                            // the sublayer output that has yet to join the residual stream
    const float* y_norm = nullptr;
    RoutedOutput<T> routed = {};
    bool embedded = false;
    auto source = [&](const float* step) {
        ResidualSource<T> s;
        s.tokens = embedded ? nullptr : b->tokens;
        s.embed = (const T*)m->embed;
        s.pos_embed = (const T*)m->pos_embed;
        s.x_in = x; s.y = y; s.y_norm = y_norm; s.step = step; s.routed = routed;
        s.eps = m->eps; s.embed_scale = m->embed_scale; s.width = m->width; s.wp = wp;
        return s;
    };
    // the residual stream brought up to date, with the next sublayer's input beside it
    struct Next { const float *shift, *shift_state, *pre_norm, *step; int* clear; int n_clear; };
    auto join = [&](const Next& next, bool want_a) {
        // rows per CTA: enough CTAs to fill the machine several times; a shifted run computes one row more than it has
        const int rpc = next.shift ? (rows >= 4096 ? 8 : rows >= 1024 ? 4 : rows >= 256 ? 2 : 1) : 1;
        const int per = (wp / 4 + ROW_THREADS - 1) / ROW_THREADS;
        const bool full = next.pre_norm || next.step || next.n_clear || routed.rows;
        auto pick = [&](auto f) {
            constexpr bool F = decltype(f)::value;
            return per <= 1 ? residual_rows_kernel<T, 1, F> : per <= 2 ? residual_rows_kernel<T, 2, F> : per <= 4 ? residual_rows_kernel<T, 4, F> :
                   per <= 8 ? residual_rows_kernel<T, 8, F> : residual_rows_kernel<T, 0, F>;
        };
        auto kernel = full ? pick(std::true_type()) : pick(std::false_type());
        const twm_status st = launch("residual_rows", kernel, dim3((rows + rpc - 1) / rpc), ROW_THREADS,
                                     per <= 8 ? 0 : sizeof(float) * (size_t)wp, flags, stream, 0, source(next.step), x_next,
                                     want_a ? (T*)b->a : (T*)nullptr, next.shift, next.shift_state, next.pre_norm, b->meta, rows, rpc,
                                     next.clear, next.n_clear);
        std::swap(x, x_next);
        embedded = true;
        y = nullptr;
        routed.rows = nullptr;
        return st;
    };
    auto trace = [&](int layer) -> twm_status {
        if (!layer_trace) return TWM_OK;
        const cudaError_t e = cudaMemcpyAsync(layer_trace + (size_t)layer * rows * wp, x, sizeof(float) * (size_t)rows * wp,
                                              cudaMemcpyDeviceToDevice, (cudaStream_t)stream);
        return e == cudaSuccess ? TWM_OK : fail("layer trace", e);
    };
    for (int i = 0; i < m->n_layers; ++i) {
        const twm_dense_layer& l = m->layers[i];
        const Sizes s = sizes_of(l);
        const bool traced = layer_trace && i > 0;
        if (traced && l.step) {                          // what the trace shows comes before the step vector
            TRY(join({}, false));
            TRY(trace(i - 1));
        }
        TRY(join({l.shift, l.shift_state, l.pre1, l.step, nullptr, 0}, true));
        if (traced && !l.step) TRY(trace(i - 1));
        TRY(gemm<T>((const T*)b->a, wp, (const T*)l.w_in, wp, b->proj, s.in, rows, s.in, wp, TWM_EPI_STORE, 0, flags, stream));
        if (l.mixer == TWM_MIX_LATENT) {
            TRY(latent_mixer<T>(m, l, b, rows, first_pos, 0, flags, stream));
        } else if (l.mixer == TWM_MIX_GLA) {
            TRY(gla_mixer<T>(m, l, b, rows, 0, flags, stream));
        } else {
            TRY(launch("qk_norm_append", qk_norm_append_kernel<T>, dim3(rows), ROW_THREADS, 0, flags, stream, 0, (T*)b->proj, s.in,
                       l.q_norm, l.k_norm, (T*)l.k_cache, (T*)l.v_cache, s.q, s.k, s.v, l.heads * l.dim, l.kv_heads * l.dim, m->eps,
                       m->capacity, (const float*)x, wp, l.shift ? l.shift_state : (float*)nullptr, b->meta));
            TRY(attention<T>(m, l, b, rows, first_pos, 0, flags, stream));
        }
        TRY(gemm<T>((const T*)b->att, s.out, (const T*)l.w_out, s.out, b->y, wp, rows, m->width, s.out, TWM_EPI_STORE_F32, 0, flags,
                    stream));
        y = b->y; y_norm = l.norm1;
        if (l.experts > 0) {
            const RouteBuffers rb = route_buffers(b, l.experts);
            TRY(join({nullptr, nullptr, l.pre2, nullptr, rb.counts, l.experts}, true));
            TRY(routed_ff<T>(m, l, b, rows, flags, stream));
            routed = RoutedOutput<T>{(const T*)b->expert_out, rb.row, b->route_weight, l.top};
            y_norm = l.norm2;
        } else if (l.ff_pad > 0) {
            TRY(join({nullptr, nullptr, l.pre2, nullptr, nullptr, 0}, true));
            TRY(gemm<T>((const T*)b->a, wp, (const T*)l.w_gate_up, wp, b->act, l.ff_pad, rows, l.ff_pad, wp, TWM_EPI_GELU_GLU, 0,
                        flags, stream));
            TRY(gemm<T>((const T*)b->act, l.ff_pad, (const T*)l.w_down, l.ff_pad, b->y, wp, rows, m->width, l.ff_pad,
                        TWM_EPI_STORE_F32, 0, flags, stream));
            y = b->y; y_norm = l.norm2;
        }
    }
    if (layer_trace && m->n_layers > 0) {
        TRY(join({}, false));
        TRY(trace(m->n_layers - 1));
    }
    if (n_want > 0) {
        TRY(launch("final_rows", final_rows_kernel<T>, dim3(n_want), ROW_THREADS, sizeof(float) * (size_t)wp, flags, stream, 0,
                   source(nullptr), (T*)b->a, m->final_norm, (const int*)b->want, (const int*)b->meta));
        TRY(gemm<T>((const T*)b->a, wp, (const T*)m->head, wp, b->logits, m->vocab, n_want, m->vocab, wp, TWM_EPI_STORE_F32, 0,
                    flags, stream));
    }
    return TWM_OK;
}

template <typename T, int PRO, int EPI = TWM_EPI_STORE_F32, int ROUTE = ROUTE_NONE>
twm_status gemv(GemvArgs<T> g, int sms, int flags, void* stream)
{
    constexpr bool GATED = EPI == TWM_EPI_GELU_GLU;
    const int rows = GV_ROWS / 2, stream_rows = GATED ? g.N : (g.N + 1) / 2;      // of each of the two streams
    const int grid = std::min(sms, (stream_rows + rows - 1) / rows);
    g.rounds = stream_rows / (grid * rows);
    // a full round of an undivided product's second stream must exist in it too: an odd row count leaves its last row out
    while (!GATED && g.rounds > 0 && g.rounds * grid * rows > g.N - stream_rows) --g.rounds;
    const int left = stream_rows - g.rounds * grid * rows;
    g.last_rows = (left + grid - 1) / grid;
    const long words = (long)g.ldw * sizeof(T) / 8;
    const long w_rows = ROUTE != ROUTE_NONE ? (long)g.router.experts * g.expert_rows : GATED ? 2L * g.N : g.N;
    if (!word_rows_map(&g.w_map, g.w, w_rows, words, GV_PIECE / 8, rows))
        return invalid("cuTensorMapEncodeTiled refused a map of the decode product");
    const size_t row_bytes = (size_t)g.ldw * sizeof(T);
    const int parts = ROUTE == ROUTE_COLUMNS ? g.router.top : 1;
    const size_t act = gemv_smem_bytes(row_bytes, parts, 0), limit = kSmemLimit - 8 * 1024;      // static shared memory beside it
    if (act + 2 * GV_STAGE > limit) return invalid("an input row does not fit shared memory");
    g.stages = (int)std::min<size_t>(GV_MAX_STAGES, (limit - act) / GV_STAGE);
    return launch("gemv", gemv_kernel<T, PRO, EPI, ROUTE>, dim3(grid), GV_THREADS, gemv_smem_bytes(row_bytes, parts, g.stages), flags, stream, 0, g);
}

// --------------------------------------------- one decoded token's mixers --
template <typename T>
twm_status sigmoid_decode(const twm_dense_model* m, const twm_dense_layer& l, const twm_dense_buffers* b, const float* proj, float* att, int sms,
                          int flags, void* stream)
{
    AttnDecodeArgs<T> t;
    t.proj = proj; t.out = att; t.q_norm = l.q_norm; t.k_norm = l.k_norm;
    t.k_cache = (T*)l.k_cache; t.v_cache = (T*)l.v_cache; t.bias_table = l.bias_table; t.meta = b->meta;
    t.heads = l.heads; t.kv_heads = l.kv_heads; t.dim = l.dim; t.dim_pad = l.dim_pad; t.vdim_pad = l.vdim_pad;
    t.window = l.window; t.keep_first = l.keep_first; t.capacity = m->capacity; t.bias_len = m->bias_len; t.gated = 1;
    t.scale = l.scale; t.eps = m->eps;
    // about 64 visible keys per CTA, up to 16 CTAs a head (a cluster; more than 8 is the non-portable size), and no
    // more CTAs than one wave
    const long visible = std::min<long>((long)l.window + l.keep_first, m->capacity);
    int splits = 1;
    while (splits < 16 && visible > 64L * splits && l.kv_heads * splits * 2 <= sms) splits *= 2;
    // a chunk of keys and values that leaves room for a product's CTA on the same SM, where heads are not too wide
    auto bytes = [&](int chunk) { return attn_decode_smem_bytes<T>(l.heads / l.kv_heads, l.dim_pad, l.vdim_pad, chunk, splits); };
    t.parts = attn_decode_parts(l.heads / l.kv_heads, l.vdim_pad);
    t.chunk = AD_MAX_CHUNK;
    while (t.chunk > 8 && bytes(t.chunk) > 80 * 1024) t.chunk /= 2;
    return launch("attn_decode", attn_decode_kernel<T>, dim3(splits, l.kv_heads), AD_THREADS, bytes(t.chunk), flags, stream, splits, t);
}

template <typename T>
twm_status latent_decode(const twm_dense_model* m, const twm_dense_layer& l, const twm_dense_buffers* b, const float* proj, float* att, int sms,
                         int flags, void* stream)
{
    LatentDecodeArgs<T> t;
    t.proj = proj; t.out = att; t.w_expand = (const T*)l.w_expand; t.norm = l.latent_norm; t.rot_table = (const float2*)l.rot_table;
    t.cache = (T*)l.latent_cache; t.meta = b->meta; t.heads = l.heads; t.dim_pad = l.dim_pad; t.rot_pad = l.rot_pad; t.rank = l.rank;
    t.rank_pad = l.rank_pad; t.vdim_pad = l.vdim_pad; t.window = l.window; t.capacity = m->capacity; t.scale = l.scale; t.eps = m->eps;
    int splits = 1;                                      // CTAs a head, one wave of them
    while (splits < LD_MAX_SPLITS && l.heads * splits * 2 <= sms) splits *= 2;
    t.parts = latent_decode_parts(l.rank_pad);
    const long visible = std::min(l.window, m->capacity), share = (visible + splits - 1) / splits;
    auto bytes = [&](int chunk) { return latent_decode_smem_bytes<T>(l.dim_pad, l.rot_pad, l.rank_pad, chunk, t.parts, splits); };
    t.chunk = (int)std::min<long>(LD_MAX_CHUNK, (share + 7) / 8 * 8);
    while (t.chunk > 8 && bytes(t.chunk) > 200 * 1024) t.chunk = (t.chunk / 2 + 7) / 8 * 8;
    return launch("latent_decode", latent_decode_kernel<T>, dim3(splits, l.heads), LD_THREADS, bytes(t.chunk), flags, stream, splits, t);
}

template <typename T>
twm_status gla_decode(const twm_dense_model* m, const twm_dense_layer& l, const twm_dense_buffers* b, const float* proj, float* att, int sms,
                      int flags, void* stream)
{
    GlaDecodeArgs<T> t;
    t.proj = proj; t.out = att; t.state = l.gla_state; t.w_decay = (const T*)l.w_decay; t.decay_bias = l.decay_bias; t.head_norm = l.head_norm;
    t.meta = b->meta; t.heads = l.heads; t.dim_pad = l.dim_pad; t.vdim = l.vdim; t.vdim_pad = l.vdim_pad; t.rank_pad = l.rank_pad;
    t.inv_tau = l.inv_tau; t.q_scale = l.scale; t.eps = m->eps;
    int splits = 1;
    while (splits < GX_MAX_SPLITS && l.heads * splits * 2 <= sms && l.vdim_pad / (2 * splits) >= 16) splits *= 2;
    return launch("gla_decode", gla_decode_kernel<T>, dim3(splits, l.heads), GX_THREADS, gla_decode_smem_bytes(l.dim_pad, l.vdim_pad, splits), flags,
                  stream, splits, t);
}

template <typename T>
twm_status decode(const twm_dense_model* m, const twm_dense_buffers* b, int want_logits, int flags, void* stream, int sms)
{
    const int wp = m->width_pad;
    float *x = b->x0, *x_next = b->x1;
    const float* y = nullptr;
    const float* y_norm = nullptr;
    bool embedded = false;
    int widest_in = 0, widest_out = 0, widest_act = 0;
    for (int i = 0; i < m->n_layers; ++i) {
        const Sizes s = sizes_of(m->layers[i]);
        widest_in = std::max(widest_in, s.in);
        widest_out = std::max(widest_out, s.out);
        widest_act = std::max(widest_act, act_columns(m->layers[i]));
    }
    float* proj = b->vec;
    float* att = proj + widest_in;
    float* act = att + widest_out;
    float* h = act + widest_act;                         // a routed feed-forward's input row
    auto args = [&](const void* w, int N, int ldw, float* out) {
        GemvArgs<T> g = {};
        g.w = (const T*)w; g.N = N; g.ldw = ldw; g.out = out; g.meta = b->meta;
        return g;
    };
    auto with_residual = [&](GemvArgs<T> g, const float* step) {
        g.src.tokens = embedded ? nullptr : b->tokens;
        g.src.embed = (const T*)m->embed;
        g.src.pos_embed = (const T*)m->pos_embed;
        g.src.x_in = x; g.src.y = y; g.src.y_norm = y_norm; g.src.step = step;
        g.src.eps = m->eps; g.src.embed_scale = m->embed_scale; g.src.width = m->width; g.src.wp = wp;
        g.x_out = x_next;
        std::swap(x, x_next);
        embedded = true;
        y = nullptr;
        return g;
    };
    for (int i = 0; i < m->n_layers; ++i) {
        const twm_dense_layer& l = m->layers[i];
        const Sizes s = sizes_of(l);
        GemvArgs<T> g = with_residual(args(l.w_in, s.in, wp, proj), l.step);
        g.shift = l.shift;
        g.shift_state = l.shift_state;
        g.pre_norm = l.pre1;
        if (l.shift) TRY((gemv<T, PRO_SHIFT>(g, sms, flags, stream)));
        else if (l.pre1) TRY((gemv<T, PRO_NORM>(g, sms, flags, stream)));
        else TRY((gemv<T, PRO_RESIDUAL>(g, sms, flags, stream)));
        if (l.mixer == TWM_MIX_LATENT) TRY(latent_decode<T>(m, l, b, proj, att, sms, flags, stream));
        else if (l.mixer == TWM_MIX_GLA) TRY(gla_decode<T>(m, l, b, proj, att, sms, flags, stream));
        else TRY(sigmoid_decode<T>(m, l, b, proj, att, sms, flags, stream));
        GemvArgs<T> o = args(l.w_out, m->width, s.out, b->y);
        o.vec = att;
        TRY((gemv<T, PRO_VEC>(o, sms, flags, stream)));
        y = b->y; y_norm = l.norm1;
        if (l.experts > 0) {
            const RouterArgs r = {l.experts, l.top, l.groups, l.keep};
            g = with_residual(args(nullptr, 0, wp, nullptr), nullptr);
            RouterDecodeArgs<T> q;
            q.src = g.src; q.x_out = g.x_out; q.h_out = h; q.pre_norm = l.pre2; q.w = (const T*)l.w_router; q.meta = b->meta; q.router = r;
            q.ids = b->route; q.weights = b->route_weight;
            TRY(launch("router_decode", router_decode_kernel<T>, dim3(RD_CTAS), RD_THREADS, router_decode_smem_bytes<T>(wp), flags, stream, RD_CTAS, q));
            g = args(l.w_gate_up, l.top * l.ff_pad, wp, act);
            g.vec = h;
            g.router = r; g.expert_rows = l.ff_pad; g.ids = b->route; g.weights = b->route_weight;
            TRY((gemv<T, PRO_VEC, TWM_EPI_RELU2, ROUTE_ROWS>(g, sms, flags, stream)));
            GemvArgs<T> d = args(l.w_down, m->width, l.ff_pad, b->y);
            d.vec = act;
            d.router = r; d.expert_rows = m->width; d.ids = b->route; d.weights = b->route_weight;
            TRY((gemv<T, PRO_VEC, TWM_EPI_STORE_F32, ROUTE_COLUMNS>(d, sms, flags, stream)));
            y = b->y; y_norm = l.norm2;
        } else if (l.ff_pad > 0) {
            g = with_residual(args(l.w_gate_up, l.ff_pad, wp, act), nullptr);
            g.pre_norm = l.pre2;
            if (l.pre2) TRY((gemv<T, PRO_NORM, TWM_EPI_GELU_GLU>(g, sms, flags, stream)));
            else TRY((gemv<T, PRO_RESIDUAL, TWM_EPI_GELU_GLU>(g, sms, flags, stream)));
            GemvArgs<T> d = args(l.w_down, m->width, l.ff_pad, b->y);
            d.vec = act;
            TRY((gemv<T, PRO_VEC>(d, sms, flags, stream)));
            y = b->y; y_norm = l.norm2;
        }
    }
    if (want_logits) {
        GemvArgs<T> g = with_residual(args(m->head, m->vocab, wp, b->logits), nullptr);
        g.pre_norm = m->final_norm;
        TRY((gemv<T, PRO_NORM>(g, sms, flags, stream)));
    }
    return TWM_OK;
}

}  // namespace

extern "C" {

twm_status twm_dense_prefill(const twm_dense_model* m, const twm_dense_buffers* b, int rows, int first_pos, int n_want,
                             float* layer_trace, int flags, void* stream)
{
    t_launches = 0;
    TRY(check_model(m, b));
    if (rows < 1 || rows > b->max_rows || n_want < 0 || n_want > rows || n_want > b->max_want) return invalid("rows or n_want");
    if (first_pos < 0 || first_pos > m->capacity - rows) return invalid("the step runs past the slot's capacity");
    TRY(device(nullptr));
    return m->dtype == TWM_DENSE_F32 ? prefill<float>(m, b, rows, first_pos, n_want, layer_trace, flags, stream)
                                     : prefill<bf16>(m, b, rows, first_pos, n_want, layer_trace, flags, stream);
}

twm_status twm_dense_decode(const twm_dense_model* m, const twm_dense_buffers* b, int want_logits, int flags, void* stream)
{
    t_launches = 0;
    TRY(check_model(m, b));
    int sms = 148;
    TRY(device(&sms));
    return m->dtype == TWM_DENSE_F32 ? decode<float>(m, b, want_logits, flags, stream, sms)
                                     : decode<bf16>(m, b, want_logits, flags, stream, sms);
}

int twm_dense_launches(void) { return t_launches; }

twm_status twm_dense_set_step(const twm_dense_buffers* b, int first_pos, int slot, int token, void* stream)
{
    if (!b || !b->meta || !b->tokens || first_pos < 0 || slot < 0) return invalid("set_step");
    TRY(device(nullptr));
    return launch("set_step", set_step_kernel, dim3(1), 1, 0, 0, stream, 0, b->meta, b->tokens, first_pos, slot, token);
}

size_t twm_dense_argmax_scratch_bytes(void) { return (size_t)kArgmaxParts * 8; }

twm_status twm_dense_argmax_advance(const twm_dense_buffers* b, int vocab, int row, int* history, int history_capacity, void* scratch,
                                    size_t scratch_bytes, int flags, void* stream)
{
    if (!b || vocab < 1 || row < 0 || row >= b->max_want || !scratch || (history && history_capacity < 1)) return invalid("argmax");
    if (scratch_bytes < twm_dense_argmax_scratch_bytes()) return TWM_EWORKSPACE;
    TRY(device(nullptr));
    float* pval = (float*)scratch;
    int* pidx = (int*)((char*)scratch + (size_t)kArgmaxParts * 4);
    TRY(launch("argmax(partial)", ops::argmax_partial_kernel, dim3(kArgmaxParts), 256, 0, flags, stream, 0, pval, pidx,
               (const float*)b->logits + (size_t)row * vocab, vocab));
    return launch("argmax(final)", ops::argmax_final_kernel, dim3(1), 256, 0, flags, stream, 0, b->tokens, history, history_capacity,
                  b->meta, b->meta + 2, b->meta + 3, (const float*)pval, (const int*)pidx, kArgmaxParts, vocab);
}

twm_status twm_dense_gemm(int dtype, const void* a, int lda, const void* w, int ldw, void* c, int ldc, int M, int N, int K,
                          int epilogue, int kernel, int flags, void* stream)
{
    if (!a || !w || !c || M < 1 || N < 1 || K < 1 || lda < K || ldw < K || ldc < N) return invalid("gemm");
    TRY(device(nullptr));
    if (dtype == TWM_DENSE_F32)
        return gemm<float>((const float*)a, lda, (const float*)w, ldw, c, ldc, M, N, K, epilogue, kernel, flags, stream);
    if (dtype == TWM_DENSE_BF16)
        return gemm<bf16>((const bf16*)a, lda, (const bf16*)w, ldw, c, ldc, M, N, K, epilogue, kernel, flags, stream);
    return invalid("dtype");
}

twm_status twm_dense_attention(const twm_dense_model* m, int layer, const twm_dense_buffers* b, int rows, int first_pos, int kernel,
                               int flags, void* stream)
{
    TRY(check_model(m, b));
    if (layer < 0 || layer >= m->n_layers || rows < 1 || rows > b->max_rows || first_pos < 0 || first_pos > m->capacity - rows)
        return invalid("attention");
    TRY(device(nullptr));
    const twm_dense_layer& l = m->layers[layer];
    if (l.mixer == TWM_MIX_GLA) return invalid("the layer has no attention");
    if (l.mixer == TWM_MIX_LATENT)
        return m->dtype == TWM_DENSE_F32 ? latent_mixer<float>(m, l, b, rows, first_pos, kernel, flags, stream)
                                         : latent_mixer<bf16>(m, l, b, rows, first_pos, kernel, flags, stream);
    return m->dtype == TWM_DENSE_F32 ? attention<float>(m, m->layers[layer], b, rows, first_pos, kernel, flags, stream)
                                     : attention<bf16>(m, m->layers[layer], b, rows, first_pos, kernel, flags, stream);
}

twm_status twm_dense_gla(const twm_dense_model* m, int layer, const twm_dense_buffers* b, int rows, int kernel, int flags, void* stream)
{
    TRY(check_model(m, b));
    if (layer < 0 || layer >= m->n_layers || rows < 1 || rows > b->max_rows || m->layers[layer].mixer != TWM_MIX_GLA) return invalid("gla");
    TRY(device(nullptr));
    return m->dtype == TWM_DENSE_F32 ? gla_mixer<float>(m, m->layers[layer], b, rows, kernel, flags, stream)
                                     : gla_mixer<bf16>(m, m->layers[layer], b, rows, kernel, flags, stream);
}

twm_status twm_dense_route(const float* logits, int experts, int top, int groups, int keep, int rows, int* ids, float* weights, int flags,
                           void* stream)
{
    if (!logits || !ids || !weights || experts < 1 || experts > MOE_MAX_EXPERTS || top < 1 || top > MOE_MAX_TOP || groups < 1 || experts % groups ||
        keep < 1 || keep > groups || top > keep * (experts / groups) || rows < 1)
        return invalid("route");
    TRY(device(nullptr));
    return route(logits, RouterArgs{experts, top, groups, keep}, rows, ids, weights, nullptr, nullptr, flags, stream);
}

twm_status twm_dense_grouped_gemm(int dtype, const void* a, int lda, const void* w, int ldw, void* c, int ldc, const int* offsets, int experts,
                                  int rows, int N, int K, int epilogue, int kernel, int flags, void* stream)
{
    if (!a || !w || !c || !offsets || experts < 1 || experts > MOE_MAX_EXPERTS || rows < 1 || N < 1 || K < 1 || lda < K || ldw < K || ldc < N)
        return invalid("grouped_gemm");
    TRY(device(nullptr));
    if (dtype == TWM_DENSE_F32)
        return grouped_gemm<float>((const float*)a, lda, (const float*)w, ldw, c, ldc, offsets, experts, rows, N, K, epilogue, kernel, flags, stream);
    if (dtype == TWM_DENSE_BF16)
        return grouped_gemm<bf16>((const bf16*)a, lda, (const bf16*)w, ldw, c, ldc, offsets, experts, rows, N, K, epilogue, kernel, flags, stream);
    return invalid("dtype");
}

twm_status twm_dense_device_error(void* stream, unsigned int* word)
{
    if (!word) return invalid("device_error");
    cudaError_t e = cudaMemcpyFromSymbolAsync(word, g_error_word, sizeof(unsigned int), 0, cudaMemcpyDeviceToHost, (cudaStream_t)stream);
    if (e == cudaSuccess) e = cudaStreamSynchronize((cudaStream_t)stream);
    if (e == cudaSuccess && *word != 0) {
        const unsigned int zero = 0;
        e = cudaMemcpyToSymbol(g_error_word, &zero, sizeof(zero));
    }
    if (e != cudaSuccess) return fail("device_error", e);
    return *word ? TWM_ETIMEOUT : TWM_OK;
}

const char* twm_dense_status_string(int s)
{
    switch (s) {
        case TWM_OK: return "ok";
        case TWM_EINVAL: return "invalid argument";
        case TWM_EWORKSPACE: return "scratch missing or too small";
        case TWM_ELAUNCH: return "CUDA launch or copy failed";
        case TWM_EARCH: return "device is not sm_100 (B200)";
        case TWM_ETIMEOUT: return "a bounded device-side wait expired";
    }
    return "unknown status";
}

const char* twm_dense_last_error(void) { return t_last_error; }

}  // extern "C"
