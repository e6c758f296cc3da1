// twm_dense_latent.cuh — latent attention: per token the cache holds one normed latent (all heads' keys and
// values are linear maps of it) and one rotated key part that all heads share.
//
// A step of several tokens expands the latents its queries can see into keys and values (one product), and
// attends with ordinary softmax attention: plain tiles here, tcgen05 in twm_dense_softmax_tc.cuh.  A decoded
// token goes the other way: the query is mapped into latent space, so the cache is read as it lies.
#pragma once

#include "twm_dense_rows.cuh"
#include "twm_dense_simt.cuh"

namespace twm {
namespace dense {

// (u, v) = elements 2i and 2i + 1 turned by the angle whose (cos, sin) is cs
__device__ __forceinline__ float2 rotate_pair(const float2 uv, const float2 cs) {
    return make_float2(uv.x * cs.x - uv.y * cs.y, uv.y * cs.x + uv.x * cs.y);
}

// Prompt steps.  CTAs 0 .. rows - 1 take a new token each: its latent is normed and its shared key part rotated, into
// the cache and into `lat`, where the step's visible tokens stand in order; its heads' rotated query parts are
// turned in place.  The CTAs after them copy the older visible tokens from the cache to `lat`.
template <typename T>
struct LatentRowsArgs {
    T* proj;                    // [rows][ld]: per head [dim_pad | rot_pad], then latent, shared key part
    T* cache;                   // [slots][capacity][rank_pad + rot_pad]
    T* lat;                     // [older + rows][rank_pad + rot_pad]
    const float* norm;          // [rank_pad]
    const float2* rot_table;    // [positions][rot_pad / 2] (cos, sin)
    const int* meta;
    int ld, heads, dim_pad, rot_pad, rank, rank_pad, capacity, rows, older;
    float eps;
};
template <typename T>
__global__ void __launch_bounds__(ROW_THREADS)
latent_rows_kernel(const LatentRowsArgs<T> g)
{
    __shared__ float red[32];
    pdl_wait_prior_grids();
    pdl_launch_dependents();
    const int width = g.rank_pad + g.rot_pad, pos0 = g.meta[0];
    T* cache = g.cache + (size_t)g.meta[1] * g.capacity * width;
    if ((int)blockIdx.x >= g.rows) {
        const int i = (int)blockIdx.x - g.rows;             // older token: position pos0 - older + i
        const uint4* src = reinterpret_cast<const uint4*>(cache + (size_t)(pos0 - g.older + i) * width);
        uint4* dst = reinterpret_cast<uint4*>(g.lat + (size_t)i * width);
        for (int c = threadIdx.x; c < width * (int)sizeof(T) / 16; c += ROW_THREADS) dst[c] = src[c];
        return;
    }
    const int r = blockIdx.x, p = pos0 + r;
    T* row = g.proj + (size_t)r * g.ld;
    const int qw = g.dim_pad + g.rot_pad, half = g.rot_pad / 2;
    T* down = row + g.heads * qw;
    T* to_cache = cache + (size_t)p * width;
    T* to_lat = g.lat + (size_t)(g.older + r) * width;
    const float2* cs = g.rot_table + (size_t)p * half;
    float ss = 0.0f;
    for (int i = threadIdx.x; i < g.rank_pad; i += ROW_THREADS) { const float v = to_f32(down[i]); ss = fmaf(v, v, ss); }
    const float ir = inv_rms(group_sum(ss, red, ROW_THREADS, 1), g.rank, g.eps);
    for (int i = threadIdx.x; i < g.rank_pad; i += ROW_THREADS) {
        const T v = from_f32<T>(to_f32(down[i]) * ir * __ldg(g.norm + i));
        to_cache[i] = v;
        to_lat[i] = v;
    }
    for (int i = threadIdx.x; i < half; i += ROW_THREADS) {
        const T* k = down + g.rank_pad + 2 * i;
        const float2 o = rotate_pair(make_float2(to_f32(k[0]), to_f32(k[1])), cs[i]);
        const T a = from_f32<T>(o.x), b = from_f32<T>(o.y);
        to_cache[g.rank_pad + 2 * i] = a; to_cache[g.rank_pad + 2 * i + 1] = b;
        to_lat[g.rank_pad + 2 * i] = a; to_lat[g.rank_pad + 2 * i + 1] = b;
    }
    for (int i = threadIdx.x; i < g.heads * half; i += ROW_THREADS) {
        const int h = i / half, j = i - h * half;
        T* q = row + h * qw + g.dim_pad + 2 * j;
        const float2 o = rotate_pair(make_float2(to_f32(q[0]), to_f32(q[1])), cs[j]);
        q[0] = from_f32<T>(o.x);
        q[1] = from_f32<T>(o.y);
    }
}

// What a softmax attention launch over expanded keys reads.  Key j of the step's visible tokens stands in row j - first_key.
template <typename T>
struct SoftmaxArgs {
    const T* proj;              // [rows][ld]: per head [dim_pad | rot_pad] queries
    const T* kv;                // [keys][heads * dim_pad | heads * vdim_pad]
    const T* shared;            // [keys][shared_ld]: the key part all heads share, rot_pad columns
    T* out;                     // [rows][heads * vdim_pad]
    int ld, gate_off;           // one gate per head at proj[row][gate_off + h]; < 0: none
    int shared_ld, heads, dim_pad, rot_pad, vdim_pad, window, rows;
    int first_pos, first_key;
    float scale;
};

// One query of one head per CTA: scores one key per thread, 128 keys at a time with a running maximum, threads
// along the value columns (grid z: blocks of 512).
template <typename T>
__global__ void __launch_bounds__(AS_THREADS)
attn_softmax_simt_kernel(const SoftmaxArgs<T> g)
{
    using V = Vec<T>;
    extern __shared__ __align__(16) float attn_smem[];
    __shared__ float red[32];
    const int qw = g.dim_pad + g.rot_pad;
    float* qs = attn_smem;                      // [dim_pad + rot_pad]
    float* ws = qs + qw;                        // [AS_THREADS]
    pdl_wait_prior_grids();
    pdl_launch_dependents();
    const int r = blockIdx.x, h = blockIdx.y, p = g.first_pos + r;
    const int kv_ld = g.heads * (g.dim_pad + g.vdim_pad);
    const T* k_base = g.kv + h * g.dim_pad;
    const T* v_base = g.kv + g.heads * g.dim_pad + h * g.vdim_pad;
    for (int d = threadIdx.x; d < qw; d += AS_THREADS) qs[d] = to_f32(g.proj[(size_t)r * g.ld + h * qw + d]);
    const int lo = g.window > p ? 0 : p - g.window + 1;
    const int c0 = blockIdx.z * AS_VPT * AS_THREADS + threadIdx.x;
    float acc[AS_VPT] = {};
    float m = -INFINITY, l = 0.0f;
    for (int t0 = lo; t0 <= p; t0 += AS_THREADS) {
        __syncthreads();                        // qs written / the previous chunk's weights read
        const int j = t0 + threadIdx.x;
        float s = -INFINITY;
        if (j <= p) {
            const uint4* kr = reinterpret_cast<const uint4*>(k_base + (size_t)(j - g.first_key) * kv_ld);
            const uint4* sr = reinterpret_cast<const uint4*>(g.shared + (size_t)(j - g.first_key) * g.shared_ld);
            s = 0.0f;
            for (int d = 0; d < g.dim_pad / V::N; ++d) {
                float f[V::N];
                V::unpack(kr[d], f);
#pragma unroll
                for (int e = 0; e < V::N; ++e) s = fmaf(f[e], qs[d * V::N + e], s);
            }
            for (int d = 0; d < g.rot_pad / V::N; ++d) {
                float f[V::N];
                V::unpack(sr[d], f);
#pragma unroll
                for (int e = 0; e < V::N; ++e) s = fmaf(f[e], qs[g.dim_pad + d * V::N + e], s);
            }
            s *= g.scale;
        }
        // every thread keeps the maximum of the whole chunk
        float cm = ops::warp_max(s);
        if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = cm;
        __syncthreads();
        cm = fmaxf(fmaxf(red[0], red[1]), fmaxf(red[2], red[3]));
        const float m_new = fmaxf(m, cm), before = expf(m - m_new);
        m = m_new;
        ws[threadIdx.x] = expf(s - m);
        __syncthreads();
        const int n = min(AS_THREADS, p + 1 - t0);
        l *= before;
#pragma unroll
        for (int i = 0; i < AS_VPT; ++i) acc[i] *= before;
        for (int tt = 0; tt < n; ++tt) {
            const float pw = ws[tt];
            const T* v = v_base + (size_t)(t0 + tt - g.first_key) * kv_ld;
            l += pw;
#pragma unroll
            for (int i = 0; i < AS_VPT; ++i) {
                const int d = c0 + i * AS_THREADS;
                if (d < g.vdim_pad) acc[i] = fmaf(pw, to_f32(v[d]), acc[i]);
            }
        }
    }
    const float gate = g.gate_off >= 0 ? sigmoid_f32(to_f32(g.proj[(size_t)r * g.ld + g.gate_off + h])) : 1.0f;
#pragma unroll
    for (int i = 0; i < AS_VPT; ++i) {
        const int d = c0 + i * AS_THREADS;
        if (d < g.vdim_pad) g.out[(size_t)r * g.heads * g.vdim_pad + h * g.vdim_pad + d] = from_f32<T>(acc[i] / l * gate);
    }
}

// One decoded token.  A cluster of CTAs per head: each maps a share of the query into latent space (W_uk^T q, pushed to
// the whole cluster), scores a share of the visible latents, and pushes its partial (maximum, sum, weighted latents) to
// all; then each makes a share of the head's value columns (W_uv times the combined latent) and gates them.  The
// CTA with the newest token norms and rotates it for itself; head 0's also appends it to the cache.
constexpr int LD_THREADS = 256, LD_MAX_SPLITS = 8, LD_MAX_CHUNK = 128;

template <typename T>
struct LatentDecodeArgs {
    const float* proj;          // f32: per head [dim_pad | rot_pad], latent, shared key part, one gate per head
    float* out;                 // f32 [heads * vdim_pad]
    const T* w_expand;          // [heads * dim_pad | heads * vdim_pad][rank_pad]
    const float* norm;
    const float2* rot_table;
    T* cache;
    const int* meta;
    int heads, dim_pad, rot_pad, rank, rank_pad, vdim_pad, window, capacity;
    int chunk;                  // tokens in shared memory at a time
    int parts;                  // threads that share the tokens of one column quad
    float scale, eps;
};

__host__ __device__ inline int latent_decode_slice(int rank_pad, int splits) { return ((rank_pad + splits - 1) / splits + 7) / 8 * 8; }
__host__ inline int latent_decode_parts(int rank_pad) {
    const int n = LD_THREADS / (rank_pad / 4);
    return n < 1 ? 1 : n > 8 ? 8 : n;
}
// floats in front of the token rows
__host__ __device__ inline int latent_decode_floats(int dim_pad, int rot_pad, int rank_pad, int chunk, int parts, int splits) {
    const int width = rank_pad + rot_pad;
    const int absorb = LD_THREADS * 8;                      // partial sums of the query's map: at most 8 columns a thread
    const int share = parts * rank_pad > absorb ? parts * rank_pad : absorb;
    return dim_pad + width + chunk + share + splits * rank_pad + 2 * LD_MAX_SPLITS;
}
template <typename T>
__host__ inline size_t latent_decode_smem_bytes(int dim_pad, int rot_pad, int rank_pad, int chunk, int parts, int splits) {
    return sizeof(float) * (size_t)latent_decode_floats(dim_pad, rot_pad, rank_pad, chunk, parts, splits) +
           (size_t)chunk * ((rank_pad + rot_pad) * sizeof(T) + 16);
}
__device__ __forceinline__ void st_cluster_f32x4(uint32_t cluster_addr, const float4 v) {
    asm volatile("st.shared::cluster.v4.f32 [%0], {%1, %2, %3, %4};" ::"r"(cluster_addr), "f"(v.x), "f"(v.y), "f"(v.z), "f"(v.w) : "memory");
}

template <typename T>
__global__ void __launch_bounds__(LD_THREADS)
latent_decode_kernel(const LatentDecodeArgs<T> g)
{
    using V = Vec<T>;
    pdl_launch_dependents();
    asm volatile("barrier.cluster.arrive.relaxed.aligned;" ::: "memory");      // waited for before the first push
    extern __shared__ __align__(16) float ld_smem[];
    __shared__ float red[32];
    const int splits = gridDim.x, rank = blockIdx.x, h = blockIdx.y;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int width = g.rank_pad + g.rot_pad, qw = g.dim_pad + g.rot_pad, half = g.rot_pad / 2;
    const int slice = latent_decode_slice(g.rank_pad, splits);
    float* qu = ld_smem;                                   // [dim_pad] the head's unrotated query
    float* qa = qu + g.dim_pad;                            // [width] the query against a cache row
    float* ws = qa + width;                                // [chunk]
    float* os = ws + g.chunk;                              // [parts][rank_pad]; before that, partial sums of the query's map
    const int share = max(g.parts * g.rank_pad, LD_THREADS * 8);
    float* recv = os + share;                              // [splits][rank_pad] the cluster's weighted latents
    float* recv_ml = recv + splits * g.rank_pad;           // [splits][2] their maxima and sums
    uint8_t* rows = reinterpret_cast<uint8_t*>(recv_ml + 2 * LD_MAX_SPLITS);
    const int row_bytes = width * (int)sizeof(T), stride = row_bytes + 16;     // a padded row: keys start in distinct banks
    const int pieces = row_bytes / 16;
    // What this CTA will read, into L2 while the kernel before runs.  Position and slot are read as they are now: a stale one
    // prefetches other rows of the cache.
    const int first = rank * slice, own = min(slice, g.rank_pad - first);          // this CTA's latent columns; own may be <= 0
    const int per_cta = (g.vdim_pad + splits - 1) / splits;
    const T* w_uk = g.w_expand + (size_t)h * g.dim_pad * g.rank_pad + first;
    const T* w_uv = g.w_expand + (size_t)g.heads * g.dim_pad * g.rank_pad + (size_t)h * g.vdim_pad * g.rank_pad;
    if (own > 0)
        for (int i = tid; i < g.dim_pad; i += LD_THREADS)
            for (int c = 0; c < own * (int)sizeof(T); c += 128) l2_prefetch(reinterpret_cast<const uint8_t*>(w_uk + (size_t)i * g.rank_pad) + c);
    for (int e = rank * per_cta + tid; e < min(g.vdim_pad, (rank + 1) * per_cta); e += LD_THREADS)
        l2_prefetch_bulk(w_uv + (size_t)e * g.rank_pad, (uint32_t)(g.rank_pad * sizeof(T)));
    if (h == 0) {
        const int now = min(max(*(volatile const int*)g.meta, 0), g.capacity - 1), from = max(0, now - g.window + 1), share_now = (now - from) / splits + 1;
        const T* rows_now = g.cache + (size_t)*(volatile const int*)(g.meta + 1) * g.capacity * width;
        for (int i = tid; i < share_now; i += LD_THREADS) {
            const int j = from + rank * share_now + i;
            if (j < now) l2_prefetch_bulk(rows_now + (size_t)j * width, (uint32_t)row_bytes);
        }
    }
    pdl_wait_prior_grids();
    const int p = g.meta[0];
    T* cache = g.cache + (size_t)g.meta[1] * g.capacity * width;
    const int lo = g.window > p ? 0 : p - g.window + 1;
    const int total = p - lo + 1, per = (total + splits - 1) / splits;
    const int t_begin = min(total, rank * per), t_end = min(total, t_begin + per);
    const bool newest = t_begin < t_end && t_end == total;
    auto load_share = [&](int t0, int n) {                 // all but the newest token, which is not in the cache yet
        for (int i = tid; i < n * pieces; i += LD_THREADS) {
            const int r = i / pieces, c = i - r * pieces, j = lo + t0 + r;
            if (j < p) ops::att_cp_async16(smem_u32(rows + (size_t)r * stride + c * 16), cache + (size_t)j * width + c * V::N, 16);
        }
        ops::att_cp_async_commit();
    };
    load_share(t_begin, min(g.chunk, t_end - t_begin));

    // ---- the query: rotated part, and this CTA's share of the mapped part ----
    const float* q = g.proj + h * qw;
    for (int d = tid; d < g.dim_pad; d += LD_THREADS) qu[d] = q[d];
    for (int i = tid; i < half; i += LD_THREADS) {
        const float2 o = rotate_pair(make_float2(q[g.dim_pad + 2 * i], q[g.dim_pad + 2 * i + 1]), g.rot_table[(size_t)p * half + i]);
        qa[g.rank_pad + 2 * i] = o.x * g.scale;
        qa[g.rank_pad + 2 * i + 1] = o.y * g.scale;
    }
    __syncthreads();
    asm volatile("barrier.cluster.wait.aligned;" ::: "memory");    // every CTA of the cluster has started
    {
        const int vecs = own > 0 ? (own + V::N - 1) / V::N : 1;
        const int vpp = min(vecs, LD_THREADS);                     // column vectors at a time
        const int groups = max(1, LD_THREADS / vpp);
        for (int v0 = 0; v0 * V::N < own; v0 += vpp) {
            const int vi = v0 + tid % vpp, dg = tid / vpp;
            float acc[V::N] = {};
            if (dg < groups && vi < vecs) {
                const T* w = w_uk + vi * V::N;
#pragma unroll 4
                for (int d = dg; d < g.dim_pad; d += groups) {
                    float f[V::N];
                    V::unpack(__ldg(reinterpret_cast<const uint4*>(w + (size_t)d * g.rank_pad)), f);
                    const float qd = qu[d];
#pragma unroll
                    for (int e = 0; e < V::N; ++e) acc[e] = fmaf(f[e], qd, acc[e]);
                }
            }
            if (dg < groups) {
#pragma unroll
                for (int e = 0; e < V::N; ++e) os[(dg * vpp + tid % vpp) * V::N + e] = acc[e];
            }
            __syncthreads();
            for (int i = tid; i < vpp * V::N; i += LD_THREADS) {
                const int col = v0 * V::N + i;
                float s = 0.0f;
                for (int k = 0; k < groups; ++k) s += os[k * vpp * V::N + i];
                if (col < own)
                    for (int c = 0; c < splits; ++c) st_cluster_f32(mapa_shared(smem_u32(qa + first + col), c), s * g.scale);
            }
            __syncthreads();
        }
    }
    // ---- the newest token ----
    float kir = 1.0f;
    const float* down = g.proj + g.heads * qw;
    if (newest) {
        float ss = 0.0f;
        for (int i = tid; i < g.rank_pad; i += LD_THREADS) ss = fmaf(down[i], down[i], ss);
        kir = inv_rms(group_sum(ss, red, LD_THREADS, 1), g.rank, g.eps);
    }
    for (int i = tid; i < share; i += LD_THREADS) os[i] = 0.0f;
    cluster_sync_all();                                            // the whole mapped query is here

    float m = -INFINITY, l = 0.0f;
    for (int t0 = t_begin; t0 < t_end; t0 += g.chunk) {
        const int n = min(g.chunk, t_end - t0);
        if (t0 > t_begin) {
            __syncthreads();                                       // the chunk before has been used
            load_share(t0, n);
        }
        if (newest && t0 + n == t_end) {
            T* mine = reinterpret_cast<T*>(rows + (size_t)(n - 1) * stride);
            T* kept = h == 0 && p < g.capacity ? cache + (size_t)p * width : nullptr;
            for (int i = tid; i < g.rank_pad; i += LD_THREADS) {
                const T v = from_f32<T>(down[i] * kir * __ldg(g.norm + i));
                mine[i] = v;
                if (kept != nullptr) kept[i] = v;
            }
            for (int i = tid; i < half; i += LD_THREADS) {
                const float* k = down + g.rank_pad + 2 * i;
                const float2 o = rotate_pair(make_float2(k[0], k[1]), g.rot_table[(size_t)p * half + i]);
                const T a = from_f32<T>(o.x), b = from_f32<T>(o.y);
                mine[g.rank_pad + 2 * i] = a; mine[g.rank_pad + 2 * i + 1] = b;
                if (kept != nullptr) { kept[g.rank_pad + 2 * i] = a; kept[g.rank_pad + 2 * i + 1] = b; }
            }
        }
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();
        // scores: eight lanes a token
        for (int t = tid >> 3; t < ((n + 31) & ~31); t += LD_THREADS / 8) {
            float s = 0.0f;
            if (t < n) {
                const uint8_t* row = rows + (size_t)t * stride;
#pragma unroll 3
                for (int c = lane & 7; c < pieces; c += 8) {
                    float f[V::N];
                    V::unpack(lds128(row + c * 16), f);
#pragma unroll
                    for (int e = 0; e < V::N; e += 4) {
                        const float4 qv = *reinterpret_cast<const float4*>(qa + c * V::N + e);
                        s = fmaf(f[e], qv.x, fmaf(f[e + 1], qv.y, fmaf(f[e + 2], qv.z, fmaf(f[e + 3], qv.w, s))));
                    }
                }
            }
#pragma unroll
            for (int d = 4; d > 0; d >>= 1) s += __shfl_xor_sync(0xffffffffu, s, d);
            if (t < n && (lane & 7) == 0) ws[t] = s;
        }
        __syncthreads();
        float cm = -INFINITY;
        for (int t = lane; t < n; t += 32) cm = fmaxf(cm, ws[t]);
        cm = ops::warp_max(cm);                                    // every warp: the same maximum
        const float m_new = fmaxf(m, cm), before = expf(m - m_new);
        __syncthreads();
        for (int t = tid; t < n; t += LD_THREADS) ws[t] = expf(ws[t] - m_new);
        __syncthreads();
        float cl = 0.0f;
        for (int t = lane; t < n; t += 32) cl += ws[t];
        l = l * before + ops::warp_sum(cl);
        m = m_new;
        const int quads = g.rank_pad / 4;
        for (int i = tid; i < quads * g.parts; i += LD_THREADS) {
            const int part = i / quads, c = (i - part * quads) * 4;
            float o0 = 0.f, o1 = 0.f, o2 = 0.f, o3 = 0.f;
#pragma unroll 8
            for (int t = part; t < n; t += g.parts) {
                const float4 vf = load4(reinterpret_cast<const T*>(rows + (size_t)t * stride) + c);
                const float w = ws[t];
                o0 = fmaf(w, vf.x, o0); o1 = fmaf(w, vf.y, o1); o2 = fmaf(w, vf.z, o2); o3 = fmaf(w, vf.w, o3);
            }
            float4* o = reinterpret_cast<float4*>(os + part * g.rank_pad + c);          // this thread's own columns
            const float4 b = *o;
            *o = make_float4(fmaf(b.x, before, o0), fmaf(b.y, before, o1), fmaf(b.z, before, o2), fmaf(b.w, before, o3));
        }
    }
    __syncthreads();
    for (int i = tid; i < g.rank_pad / 4; i += LD_THREADS) {
        float4 o = reinterpret_cast<const float4*>(os)[i];
        for (int part = 1; part < g.parts; ++part) {
            const float4 b = reinterpret_cast<const float4*>(os + part * g.rank_pad)[i];
            o.x += b.x; o.y += b.y; o.z += b.z; o.w += b.w;
        }
        for (int c = 0; c < splits; ++c) st_cluster_f32x4(mapa_shared(smem_u32(recv + rank * g.rank_pad + i * 4), c), o);
    }
    if (tid < splits) {
        st_cluster_f32(mapa_shared(smem_u32(recv_ml + rank * 2), tid), m);
        st_cluster_f32(mapa_shared(smem_u32(recv_ml + rank * 2 + 1), tid), l);
    }
    cluster_sync_all();
    // ---- the combined latent, over qa, then this CTA's value columns ----
    float top = -INFINITY, sum = 0.0f;
    for (int s = 0; s < splits; ++s) top = fmaxf(top, recv_ml[2 * s]);
    for (int s = 0; s < splits; ++s) sum += recv_ml[2 * s + 1] * expf(recv_ml[2 * s] - top);
    for (int i = tid; i < g.rank_pad; i += LD_THREADS) {
        float o = 0.0f;
        for (int s = 0; s < splits; ++s) o = fmaf(expf(recv_ml[2 * s] - top), recv[s * g.rank_pad + i], o);
        qa[i] = o / sum;
    }
    __syncthreads();
    const float gate = sigmoid_f32(g.proj[g.heads * qw + width + h]);
    for (int e = rank * per_cta + warp; e < min(g.vdim_pad, (rank + 1) * per_cta); e += LD_THREADS / 32) {
        float s = 0.0f;
        for (int c = lane; c < g.rank_pad / V::N; c += 32) {
            float f[V::N];
            V::unpack(__ldg(reinterpret_cast<const uint4*>(w_uv + (size_t)e * g.rank_pad) + c), f);
#pragma unroll
            for (int k = 0; k < V::N; ++k) s = fmaf(f[k], qa[c * V::N + k], s);
        }
        s = ops::warp_sum(s);
        if (lane == 0) g.out[h * g.vdim_pad + e] = s * gate;
    }
}

}  // namespace dense
}  // namespace twm
