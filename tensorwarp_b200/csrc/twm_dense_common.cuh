// twm_dense_common.cuh — element types, reductions and activations shared by the dense-weight kernels.
#pragma once

#include <cuda_bf16.h>

#include "../../include/twm_dense.h"
#include "twm_common.cuh"
#include "twm_decode_ops.cuh"

namespace twm {
namespace dense {

using bf16 = __nv_bfloat16;

__device__ __forceinline__ float to_f32(float v) { return v; }
__device__ __forceinline__ float to_f32(bf16 v) { return __bfloat162float(v); }
template <typename T> __device__ __forceinline__ T from_f32(float v);
template <> __device__ __forceinline__ float from_f32<float>(float v) { return v; }
template <> __device__ __forceinline__ bf16 from_f32<bf16>(float v) { return __float2bfloat16_rn(v); }

// 16 bytes of T (8 bf16 or 4 f32) as floats
template <typename T> struct Vec;
template <> struct Vec<bf16> {
    static constexpr int N = 8;
    static __device__ __forceinline__ void unpack(const uint4& v, float (&f)[8]) {
        const uint32_t w[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            f[2 * i] = __uint_as_float(w[i] << 16);
            f[2 * i + 1] = __uint_as_float(w[i] & 0xffff0000u);
        }
    }
    static __device__ __forceinline__ uint4 pack(const float (&f)[8]) {
        uint4 o;
        uint32_t* w = &o.x;
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const __nv_bfloat162 h = __floats2bfloat162_rn(f[2 * i], f[2 * i + 1]);
            w[i] = *reinterpret_cast<const uint32_t*>(&h);
        }
        return o;
    }
};
template <> struct Vec<float> {
    static constexpr int N = 4;
    static __device__ __forceinline__ void unpack(const uint4& v, float (&f)[4]) {
        f[0] = __uint_as_float(v.x); f[1] = __uint_as_float(v.y); f[2] = __uint_as_float(v.z); f[3] = __uint_as_float(v.w);
    }
    static __device__ __forceinline__ uint4 pack(const float (&f)[4]) {
        return make_uint4(__float_as_uint(f[0]), __float_as_uint(f[1]), __float_as_uint(f[2]), __float_as_uint(f[3]));
    }
};

__device__ __forceinline__ float gelu_tanh(float z) {
    const float u = 0.7978845608028654f * fmaf(0.044715f * z * z, z, z);
    return 0.5f * z * (1.0f + tanhf(u));
}
__device__ __forceinline__ float sigmoid_f32(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float silu_f32(float z) { return z * sigmoid_f32(z); }
__device__ __forceinline__ float log_sigmoid_f32(float z) { return fminf(z, 0.0f) - log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float squared_relu(float z) { const float p = fmaxf(z, 0.0f); return p * p; }
// what a product's epilogue does to a single sum
template <int EPI>
__device__ __forceinline__ float epilogue_value(float v) { return EPI == TWM_EPI_RELU2 ? squared_relu(v) : v; }

// Sum over the `threads` threads (a multiple of 32, all taking part) that share named barrier `bar`; `red` holds 32
// floats.  Every thread gets the sum, added in warp order.
__device__ __forceinline__ float group_sum(float v, float* red, int threads, int bar) {
    v = ops::warp_sum(v);
    named_bar_sync(bar, threads);                       // `red` may still be read from the sum before
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
    named_bar_sync(bar, threads);
    float t = 0.0f;
    for (int w = 0; w < (threads >> 5); ++w) t += red[w];
    return t;
}
__device__ __forceinline__ float inv_rms(float sumsq, int n, float eps) { return 1.0f / sqrtf(sumsq / (float)n + eps); }

// True in one lane of a converged warp.  Code under it is known to run in one thread, which the tensor-core and TMA
// instructions (uniform operands) issue faster from than from a lane-number test.
__device__ __forceinline__ bool elect_one() {
    uint32_t p;
    asm volatile("{\n\t.reg .pred p;\n\telect.sync _|p, 0xffffffff;\n\tselp.u32 %0, 1, 0, p;\n\t}" : "=r"(p));
    return p != 0;
}

__device__ __forceinline__ void l2_prefetch(const void* p) { asm volatile("prefetch.global.L2 [%0];" ::"l"(p) : "memory"); }

// Ask for a tensor map (kernel-parameter space) ahead of the first load that uses it.
__device__ __forceinline__ void prefetch_map(const CUtensorMap* map) {
    asm volatile("prefetch.tensormap [%0];" ::"l"(reinterpret_cast<uint64_t>(map)) : "memory");
}

// Which keys the query at position p sees: [0, sinks) and [lo, p].
__device__ __forceinline__ void visible_range(int p, int window, int keep_first, int& sinks, int& lo) {
    lo = window > p ? 0 : p - window + 1;               // p - j < window
    sinks = min(keep_first, lo);
}

}  // namespace dense
}  // namespace twm
