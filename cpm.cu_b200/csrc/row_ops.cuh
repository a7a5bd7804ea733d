// Device helpers of the row-wise kernels: typed vector access and sums.
#pragma once
#include "layered.cuh"

namespace {

template <typename T>
__device__ __forceinline__ float to_float(T v);
template <>
__device__ __forceinline__ float to_float<float>(float v) { return v; }
template <>
__device__ __forceinline__ float to_float<bf16>(bf16 v) { return __bfloat162float(v); }
template <typename T>
__device__ __forceinline__ T from_float(float v);
template <>
__device__ __forceinline__ float from_float<float>(float v) { return v; }
template <>
__device__ __forceinline__ bf16 from_float<bf16>(float v) { return __float2bfloat16(v); }

// VEC consecutive elements (8: 16-byte accesses)
template <int VEC, typename T>
__device__ __forceinline__ void load_vec(const T* p, float* f) {
    if constexpr (VEC == 8 && sizeof(T) == 2) {
        const uint4 v = *reinterpret_cast<const uint4*>(p);
        const bf16* e = reinterpret_cast<const bf16*>(&v);
#pragma unroll
        for (int i = 0; i < 8; ++i) f[i] = __bfloat162float(e[i]);
    } else if constexpr (VEC == 8) {
        const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
        f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w;
        f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
    } else {
        f[0] = to_float<T>(*p);
    }
}
template <int VEC, typename T>
__device__ __forceinline__ void store_vec(T* p, const float* f) {
    if constexpr (VEC == 8 && sizeof(T) == 2) {
        uint4 v;
        bf16* e = reinterpret_cast<bf16*>(&v);
#pragma unroll
        for (int i = 0; i < 8; ++i) e[i] = __float2bfloat16(f[i]);
        *reinterpret_cast<uint4*>(p) = v;
    } else if constexpr (VEC == 8) {
        *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]);
        *reinterpret_cast<float4*>(p + 4) = make_float4(f[4], f[5], f[6], f[7]);
    } else {
        *p = from_float<T>(f[0]);
    }
}

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}
// sums of two values over the CTA; sh: 64 floats
__device__ __forceinline__ float2 block_sum2(float a, float b, float* sh) {
    a = warp_sum(a);
    b = warp_sum(b);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
    if (lane == 0) { sh[warp] = a; sh[32 + warp] = b; }
    __syncthreads();
    a = warp_sum(lane < nw ? sh[lane] : 0.f);
    b = warp_sum(lane < nw ? sh[32 + lane] : 0.f);
    return make_float2(a, b);
}

// asks for the cache line at p ahead of its use (weights, before the wait for the previous kernel)
__device__ __forceinline__ void prefetch_l2(const void* p) { asm volatile("prefetch.global.L2 [%0];" ::"l"(p)); }

__device__ __forceinline__ float silu_f32(float v) { return v / (1.f + expf(-v)); }
// of a value that is known to bf16 precision only: the approximate exponential and division are far finer than that
__device__ __forceinline__ float silu_fast(float v) { return __fdividef(v, 1.f + __expf(-v)); }
template <typename T>
__device__ __forceinline__ float silu_of(float v) { return sizeof(T) == 2 ? silu_fast(v) : silu_f32(v); }

// ---- pairs of fp32 for the packed instructions
typedef unsigned long long f32x2;
__device__ __forceinline__ f32x2 pair(float lo, float hi) {
    f32x2 r;
    asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(lo), "f"(hi));
    return r;
}
__device__ __forceinline__ float2 unpair(f32x2 p) {
    float2 f;
    asm("mov.b64 {%0, %1}, %2;" : "=f"(f.x), "=f"(f.y) : "l"(p));
    return f;
}
__device__ __forceinline__ f32x2 fma2(f32x2 a, f32x2 b, f32x2 c) {
    f32x2 d;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
    return d;
}
__device__ __forceinline__ f32x2 mul2(f32x2 a, f32x2 b) {
    f32x2 d;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
    return d;
}

}  // namespace
