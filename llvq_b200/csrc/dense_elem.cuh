// Element types of the dense-weight path: bf16 (serving) and f32 (the exact path). A kernel is written once
// over T; loads widen to f32, stores round to nearest once.
#pragma once
#include <cuda_bf16.h>

#include <cstdint>

#include "warp_reduce.cuh"

namespace llvq {

using bf16 = __nv_bfloat16;

__device__ __forceinline__ float to_f32(float v) { return v; }
__device__ __forceinline__ float to_f32(bf16 v) { return __bfloat162float(v); }
template <typename T>
__device__ __forceinline__ T from_f32(float v);
template <>
__device__ __forceinline__ float from_f32<float>(float v) { return v; }
template <>
__device__ __forceinline__ bf16 from_f32<bf16>(float v) { return __float2bfloat16_rn(v); }

// Elements of T in a 16-byte vector, and the vector widened.
template <typename T>
struct Vec16;
template <>
struct Vec16<bf16> {
    static constexpr int N = 8;
    static __device__ __forceinline__ void widen(const uint4& u, float (&f)[8]) {
        const unsigned int w[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            f[2 * i] = __uint_as_float(w[i] << 16);
            f[2 * i + 1] = __uint_as_float(w[i] & 0xffff0000u);
        }
    }
    static __device__ __forceinline__ uint4 narrow(const float (&f)[8]) {
        unsigned int w[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const __nv_bfloat162 v = __floats2bfloat162_rn(f[2 * i], f[2 * i + 1]);
            w[i] = *reinterpret_cast<const unsigned int*>(&v);
        }
        return make_uint4(w[0], w[1], w[2], w[3]);
    }
};
template <>
struct Vec16<float> {
    static constexpr int N = 4;
    static __device__ __forceinline__ void widen(const uint4& u, float (&f)[4]) {
        f[0] = __uint_as_float(u.x), f[1] = __uint_as_float(u.y), f[2] = __uint_as_float(u.z), f[3] = __uint_as_float(u.w);
    }
    static __device__ __forceinline__ uint4 narrow(const float (&f)[4]) {
        return make_uint4(__float_as_uint(f[0]), __float_as_uint(f[1]), __float_as_uint(f[2]), __float_as_uint(f[3]));
    }
};
// A vector at p (16-byte aligned), widened, and back.
template <typename T>
__device__ __forceinline__ void load_vec(const T* p, float (&f)[Vec16<T>::N]) { Vec16<T>::widen(*reinterpret_cast<const uint4*>(p), f); }
template <typename T>
__device__ __forceinline__ void store_vec(T* p, const float (&f)[Vec16<T>::N]) { *reinterpret_cast<uint4*>(p) = Vec16<T>::narrow(f); }

// Four consecutive values as f32 and back.
template <typename T>
__device__ __forceinline__ float4 load4(const T* p) {
    if constexpr (sizeof(T) == 4) {
        return *reinterpret_cast<const float4*>(p);
    } else {
        const uint2 u = *reinterpret_cast<const uint2*>(p);
        return make_float4(__uint_as_float(u.x << 16), __uint_as_float(u.x & 0xffff0000u), __uint_as_float(u.y << 16), __uint_as_float(u.y & 0xffff0000u));
    }
}
template <typename T>
__device__ __forceinline__ void store4(T* p, float4 v) {
    if constexpr (sizeof(T) == 4) {
        *reinterpret_cast<float4*>(p) = v;
    } else {
        __align__(16) const T r[4] = {from_f32<T>(v.x), from_f32<T>(v.y), from_f32<T>(v.z), from_f32<T>(v.w)};
        *reinterpret_cast<uint2*>(p) = *reinterpret_cast<const uint2*>(r);
    }
}

// Sum over the CTA, the same value in every thread. `red` holds one float per warp; two barriers.
__device__ __forceinline__ float block_sum_f(float v, float* red) {
    v = warp_sum_f(v);
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
    __syncthreads();
    float t = 0.0f;
    for (int w = 0; w < (int)(blockDim.x >> 5); ++w) t += red[w];
    __syncthreads();
    return t;
}

// Clamped gated unit: g = min(gate, limit), u = clamp(up, -limit, limit); g * sigmoid(gain * g) * (u + shift).
__device__ __forceinline__ float clamped_glu(float gate, float up, float limit, float gain, float shift) {
    const float g = fminf(gate, limit), u = fminf(fmaxf(up, -limit), limit);
    return g / (1.0f + expf(-gain * g)) * (u + shift);
}

}  // namespace llvq
