// Elements of either activation type (bf16 when serving, float on the 32-bit path) read and written as floats.
#pragma once
#include "common.cuh"

namespace pie {

template <typename T> __device__ __forceinline__ float to_f(T v);
template <> __device__ __forceinline__ float to_f<float>(float v) { return v; }
template <> __device__ __forceinline__ float to_f<bf16>(bf16 v) { return __bfloat162float(v); }
template <typename T> __device__ __forceinline__ T from_f(float v);
template <> __device__ __forceinline__ float from_f<float>(float v) { return v; }
template <> __device__ __forceinline__ bf16 from_f<bf16>(float v) { return __float2bfloat16(v); }

// VEC consecutive elements as floats (VEC 4: one 8- or 16-byte access)
template <int VEC, typename T>
__device__ __forceinline__ void load_vec(const T* p, float (&f)[VEC]) {
    if constexpr (VEC == 1) {
        f[0] = to_f(*p);
    } else if constexpr (sizeof(T) == 4) {
        const float4 v = *reinterpret_cast<const float4*>(p);
        f[0] = v.x; f[1] = v.y; f[2] = v.z; f[3] = v.w;
    } else {
        const uint2 v = *reinterpret_cast<const uint2*>(p);
        const float2 a = __bfloat1622float2(*reinterpret_cast<const bf162*>(&v.x));
        const float2 b = __bfloat1622float2(*reinterpret_cast<const bf162*>(&v.y));
        f[0] = a.x; f[1] = a.y; f[2] = b.x; f[3] = b.y;
    }
}
template <int VEC, typename T>
__device__ __forceinline__ void store_vec(T* p, const float (&f)[VEC]) {
    if constexpr (VEC == 1) {
        *p = from_f<T>(f[0]);
    } else if constexpr (sizeof(T) == 4) {
        *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]);
    } else {
        const bf162 a = __floats2bfloat162_rn(f[0], f[1]), b = __floats2bfloat162_rn(f[2], f[3]);
        *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&a), *reinterpret_cast<const uint32_t*>(&b));
    }
}

}  // namespace pie
