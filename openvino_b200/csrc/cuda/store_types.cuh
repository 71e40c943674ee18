// Storage types of the kernels that run both in 32-bit (float) and in the serving precision (bf16): arithmetic is always fp32.
#pragma once
#include <cuda_bf16.h>

#include "common.cuh"

namespace ovb {

__device__ __forceinline__ float ld_f32(const float* p) { return *p; }
__device__ __forceinline__ float ld_f32(const __nv_bfloat16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void st_f32(float* p, float v) { *p = v; }
__device__ __forceinline__ void st_f32(__nv_bfloat16* p, float v) { *p = __float2bfloat16_rn(v); }

// Four consecutive elements (16-byte aligned for float, 8-byte aligned for bf16).
__device__ __forceinline__ float4 ld4_f32(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 ld4_f32(const __nv_bfloat16* p) {
    const uint2 r = *reinterpret_cast<const uint2*>(p);
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&r.x));
    const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&r.y));
    return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ void st4_f32(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void st4_f32(__nv_bfloat16* p, float4 v) {
    __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
    uint2 r;
    r.x = *reinterpret_cast<uint32_t*>(&a);
    r.y = *reinterpret_cast<uint32_t*>(&b);
    *reinterpret_cast<uint2*>(p) = r;
}

// Four elements as they lie in memory.
template <class E>
struct Raw4;
template <>
struct Raw4<float> {
    float4 v;
    __device__ __forceinline__ float4 get() const { return v; }
    __device__ __forceinline__ void load(const float* p) { v = *reinterpret_cast<const float4*>(p); }
    __device__ __forceinline__ void set(float4 x) { v = x; }
};
template <>
struct Raw4<__nv_bfloat16> {
    uint2 v;
    __device__ __forceinline__ float4 get() const {
        return make_float4(__uint_as_float(v.x << 16), __uint_as_float(v.x & 0xffff0000u), __uint_as_float(v.y << 16), __uint_as_float(v.y & 0xffff0000u));
    }
    __device__ __forceinline__ void load(const __nv_bfloat16* p) { v = *reinterpret_cast<const uint2*>(p); }
    __device__ __forceinline__ void set(float4 x) { st4_f32(reinterpret_cast<__nv_bfloat16*>(&v), x); }
};

// Host side: call `f` with a value of the element type that `dtype` (OVB_DT_F32 / OVB_DT_BF16) names.
template <class F>
inline int dispatch_store(int dtype, const char* what, F f) {
    if (dtype == OVB_DT_F32) return f(float());
    if (dtype == OVB_DT_BF16) return f(__nv_bfloat16());
    set_error("%s: storage type %d is neither fp32 nor bf16", what, dtype);
    return ERR_UNSUPPORTED;
}

}  // namespace ovb
