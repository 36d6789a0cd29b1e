// Eight-element loads and stores as fp32 for kernels that exist for bf16 and fp32 activations.
#pragma once
#include "common.cuh"

typedef __nv_bfloat16 bf16;

__device__ __forceinline__ void load8(const bf16* p, float* f) { unpack8(ld8(p), f); }
__device__ __forceinline__ void load8(const float* p, float* f) {
    *reinterpret_cast<float4*>(f) = *reinterpret_cast<const float4*>(p);
    *reinterpret_cast<float4*>(f + 4) = *reinterpret_cast<const float4*>(p + 4);
}
__device__ __forceinline__ void store8(bf16* p, const float* f) { st8(p, pack8(f)); }
__device__ __forceinline__ void store8(float* p, const float* f) {
    *reinterpret_cast<float4*>(p) = *reinterpret_cast<const float4*>(f);
    *reinterpret_cast<float4*>(p + 4) = *reinterpret_cast<const float4*>(f + 4);
}
__device__ __forceinline__ float to_float(bf16 v) { return __bfloat162float(v); }
__device__ __forceinline__ float to_float(float v) { return v; }
__device__ __forceinline__ void from_float(bf16* p, float v) { *p = __float2bfloat16(v); }
__device__ __forceinline__ void from_float(float* p, float v) { *p = v; }
