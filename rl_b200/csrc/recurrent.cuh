// Pieces shared by the kernels of recurrent mixers.
#pragma once
#include "common.cuh"

#include <math.h>

namespace rlb {
__device__ __forceinline__ float rc_ld(const float* p) { return *p; }
__device__ __forceinline__ float rc_ld(const __nv_bfloat16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void rc_st(float* p, float v) { *p = v; }
__device__ __forceinline__ void rc_st(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }
__device__ __forceinline__ float rc_softplus(float x) { return x > 20.f ? x : log1pf(expf(x)); }
}  // namespace rlb
