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
__device__ __forceinline__ float rc_silu(float x) { return x / (1.f + expf(-x)); }

// For activations that are rounded to bf16 right away (the approximate exponential and quotient err by a few units of 2^-22).
__device__ __forceinline__ float rc_silu_bf16(float x) { return __fdividef(x, 1.f + __expf(-x)); }

// Shared-memory operand tiles of the chunked forms: rows of 64 bf16 (128 bytes, 128-byte swizzle), one atom per 64 columns. The same tile is
// a K-major operand (rows along M or N) or an MN-major one (rows along K).
constexpr int RT_C = 128;                 // tokens per chunk
constexpr int RT_ATOM = RT_C * 128;       // 128 rows x 64 columns of bf16
constexpr int RT_SATOM = 64 * 128;        // 64 state rows x 64 value columns
__device__ __forceinline__ uint32_t rt_sw(int row, int piece) { return row * 128 + ((piece ^ (row & 7)) << 4); }

// Splits 8 fp32 values into bf16 high and low parts.
__device__ __forceinline__ void split8(const float (&v)[8], uint4& hi, uint4& lo) {
  uint32_t h[4], l[4];
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    h[i] = pack_bf16x2(v[2 * i], v[2 * i + 1]);
    const float2 hf = unpack_bf16x2(h[i]);
    l[i] = pack_bf16x2(v[2 * i] - hf.x, v[2 * i + 1] - hf.y);
  }
  hi = make_uint4(h[0], h[1], h[2], h[3]);
  lo = make_uint4(l[0], l[1], l[2], l[3]);
}
// ... and stores them as 16-byte pieces.
__device__ __forceinline__ void store_split(uint8_t* hi, uint8_t* lo, uint32_t off, const float (&v)[8]) {
  uint4 h, l;
  split8(v, h, l);
  *reinterpret_cast<uint4*>(hi + off) = h;
  *reinterpret_cast<uint4*>(lo + off) = l;
}
__device__ __forceinline__ void unpack8(const uint4& r, float (&v)[8]) {
  const uint32_t w[4] = {r.x, r.y, r.z, r.w};
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const float2 f = unpack_bf16x2(w[i]);
    v[2 * i] = f.x;
    v[2 * i + 1] = f.y;
  }
}
}  // namespace rlb
