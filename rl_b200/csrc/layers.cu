// Row kernels of post-norm and pre-norm layers (models/post_norm.py, models/pre_norm.py), for every size and for bf16 and fp32 models: the step that norms a sublayer's
// output and joins it to the residual stream, the sigmoid router with group-limited choice, the placement of the tokens' copies in
// per-expert row ranges, and the soft cap of the logits.
//
//   add_normed   x += m * rms(y) * w (post-norm layers) or x += y (pre-norm layers) on the fp32 stream, and what the next sublayer reads: x
//                itself in the model's type, or its RMS norm. y is a product's output or the weighted sum of a token's expert rows (combined here, never stored).
//   moe_choose   one warp per token: scores, group choice, top-k; every copy takes a number among its expert's copies.
//   moe_place    row ranges of the experts (multiples of 128 rows) from their counts, the row of every copy, and its token's row moved there.
//
// This file is compiled without fast math.
#include "common.cuh"

#include <math.h>

namespace {
using namespace rlb;

template <typename T>
__device__ __forceinline__ float ldv(const T* p) {
  return static_cast<float>(*p);
}
template <>
__device__ __forceinline__ float ldv<__nv_bfloat16>(const __nv_bfloat16* p) {
  return __bfloat162float(*p);
}
__device__ __forceinline__ float4 ld4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 ld4(const __nv_bfloat16* p) {
  const uint2 r = *reinterpret_cast<const uint2*>(p);
  const float2 a = unpack_bf16x2(r.x), b = unpack_bf16x2(r.y);
  return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ void st4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void st4(__nv_bfloat16* p, float4 v) {
  *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(v.x, v.y), pack_bf16x2(v.z, v.w));
}
__device__ __forceinline__ void st1(float* p, float v) { *p = v; }
__device__ __forceinline__ void st1(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }

struct AddNormed {
  float* x;                // [rows, d]
  const void* y;           // [rows, ldy], or the experts' rows when copy_row is set
  long long ldy;
  const int* copy_row;     // [rows, k] row of each of a token's copies in y (out of [0, y_rows): skipped)
  const float* weight;     // [rows, k] (null: 1)
  int k, y_rows;
  int* counts;             // the experts' counts [experts], set to zero for the next layer
  int experts;
  const void* w;           // norm weight of the sublayer (null: its output joins as it is)
  const void* next_w;      // weight of the next norm (null: h is x)
  void* h;                 // [rows, d]
  int d;
  float mult, eps;
  const void* also;        // [rows, ld_also] or null: added to the sublayer's output
  long long ld_also;
};

// AN_KEEP: groups of four columns that a thread keeps in registers
template <typename T, int THREADS, int AN_KEEP>
__global__ void __launch_bounds__(THREADS) add_normed_kernel(AddNormed a) {
  __shared__ float red[32];
  pdl_sync();
  const long long row = blockIdx.x;
  if (row == 0 && a.counts)
    for (int e = threadIdx.x; e < a.experts; e += THREADS) a.counts[e] = 0;
  const T* Y = static_cast<const T*>(a.y);
  float* x = a.x + row * a.d;
  T* h = static_cast<T*>(a.h) + row * a.d;
  const T *w = static_cast<const T*>(a.w), *nw = static_cast<const T*>(a.next_w), *also = static_cast<const T*>(a.also);
  if (a.d % 4 == 0 && a.d <= AN_KEEP * 4 * THREADS) {
    float4 v[AN_KEEP], xv[AN_KEEP];
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < AN_KEEP; ++i) {
      const int c = (threadIdx.x + i * THREADS) * 4;
      v[i] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (c >= a.d) continue;
      xv[i] = ld4(x + c);
      if (!a.copy_row) v[i] = ld4(Y + row * a.ldy + c);
      if (also) {
        const float4 t = ld4(also + row * a.ld_also + c);
        v[i].x += t.x; v[i].y += t.y; v[i].z += t.z; v[i].w += t.w;
      }
    }
    if (a.copy_row) {
      constexpr int AHEAD = AN_KEEP <= 2 ? 4 : 2;      // copies in flight
      for (int j0 = 0; j0 < a.k; j0 += AHEAD) {
        float4 e[AHEAD][AN_KEEP];
        float wt[AHEAD];
#pragma unroll
        for (int j = 0; j < AHEAD; ++j) {
          const int r = j0 + j < a.k ? a.copy_row[row * a.k + j0 + j] : -1;
          const bool live = r >= 0 && r < a.y_rows;
          wt[j] = live ? (a.weight ? a.weight[row * a.k + j0 + j] : 1.f) : 0.f;
#pragma unroll
          for (int i = 0; i < AN_KEEP; ++i) {
            const int c = (threadIdx.x + i * THREADS) * 4;
            e[j][i] = live && c < a.d ? ld4(Y + r * a.ldy + c) : make_float4(0.f, 0.f, 0.f, 0.f);
          }
        }
#pragma unroll
        for (int j = 0; j < AHEAD; ++j)
#pragma unroll
          for (int i = 0; i < AN_KEEP; ++i) {
            v[i].x = fmaf(wt[j], e[j][i].x, v[i].x);
            v[i].y = fmaf(wt[j], e[j][i].y, v[i].y);
            v[i].z = fmaf(wt[j], e[j][i].z, v[i].z);
            v[i].w = fmaf(wt[j], e[j][i].w, v[i].w);
          }
      }
    }
    float f = a.mult;
    if (w) {
#pragma unroll
      for (int i = 0; i < AN_KEEP; ++i) ss += v[i].x * v[i].x + v[i].y * v[i].y + v[i].z * v[i].z + v[i].w * v[i].w;
      ss = block_sum(ss, red);
      f = a.mult / sqrtf(ss / static_cast<float>(a.d) + a.eps);
    }
    float s2 = 0.f;
#pragma unroll
    for (int i = 0; i < AN_KEEP; ++i) {
      const int c = (threadIdx.x + i * THREADS) * 4;
      if (c >= a.d) continue;
      const float4 wv = w ? ld4(w + c) : make_float4(1.f, 1.f, 1.f, 1.f);
      xv[i].x = fmaf(v[i].x * f, wv.x, xv[i].x);
      xv[i].y = fmaf(v[i].y * f, wv.y, xv[i].y);
      xv[i].z = fmaf(v[i].z * f, wv.z, xv[i].z);
      xv[i].w = fmaf(v[i].w * f, wv.w, xv[i].w);
      st4(x + c, xv[i]);
      if (!nw) st4(h + c, xv[i]);
      s2 += xv[i].x * xv[i].x + xv[i].y * xv[i].y + xv[i].z * xv[i].z + xv[i].w * xv[i].w;
    }
    if (nw) {
      s2 = block_sum(s2, red);
      const float g = 1.f / sqrtf(s2 / static_cast<float>(a.d) + a.eps);
#pragma unroll
      for (int i = 0; i < AN_KEEP; ++i) {
        const int c = (threadIdx.x + i * THREADS) * 4;
        if (c >= a.d) continue;
        const float4 wv = ld4(nw + c);
        st4(h + c, make_float4(xv[i].x * g * wv.x, xv[i].y * g * wv.y, xv[i].z * g * wv.z, xv[i].w * g * wv.w));
      }
    }
    return;
  }
  auto value = [&](int c) {
    float v = also ? ldv(also + row * a.ld_also + c) : 0.f;
    if (!a.copy_row) return v + ldv(Y + row * a.ldy + c);
    for (int j = 0; j < a.k; ++j) {
      const int r = a.copy_row[row * a.k + j];
      if (r >= 0 && r < a.y_rows) v = fmaf(a.weight ? a.weight[row * a.k + j] : 1.f, ldv(Y + r * a.ldy + c), v);
    }
    return v;
  };
  float ss = 0.f, s2 = 0.f;
  float f = a.mult;
  if (w) {
    for (int c = threadIdx.x; c < a.d; c += THREADS) {
      const float v = value(c);
      ss += v * v;
    }
    ss = block_sum(ss, red);
    f = a.mult / sqrtf(ss / static_cast<float>(a.d) + a.eps);
  }
  for (int c = threadIdx.x; c < a.d; c += THREADS) {
    const float v = fmaf(value(c) * f, w ? ldv(w + c) : 1.f, x[c]);
    x[c] = v;
    if (!nw) st1(h + c, v);
    s2 += v * v;
  }
  if (!nw) return;
  s2 = block_sum(s2, red);
  const float g = 1.f / sqrtf(s2 / static_cast<float>(a.d) + a.eps);
  for (int c = threadIdx.x; c < a.d; c += THREADS) st1(h + c, x[c] * g * ldv(nw + c));
}

// Divides `groups` equal parts of each row by their root mean square and multiplies by w, in place.
template <typename T>
__global__ void __launch_bounds__(256) group_norm_rows_kernel(T* __restrict__ y, long long ldy, const T* __restrict__ w, int groups, int n, float eps) {
  __shared__ float red[32];
  pdl_sync();
  const long long row = blockIdx.x;
  const int g = blockIdx.y;
  (void)groups;
  T* p = y + row * ldy + static_cast<long long>(g) * n;
  const T* wg = w + static_cast<long long>(g) * n;
  float ss = 0.f;
  if (n % 4 == 0 && ldy % 4 == 0 && n <= 8192) {
    float4 v[8];
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      const int c = (threadIdx.x + i * 256) * 4;
      v[i] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (c < n) v[i] = ld4(p + c);
      ss += v[i].x * v[i].x + v[i].y * v[i].y + v[i].z * v[i].z + v[i].w * v[i].w;
    }
    ss = block_sum(ss, red);
    const float f = 1.f / sqrtf(ss / static_cast<float>(n) + eps);
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      const int c = (threadIdx.x + i * 256) * 4;
      if (c >= n) continue;
      const float4 wv = ld4(wg + c);
      st4(p + c, make_float4(v[i].x * f * wv.x, v[i].y * f * wv.y, v[i].z * f * wv.z, v[i].w * f * wv.w));
    }
    return;
  }
  for (int c = threadIdx.x; c < n; c += 256) {
    const float v = ldv(p + c);
    ss += v * v;
  }
  ss = block_sum(ss, red);
  const float f = 1.f / sqrtf(ss / static_cast<float>(n) + eps);
  for (int c = threadIdx.x; c < n; c += 256) st1(p + c, ldv(p + c) * f * ldv(wg + c));
}

// The same for bf16 parts of at most 2048 columns: one warp per part.
__global__ void __launch_bounds__(256)
group_norm_warp_kernel(__nv_bfloat16* __restrict__ y, long long ldy, const __nv_bfloat16* __restrict__ w, long long parts, int groups, int n, float eps) {
  pdl_sync();
  const int lane = threadIdx.x & 31;
  const long long i = static_cast<long long>(blockIdx.x) * 8 + (threadIdx.x >> 5);
  if (i >= parts) return;
  const long long row = i / groups;
  const int g = static_cast<int>(i - row * groups);
  __nv_bfloat16* p = y + row * ldy + static_cast<long long>(g) * n;
  const __nv_bfloat16* wg = w + static_cast<long long>(g) * n;
  uint4 raw[8];
  float ss = 0.f;
#pragma unroll
  for (int q = 0; q < 8; ++q) {
    const int c = (lane + q * 32) * 8;
    raw[q] = c < n ? *reinterpret_cast<const uint4*>(p + c) : make_uint4(0, 0, 0, 0);
  }
#pragma unroll
  for (int q = 0; q < 8; ++q) {
    const float2 a = unpack_bf16x2(raw[q].x), b = unpack_bf16x2(raw[q].y), c = unpack_bf16x2(raw[q].z), d = unpack_bf16x2(raw[q].w);
    ss += a.x * a.x + a.y * a.y + b.x * b.x + b.y * b.y + c.x * c.x + c.y * c.y + d.x * d.x + d.y * d.y;
  }
  ss = warp_sum(ss);
  const float f = 1.f / sqrtf(ss / static_cast<float>(n) + eps);
#pragma unroll
  for (int q = 0; q < 8; ++q) {
    const int c = (lane + q * 32) * 8;
    if (c >= n) continue;
    const uint4 wr = *reinterpret_cast<const uint4*>(wg + c);
    const uint32_t in[4] = {raw[q].x, raw[q].y, raw[q].z, raw[q].w}, wv[4] = {wr.x, wr.y, wr.z, wr.w};
    uint32_t o[4];
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      const float2 a = unpack_bf16x2(in[k]), b = unpack_bf16x2(wv[k]);
      o[k] = pack_bf16x2(a.x * f * b.x, a.y * f * b.y);
    }
    *reinterpret_cast<uint4*>(p + c) = make_uint4(o[0], o[1], o[2], o[3]);
  }
}

__global__ void __launch_bounds__(256) cap_rows_kernel(float* __restrict__ z, long long n, float scale, float cap) {
  for (long long i = static_cast<long long>(blockIdx.x) * 256 + threadIdx.x; i < n; i += static_cast<long long>(gridDim.x) * 256) {
    const float v = z[i] * scale;
    z[i] = cap > 0.f ? cap * tanhf(v / cap) : v;
  }
}

// ---------------------------------------------------------------- router
constexpr int MC_WARPS = 4;

// Largest of v over the warp, the lowest index of equal values; index 0x7fffffff where no lane has a value.
__device__ __forceinline__ void warp_best(float& v, int& i) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    const float ov = __shfl_xor_sync(0xffffffffu, v, o);
    const int oi = __shfl_xor_sync(0xffffffffu, i, o);
    if (ov > v || (ov == v && oi < i)) {
      v = ov;
      i = oi;
    }
  }
}

__global__ void __launch_bounds__(MC_WARPS * 32)
moe_choose_kernel(const float* __restrict__ logits, long long ld, int T, int E, const float* __restrict__ correction, int groups, int keep, int k,
                  float* __restrict__ out_w, int* __restrict__ out_idx, int* __restrict__ out_rank, int* __restrict__ counts) {
  extern __shared__ float sm[];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int t = blockIdx.x * MC_WARPS + warp;
  pdl_sync();
  if (t >= T) return;
  float* s = sm + warp * (2 * E + groups);
  float* c = s + E;
  float* gs = c + E;
  for (int e = lane; e < E; e += 32) {
    const float v = 1.f / (1.f + expf(-logits[static_cast<long long>(t) * ld + e]));
    s[e] = v;
    c[e] = correction ? v + correction[e] : v;
  }
  __syncwarp();
  if (groups > 1) {
    const int size = E / groups;
    for (int g = lane; g < groups; g += 32) {
      float a = -INFINITY, b = -INFINITY;      // the two largest
      for (int e = g * size; e < (g + 1) * size; ++e) {
        const float v = c[e];
        if (v > a) {
          b = a;
          a = v;
        } else if (v > b) {
          b = v;
        }
      }
      gs[g] = size > 1 ? a + b : a;
    }
    __syncwarp();
    for (int n = 0; n < keep; ++n) {           // chosen groups are marked with NaN
      float best = -INFINITY;
      int bi = 0x7fffffff;
      for (int g = lane; g < groups; g += 32)
        if (gs[g] > best) {
          best = gs[g];
          bi = g;
        }
      warp_best(best, bi);
      if (lane == 0 && bi < groups) gs[bi] = __int_as_float(0x7fc00000);
      __syncwarp();
    }
    for (int e = lane; e < E; e += 32)
      if (gs[e / size] == gs[e / size]) c[e] = -INFINITY;
    __syncwarp();
  }
  float wsel = 0.f;
  int isel = 0;
  for (int j = 0; j < k; ++j) {
    float best = -INFINITY;
    int bi = 0x7fffffff;
    for (int e = lane; e < E; e += 32)
      if (c[e] > best) {
        best = c[e];
        bi = e;
      }
    warp_best(best, bi);
    if (bi >= E) bi = 0;                        // (not a number everywhere)
    if (lane == j) {
      isel = bi;
      wsel = s[bi];
    }
    __syncwarp();
    if (lane == 0) c[bi] = -INFINITY;
    __syncwarp();
  }
  if (lane < k) {
    const long long o = static_cast<long long>(t) * k + lane;
    out_w[o] = wsel;
    out_idx[o] = isel;
    out_rank[o] = atomicAdd(counts + isel, 1);
  }
}

// Every CTA sums the experts' padded counts for itself; CTA 0 writes the tile table. One warp per copy moves its token's row (x_out null:
// the rows stay where they are and a_rows says which token each padded row reads).
constexpr int MP_MAX_E = 1024;
__global__ void __launch_bounds__(256)
moe_place_kernel(const int* __restrict__ idx, const int* __restrict__ rank, long long copies, int k, const int* __restrict__ counts, int E, int mpad,
                 int* __restrict__ copy_row, int* __restrict__ tile_expert, int* __restrict__ a_rows,
                 const uint4* __restrict__ x, long long x_vecs, uint4* __restrict__ x_out, int vecs, const float* __restrict__ weight,
                 float* __restrict__ row_weight, int* status) {
  __shared__ int row0[MP_MAX_E + 1];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  pdl_sync();
  for (int e = tid; e < E; e += 256) row0[e] = (counts[e] + 127) / 128;     // (in tiles)
  __syncthreads();
  if (warp == 0) {                                                          // exclusive sums, 32 experts at a time
    int at = 0;
    for (int e0 = 0; e0 < E; e0 += 32) {
      const int mine = e0 + lane < E ? row0[e0 + lane] : 0;
      int inc = mine;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const int up = __shfl_up_sync(0xffffffffu, inc, o);
        if (lane >= o) inc += up;
      }
      if (e0 + lane < E) row0[e0 + lane] = at + inc - mine;
      at += __shfl_sync(0xffffffffu, inc, 31);
    }
    if (lane == 0) row0[E] = at;
  }
  __syncthreads();
  const int tiles = mpad / 128;
  if (blockIdx.x == 0) {
    for (int e = tid; e < E; e += 256) {
      for (int t = row0[e]; t < row0[e + 1] && t < tiles; ++t) tile_expert[t] = e;
    }
    for (int t = row0[E] + tid; t < tiles; t += 256) tile_expert[t] = -1;
    if (tid == 0 && row0[E] > tiles && status) atomicCAS(status, 0, RLB_ERR_BOUNDS);
  }
  for (long long c = static_cast<long long>(blockIdx.x) * 8 + warp; c < copies; c += static_cast<long long>(gridDim.x) * 8) {
    const int e = idx[c];
    int row = row0[e] * 128 + rank[c];
    if (row >= mpad) row = -1;
    if (lane == 0) {
      copy_row[c] = row;
      if (a_rows && row >= 0) a_rows[row] = static_cast<int>(c / k);
      if (row_weight && row >= 0) row_weight[row] = weight[c];
    }
    if (x_out && row >= 0) {
      const uint4* src = x + (c / k) * x_vecs;
      uint4* dst = x_out + static_cast<long long>(row) * vecs;
      for (int v = lane; v < vecs; v += 32) dst[v] = src[v];
    }
  }
}
}  // namespace

// x [rows, d] fp32 += mult * rms(y) * w (w null: mult * y); h [rows, d] = x, or rms(x) * next_w. With copy_row [rows, k]: y of a row is the
// sum of its k weighted (weight null: plain) rows of y [y_rows, ldy], and counts [experts] are set to zero. also [rows, ld_also]: added to y.
RLB_API int rlb_add_normed(float* x, const void* y, long long ldy, int f32, const int* copy_row, const float* weight, int k, int y_rows, int* counts, int experts,
                           const void* also, long long ld_also, const void* w, const void* next_w, void* h, long long rows, int d, float mult, float eps, void* stream) {
  if (rows <= 0) return 0;
  if (d % 4 == 0 && (ldy % 4 || (also && ld_also % 4))) return -2;
  AddNormed a{x, y, ldy, copy_row, weight, k, y_rows, counts, experts, w, next_w, h, d, mult, eps, also, ld_also};
  const dim3 grid(static_cast<unsigned>(rows));
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (f32) return static_cast<int>(rlb_launch_pdl(add_normed_kernel<float, 256, 8>, grid, dim3(256), 0, s, a));
  const bool few = rows < 148 * 4;      // few rows: more threads per row
  auto kernel = few && d > 1024 ? (d <= 2048 ? add_normed_kernel<__nv_bfloat16, 512, 1> : (d <= 4096 ? add_normed_kernel<__nv_bfloat16, 512, 2>
                                                                                                : add_normed_kernel<__nv_bfloat16, 512, 4>))
                           : (d <= 1024 ? add_normed_kernel<__nv_bfloat16, 256, 1> : (d <= 2048 ? add_normed_kernel<__nv_bfloat16, 256, 2>
                              : (d <= 4096 ? add_normed_kernel<__nv_bfloat16, 256, 4> : add_normed_kernel<__nv_bfloat16, 256, 8>)));
  return static_cast<int>(rlb_launch_pdl(kernel, grid, dim3(few && d > 1024 ? 512 : 256), 0, s, a));
}

// y [rows, ldy]: each of `groups` neighbouring parts of n columns divided by its root mean square, times w [groups * n]; in place.
RLB_API int rlb_group_norm_rows(void* y, long long ldy, int f32, const void* w, long long rows, int groups, int n, float eps, void* stream) {
  if (rows <= 0) return 0;
  if (groups > 65535) return -2;
  const dim3 grid(static_cast<unsigned>(rows), groups);
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (f32)
    return static_cast<int>(rlb_launch_pdl(group_norm_rows_kernel<float>, grid, dim3(256), 0, s, static_cast<float*>(y), ldy, static_cast<const float*>(w),
                                           groups, n, eps));
  const bool few = rows * groups < 148 * 2 && n >= 256;      // few parts: a CTA each
  if (!few && n % 8 == 0 && n <= 2048 && ldy % 8 == 0 && !((reinterpret_cast<uintptr_t>(y) | reinterpret_cast<uintptr_t>(w)) & 15)) {
    const long long parts = rows * groups;
    return static_cast<int>(rlb_launch_pdl(group_norm_warp_kernel, dim3(static_cast<unsigned>((parts + 7) / 8)), dim3(256), 0, s,
                                           static_cast<__nv_bfloat16*>(y), ldy, static_cast<const __nv_bfloat16*>(w), parts, groups, n, eps));
  }
  return static_cast<int>(rlb_launch_pdl(group_norm_rows_kernel<__nv_bfloat16>, grid, dim3(256), 0, s, static_cast<__nv_bfloat16*>(y), ldy,
                                         static_cast<const __nv_bfloat16*>(w), groups, n, eps));
}

RLB_API int rlb_cap_rows(float* z, long long n, float scale, float cap, void* stream) {
  if (n <= 0) return 0;
  const long long want = (n + 255) / 256;
  cap_rows_kernel<<<static_cast<unsigned>(want < 148 * 16 ? want : 148 * 16), 256, 0, static_cast<cudaStream_t>(stream)>>>(z, n, scale, cap);
  return static_cast<int>(cudaGetLastError());
}

// Scores sigmoid(logits [T, E]), choice by score + correction (null: none) among the `keep` best of `groups` groups. counts [E] (zero before the call)
// receives the experts' copies, out_rank each copy's number among them.
RLB_API int rlb_moe_choose(const float* logits, long long ld, int T, int E, const float* correction, int groups, int keep, int k, float* out_w,
                           int* out_idx, int* out_rank, int* counts, void* stream) {
  if (T <= 0) return 0;
  if (E < 1 || E > MP_MAX_E || k < 1 || k > 32 || k > E || groups < 1 || E % groups || keep < 1 || keep > groups) return -2;
  const size_t smem = sizeof(float) * MC_WARPS * (2 * E + groups);
  return static_cast<int>(rlb_launch_pdl(moe_choose_kernel, dim3((T + MC_WARPS - 1) / MC_WARPS), dim3(MC_WARPS * 32), smem, static_cast<cudaStream_t>(stream),
                                         logits, ld, T, E, correction, groups, keep, k, out_w, out_idx, out_rank, counts));
}

// mpad: a multiple of 128, at least copies + E * 127. a_rows (with x_out null) must hold -1 everywhere before the call. row_bytes and the
// row stride of x: multiples of 16 (only with x_out). row_weight [mpad] (or null): each copy's weight [copies] at its row.
RLB_API int rlb_moe_place(const int* idx, const int* rank, long long copies, int k, const int* counts, int E, int mpad, int* copy_row,
                          int* tile_expert, int* a_rows, const void* x, long long x_stride_bytes, void* x_out, int row_bytes, const float* weight,
                          float* row_weight, int* status, void* stream) {
  if (copies <= 0) return 0;
  if (E < 1 || E > MP_MAX_E || mpad % 128 || mpad < copies + static_cast<long long>(E) * 127) return -2;
  if (x_out && ((row_bytes % 16) || (x_stride_bytes % 16) || ((reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(x_out)) & 15))) return -3;
  const long long want = (copies + 7) / 8;
  return static_cast<int>(rlb_launch_pdl(moe_place_kernel, dim3(static_cast<unsigned>(want < 148 * 4 ? want : 148 * 4)), dim3(256), 0,
                                         static_cast<cudaStream_t>(stream), idx, rank, copies, k, counts, E, mpad, copy_row, tile_expert, a_rows,
                                         static_cast<const uint4*>(x), x_stride_bytes / 16, static_cast<uint4*>(x_out), row_bytes / 16, weight, row_weight, status));
}
