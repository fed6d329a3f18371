// Grouped-query attention of layer-list models (GroupedAttentionMixer): the step between the projection and the attention kernels, the gather
// of cached keys and values for prompt portions, and attention one row at a time for every size and for bf16 and fp32 models.
//
// Keys and values live in pages [page, kv head, token, dim] / [page, kv head, token, vdim]. The tensor-core forms are in
// latent_attention.cu (portions of prompts) and paged_decode_mma.cu (single rows, head dimension 128).
//
// This file is compiled without fast math.
#include "common.cuh"

#include <math.h>

namespace {
using namespace rlb;

template <typename T>
__device__ __forceinline__ float ldf(const T* p) {
  return static_cast<float>(*p);
}
template <>
__device__ __forceinline__ float ldf<__nv_bfloat16>(const __nv_bfloat16* p) {
  return __bfloat162float(*p);
}
__device__ __forceinline__ void stf(float* p, float v) { *p = v; }
__device__ __forceinline__ void stf(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }

struct GqaShape {
  long long ldp;
  int q_off, k_off, v_off;
  int heads, kv_heads, dim, vdim;
  int block_size, num_blocks;
  int halves;            // rotated pairs are (i, i + half) instead of (2i, 2i + 1)
  int own_kv;            // the rows hold keys and values of the layer's own
};

// Values of a layer that mixes them with an earlier layer's: v <- (1 - share) v + share v_first.
template <typename T>
struct ValueMix {
  const T* first;        // column of kv head 0 of the earlier layer's projected rows (null: no mixing)
  long long ld;
  const T* share;        // one number
};

// One CTA per row, a warp per head in turn: RMS norm and rotation of the query and key heads in place, keys and values into the cache. The
// row's cosines and sines are computed once for all heads. A lane keeps pairs (2i, 2i + 1), which is also what the interleaved rotation
// turns. Few rows are spread over several CTAs each (blockIdx.y).
constexpr int GP_WARPS = 8, GP_KEEP = 4;      // pairs a lane keeps in registers
template <typename T>
struct Pair;
template <>
struct Pair<float> {
  static __device__ __forceinline__ float2 load(const float* p, bool aligned) { return aligned ? *reinterpret_cast<const float2*>(p) : make_float2(p[0], p[1]); }
  static __device__ __forceinline__ void store(float* p, float a, float b, bool aligned) {
    if (aligned) {
      *reinterpret_cast<float2*>(p) = make_float2(a, b);
    } else {
      p[0] = a;
      p[1] = b;
    }
  }
};
template <>
struct Pair<__nv_bfloat16> {
  static __device__ __forceinline__ float2 load(const __nv_bfloat16* p, bool aligned) {
    return aligned ? unpack_bf16x2(*reinterpret_cast<const uint32_t*>(p)) : make_float2(__bfloat162float(p[0]), __bfloat162float(p[1]));
  }
  static __device__ __forceinline__ void store(__nv_bfloat16* p, float a, float b, bool aligned) {
    if (aligned) {
      *reinterpret_cast<uint32_t*>(p) = pack_bf16x2(a, b);
    } else {
      p[0] = __float2bfloat16(a);
      p[1] = __float2bfloat16(b);
    }
  }
};

template <typename T>
__global__ void __launch_bounds__(GP_WARPS * 32)
gqa_prep_kernel(T* __restrict__ p, GqaShape s, ValueMix<T> mix, const int* __restrict__ positions, const long long* __restrict__ slots,
                const T* __restrict__ q_norm, const T* __restrict__ k_norm, const float* __restrict__ freq, int half, float gain, float eps, T* __restrict__ k_cache,
                T* __restrict__ v_cache, int* status) {
  extern __shared__ float2 turn[];      // [half] (cosine, sine)
  const int lane = threadIdx.x & 31;
  const long long row = blockIdx.x;
  pdl_sync();
  const float pos = static_cast<float>(positions[row]);
  const long long slot = slots[row];
  for (int i = threadIdx.x; i < half; i += GP_WARPS * 32) {
    float sn, cs;
    sincosf(pos * freq[i], &sn, &cs);
    turn[i] = make_float2(cs * gain, sn * gain);
  }
  T* pr = p + row * s.ldp;
  const bool bad = slot >= static_cast<long long>(s.num_blocks) * s.block_size;
  if (bad && threadIdx.x == 0 && status) atomicCAS(status, 0, RLB_ERR_BOUNDS);
  const bool cached = slot >= 0 && !bad;
  const long long page = cached ? slot / s.block_size : 0, off = cached ? slot % s.block_size : 0;
  const bool even = s.dim % 2 == 0 && s.ldp % 2 == 0, veven = s.vdim % 2 == 0 && s.ldp % 2 == 0;      // pairs are aligned
  const int pairs = (s.dim + 1) / 2;
  __syncthreads();
  for (int unit = blockIdx.y * GP_WARPS + (threadIdx.x >> 5); unit < s.heads + (s.own_kv ? 2 * s.kv_heads : 0); unit += gridDim.y * GP_WARPS) {
    const bool is_q = unit < s.heads, is_k = !is_q && unit < s.heads + s.kv_heads;
    const int head = is_q ? unit : (is_k ? unit - s.heads : unit - s.heads - s.kv_heads);
    if (!is_q && !is_k) {
      T* v = pr + s.v_off + head * s.vdim;
      if (mix.first) {
        const T* f = mix.first + row * mix.ld + head * s.vdim;
        const float share = ldf(mix.share);
        for (int i = lane; i < s.vdim; i += 32) stf(v + i, (1.f - share) * ldf(v + i) + share * ldf(f + i));
        __syncwarp();
      }
      if (!cached) continue;
      T* c = v_cache + ((page * s.kv_heads + head) * s.block_size + off) * s.vdim;
      if (veven) {
        for (int i = lane * 2; i < s.vdim; i += 64) {
          const float2 t = Pair<T>::load(v + i, true);
          Pair<T>::store(c + i, t.x, t.y, true);
        }
      } else {
        for (int i = lane; i < s.vdim; i += 32) c[i] = v[i];
      }
      continue;
    }
    T* x = pr + (is_q ? s.q_off : s.k_off) + head * s.dim;
    const T* w = is_q ? q_norm : k_norm;      // null: no norm
    auto weight = [&](int i) { return w ? ldf(w + i) : 1.f; };
    T* c = is_k && cached ? k_cache + ((page * s.kv_heads + head) * s.block_size + off) * s.dim : nullptr;
    auto load = [&](int i) {      // pair i, zeros past the end
      if (2 * i + 1 < s.dim) return Pair<T>::load(x + 2 * i, even);
      return make_float2(2 * i < s.dim ? ldf(x + 2 * i) : 0.f, 0.f);
    };
    float2 u[GP_KEEP];
    float ss = 0.f;
#pragma unroll
    for (int j = 0; j < GP_KEEP; ++j) {
      u[j] = load(lane + j * 32);
      ss += u[j].x * u[j].x + u[j].y * u[j].y;
    }
    for (int i = lane + GP_KEEP * 32; i < pairs; i += 32) {
      const float2 t = load(i);
      ss += t.x * t.x + t.y * t.y;
    }
    ss = warp_sum(ss);
    const float rstd = w ? 1.f / sqrtf(ss / static_cast<float>(s.dim) + eps) : 1.f;
    if (s.halves) {      // a lane turns entries i and i + half; the sum's shuffles stand between the loads above and these stores
      auto put = [&](int i, float t) {
        stf(x + i, t);
        if (c) stf(c + i, t);
      };
      for (int i = lane; i < half; i += 32) {
        const float a = ldf(x + i) * rstd * weight(i), b = ldf(x + i + half) * rstd * weight(i + half);
        const float2 r = turn[i];
        put(i, a * r.x - b * r.y);
        put(i + half, b * r.x + a * r.y);
      }
      for (int i = 2 * half + lane; i < s.dim; i += 32) put(i, ldf(x + i) * rstd * weight(i));
      continue;
    }
    auto finish = [&](int i, float2 t) {
      if (2 * i >= s.dim) return;
      const bool two = 2 * i + 1 < s.dim;
      t.x *= rstd * weight(2 * i);
      if (two) t.y *= rstd * weight(2 * i + 1);
      if (i < half) {
        const float2 r = turn[i];
        t = make_float2(t.x * r.x - t.y * r.y, t.y * r.x + t.x * r.y);
      }
      if (two) {
        Pair<T>::store(x + 2 * i, t.x, t.y, even);
        if (c) Pair<T>::store(c + 2 * i, t.x, t.y, even);
      } else {
        stf(x + 2 * i, t.x);
        if (c) stf(c + 2 * i, t.x);
      }
    };
#pragma unroll
    for (int j = 0; j < GP_KEEP; ++j) finish(lane + j * 32, u[j]);
    for (int i = lane + GP_KEEP * 32; i < pairs; i += 32) finish(i, load(i));
  }
}

// The same for bf16 rows with even dim <= 64 * KEEP and even vdim: one warp per row (and share of its heads). A lane keeps the same 32-bit words
// (two entries) of every head, so cosines, sines and norm weights stay in its registers; four heads are in flight. Interleaved pairs: word
// lane + 32 j is one pair. HALVES (half even): words 2 s and 2 s + 1 of a lane are r and r + half / 2 with r = lane + 32 s, two pairs, or two
// neighbours behind the rotated part.
template <int KEEP, bool HALVES>
__global__ void __launch_bounds__(GP_WARPS * 32)
gqa_prep_rows_kernel(__nv_bfloat16* __restrict__ p, GqaShape s, ValueMix<__nv_bfloat16> mix, long long rows, const int* __restrict__ positions, const long long* __restrict__ slots,
                     const __nv_bfloat16* __restrict__ q_norm, const __nv_bfloat16* __restrict__ k_norm, const float* __restrict__ freq, int half,
                     float gain, float eps, __nv_bfloat16* __restrict__ k_cache, __nv_bfloat16* __restrict__ v_cache, int* status) {
  constexpr int AHEAD = 4;
  const int lane = threadIdx.x & 31;
  const long long row = static_cast<long long>(blockIdx.x) * GP_WARPS + (threadIdx.x >> 5);
  float2 wq[KEEP], wk[KEEP], turn[KEEP];
  auto word = [&](int j) {      // may lie behind the head
    if (!HALVES) return lane + j * 32;
    const int r = lane + (j >> 1) * 32, hw = half / 2;
    return r < hw ? r + (j & 1) * hw : half + 2 * (r - hw) + (j & 1);
  };
#pragma unroll
  for (int j = 0; j < KEEP; ++j) {
    const int i = word(j);
    const bool live = 2 * i < s.dim;
    wq[j] = live && q_norm ? Pair<__nv_bfloat16>::load(q_norm + 2 * i, true) : make_float2(1.f, 1.f);
    wk[j] = live && k_norm ? Pair<__nv_bfloat16>::load(k_norm + 2 * i, true) : make_float2(1.f, 1.f);
  }
  pdl_sync();
  if (row >= rows) return;
  const float pos = static_cast<float>(positions[row]);
  const long long slot = slots[row];
  const bool bad = slot >= static_cast<long long>(s.num_blocks) * s.block_size;
  if (bad && lane == 0 && status) atomicCAS(status, 0, RLB_ERR_BOUNDS);
  const bool cached = slot >= 0 && !bad;
  const unsigned at = cached ? static_cast<unsigned>(slot) : 0u, page = at / s.block_size, off = at - page * s.block_size;
#pragma unroll
  for (int j = 0; j < KEEP; ++j) {
    const int i = HALVES ? 2 * (lane + (j >> 1) * 32) + (j & 1) : lane + j * 32;      // pair
    turn[j] = make_float2(1.f, 0.f);
    if (i < half) {
      float sn, cs;
      sincosf(pos * freq[i], &sn, &cs);
      turn[j] = make_float2(cs * gain, sn * gain);
    }
  }
  __nv_bfloat16* pr = p + row * s.ldp;
  const int units = s.heads + (s.own_kv ? s.kv_heads : 0);
  for (int u0 = blockIdx.y * AHEAD; u0 < units; u0 += gridDim.y * AHEAD) {
    float2 v[AHEAD][KEEP];
    float ss[AHEAD];
#pragma unroll
    for (int a = 0; a < AHEAD; ++a) {
      const int unit = u0 + a;
      const __nv_bfloat16* x = pr + (unit < s.heads ? s.q_off + unit * s.dim : s.k_off + (unit - s.heads) * s.dim);
#pragma unroll
      for (int j = 0; j < KEEP; ++j) {
        const int i = word(j);
        v[a][j] = unit < units && 2 * i < s.dim ? Pair<__nv_bfloat16>::load(x + 2 * i, true) : make_float2(0.f, 0.f);
      }
    }
#pragma unroll
    for (int a = 0; a < AHEAD; ++a) {
      ss[a] = 0.f;
#pragma unroll
      for (int j = 0; j < KEEP; ++j) ss[a] += v[a][j].x * v[a][j].x + v[a][j].y * v[a][j].y;
    }
#pragma unroll
    for (int a = 0; a < AHEAD; ++a) ss[a] = warp_sum(ss[a]);
#pragma unroll
    for (int a = 0; a < AHEAD; ++a) {
      const int unit = u0 + a;
      if (unit >= units) break;
      const bool is_q = unit < s.heads;
      const int head = is_q ? unit : unit - s.heads;
      const float rstd = (is_q ? q_norm : k_norm) ? 1.f / sqrtf(ss[a] / static_cast<float>(s.dim) + eps) : 1.f;
      __nv_bfloat16* x = pr + (is_q ? s.q_off : s.k_off) + head * s.dim;
      __nv_bfloat16* c = k_cache + ((static_cast<long long>(page) * s.kv_heads + head) * s.block_size + off) * s.dim;
      if (HALVES) {
#pragma unroll
        for (int j = 0; j < KEEP; j += 2) {
          const int i0 = word(j), i1 = word(j + 1);
          const float2 w0 = is_q ? wq[j] : wk[j], w1 = is_q ? wq[j + 1] : wk[j + 1], t0 = turn[j], t1 = turn[j + 1];
          const float2 e = make_float2(v[a][j].x * rstd * w0.x, v[a][j].y * rstd * w0.y), f = make_float2(v[a][j + 1].x * rstd * w1.x, v[a][j + 1].y * rstd * w1.y);
          const uint32_t o0 = pack_bf16x2(e.x * t0.x - f.x * t0.y, e.y * t1.x - f.y * t1.y), o1 = pack_bf16x2(f.x * t0.x + e.x * t0.y, f.y * t1.x + e.y * t1.y);
          if (2 * i0 < s.dim) {
            *reinterpret_cast<uint32_t*>(x + 2 * i0) = o0;
            if (!is_q && cached) *reinterpret_cast<uint32_t*>(c + 2 * i0) = o0;
          }
          if (2 * i1 < s.dim) {
            *reinterpret_cast<uint32_t*>(x + 2 * i1) = o1;
            if (!is_q && cached) *reinterpret_cast<uint32_t*>(c + 2 * i1) = o1;
          }
        }
        continue;
      }
#pragma unroll
      for (int j = 0; j < KEEP; ++j) {
        const int i = lane + j * 32;
        if (2 * i >= s.dim) continue;
        const float2 w = is_q ? wq[j] : wk[j];
        const float a0 = v[a][j].x * rstd * w.x, b0 = v[a][j].y * rstd * w.y;
        const uint32_t o = pack_bf16x2(a0 * turn[j].x - b0 * turn[j].y, b0 * turn[j].x + a0 * turn[j].y);
        *reinterpret_cast<uint32_t*>(x + 2 * i) = o;
        if (!is_q && cached) *reinterpret_cast<uint32_t*>(c + 2 * i) = o;
      }
    }
  }
  if (!s.own_kv || (!cached && !mix.first)) return;
  const float share = mix.first ? __bfloat162float(*mix.share) : 0.f;
  for (int g = blockIdx.y; g < s.kv_heads; g += gridDim.y) {
    __nv_bfloat16* x = pr + s.v_off + g * s.vdim;
    const __nv_bfloat16* f = mix.first + row * mix.ld + g * s.vdim;
    __nv_bfloat16* c = v_cache + ((static_cast<long long>(page) * s.kv_heads + g) * s.block_size + off) * s.vdim;
    for (int i = lane * 2; i < s.vdim; i += 64) {
      uint32_t t = *reinterpret_cast<const uint32_t*>(x + i);
      if (mix.first) {
        const float2 own = unpack_bf16x2(t), old = unpack_bf16x2(*reinterpret_cast<const uint32_t*>(f + i));
        t = pack_bf16x2((1.f - share) * own.x + share * old.x, (1.f - share) * own.y + share * old.y);
        *reinterpret_cast<uint32_t*>(x + i) = t;
      }
      if (cached) *reinterpret_cast<uint32_t*>(c + i) = t;
    }
  }
}

// One CTA per (row, query head): tiles of 128 keys, everything in fp32; online softmax, or with `offset` the weights sigmoid(score + offset[head]).
// What a row at position i sees: chunk > 0: the keys of its own run of `chunk` positions; window > 0: keys j with i - j < window or j < keep.
// gated: the output's place holds gates, out = y * sigmoid(gate).
struct RowsMask {
  int chunk, window, keep, gated;
};
constexpr int GR_TILE = 128;
template <typename T>
__global__ void __launch_bounds__(128)
gqa_rows_kernel(const T* p, GqaShape s, const T* __restrict__ k_cache, const T* __restrict__ v_cache, const int* __restrict__ block_table,
                int bt_stride, const int* __restrict__ seq_lens, RowsMask mask, const T* __restrict__ offset, float scale, T* y, long long ldy, int* status) {
  extern __shared__ float sm[];
  __shared__ float red[32];
  float* q = sm;                        // [dim]
  float* o = q + s.dim;                 // [vdim]
  float* sc = o + s.vdim;               // [GR_TILE]
  long long* rows = reinterpret_cast<long long*>(sm + ((s.dim + s.vdim + GR_TILE + 1) & ~1));   // [GR_TILE] token row of the head in the cache
  const int row = blockIdx.x, h = blockIdx.y, g = h / (s.heads / s.kv_heads), tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const T* qp = p + row * s.ldp + s.q_off + h * s.dim;
  for (int i = tid; i < s.dim; i += 128) q[i] = ldf(qp + i) * scale;
  for (int i = tid; i < s.vdim; i += 128) o[i] = 0.f;
  const int len = min(seq_lens[row], bt_stride * s.block_size);
  const float off = offset ? ldf(offset + h) : 0.f;
  float m = -INFINITY, l = 0.f;
  int first = 0;                        // first visible key behind the kept ones
  if (len > 0 && mask.chunk > 0) first = (len - 1) / mask.chunk * mask.chunk;
  if (mask.window > 0) first = max(0, len - mask.window);
  const int kept = mask.window > 0 ? min(mask.keep, first) : 0;
  int t0 = kept > 0 ? 0 : first;
  while (t0 < len) {
    const int n = min(GR_TILE, (t0 < kept ? kept : len) - t0);
    __syncthreads();
    if (tid < n) {
      const int t = t0 + tid;
      int blk = block_table[static_cast<long long>(row) * bt_stride + t / s.block_size];
      if (blk < 0 || blk >= s.num_blocks) {
        if (status) atomicCAS(status, 0, RLB_ERR_BOUNDS);
        blk = 0;
      }
      rows[tid] = (static_cast<long long>(blk) * s.kv_heads + g) * s.block_size + t % s.block_size;
    }
    __syncthreads();
    for (int j = warp; j < n; j += 4) {
      const T* k = k_cache + rows[j] * s.dim;
      float v = 0.f;
      for (int i = lane; i < s.dim; i += 32) v = fmaf(q[i], ldf(k + i), v);
      v = warp_sum(v);
      if (lane == 0) sc[j] = v;
    }
    __syncthreads();
    float c = 1.f;
    if (offset) {
      if (tid < n) sc[tid] = 1.f / (1.f + expf(-(sc[tid] + off)));
    } else {
      const float mine = tid < n ? sc[tid] : -INFINITY;
      const float mn = fmaxf(m, block_max(mine, red));
      const float pj = tid < n ? expf(mine - mn) : 0.f;
      c = m == -INFINITY ? 0.f : expf(m - mn);
      l = l * c + block_sum(pj, red);
      m = mn;
      if (tid < n) sc[tid] = pj;
    }
    __syncthreads();
    for (int i = tid; i < s.vdim; i += 128) {
      float v[4] = {0.f, 0.f, 0.f, 0.f};
      int j = 0;
      for (; j + 4 <= n; j += 4)
#pragma unroll
        for (int q = 0; q < 4; ++q) v[q] = fmaf(sc[j + q], ldf(v_cache + rows[j + q] * s.vdim + i), v[q]);
      for (; j < n; ++j) v[0] = fmaf(sc[j], ldf(v_cache + rows[j] * s.vdim + i), v[0]);
      o[i] = fmaf(o[i], c, (v[0] + v[1]) + (v[2] + v[3]));
    }
    t0 = t0 < kept && t0 + n >= kept ? first : t0 + n;
  }
  const float inv = offset ? 1.f : (l > 0.f ? 1.f / l : 0.f);
  for (int i = tid; i < s.vdim; i += 128) {     // (each thread reads what it wrote)
    T* d = y + row * ldy + h * s.vdim + i;
    stf(d, mask.gated ? o[i] * inv / (1.f + expf(-ldf(d))) : o[i] * inv);
  }
}

// out[i] = [keys of all kv heads | values of all kv heads] of cache slot slots[i]; dim and vdim in 16-byte pieces.
__global__ void gqa_gather_kernel(const uint4* __restrict__ k_cache, const uint4* __restrict__ v_cache, const long long* __restrict__ slots,
                                  uint4* __restrict__ out, long long n, int kv_heads, int dv, int vv, int block_size, long long num_slots, int* status) {
  const int per = kv_heads * (dv + vv);
  for (long long i = static_cast<long long>(blockIdx.x) * blockDim.x + threadIdx.x; i < n * per; i += static_cast<long long>(gridDim.x) * blockDim.x) {
    const long long t = i / per;
    int c = static_cast<int>(i - t * per);
    const long long s = slots[t];
    if (s < 0 || s >= num_slots) {
      if (status) atomicCAS(status, 0, RLB_ERR_BOUNDS);
      out[i] = make_uint4(0, 0, 0, 0);
      continue;
    }
    const bool is_k = c < kv_heads * dv;
    if (!is_k) c -= kv_heads * dv;
    const int w = is_k ? dv : vv, g = c / w;
    out[i] = (is_k ? k_cache : v_cache)[((s / block_size * kv_heads + g) * block_size + s % block_size) * w + (c - g * w)];
  }
}
}  // namespace

// In place on the projected rows p: RMS norm (weight [dim]; null: none) and rotation of the first 2 * half dimensions (pairs (2i, 2i + 1), or (i, i + half)
// when `halves`) of every query and key head; v_first (row stride ld_first, null: none): values become (1 - share) v + share v_first; keys and
// values of rows with a slot go to the cache. own_kv 0: the rows hold queries only.
RLB_API int rlb_gqa_prep(void* p, int f32, long long rows, long long ldp, int q_off, int k_off, int v_off, int heads, int kv_heads, int dim, int vdim,
                         int block_size, int num_blocks, const int* positions, const long long* slots, const void* q_norm, const void* k_norm,
                         const float* freq, int half, int halves, float gain, float eps, const void* v_first, long long ld_first, const void* share, int own_kv,
                         void* k_cache, void* v_cache, int* status, void* stream) {
  if (rows <= 0) return 0;
  if (2 * half > dim || kv_heads < 1 || heads % kv_heads || (v_first && !share)) return -2;
  GqaShape s{ldp, q_off, k_off, v_off, heads, kv_heads, dim, vdim, block_size, num_blocks, halves, own_kv};
  const ValueMix<float> mix32{static_cast<const float*>(v_first), ld_first, static_cast<const float*>(share)};
  const ValueMix<__nv_bfloat16> mix16{static_cast<const __nv_bfloat16*>(v_first), ld_first, static_cast<const __nv_bfloat16*>(share)};
  const int per_row = (heads + (own_kv ? 2 * kv_heads : 0) + GP_WARPS - 1) / GP_WARPS;
  const dim3 grid(static_cast<unsigned>(rows), rows >= 148 * 8 ? 1 : (per_row < 64 ? per_row : 64)), block(GP_WARPS * 32);
  const size_t sm = sizeof(float2) * half;
  if (sm > 48 * 1024) return -2;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (!f32 && dim % 2 == 0 && vdim % 2 == 0 && ldp % 2 == 0 && dim <= 256 && (q_off | k_off | v_off) % 2 == 0 && (!halves || half % 2 == 0) &&
      ld_first % 2 == 0 && reinterpret_cast<uintptr_t>(v_first) % 4 == 0 &&
      static_cast<long long>(num_blocks) * block_size < 0x7fffffffll) {
    const int share = (heads + (own_kv ? kv_heads : 0) + 3) / 4;
    const dim3 g(static_cast<unsigned>((rows + GP_WARPS - 1) / GP_WARPS), rows >= 148 * 16 ? 1 : (share < 64 ? share : 64));
    auto k = halves ? (dim <= 128 ? gqa_prep_rows_kernel<2, true> : gqa_prep_rows_kernel<4, true>)
                    : (dim <= 128 ? gqa_prep_rows_kernel<2, false> : gqa_prep_rows_kernel<4, false>);
    return static_cast<int>(rlb_launch_pdl(k, g, block, 0, st, static_cast<__nv_bfloat16*>(p), s, mix16, rows, positions, slots,
                                           static_cast<const __nv_bfloat16*>(q_norm), static_cast<const __nv_bfloat16*>(k_norm), freq, half, gain, eps,
                                           static_cast<__nv_bfloat16*>(k_cache), static_cast<__nv_bfloat16*>(v_cache), status));
  }
  if (f32)
    return static_cast<int>(rlb_launch_pdl(gqa_prep_kernel<float>, grid, block, sm, st, static_cast<float*>(p), s, mix32, positions, slots,
                                           static_cast<const float*>(q_norm), static_cast<const float*>(k_norm), freq, half, gain, eps,
                                           static_cast<float*>(k_cache), static_cast<float*>(v_cache), status));
  return static_cast<int>(rlb_launch_pdl(gqa_prep_kernel<__nv_bfloat16>, grid, block, sm, st, static_cast<__nv_bfloat16*>(p), s, mix16, positions, slots,
                                         static_cast<const __nv_bfloat16*>(q_norm), static_cast<const __nv_bfloat16*>(k_norm), freq, half, gain, eps,
                                         static_cast<__nv_bfloat16*>(k_cache), static_cast<__nv_bfloat16*>(v_cache), status));
}

RLB_API int rlb_gqa_rows(const void* p, int f32, int rows, long long ldp, int q_off, int heads, int kv_heads, int dim, int vdim, int block_size,
                         int num_blocks, const void* k_cache, const void* v_cache, const int* block_table, int bt_stride, const int* seq_lens,
                         int chunk, int window, int keep, const void* offset, int gated, float scale, void* y, long long ldy, int* status, void* stream) {
  if (rows <= 0) return 0;
  if (kv_heads < 1 || heads % kv_heads || heads > 65535 || dim + vdim > 12000 || (chunk > 0 && window > 0)) return -2;
  GqaShape s{ldp, q_off, 0, 0, heads, kv_heads, dim, vdim, block_size, num_blocks, 0, 0};
  const RowsMask mask{chunk, window, keep, gated};
  const size_t sm = sizeof(float) * ((dim + vdim + GR_TILE + 1) & ~1) + sizeof(long long) * GR_TILE;
  if (sm > 48 * 1024) return -2;
  const dim3 grid(rows, heads);
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (f32)
    gqa_rows_kernel<float><<<grid, 128, sm, st>>>(static_cast<const float*>(p), s, static_cast<const float*>(k_cache), static_cast<const float*>(v_cache),
                                                  block_table, bt_stride, seq_lens, mask, static_cast<const float*>(offset), scale, static_cast<float*>(y),
                                                  ldy, status);
  else
    gqa_rows_kernel<__nv_bfloat16><<<grid, 128, sm, st>>>(static_cast<const __nv_bfloat16*>(p), s, static_cast<const __nv_bfloat16*>(k_cache),
                                                          static_cast<const __nv_bfloat16*>(v_cache), block_table, bt_stride, seq_lens, mask,
                                                          static_cast<const __nv_bfloat16*>(offset), scale, static_cast<__nv_bfloat16*>(y), ldy, status);
  return static_cast<int>(cudaGetLastError());
}

RLB_API int rlb_gqa_gather(const void* k_cache, const void* v_cache, const long long* slots, void* out, long long n, int kv_heads, int dim, int vdim,
                           int block_size, long long num_slots, int* status, void* stream) {
  if (n <= 0) return 0;
  if (dim % 8 || vdim % 8) return -2;
  const long long want = (n * kv_heads * ((dim + vdim) / 8) + 255) / 256;
  gqa_gather_kernel<<<static_cast<unsigned>(want < 148 * 16 ? want : 148 * 16), 256, 0, static_cast<cudaStream_t>(stream)>>>(
      static_cast<const uint4*>(k_cache), static_cast<const uint4*>(v_cache), slots, static_cast<uint4*>(out), n, kv_heads, dim / 8, vdim / 8, block_size,
      num_slots, status);
  return static_cast<int>(cudaGetLastError());
}
