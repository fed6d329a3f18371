// Kernels of parallel mixer layers (models/mixers.py) that run for every size and for bf16 and fp32 models alike: the residual
// stream's start, a plain product with the layer epilogues, the latent-attention and retention mixers one row at a time.
//
// The batch of an engine step mixes single decoded tokens and portions of prompts; every row knows its position, its cache slot and
// its sequence's pages or state row, so nothing here depends on how a prompt was cut or on what else is in the batch. The mixers
// read their projections from the rows of the fused input product and write their gated output over the gate columns of the same
// rows, which the output product then reads in place.
//
// This file is compiled without fast math: tanh, sine, cosine, exponentials, square roots and divisions are the accurate ones.
// The tensor-core forms for bf16 are in latent_attention.cu, latent_decode.cu and retention.cu.
#include "common.cuh"

#include <math.h>

namespace {
using namespace rlb;

template <typename T>
__device__ __forceinline__ float ld(const T* p) {
  return static_cast<float>(*p);
}
template <>
__device__ __forceinline__ float ld<__nv_bfloat16>(const __nv_bfloat16* p) {
  return __bfloat162float(*p);
}
template <typename T>
__device__ __forceinline__ void st(T* p, float v) {
  *p = static_cast<T>(v);
}
template <>
__device__ __forceinline__ void st<__nv_bfloat16>(__nv_bfloat16* p, float v) {
  *p = __float2bfloat16(v);
}

// ---------------------------------------------------------------- start of the residual stream
// x = table[id] * scale (kept in e), + step; h = w * tanh(alpha x) + b, or x / rms(x) * w (alpha null), or x itself (no norm)
template <typename T>
__global__ void embed_rows_kernel(const void* ids, int ids64, const T* __restrict__ table, float* __restrict__ x, float* __restrict__ e,
                                  T* __restrict__ h, const T* __restrict__ step, const T* __restrict__ alpha, const T* __restrict__ nw,
                                  const T* __restrict__ nb, int d, int vocab, float scale, float eps, int* status) {
  __shared__ float red[32];
  const long long row = blockIdx.x;
  long long id = ids64 ? static_cast<const long long*>(ids)[row] : static_cast<const int*>(ids)[row];
  if (id < 0 || id >= vocab) {
    if (threadIdx.x == 0 && status) atomicCAS(status, 0, RLB_ERR_BOUNDS);
    id = 0;
  }
  const float a = alpha ? ld(alpha) : 0.f;
  float ss = 0.f;
  for (int c = threadIdx.x; c < d; c += blockDim.x) {
    float v = ld(table + id * d + c) * scale;
    if (e) e[row * d + c] = v;
    if (step) v += ld(step + c);
    x[row * d + c] = v;
    ss += v * v;
    if (alpha || !nw) st(h + row * d + c, alpha ? tanhf(a * v) * ld(nw + c) + ld(nb + c) : v);
  }
  if (alpha || !nw) return;
  ss = block_sum(ss, red);
  const float rstd = 1.f / sqrtf(ss / static_cast<float>(d) + eps);
  for (int c = threadIdx.x; c < d; c += blockDim.x) st(h + row * d + c, x[row * d + c] * rstd * ld(nw + c));     // (each thread reads what it wrote)
}

// The same without a loop's copies and steps, d a multiple of 4 and at most 4 * EM_KEEP * EM_THREADS: h = x, or x / rms(x) * w. A thread keeps its
// columns in registers, all loads are issued before the first is used.
constexpr int EM_THREADS = 512, EM_KEEP = 4;
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
template <typename T>
__global__ void __launch_bounds__(EM_THREADS)
embed_wide_kernel(const void* ids, int ids64, const T* __restrict__ table, float* __restrict__ x, T* __restrict__ h, const T* __restrict__ nw, int d,
                  int vocab, float scale, float eps, int* status) {
  __shared__ float red[32];
  const long long row = blockIdx.x;
  const int n = blockDim.x;
  float4 w[EM_KEEP], v[EM_KEEP];
#pragma unroll
  for (int i = 0; i < EM_KEEP; ++i) {
    const int c = (threadIdx.x + i * n) * 4;
    w[i] = nw && c < d ? ld4(nw + c) : make_float4(1.f, 1.f, 1.f, 1.f);
  }
  long long id = ids64 ? static_cast<const long long*>(ids)[row] : static_cast<const int*>(ids)[row];
  if (id < 0 || id >= vocab) {
    if (threadIdx.x == 0 && status) atomicCAS(status, 0, RLB_ERR_BOUNDS);
    id = 0;
  }
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < EM_KEEP; ++i) {
    const int c = (threadIdx.x + i * n) * 4;
    v[i] = c < d ? ld4(table + id * d + c) : make_float4(0.f, 0.f, 0.f, 0.f);
  }
#pragma unroll
  for (int i = 0; i < EM_KEEP; ++i) {
    const int c = (threadIdx.x + i * n) * 4;
    v[i] = make_float4(v[i].x * scale, v[i].y * scale, v[i].z * scale, v[i].w * scale);
    ss += v[i].x * v[i].x + v[i].y * v[i].y + v[i].z * v[i].z + v[i].w * v[i].w;
    if (c < d) st4(x + row * d + c, v[i]);
  }
  float f = 1.f;
  if (nw) f = 1.f / sqrtf(block_sum(ss, red) / static_cast<float>(d) + eps);
#pragma unroll
  for (int i = 0; i < EM_KEEP; ++i) {
    const int c = (threadIdx.x + i * n) * 4;
    if (c < d) st4(h + row * d + c, make_float4(v[i].x * f * w[i].x, v[i].y * f * w[i].y, v[i].z * f * w[i].z, v[i].w * f * w[i].w));
  }
}

// ---------------------------------------------------------------- product with the layer epilogues
struct RowsGemm {
  const void* a;
  const void* w;
  void* out;
  int M, N, K;
  long long lda, ldw, ldo;
  int act_from;        // squared ReLU on columns >= act_from
  float* x;            // residual stream (null: plain store): x += acc (+ e) (+ step), out = dynamic tanh of x
  long long ldx;
  const float* e;
  const void* step;
  const void* alpha;
  const void* nw;
  const void* nb;
  LinearEpi lin;
  const int* tile_expert;   // expert of each 128-row tile (null: one weight); its weight starts expert * N * ldw further on
  const int* a_rows;        // row of `a` that each row reads (-1 or out of range: zeros); null: its own
  int num_a_rows;
};

constexpr int RG_T = 64, RG_K = 16;

template <typename TI, typename TO>
__global__ void __launch_bounds__(256) gemm_rows_kernel(RowsGemm g) {
  __shared__ float as[RG_K][RG_T + 4], ws[RG_K][RG_T + 4];
  const TI* A = static_cast<const TI*>(g.a);
  const TI* W = static_cast<const TI*>(g.w);
  const int m0 = blockIdx.y * RG_T, n0 = blockIdx.x * RG_T;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  if (g.tile_expert) {
    const int e = g.tile_expert[m0 / 128];
    if (e < 0) return;
    W += static_cast<long long>(e) * g.N * g.ldw;
  }
  float acc[4][4] = {};
  for (int k0 = 0; k0 < g.K; k0 += RG_K) {
    for (int i = threadIdx.x; i < RG_T * RG_K; i += 256) {
      const int r = i / RG_K, k = i % RG_K;
      int row = m0 + r < g.M ? m0 + r : -1;
      if (g.a_rows && row >= 0) {
        row = g.a_rows[row];
        if (row >= g.num_a_rows) row = -1;
      }
      as[k][r] = (row >= 0 && k0 + k < g.K) ? ld(A + static_cast<long long>(row) * g.lda + k0 + k) : 0.f;
      ws[k][r] = (n0 + r < g.N && k0 + k < g.K) ? ld(W + static_cast<long long>(n0 + r) * g.ldw + k0 + k) : 0.f;
    }
    __syncthreads();
    float part[4][4] = {};      // summed apart: chains of RG_K terms round less than one of K
#pragma unroll
    for (int k = 0; k < RG_K; ++k) {
      float av[4], wv[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        av[i] = as[k][ty * 4 + i];
        wv[i] = ws[k][tx * 4 + i];
      }
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) part[i][j] = fmaf(av[i], wv[j], part[i][j]);
    }
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) acc[i][j] += part[i][j];
    __syncthreads();
  }
  const float alpha = g.x ? ld(static_cast<const TI*>(g.alpha)) : 0.f;
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int m = m0 + ty * 4 + i;
    if (m >= g.M) continue;
    if (g.lin.row_scale) {
      const float f = g.lin.row_scale[m];
#pragma unroll
      for (int j = 0; j < 4; ++j) acc[i][j] *= f;
    }
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int n = n0 + tx * 4 + j;
      if (n >= g.N) continue;
      float v = acc[i][j];
      if (g.lin.bias) v += ld(static_cast<const TI*>(g.lin.bias) + n);
      if (lin_gated(g.lin.act)) {          // N is even: the pair of an even column is there
        if (j & 1) continue;
        float u = acc[i][j + 1];
        if (g.lin.bias) u += ld(static_cast<const TI*>(g.lin.bias) + n + 1);
        st(static_cast<TO*>(g.out) + static_cast<long long>(m) * g.ldo + n / 2, gated_unit(g.lin.act, v, u, g.lin.limit));
        continue;
      }
      if (g.lin.act == LIN_GELU_MUL) {
        const TI* t = static_cast<const TI*>(g.lin.table) + lin_token(g.lin, m) * g.lin.ld_table + g.lin.table_off;
        v = n < g.lin.table_cols ? 0.5f * v * (1.f + tanhf(0.7978845608028654f * (v + 0.044715f * v * v * v))) * ld(t + n) : 0.f;
      } else if (g.lin.act == LIN_CAP) {
        v *= g.lin.scale;
        if (g.lin.cap > 0.f) v = g.lin.cap * tanhf(v / g.lin.cap);
      }
      TO* o = static_cast<TO*>(g.out) + static_cast<long long>(m) * g.ldo + n;
      if (g.x) {
        float* xp = g.x + static_cast<long long>(m) * g.ldx + n;
        v += *xp;
        if (g.e) v += g.e[static_cast<long long>(m) * g.ldx + n];
        if (g.step) v += ld(static_cast<const TI*>(g.step) + n);
        *xp = v;
        v = tanhf(alpha * v) * ld(static_cast<const TI*>(g.nw) + n) + ld(static_cast<const TI*>(g.nb) + n);
      } else if (n >= g.act_from) {
        v = fmaxf(v, 0.f);
        v *= v;
      }
      st(o, v);
    }
  }
}

// ---------------------------------------------------------------- latent attention
struct LatentShape {
  long long ldp, ldq, ldo;             // row strides of the rows with the latent, of the queries, of the output
  int q_off, lat_off, mix_off;         // columns of queries, latent and output
  int heads, dim, rot_dim, vdim, rank; // per head: dim unrotated + rot_dim rotated query / key dimensions
  int width;                           // row width of the latent cache
  int block_size, num_blocks;
  int halves;                          // rotated pairs are (i, i + half) instead of (2i, 2i + 1)
  int gated;                           // the output columns hold gates: out = y * sigmoid(gate)
};

// Two CTAs per row. blockIdx.y 0: latent / rms * w and the rotated shared key into the cache row of the token. blockIdx.y 1: the
// rotated query parts, in place, and for the first `q_rows` rows also behind the latent columns of q_lat [rows, heads, width]
// (the decode kernels' queries). Few rows are a matter of latency: every load is issued before the first is used, angles are computed
// by the thread that needs them.
constexpr int LP_KEEP = 8;     // latent columns a thread keeps in registers
template <typename T>
__global__ void __launch_bounds__(128)
latent_prep_kernel(const T* __restrict__ p, T* __restrict__ queries, LatentShape s, const int* __restrict__ positions, const long long* __restrict__ slots,
                   const T* __restrict__ norm_w, const float* __restrict__ freq, int half, float gain, float eps,
                   T* __restrict__ cache, T* __restrict__ q_lat, int q_rows, int* status) {
  __shared__ float red[32];
  const int tid = threadIdx.x;
  pdl_sync();
  const long long row = blockIdx.x;
  const float pos = static_cast<float>(positions[row]);
  if (blockIdx.y == 1) {
    const int tail = s.width - s.rank, pairs = (tail + 1) / 2, qd = s.dim + s.rot_dim;
    const bool decode = q_lat && row < q_rows;
    T* qr = queries + row * s.ldq + s.q_off + s.dim;
    if (s.halves) {      // a thread turns pairs (f, f + half), or passes on a column behind the rotated ones
      const int units = tail - half;
      for (int i = tid; i < s.heads * units; i += 128) {
        const int h = i / units, f = i % units;
        T* q = qr + h * qd;
        T* o = q_lat + (row * s.heads + h) * s.width + s.rank;
        if (f >= half) {
          if (decode) st(o + f + half, f + half < s.rot_dim ? ld(q + f + half) : 0.f);
          continue;
        }
        const float u = ld(q + f), v = ld(q + f + half);
        float sn, c;
        sincosf(pos * freq[f], &sn, &c);
        c *= gain;
        sn *= gain;
        const float a = u * c - v * sn, b = v * c + u * sn;
        st(q + f, a);
        st(q + f + half, b);
        if (decode) {
          st(o + f, a);
          st(o + f + half, b);
        }
      }
      return;
    }
    for (int i = tid; i < s.heads * pairs; i += 128) {
      const int h = i / pairs, f = i % pairs, j = 2 * f;
      T* q = qr + h * qd + j;
      float u = j < s.rot_dim ? ld(q) : 0.f, v = j + 1 < s.rot_dim ? ld(q + 1) : 0.f;
      if (f < half) {
        float sn, c;
        sincosf(pos * freq[f], &sn, &c);
        c *= gain;
        sn *= gain;
        const float a = u * c - v * sn, b = v * c + u * sn;
        st(q, a);
        st(q + 1, b);
        u = a;
        v = b;
      }
      if (decode) {
        T* o = q_lat + (row * s.heads + h) * s.width + s.rank + j;
        st(o, u);
        if (j + 1 < tail) st(o + 1, v);
      }
    }
    return;
  }
  const long long slot = slots[row];
  const T* lat = p + row * s.ldp + s.lat_off;
  float keep[LP_KEEP];
  float ss = 0.f;
#pragma unroll
  for (int k = 0; k < LP_KEEP; ++k) {
    const int r = tid + k * 128;
    keep[k] = r < s.rank ? ld(lat + r) : 0.f;
  }
#pragma unroll
  for (int k = 0; k < LP_KEEP; ++k) ss += keep[k] * keep[k];
  for (int r = tid + LP_KEEP * 128; r < s.rank; r += 128) {
    const float v = ld(lat + r);
    ss += v * v;
  }
  const bool bad = slot >= static_cast<long long>(s.num_blocks) * s.block_size;
  if (bad && tid == 0 && status) atomicCAS(status, 0, RLB_ERR_BOUNDS);
  T* cr = cache + slot * s.width;
  if (slot >= 0 && !bad) {
    for (int j = tid; j < s.width - s.rank; j += 128) {      // rotated key part, then padding
      float v = j < s.rot_dim ? ld(lat + s.rank + j) : 0.f;
      if (j < 2 * half) {
        const bool second = s.halves ? j >= half : (j & 1);
        float sn, c;
        sincosf(pos * freq[s.halves ? j - (second ? half : 0) : j >> 1], &sn, &c);
        const float o = ld(lat + s.rank + (s.halves ? (second ? j - half : j + half) : (j ^ 1)));
        v = (second ? v * c + o * sn : v * c - o * sn) * gain;
      }
      st(cr + s.rank + j, v);
    }
  }
  ss = block_sum(ss, red);
  if (slot < 0 || bad) return;
  const float rstd = 1.f / sqrtf(ss / static_cast<float>(s.rank) + eps);
#pragma unroll
  for (int k = 0; k < LP_KEEP; ++k) {
    const int r = tid + k * 128;
    if (r < s.rank) st(cr + r, keep[k] * rstd * ld(norm_w + r));
  }
  for (int r = tid + LP_KEEP * 128; r < s.rank; r += 128) st(cr + r, ld(lat + r) * rstd * ld(norm_w + r));
}

// One CTA per (row, head): the query is carried into the latent space (q^T W_uk), the keys are the cached rows, the weighted
// latent is carried to the values (W_uv), and gated where the output columns hold gates. Everything in fp32.
constexpr int LR_TILE = 128;
template <typename T>
__global__ void __launch_bounds__(128)
latent_rows_kernel(const T* queries, T* out, LatentShape s, const T* __restrict__ cache, const int* __restrict__ block_table, int bt_stride,
                   const int* __restrict__ seq_lens, const T* __restrict__ kv_up, float scale, int* status) {
  extern __shared__ float sm[];
  __shared__ float red[32];
  float* qa = sm;                       // [width]
  float* o = qa + s.width;              // [rank]
  float* sc = o + s.rank;               // [LR_TILE]
  long long* rows = reinterpret_cast<long long*>(sm + ((s.width + s.rank + LR_TILE + 1) & ~1));   // [LR_TILE]
  const int row = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const T* q = queries + row * s.ldq + s.q_off + h * (s.dim + s.rot_dim);
  for (int r = tid; r < s.width; r += 128) {
    float v = 0.f;
    if (r < s.rank) {
      for (int d = 0; d < s.dim; ++d) v = fmaf(ld(q + d), ld(kv_up + static_cast<long long>(h * s.dim + d) * s.rank + r), v);
    } else if (r < s.rank + s.rot_dim) {
      v = ld(q + s.dim + r - s.rank);
    }
    qa[r] = v * scale;
  }
  for (int r = tid; r < s.rank; r += 128) o[r] = 0.f;
  const int len = min(seq_lens[row], bt_stride * s.block_size);
  float m = -INFINITY, l = 0.f;
  for (int t0 = 0; t0 < len; t0 += LR_TILE) {
    const int n = min(LR_TILE, len - t0);
    __syncthreads();
    if (tid < n) {
      const int t = t0 + tid;
      int blk = block_table[static_cast<long long>(row) * bt_stride + t / s.block_size];
      if (blk < 0 || blk >= s.num_blocks) {
        if (status) atomicCAS(status, 0, RLB_ERR_BOUNDS);
        blk = 0;
      }
      rows[tid] = (static_cast<long long>(blk) * s.block_size + t % s.block_size) * s.width;
    }
    __syncthreads();
    for (int j = warp; j < n; j += 4) {
      const T* cr = cache + rows[j];
      float v = 0.f;
      for (int r = lane; r < s.width; r += 32) v = fmaf(qa[r], ld(cr + r), v);
      v = warp_sum(v);
      if (lane == 0) sc[j] = v;
    }
    __syncthreads();
    const float mine = tid < n ? sc[tid] : -INFINITY;
    const float mn = fmaxf(m, block_max(mine, red));
    const float pj = tid < n ? expf(mine - mn) : 0.f;
    const float c = m == -INFINITY ? 0.f : expf(m - mn);
    l = l * c + block_sum(pj, red);
    m = mn;
    if (tid < n) sc[tid] = pj;
    __syncthreads();
    for (int r = tid; r < s.rank; r += 128) {
      float v = o[r] * c;
      for (int j = 0; j < n; ++j) v = fmaf(sc[j], ld(cache + rows[j] + r), v);
      o[r] = v;
    }
  }
  __syncthreads();
  const float inv = l > 0.f ? 1.f / l : 0.f;
  for (int v = warp; v < s.vdim; v += 4) {
    const T* w = kv_up + static_cast<long long>(s.heads * s.dim + h * s.vdim + v) * s.rank;
    float y = 0.f;
    for (int r = lane; r < s.rank; r += 32) y = fmaf(o[r], ld(w + r), y);
    y = warp_sum(y) * inv;
    if (lane == 0) {
      T* g = out + row * s.ldo + s.mix_off + h * s.vdim + v;
      st(g, s.gated ? y / (1.f + expf(-ld(g))) : y);
    }
  }
}

// ---------------------------------------------------------------- retention
struct RetentionShape {
  long long ldp;
  int q_off, k_off, v_off, mix_off;
  int heads, dim, vdim;
};

// One CTA per (sequence piece, head), token after token: S = decay S + k v^T, o = S^T q, unit RMS over the head, SiLU gate. A piece
// whose first token stands at position 0 starts from a zero state, whatever its state row held before.
template <typename T>
__global__ void __launch_bounds__(256)
retention_rows_kernel(T* __restrict__ p, RetentionShape s, int row0, const int* __restrict__ cu, const int* __restrict__ positions,
                      const long long* __restrict__ state_rows, float* __restrict__ state, long long num_states,
                      const float* __restrict__ decay, const float* __restrict__ freq, int half, float gain, float kscale, float eps, int* status) {
  extern __shared__ float sm[];
  __shared__ float red[32];
  float* q = sm;                 // [dim]
  float* k = q + s.dim;          // [dim]
  float* o = k + s.dim;          // [vdim]
  float* part = o + s.vdim;      // [256] partial sums over slices of dim (vdim < 256)
  const int seq = blockIdx.x, h = blockIdx.y, tid = threadIdx.x;
  const int begin = cu ? cu[seq] : seq, end = cu ? cu[seq + 1] : seq + 1;
  const long long sr = state_rows[seq];
  if (sr < 0 || sr >= num_states) {
    if (tid == 0 && status) atomicCAS(status, 0, RLB_ERR_BOUNDS);
    return;
  }
  float* S = state + (sr * s.heads + h) * static_cast<long long>(s.dim) * s.vdim;
  const float dec = decay[h];
  const int slices = s.vdim >= 256 ? 1 : 256 / s.vdim;
  const int slice = s.vdim >= 256 ? 0 : tid / s.vdim;
  for (int t = begin; t < end; ++t) {
    T* pr = p + (row0 + t) * s.ldp;
    const float pos = static_cast<float>(positions[row0 + t]);
    const bool fresh = positions[row0 + t] == 0;
    for (int i = tid; i < s.dim; i += 256) {
      float qv = ld(pr + s.q_off + h * s.dim + i), kv = ld(pr + s.k_off + h * s.dim + i);
      if (i < 2 * half) {
        const int f = i < half ? i : i - half, oi = i < half ? i + half : i - half;
        float sn, c;
        sincosf(pos * freq[f], &sn, &c);
        c *= gain;
        sn *= i < half ? -gain : gain;
        qv = qv * c + ld(pr + s.q_off + h * s.dim + oi) * sn;
        kv = kv * c + ld(pr + s.k_off + h * s.dim + oi) * sn;
      }
      q[i] = qv;
      k[i] = kv * kscale;
    }
    __syncthreads();
    if (slice < slices) {
      for (int v = s.vdim >= 256 ? tid : tid % s.vdim; v < s.vdim; v += 256) {
        const float vv = ld(pr + s.v_off + h * s.vdim + v);
        float acc = 0.f;
        for (int i = slice; i < s.dim; i += slices) {
          float* sp = S + static_cast<long long>(i) * s.vdim + v;
          const float nv = fresh ? k[i] * vv : fmaf(dec, *sp, k[i] * vv);
          *sp = nv;
          acc = fmaf(nv, q[i], acc);
        }
        if (slices > 1) {
          part[tid] = acc;
          break;
        }
        o[v] = acc;
      }
    }
    __syncthreads();
    if (slices > 1 && tid < s.vdim) {
      float acc = 0.f;
      for (int j = 0; j < slices; ++j) acc += part[j * s.vdim + tid];
      o[tid] = acc;
    }
    float ss = 0.f;
    for (int v = tid; v < s.vdim; v += 256) ss += o[v] * o[v];   // each thread reads what it wrote
    ss = block_sum(ss, red);
    const float rstd = 1.f / sqrtf(ss / static_cast<float>(s.vdim) + eps);
    for (int v = tid; v < s.vdim; v += 256) {
      T* g = pr + s.mix_off + h * s.vdim + v;
      const float gv = ld(g);
      st(g, o[v] * rstd * (gv / (1.f + expf(-gv))));
    }
    __syncthreads();
  }
}

int launch_rows(const RowsGemm& g, int in_f32, int out_f32, cudaStream_t s) {
  const dim3 grid((g.N + RG_T - 1) / RG_T, (g.M + RG_T - 1) / RG_T);
  if (grid.y > 65535) return -2;
  if (in_f32 && out_f32) gemm_rows_kernel<float, float><<<grid, 256, 0, s>>>(g);
  else if (in_f32) gemm_rows_kernel<float, __nv_bfloat16><<<grid, 256, 0, s>>>(g);
  else if (out_f32) gemm_rows_kernel<__nv_bfloat16, float><<<grid, 256, 0, s>>>(g);
  else gemm_rows_kernel<__nv_bfloat16, __nv_bfloat16><<<grid, 256, 0, s>>>(g);
  return static_cast<int>(cudaGetLastError());
}

int smem_attr(const void* kernel, size_t bytes) {
  if (bytes <= 48 * 1024) return 0;
  if (bytes > 220 * 1024) return -2;
  return static_cast<int>(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(bytes)));
}
}  // namespace

RLB_API int rlb_embed_rows(const void* ids, int ids64, const void* table, int f32, float* x, float* e, void* h, const void* step,
                           const void* alpha, const void* nw, const void* nb, long long rows, int d, int vocab, float scale, float eps, int* status,
                           void* stream) {
  if (rows <= 0) return 0;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (!e && !step && !alpha && d % 4 == 0 && d <= 4 * EM_KEEP * EM_THREADS) {
    const int threads = d > 4096 ? EM_THREADS : (d > 1024 ? 256 : 128);
    if (f32)
      embed_wide_kernel<float><<<static_cast<unsigned>(rows), threads, 0, s>>>(ids, ids64, static_cast<const float*>(table), x, static_cast<float*>(h),
                                                                               static_cast<const float*>(nw), d, vocab, scale, eps, status);
    else
      embed_wide_kernel<__nv_bfloat16><<<static_cast<unsigned>(rows), threads, 0, s>>>(ids, ids64, static_cast<const __nv_bfloat16*>(table), x,
                                                                                       static_cast<__nv_bfloat16*>(h), static_cast<const __nv_bfloat16*>(nw), d,
                                                                                       vocab, scale, eps, status);
    return static_cast<int>(cudaGetLastError());
  }
  if (f32)
    embed_rows_kernel<float><<<static_cast<unsigned>(rows), 256, 0, s>>>(ids, ids64, static_cast<const float*>(table), x, e, static_cast<float*>(h),
        static_cast<const float*>(step), static_cast<const float*>(alpha), static_cast<const float*>(nw), static_cast<const float*>(nb), d, vocab, scale, eps, status);
  else
    embed_rows_kernel<__nv_bfloat16><<<static_cast<unsigned>(rows), 256, 0, s>>>(ids, ids64, static_cast<const __nv_bfloat16*>(table), x, e,
        static_cast<__nv_bfloat16*>(h), static_cast<const __nv_bfloat16*>(step), static_cast<const __nv_bfloat16*>(alpha),
        static_cast<const __nv_bfloat16*>(nw), static_cast<const __nv_bfloat16*>(nb), d, vocab, scale, eps, status);
  return static_cast<int>(cudaGetLastError());
}

// out = A W^T for any sizes (A, W both bf16 or both fp32; out bf16 or fp32), squared ReLU on columns >= act_from. With `x`:
// x += A W^T (+ e) (+ step) in place (fp32, row stride ldx, as is e) and out = nw * tanh(alpha x) + nb.
RLB_API int rlb_gemm_rows(const void* a, const void* w, void* out, int M, int N, int K, long long lda, long long ldw, long long ldo, int in_f32,
                          int out_f32, int act_from, float* x, long long ldx, const float* e, const void* step, const void* alpha,
                          const void* nw, const void* nb, void* stream) {
  if (M <= 0 || N <= 0 || K <= 0) return 0;
  if (x && (!alpha || !nw || !nb)) return -2;
  RowsGemm g{a, w, out, M, N, K, lda, ldw, ldo, act_from, x, ldx, e, step, alpha, nw, nb, LinearEpi{}, nullptr, nullptr, 0};
  return launch_rows(g, in_f32, out_f32, static_cast<cudaStream_t>(stream));
}

// The product of RlbLinear for any sizes, bf16 or fp32, one weight or one per expert.
RLB_API int rlb_linear_rows(const RlbLinear* l, void* stream) {
  if (l->M <= 0 || l->N <= 0 || l->K <= 0) return 0;
  if ((lin_gated(l->act) && l->N % 2) || (l->tile_expert && l->M % 128)) return -2;
  RowsGemm g{l->a, l->w, l->out, l->M, l->N, l->K, l->lda, l->ldw, l->ldo, 1 << 30, nullptr, 0, nullptr, nullptr, nullptr, nullptr, nullptr,
             rlb_linear_epi(*l), l->tile_expert, l->a_rows, l->num_a_rows};
  return launch_rows(g, l->in_f32, l->out_f32, static_cast<cudaStream_t>(stream));
}

// p: rows with the latent (lat_off) and the shared key part behind it; q: rows with the queries (may be p). halves: rotated pairs are
// (i, i + half) instead of (2i, 2i + 1).
RLB_API int rlb_latent_prep(const void* p, int f32, long long rows, long long ldp, int lat_off, void* q, long long ldq, int q_off, int heads, int dim,
                            int rot_dim, int rank, int width, int block_size, int num_blocks, const int* positions, const long long* slots,
                            const void* norm_w, const float* freq, int half, int halves, float gain, float eps, void* cache, void* q_lat, int q_rows,
                            int* status, void* stream) {
  if (rows <= 0) return 0;
  if (2 * half > rot_dim || rank + rot_dim > width) return -2;
  LatentShape s{ldp, ldq, 0, q_off, lat_off, 0, heads, dim, rot_dim, 0, rank, width, block_size, num_blocks, halves, 0};
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const dim3 grid(static_cast<unsigned>(rows), 2), block(128);
  if (f32)
    rlb_launch_pdl(latent_prep_kernel<float>, grid, block, 0, st, static_cast<const float*>(p), static_cast<float*>(q), s, positions, slots,
                   static_cast<const float*>(norm_w), freq, half, gain, eps, static_cast<float*>(cache), static_cast<float*>(q_lat), q_rows, status);
  else
    rlb_launch_pdl(latent_prep_kernel<__nv_bfloat16>, grid, block, 0, st, static_cast<const __nv_bfloat16*>(p), static_cast<__nv_bfloat16*>(q), s, positions, slots,
        static_cast<const __nv_bfloat16*>(norm_w), freq, half, gain, eps, static_cast<__nv_bfloat16*>(cache),
        static_cast<__nv_bfloat16*>(q_lat), q_rows, status);
  return static_cast<int>(cudaGetLastError());
}

// q: prepared queries; out (row stride ldo, may be the same rows): head outputs from column mix_off, gated by what stands there when `gated`.
RLB_API int rlb_latent_rows(const void* q, int f32, int rows, long long ldq, int q_off, void* out, long long ldo, int mix_off, int gated, int heads, int dim, int rot_dim, int vdim, int rank,
                            int width, int block_size, int num_blocks, const void* cache, const int* block_table, int bt_stride,
                            const int* seq_lens, const void* kv_up, float scale, int* status, void* stream) {
  if (rows <= 0) return 0;
  if (rank + rot_dim > width || heads > 65535) return -2;
  LatentShape s{0, ldq, ldo, q_off, 0, mix_off, heads, dim, rot_dim, vdim, rank, width, block_size, num_blocks, 0, gated};
  const size_t sm = sizeof(float) * ((width + rank + LR_TILE + 1) & ~1) + sizeof(long long) * LR_TILE;
  const dim3 grid(rows, heads);
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  int rc;
  if (f32) {
    if ((rc = smem_attr(reinterpret_cast<const void*>(latent_rows_kernel<float>), sm))) return rc;
    latent_rows_kernel<float><<<grid, 128, sm, st>>>(static_cast<const float*>(q), static_cast<float*>(out), s, static_cast<const float*>(cache), block_table, bt_stride, seq_lens,
                                                     static_cast<const float*>(kv_up), scale, status);
  } else {
    if ((rc = smem_attr(reinterpret_cast<const void*>(latent_rows_kernel<__nv_bfloat16>), sm))) return rc;
    latent_rows_kernel<__nv_bfloat16><<<grid, 128, sm, st>>>(static_cast<const __nv_bfloat16*>(q), static_cast<__nv_bfloat16*>(out), s, static_cast<const __nv_bfloat16*>(cache), block_table,
                                                             bt_stride, seq_lens, static_cast<const __nv_bfloat16*>(kv_up), scale, status);
  }
  return static_cast<int>(cudaGetLastError());
}

// `cu` (offsets of the pieces, counted from row0) null: piece i is the single row row0 + i.
RLB_API int rlb_retention_rows(void* p, int f32, int row0, int pieces, long long ldp, int q_off, int k_off, int v_off, int mix_off, int heads,
                               int dim, int vdim, const int* cu, const int* positions, const long long* state_rows, float* state,
                               long long num_states, const float* decay, const float* freq, int half, float gain, float kscale, float eps,
                               int* status, void* stream) {
  if (pieces <= 0) return 0;
  if (2 * half > dim || heads > 65535) return -2;
  RetentionShape s{ldp, q_off, k_off, v_off, mix_off, heads, dim, vdim};
  const size_t sm = sizeof(float) * (2 * dim + vdim + 256);
  const dim3 grid(pieces, heads);
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  int rc;
  if (f32) {
    if ((rc = smem_attr(reinterpret_cast<const void*>(retention_rows_kernel<float>), sm))) return rc;
    retention_rows_kernel<float><<<grid, 256, sm, st>>>(static_cast<float*>(p), s, row0, cu, positions, state_rows, state, num_states, decay, freq, half,
                                                        gain, kscale, eps, status);
  } else {
    if ((rc = smem_attr(reinterpret_cast<const void*>(retention_rows_kernel<__nv_bfloat16>), sm))) return rc;
    retention_rows_kernel<__nv_bfloat16><<<grid, 256, sm, st>>>(static_cast<__nv_bfloat16*>(p), s, row0, cu, positions, state_rows, state, num_states,
                                                                decay, freq, half, gain, kscale, eps, status);
  }
  return static_cast<int>(cudaGetLastError());
}
