// Retention (linear attention with one fixed decay per head) for bf16 models: the decode step, and prompt portions chunk by chunk on
// the 5th-generation tensor cores (tcgen05 + TMEM + TMA).
//
// Chunk form, for chunks of 128 tokens with start state S0 (i, j count inside the chunk, d the head's decay):
//     out_i   = sum_{j <= i} d^(i-j) (q_i . k_j) v_j + d^(i+1) S0^T q_i
//     S0 next = d^n S0 + sum_j d^(n-1-j) k_j v_j^T
//   retention_state   per (chunk, head): the sum over j, D[dim, vdim] = (weighted K)^T V
//   retention_scan    per piece: turns the chunks' sums into their start states, advances the sequence's state row
//   retention_out     per (chunk, head): scores, decays, both output terms, unit-RMS norm over the head, SiLU gate, store
// Everything that enters the recurrence is 32-bit: rotated queries and keys, decayed weights and states are split into two bf16
// parts (hi + lo, 16 mantissa bits and more) and multiplied as hi*hi + hi*lo + lo*hi with fp32 accumulation; values are projections and exact
// in bf16. The operands are rotated, weighted, split and swizzled by the CTA that consumes them, straight from the projected rows.
//
// Decode: one CTA per (row, head) streams the fp32 state once (read, decay, rank-one update, write, dot with q).
//
// This file is compiled without fast math.
#include "recurrent.cuh"

#include <math.h>

namespace {
using namespace rlb;

struct RetShape {
  __nv_bfloat16* p;       // projected rows
  long long ldp;
  int q_off, k_off, v_off, mix_off;
  int heads, dim, vdim;
  int row0;               // first row of the portions
  const int* chunk_row;   // [chunks] first row, counted from row0
  const int* chunk_rows;  // [chunks] rows
  const float* cs;        // [rows from row0, 2 * half] cosine | sine (gain included)
  int half;
  float kscale, eps;
  const float* log2_decay;
  float* sums;            // [chunks, heads, dim, vdim]: sums of the chunks, after the scan their start states
  int* status;
};

constexpr int RT_THREADS = 512;

__global__ void rotation_table_kernel(const int* __restrict__ positions, const float* __restrict__ freq, int half, float gain, float* __restrict__ cs,
                                      long long n) {
  for (long long i = static_cast<long long>(blockIdx.x) * blockDim.x + threadIdx.x; i < n * half; i += static_cast<long long>(gridDim.x) * blockDim.x) {
    const long long t = i / half;
    const int f = static_cast<int>(i - t * half);
    float s, c;
    sincosf(static_cast<float>(positions[t]) * freq[f], &s, &c);
    cs[t * 2 * half + f] = c * gain;
    cs[t * 2 * half + half + f] = s * gain;
  }
}

// Eight consecutive dimensions d0.. of one head's row: the raw piece and, where the halves layout rotates whole pieces, its partner.
struct RawPiece {
  uint4 own, other;
};
__device__ __forceinline__ RawPiece load_piece(const __nv_bfloat16* row, int d0, int half) {
  RawPiece r;
  r.own = *reinterpret_cast<const uint4*>(row + d0);
  if (d0 < 2 * half && half % 8 == 0) r.other = *reinterpret_cast<const uint4*>(row + (d0 < half ? d0 + half : d0 - half));
  else r.other = make_uint4(0, 0, 0, 0);
  return r;
}
// The rotation of that piece in fp32 (d0 a multiple of 8).
__device__ __forceinline__ void rotate_piece(const RawPiece& raw, const __nv_bfloat16* row, int d0, int half, const float* cs, float (&v)[8]) {
  unpack8(raw.own, v);
  if (d0 >= 2 * half) return;
  if (half % 8 == 0) {
    const bool low = d0 < half;
    const int f0 = low ? d0 : d0 - half;
    const float4 c0 = *reinterpret_cast<const float4*>(cs + f0), c1 = *reinterpret_cast<const float4*>(cs + f0 + 4);
    const float4 s0 = *reinterpret_cast<const float4*>(cs + half + f0), s1 = *reinterpret_cast<const float4*>(cs + half + f0 + 4);
    const float c[8] = {c0.x, c0.y, c0.z, c0.w, c1.x, c1.y, c1.z, c1.w}, s[8] = {s0.x, s0.y, s0.z, s0.w, s1.x, s1.y, s1.z, s1.w};
    float o[8];
    unpack8(raw.other, o);
#pragma unroll
    for (int i = 0; i < 8; ++i) v[i] = low ? v[i] * c[i] - o[i] * s[i] : v[i] * c[i] + o[i] * s[i];
  } else {
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      const int d = d0 + i;
      if (d >= 2 * half) break;
      const bool low = d < half;
      const int f = low ? d : d - half;
      const float o = __bfloat162float(row[low ? d + half : d - half]);
      v[i] = low ? v[i] * cs[f] - o * cs[half + f] : v[i] * cs[f] + o * cs[half + f];
    }
  }
}

// One 64-dimension atom [128 rows x 64] of rotated, scaled queries or keys, split into hi and lo; rows past the chunk and dimensions past
// dim are zero. `weight` (null or [128]) multiplies the rows. All loads of a thread are issued before the first is used: `fetch` and
// `store` are separate so that a caller can have several atoms in flight.
constexpr int RT_FILL = RT_C * 8 / RT_THREADS;
struct AtomFill {
  RawPiece raw[RT_FILL];
  __device__ __forceinline__ const __nv_bfloat16* row(const RetShape& p, int off, int head, int row_first, int r) const {
    return p.p + static_cast<long long>(p.row0 + row_first + r) * p.ldp + off + head * p.dim;
  }
  __device__ __forceinline__ void fetch(const RetShape& p, int off, int head, int row_first, int rows, int dim0) {
#pragma unroll
    for (int n = 0; n < RT_FILL; ++n) {
      const int i = threadIdx.x + n * RT_THREADS, r = i >> 3, d0 = dim0 + (i & 7) * 8;
      if (r < rows && d0 < p.dim) raw[n] = load_piece(row(p, off, head, row_first, r), d0, p.half);
    }
  }
  __device__ __forceinline__ void store(const RetShape& p, uint8_t* hi, uint8_t* lo, int off, int head, int row_first, int rows, int dim0, float scale,
                                        const float* weight) {
#pragma unroll
    for (int n = 0; n < RT_FILL; ++n) {
      const int i = threadIdx.x + n * RT_THREADS, r = i >> 3, piece = i & 7, d0 = dim0 + piece * 8;
      float v[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
      if (r < rows && d0 < p.dim) {
        rotate_piece(raw[n], row(p, off, head, row_first, r), d0, p.half, p.cs + static_cast<long long>(row_first + r) * 2 * p.half, v);
        const float s = weight ? scale * weight[r] : scale;
#pragma unroll
        for (int k = 0; k < 8; ++k) v[k] *= s;
      }
      store_split(hi, lo, rt_sw(r, piece), v);
    }
  }
};

// ---------------------------------------------------------------- sums of the chunks
__global__ void __launch_bounds__(RT_THREADS, 1)
retention_state_kernel(const __grid_constant__ CUtensorMap tmap_v, RetShape p, int atoms_v, int tmem_cols) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* k_hi = smem;                       // two atoms (128 dimensions)
  uint8_t* k_lo = smem + 2 * RT_ATOM;
  uint8_t* v_s = smem + 4 * RT_ATOM;
  float* weight = reinterpret_cast<float*>(v_s + atoms_v * RT_ATOM);
  uint64_t* bars = reinterpret_cast<uint64_t*>(weight + RT_C);
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 2);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int chunk = blockIdx.x, head = blockIdx.y;
  const int row_first = p.chunk_row[chunk], rows = p.chunk_rows[chunk];
  const float ld = p.log2_decay[head];
  if (threadIdx.x == 0) {
    mbar_init(smem_u32(bars), 1);
    mbar_init(smem_u32(bars + 1), 1);
    *abort_flag = 0;
    mbar_fence_init();
    fence_proxy_async();
    mbar_arrive_expect_tx(smem_u32(bars), atoms_v * RT_ATOM);
    for (int a = 0; a < atoms_v; ++a)
      tma_load_2d(smem_u32(v_s + a * RT_ATOM), &tmap_v, smem_u32(bars), p.v_off + head * p.vdim + a * 64, p.row0 + row_first);
  }
  if (warp == 1) {
    tmem_alloc(smem_u32(tmem_slot), tmem_cols);
    tmem_relinquish();
  }
  if (threadIdx.x < RT_C) weight[threadIdx.x] = threadIdx.x < rows ? exp2f(static_cast<float>(rows - 1 - threadIdx.x) * ld) : 0.f;
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *tmem_slot;
  const int quarter = warp & 3, side = warp >> 2;
  const uint32_t idesc = make_idesc_bf16(128, (p.vdim + 15) / 16 * 16, true, true);
  float* out = p.sums + (static_cast<long long>(chunk) * p.heads + head) * p.dim * p.vdim;
  bool ok = true;
  for (int d0 = 0, m = 0; d0 < p.dim; d0 += 128, ++m) {
    AtomFill f[2];
#pragma unroll
    for (int a = 0; a < 2; ++a) f[a].fetch(p, p.k_off, head, row_first, rows, d0 + a * 64);
#pragma unroll
    for (int a = 0; a < 2; ++a)
      f[a].store(p, k_hi + a * RT_ATOM, k_lo + a * RT_ATOM, p.k_off, head, row_first, rows, d0 + a * 64, p.kscale, weight);
    fence_proxy_async();
    tc_fence_before();
    __syncthreads();
    if (threadIdx.x == 0) {
      ok = mbar_wait(smem_u32(bars), 0, abort_flag, p.status, RLB_ERR_WAIT_FULL);
      tc_fence_after();
      for (int part = 0; part < 2; ++part) {
        const uint32_t k = smem_u32(part ? k_lo : k_hi);
        for (int kk = 0; kk < RT_C / 16; ++kk)
          umma_f16(tmem, make_smem_desc_sw128(k + kk * 2048, RT_ATOM, 1024), make_smem_desc_sw128(smem_u32(v_s) + kk * 2048, RT_ATOM, 1024), idesc,
                   (part | kk) != 0 ? 1u : 0u);
      }
      umma_commit(smem_u32(bars + 1));
    }
    ok = mbar_wait(smem_u32(bars + 1), m & 1, abort_flag, p.status, RLB_ERR_WAIT_TMEM_FULL) && ok;
    __syncwarp();
    tc_fence_after();
    const int d = d0 + quarter * 32 + lane;
    for (int c = side * 32; c < p.vdim; c += RT_THREADS / 4) {
      uint32_t r[32];
      tmem_ld_32x32b_x32(tmem + (static_cast<uint32_t>(quarter * 32) << 16) + c, r);
      tmem_ld_wait();
      if (d < p.dim) {
        float* o = out + static_cast<long long>(d) * p.vdim + c;
#pragma unroll
        for (int q = 0; q < 8; ++q)
          if (c + q * 4 < p.vdim)
            *reinterpret_cast<float4*>(o + q * 4) = make_float4(__uint_as_float(r[q * 4]), __uint_as_float(r[q * 4 + 1]), __uint_as_float(r[q * 4 + 2]),
                                                                __uint_as_float(r[q * 4 + 3]));
      }
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
  }
  if (warp == 1) tmem_dealloc(tmem, tmem_cols);
}

// ---------------------------------------------------------------- start states
__global__ void __launch_bounds__(256)
retention_scan_kernel(float* __restrict__ sums, const int* __restrict__ piece_chunk, const int* __restrict__ chunk_rows, const int* __restrict__ chunk_row,
                      const int* __restrict__ positions, int row0, const long long* __restrict__ state_rows, float* __restrict__ state, long long num_states,
                      const float* __restrict__ log2_decay, int heads, int elems, int* status) {
  const int piece = blockIdx.y, head = blockIdx.z;
  const int e = (blockIdx.x * blockDim.x + threadIdx.x) * 4;
  const long long sr = state_rows[piece];
  if (sr < 0 || sr >= num_states) {
    if (threadIdx.x == 0 && status) atomicCAS(status, 0, RLB_ERR_BOUNDS);
    return;
  }
  if (e >= elems) return;
  const int c0 = piece_chunk[piece], c1 = piece_chunk[piece + 1];
  float4* sp = reinterpret_cast<float4*>(state + (sr * heads + head) * static_cast<long long>(elems) + e);
  float4 s = make_float4(0.f, 0.f, 0.f, 0.f);
  if (positions[row0 + chunk_row[c0]] != 0) s = *sp;
  const float ld = log2_decay[head];
  const long long step = static_cast<long long>(heads) * elems;
  float4* q = reinterpret_cast<float4*>(sums + (static_cast<long long>(c0) * heads + head) * elems + e);
  constexpr int AHEAD = 8;
  for (int c = c0; c < c1; c += AHEAD) {
    float4 add[AHEAD];
#pragma unroll
    for (int k = 0; k < AHEAD; ++k)
      if (c + k < c1) add[k] = *reinterpret_cast<const float4*>(reinterpret_cast<const float*>(q) + k * step);
#pragma unroll
    for (int k = 0; k < AHEAD; ++k) {
      if (c + k < c1) {
        *reinterpret_cast<float4*>(reinterpret_cast<float*>(q) + k * step) = s;
        const float f = exp2f(static_cast<float>(chunk_rows[c + k]) * ld);
        s = make_float4(fmaf(s.x, f, add[k].x), fmaf(s.y, f, add[k].y), fmaf(s.z, f, add[k].z), fmaf(s.w, f, add[k].w));
      }
    }
    q = reinterpret_cast<float4*>(reinterpret_cast<float*>(q) + AHEAD * step);
  }
  *sp = s;
}

// ---------------------------------------------------------------- outputs
__global__ void __launch_bounds__(RT_THREADS, 1)
retention_out_kernel(const __grid_constant__ CUtensorMap tmap_v, RetShape p, int atoms_v, int tmem_cols) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t *q_hi = smem, *q_lo = smem + RT_ATOM, *k_hi = smem + 2 * RT_ATOM, *k_lo = smem + 3 * RT_ATOM;
  uint8_t* w_hi = smem;                       // decayed weights [128 x 128], over the queries and keys once those have been read
  uint8_t* w_lo = smem + 2 * RT_ATOM;
  uint8_t* s_hi = smem + 4 * RT_ATOM;         // 64 state rows x vdim
  uint8_t* s_lo = s_hi + atoms_v * RT_SATOM;
  uint8_t* v_s = s_lo + atoms_v * RT_SATOM;
  float* pw = reinterpret_cast<float*>(v_s + atoms_v * RT_ATOM);   // [129] powers of the decay
  float* ssq = pw + 132;                                           // [column groups][128]
  uint64_t* bars = reinterpret_cast<uint64_t*>(ssq + RT_THREADS);
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 2);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int chunk = blockIdx.x, head = blockIdx.y;
  const int row_first = p.chunk_row[chunk], rows = p.chunk_rows[chunk];
  const float ld = p.log2_decay[head];
  if (threadIdx.x == 0) {
    mbar_init(smem_u32(bars), 1);
    mbar_init(smem_u32(bars + 1), 1);
    *abort_flag = 0;
    mbar_fence_init();
    fence_proxy_async();
    mbar_arrive_expect_tx(smem_u32(bars), atoms_v * RT_ATOM);
    for (int a = 0; a < atoms_v; ++a)
      tma_load_2d(smem_u32(v_s + a * RT_ATOM), &tmap_v, smem_u32(bars), p.v_off + head * p.vdim + a * 64, p.row0 + row_first);
  }
  if (warp == 1) {
    tmem_alloc(smem_u32(tmem_slot), tmem_cols);
    tmem_relinquish();
  }
  if (threadIdx.x <= RT_C) pw[threadIdx.x] = exp2f(static_cast<float>(threadIdx.x) * ld);
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_s = *tmem_slot, tmem_o = tmem_s + RT_C;
  const int vcols = (p.vdim + 15) / 16 * 16;
  const uint32_t idesc_s = make_idesc_bf16(RT_C, RT_C, false, false), idesc_o = make_idesc_bf16(RT_C, vcols, false, true);
  const float* S0 = p.sums + (static_cast<long long>(chunk) * p.heads + head) * p.dim * p.vdim;
  bool ok = true;
  int done = 0;      // commits waited for
  for (int d0 = 0; d0 < p.dim; d0 += 64) {
    // the loads of queries, keys and start state are in flight together
    AtomFill fq, fk;
    fq.fetch(p, p.q_off, head, row_first, rows, d0);
    fk.fetch(p, p.k_off, head, row_first, rows, d0);
    const int groups = atoms_v * 8;      // 8-column pieces of a state row
    float4 sx[4], sy[4];
#pragma unroll
    for (int n = 0; n < 4; ++n) {        // 64 rows x at most 32 pieces
      const int i = threadIdx.x + n * RT_THREADS, r = i / groups, v0 = (i % groups) * 8;
      sx[n] = sy[n] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (i < 64 * groups && d0 + r < p.dim && v0 < p.vdim) {
        sx[n] = *reinterpret_cast<const float4*>(S0 + static_cast<long long>(d0 + r) * p.vdim + v0);
        sy[n] = *reinterpret_cast<const float4*>(S0 + static_cast<long long>(d0 + r) * p.vdim + v0 + 4);
      }
    }
    if (d0 > 0) {    // the previous products have read the stage
      ok = mbar_wait(smem_u32(bars + 1), done & 1, abort_flag, p.status, RLB_ERR_WAIT_EMPTY) && ok;
      ++done;
      __syncthreads();
    }
    fq.store(p, q_hi, q_lo, p.q_off, head, row_first, rows, d0, 1.f, nullptr);
    fk.store(p, k_hi, k_lo, p.k_off, head, row_first, rows, d0, p.kscale, nullptr);
#pragma unroll
    for (int n = 0; n < 4; ++n) {
      const int i = threadIdx.x + n * RT_THREADS, r = i / groups, g = i % groups;
      if (i < 64 * groups) {
        const float v[8] = {sx[n].x, sx[n].y, sx[n].z, sx[n].w, sy[n].x, sy[n].y, sy[n].z, sy[n].w};
        store_split(s_hi, s_lo, (g >> 3) * RT_SATOM + rt_sw(r, g & 7), v);
      }
    }
    fence_proxy_async();
    tc_fence_before();
    __syncthreads();
    if (threadIdx.x == 0) {
      tc_fence_after();
      const int steps = min(4, (p.dim - d0 + 15) / 16);
      for (int part = 0; part < 3; ++part) {     // hi hi, hi lo, lo hi
        const uint32_t q = smem_u32(part == 2 ? q_lo : q_hi), k = smem_u32(part == 1 ? k_lo : k_hi), s = smem_u32(part == 1 ? s_lo : s_hi);
        for (int kk = 0; kk < steps; ++kk) {
          const uint32_t acc = (d0 | part | kk) != 0 ? 1u : 0u;
          umma_f16(tmem_s, make_smem_desc_sw128(q + kk * 32, 16, 1024), make_smem_desc_sw128(k + kk * 32, 16, 1024), idesc_s, acc);
          umma_f16(tmem_o, make_smem_desc_sw128(q + kk * 32, 16, 1024), make_smem_desc_sw128(s + kk * 2048, RT_SATOM, 1024), idesc_o, acc);
        }
      }
      umma_commit(smem_u32(bars + 1));
    }
  }
  ok = mbar_wait(smem_u32(bars + 1), done & 1, abort_flag, p.status, RLB_ERR_WAIT_TMEM_FULL) && ok;
  ++done;
  __syncwarp();
  tc_fence_after();
  // groups of four warps share the rows and split the columns
  const int quarter = warp & 3, side = warp >> 2, i = quarter * 32 + lane;
  const uint32_t lane_addr = static_cast<uint32_t>(quarter * 32) << 16;
  for (int c = side * 32; c < RT_C; c += RT_THREADS / 4) {
    uint32_t r[32];
    tmem_ld_32x32b_x32(tmem_s + lane_addr + c, r);
    tmem_ld_wait();
#pragma unroll
    for (int q = 0; q < 4; ++q) {
      float v[8];
#pragma unroll
      for (int k = 0; k < 8; ++k) {
        const int j = c + q * 8 + k;
        v[k] = j <= i ? __uint_as_float(r[q * 8 + k]) * pw[i - j] : 0.f;
      }
      store_split(w_hi, w_lo, (c >> 6) * RT_ATOM + rt_sw(i, ((c & 63) >> 3) + q), v);
    }
  }
  for (int c = side * 32; c < vcols; c += RT_THREADS / 4) {     // start-state term: row i is d^(i+1) times what stands in O
    uint32_t r[16];
    const float f = pw[i + 1];
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      if (c + h * 16 < vcols) {
        tmem_ld_32x32b_x16(tmem_o + lane_addr + c + h * 16, r);
        tmem_ld_wait();
#pragma unroll
        for (int k = 0; k < 16; ++k) r[k] = __float_as_uint(__uint_as_float(r[k]) * f);
        tmem_st_32x32b_x16(tmem_o + lane_addr + c + h * 16, r);
      }
    }
  }
  tmem_st_wait();
  fence_proxy_async();
  tc_fence_before();
  __syncthreads();
  if (threadIdx.x == 0) {
    ok = mbar_wait(smem_u32(bars), 0, abort_flag, p.status, RLB_ERR_WAIT_FULL) && ok;
    tc_fence_after();
    for (int part = 0; part < 2; ++part) {
      const uint32_t w = smem_u32(part ? w_lo : w_hi);
      for (int kk = 0; kk < RT_C / 16; ++kk)
        umma_f16(tmem_o, make_smem_desc_sw128(w + (kk >> 2) * RT_ATOM + (kk & 3) * 32, 16, 1024), make_smem_desc_sw128(smem_u32(v_s) + kk * 2048, RT_ATOM, 1024),
                 idesc_o, 1u);
    }
    umma_commit(smem_u32(bars + 1));
  }
  ok = mbar_wait(smem_u32(bars + 1), done & 1, abort_flag, p.status, RLB_ERR_WAIT_TMEM_FULL) && ok;
  __syncwarp();
  tc_fence_after();
  float ss = 0.f;
  for (int c = side * 32; c < p.vdim; c += RT_THREADS / 4) {
    uint32_t r[32];
    tmem_ld_32x32b_x32(tmem_o + lane_addr + c, r);
    tmem_ld_wait();
#pragma unroll
    for (int k = 0; k < 32; ++k)
      if (c + k < p.vdim) ss += __uint_as_float(r[k]) * __uint_as_float(r[k]);
  }
  ssq[side * RT_C + i] = ss;
  __syncthreads();
  ss = 0.f;
#pragma unroll
  for (int g = 0; g < RT_THREADS / 128; ++g) ss += ssq[g * RT_C + i];
  const float rstd = 1.f / sqrtf(ss / static_cast<float>(p.vdim) + p.eps);
  __nv_bfloat16* dst = p.p + static_cast<long long>(p.row0 + row_first + i) * p.ldp + p.mix_off + head * p.vdim;
  for (int c = side * 32; c < p.vdim; c += RT_THREADS / 4) {
    uint32_t r[32];
    tmem_ld_32x32b_x32(tmem_o + lane_addr + c, r);
    tmem_ld_wait();
    if (i < rows) {
#pragma unroll
      for (int q = 0; q < 4; ++q) {
        if (c + q * 8 < p.vdim) {
          uint4 g = *reinterpret_cast<uint4*>(dst + c + q * 8);
          uint32_t* gw = reinterpret_cast<uint32_t*>(&g);
#pragma unroll
          for (int w = 0; w < 4; ++w) {
            const float2 gf = unpack_bf16x2(gw[w]);
            gw[w] = pack_bf16x2(__uint_as_float(r[q * 8 + 2 * w]) * rstd * (gf.x / (1.f + expf(-gf.x))),
                                __uint_as_float(r[q * 8 + 2 * w + 1]) * rstd * (gf.y / (1.f + expf(-gf.y))));
          }
          *reinterpret_cast<uint4*>(dst + c + q * 8) = g;
        }
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem_s, tmem_cols);
  }
}

// ---------------------------------------------------------------- decode
// Rows [0, rows) of p are one token each of as many sequences. Every thread owns four value columns and every `slices`-th state row.
__global__ void __launch_bounds__(256)
retention_step_kernel(__nv_bfloat16* __restrict__ p, long long ldp, int q_off, int k_off, int v_off, int mix_off, int heads, int dim, int vdim,
                      const int* __restrict__ positions, const long long* __restrict__ state_rows, float* __restrict__ state, long long num_states,
                      const float* __restrict__ decay, const float* __restrict__ freq, int half, float gain, float kscale, float eps, int* status) {
  extern __shared__ float sm[];
  __shared__ float red[32];
  float* q = sm;
  float* k = q + dim;
  float4* part = reinterpret_cast<float4*>(k + dim);     // [256] (dim is a multiple of 8)
  const int row = blockIdx.x, head = blockIdx.y, tid = threadIdx.x;
  pdl_sync();
  const long long sr = state_rows[row];
  if (sr < 0 || sr >= num_states) {
    if (tid == 0 && status) atomicCAS(status, 0, RLB_ERR_BOUNDS);
    return;
  }
  __nv_bfloat16* pr = p + row * ldp;
  const __nv_bfloat16 *qp = pr + q_off + head * dim, *kp = pr + k_off + head * dim;
  const int pos = positions[row];
  const int c4 = vdim / 4, slices = 256 / c4, slice = tid / c4, col = tid % c4;
  const bool live = slice < slices;
  for (int i = tid; i < dim; i += 256) {
    if (i < half) {
      float s, c;
      sincosf(static_cast<float>(pos) * freq[i], &s, &c);
      s *= gain;
      c *= gain;
      const float qa = __bfloat162float(qp[i]), qb = __bfloat162float(qp[i + half]), ka = __bfloat162float(kp[i]), kb = __bfloat162float(kp[i + half]);
      q[i] = qa * c - qb * s;
      q[i + half] = qb * c + qa * s;
      k[i] = (ka * c - kb * s) * kscale;
      k[i + half] = (kb * c + ka * s) * kscale;
    } else if (i >= 2 * half) {
      q[i] = __bfloat162float(qp[i]);
      k[i] = __bfloat162float(kp[i]) * kscale;
    }
  }
  const float dec = pos == 0 ? 0.f : decay[head];
  float4 v = make_float4(0.f, 0.f, 0.f, 0.f), acc = v;
  if (live) {
    const uint2 raw = *reinterpret_cast<const uint2*>(pr + v_off + head * vdim + col * 4);
    const float2 a = unpack_bf16x2(raw.x), b = unpack_bf16x2(raw.y);
    v = make_float4(a.x, a.y, b.x, b.y);
  }
  float4* S = reinterpret_cast<float4*>(state + (sr * heads + head) * static_cast<long long>(dim) * vdim) + col;
  constexpr int U = 8;
  __syncthreads();
  if (live) {
    for (int i0 = slice; i0 < dim; i0 += U * slices) {
      float4 s[U];
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const int i = i0 + u * slices;
        s[u] = (i < dim && pos != 0) ? S[static_cast<long long>(i) * c4] : make_float4(0.f, 0.f, 0.f, 0.f);
      }
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const int i = i0 + u * slices;
        if (i < dim) {
          const float kv = k[i], qv = q[i];
          s[u] = make_float4(fmaf(dec, s[u].x, kv * v.x), fmaf(dec, s[u].y, kv * v.y), fmaf(dec, s[u].z, kv * v.z), fmaf(dec, s[u].w, kv * v.w));
          S[static_cast<long long>(i) * c4] = s[u];
          acc.x = fmaf(s[u].x, qv, acc.x);
          acc.y = fmaf(s[u].y, qv, acc.y);
          acc.z = fmaf(s[u].z, qv, acc.z);
          acc.w = fmaf(s[u].w, qv, acc.w);
        }
      }
    }
    part[tid] = acc;
  }
  __syncthreads();
  float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
  if (tid < c4)
    for (int j = 0; j < slices; ++j) {
      const float4 t = part[j * c4 + tid];
      o.x += t.x; o.y += t.y; o.z += t.z; o.w += t.w;
    }
  const float ss = block_sum(o.x * o.x + o.y * o.y + o.z * o.z + o.w * o.w, red);
  if (tid < c4) {
    const float rstd = 1.f / sqrtf(ss / static_cast<float>(vdim) + eps);
    uint2* g = reinterpret_cast<uint2*>(pr + mix_off + head * vdim + tid * 4);
    const uint2 raw = *g;
    const float2 a = unpack_bf16x2(raw.x), b = unpack_bf16x2(raw.y);
    *g = make_uint2(pack_bf16x2(o.x * rstd * (a.x / (1.f + expf(-a.x))), o.y * rstd * (a.y / (1.f + expf(-a.y)))),
                    pack_bf16x2(o.z * rstd * (b.x / (1.f + expf(-b.x))), o.w * rstd * (b.y / (1.f + expf(-b.y)))));
  }
}
}  // namespace

// Shapes both kernels take: dim and vdim multiples of 8, vdim at most 256 (decode: 1024).
RLB_API int rlb_retention_supported(int dim, int vdim) { return dim > 0 && dim % 8 == 0 && dim <= 2048 && vdim > 0 && vdim % 8 == 0 && vdim <= 256; }

RLB_API int rlb_retention_step(void* p, int rows, long long ldp, int q_off, int k_off, int v_off, int mix_off, int heads, int dim, int vdim,
                               const int* positions, const long long* state_rows, float* state, long long num_states, const float* decay,
                               const float* freq, int half, float gain, float kscale, float eps, int* status, void* stream) {
  if (rows <= 0) return 0;
  if (!rlb_retention_supported(dim, vdim) || 2 * half > dim || ldp % 8 || (q_off | k_off | v_off | mix_off) % 8 || heads > 65535) return -2;
  const size_t sm = sizeof(float) * 2 * dim + sizeof(float4) * 256;
  return static_cast<int>(rlb_launch_pdl(retention_step_kernel, dim3(rows, heads), dim3(256), sm, static_cast<cudaStream_t>(stream),
                                         static_cast<__nv_bfloat16*>(p), ldp, q_off, k_off, v_off, mix_off, heads, dim, vdim, positions, state_rows,
                                         state, num_states, decay, freq, half, gain, kscale, eps, status));
}

// Portions: rows [row0, rows) of p, cut into chunks of at most 128 rows (chunk_row: first row counted from row0, chunk_rows). Piece i owns
// chunks [piece_chunk[i], piece_chunk[i + 1]) and state row state_rows[i]. Scratch: cs [rows - row0, 2 * half], sums [chunks, heads, dim, vdim].
RLB_API int rlb_retention_portions(void* p, long long rows, long long ldp, int in_width, int row0, int q_off, int k_off, int v_off, int mix_off,
                                   int heads, int dim, int vdim, int pieces, int chunks, const int* piece_chunk, const int* chunk_row,
                                   const int* chunk_rows, const int* positions, const long long* state_rows, float* state, long long num_states,
                                   const float* log2_decay, const float* freq, int half, float gain, float kscale, float eps, float* cs, float* sums,
                                   int* status, void* stream) {
  if (pieces <= 0 || chunks <= 0) return 0;
  if (!rlb_retention_supported(dim, vdim) || 2 * half > dim || ldp % 8 || (q_off | k_off | v_off | mix_off) % 8 || heads > 65535 || pieces > 65535) return -2;
  if ((reinterpret_cast<uintptr_t>(p) | reinterpret_cast<uintptr_t>(sums) | reinterpret_cast<uintptr_t>(cs)) & 15) return -3;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (half > 0) {
    const long long n = (rows - row0) * half, want = (n + 255) / 256;
    rotation_table_kernel<<<static_cast<unsigned>(want < 148 * 8 ? want : 148 * 8), 256, 0, s>>>(positions + row0, freq, half, gain, cs, rows - row0);
  }
  RetShape r{static_cast<__nv_bfloat16*>(p), ldp, q_off, k_off, v_off, mix_off, heads, dim, vdim, row0, chunk_row, chunk_rows, cs, half, kscale, eps,
             log2_decay, sums, status};
  CUtensorMap tv;
  const int rc = rlb_make_tmap_2d(&tv, p, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, in_width, rows, ldp * 2, 64, RT_C, CU_TENSOR_MAP_SWIZZLE_128B);
  if (rc) return -100 - rc;
  const int av = (vdim + 63) / 64;
  const int smem_state = (4 + av) * RT_ATOM + RT_C * 4 + 64 + 1024;
  const int smem_out = 4 * RT_ATOM + 2 * av * RT_SATOM + av * RT_ATOM + (132 + RT_THREADS) * 4 + 64 + 1024;
  static int conf_state = 0, conf_out = 0;
  if (smem_state > conf_state) {
    cudaError_t e = cudaFuncSetAttribute(retention_state_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, smem_state);
    if (e != cudaSuccess) return static_cast<int>(e);
    conf_state = smem_state;
  }
  if (smem_out > conf_out) {
    cudaError_t e = cudaFuncSetAttribute(retention_out_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, smem_out);
    if (e != cudaSuccess) return static_cast<int>(e);
    conf_out = smem_out;
  }
  const int vpad = (vdim + 31) / 32 * 32;
  const int cols_state = vpad <= 32 ? 32 : (vpad <= 64 ? 64 : (vpad <= 128 ? 128 : 256));
  const int cols_out = vpad <= 128 ? 256 : 512;
  const dim3 grid(chunks, heads);
  retention_state_kernel<<<grid, RT_THREADS, smem_state, s>>>(tv, r, av, cols_state);
  const int elems = dim * vdim;
  retention_scan_kernel<<<dim3((elems / 4 + 255) / 256, pieces, heads), 256, 0, s>>>(sums, piece_chunk, chunk_rows, chunk_row, positions, row0, state_rows,
                                                                                     state, num_states, log2_decay, heads, elems, status);
  retention_out_kernel<<<grid, RT_THREADS, smem_out, s>>>(tv, r, av, cols_out);
  return static_cast<int>(cudaGetLastError());
}
