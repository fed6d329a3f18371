// Recurrent mixers with a short convolution for bf16 models: decode steps that stream the fp32 state once, and prompt portions chunk by chunk on
// the 5th-generation tensor cores (tcgen05 + TMEM + TMA). Chunks have 128 tokens; i, j count inside a chunk, S0 is its start state, and c_i
// the log2 of the decay from the chunk's start through token i, so that d_ij = 2^(c_i - c_j) <= 1 for j <= i.
//
//   Mamba-2 (q = C, k = B, w = dt)       y_i = sum_{j<=i} d_ij w_j (q_i . k_j) x_j + 2^c_i S0^T q_i + D x_i
//                                        S next = 2^c_end S0 + sum_j d_end,j w_j k_j x_j^T
//   Delta rule (unit q, k; w = beta)     U = V' - W S0 with T = (I + A)^-1, A_ij = w_i d_ij (k_i . k_j) for j < i,
//                                        V' = T diag(w) V, W = T diag(w 2^c) K;   the writes U then stand where x w stood above:
//                                        o_i = sum_{j<=i} d_ij (q_i . k_j) u_j + 2^c_i S0^T q_i,  S next = 2^c_end S0 + sum_j d_end,j k_j u_j^T
//
//   rec_prep      per (chunk, head): step sizes or betas and c
//   rec_unit      per (row, group): factors that make delta-rule queries and keys unit vectors
//   ssd_state, ssd_scan      per (chunk, head) the sum over j, then per piece the chunks' start states
//   delta_wy      per (chunk, head): A, its inverse (16 x 16 blocks by substitution, then block by block), W, V', decayed keys
//   delta_scan    per (piece, head, 32 or 64 value columns), chunk after chunk: U and the state; both products of a chunk on the tensor cores, the
//                 next chunk's tiles in flight under them
//   rec_out       per (chunk, head): scores, decays, both output terms, the mixer's gate (and head norm), store
//
// Everything that enters the recurrences is 32-bit: unit vectors, decayed weights, T, W, U and states are split into two bf16 parts and
// multiplied as hi*hi + hi*lo + lo*hi with fp32 accumulation; convolved channels are bf16 values and exact.
//
// This file is compiled without fast math.
#include "recurrent.cuh"

namespace {
using namespace rlb;

constexpr int RC_THREADS = 512;
constexpr float RC_LOG2E = 1.4426950408889634f;

struct RecTiles {
  const __nv_bfloat16* u;      // convolved rows
  long long ldu;
  const __nv_bfloat16* p;      // projected rows
  long long ldp;
  __nv_bfloat16* y;
  long long ldy;
  int heads, per_group, dim, vdim;
  int q_col, k_col, v_col;     // columns of u
  int gate_off;                // column of p
  int row0;                    // first row of the portions in u, p, y
  long long rows;              // rows of the portions
  const int* chunk_row;        // [chunks] first row, counted from row0
  const int* chunk_rows;
  const float* cum;            // [heads, rows]
  const float* wt;             // [heads, rows]
  const float* unit;           // delta: [2, groups, rows] factors of q (with the scale), of k
  float eps;
  const __nv_bfloat16* D;
  const __nv_bfloat16* norm;
  float* start;                // [chunks, heads, dim, vdim]: sums of the chunks, then their start states
  __nv_bfloat16 *w_hi, *w_lo, *kt_hi, *kt_lo;   // delta: [chunks * heads * 128, 128]
  float* u0;                   // delta: [chunks * heads * 128, vdim]
  __nv_bfloat16 *uu_hi, *uu_lo;                 // delta: [rows, heads * vdim]
  int* status;
};

// ---------------------------------------------------------------- convolution of runs of rows, 8 channels per thread
constexpr int CV_RUN = 16;
template <int TAPS>
__global__ void __launch_bounds__(128, 5)
conv_runs_kernel(const __nv_bfloat16* __restrict__ x, long long ldx, __nv_bfloat16* __restrict__ u, long long ldu, long long rows, int channels,
                 const __nv_bfloat16* __restrict__ w, const __nv_bfloat16* __restrict__ bias, const __nv_bfloat16* __restrict__ ring,
                 const int* __restrict__ positions, const int* __restrict__ row_off, const long long* __restrict__ row_state, long long num_states,
                 int* status) {
  const int c = (blockIdx.y * 128 + threadIdx.x) * 8;
  if (c >= channels) return;
  float wv[8][TAPS], b[8], win[TAPS][8];
  {
    float wf[8 * TAPS];      // the channels' taps are contiguous
#pragma unroll
    for (int q = 0; q < TAPS; ++q) {
      float t[8];
      unpack8(*reinterpret_cast<const uint4*>(w + static_cast<long long>(c) * TAPS + q * 8), t);
#pragma unroll
      for (int k = 0; k < 8; ++k) wf[q * 8 + k] = t[k];
    }
#pragma unroll
    for (int k = 0; k < 8; ++k)
#pragma unroll
      for (int j = 0; j < TAPS; ++j) wv[k][j] = wf[k * TAPS + j];
    unpack8(bias ? *reinterpret_cast<const uint4*>(bias + c) : make_uint4(0, 0, 0, 0), b);
  }
  const long long r0 = static_cast<long long>(blockIdx.x) * CV_RUN, r1 = min(rows, r0 + CV_RUN);
  constexpr int AHEAD = 4;
  for (long long rb = r0; rb < r1; rb += AHEAD) {
    uint4 raw[AHEAD];
    int offs[AHEAD];
#pragma unroll
    for (int a = 0; a < AHEAD; ++a) {
      raw[a] = rb + a < r1 ? *reinterpret_cast<const uint4*>(x + (rb + a) * ldx + c) : make_uint4(0, 0, 0, 0);
      offs[a] = rb + a < r1 ? row_off[rb + a] : 1;
    }
#pragma unroll
    for (int a = 0; a < AHEAD; ++a) {
      const long long r = rb + a;
      if (r >= r1) break;
      const int off = offs[a];
      if (r == r0 || off == 0) {      // the inputs before this row: of the same piece, of the ring, or none
        const int pos = positions[r];
        long long sr = row_state[r];
        if (sr < 0 || sr >= num_states) {
          if (c == 0 && status) atomicCAS(status, 0, RLB_ERR_BOUNDS);
          sr = 0;
        }
#pragma unroll
        for (int j = 0; j < TAPS - 1; ++j) {
          const int back = TAPS - 1 - j;
          uint4 before = make_uint4(0, 0, 0, 0);
          if (back <= off) before = *reinterpret_cast<const uint4*>(x + (r - back) * ldx + c);
          else if (back <= pos) before = *reinterpret_cast<const uint4*>(ring + (sr * TAPS + (pos - back) % TAPS) * channels + c);
          unpack8(before, win[j]);
        }
      }
      unpack8(raw[a], win[TAPS - 1]);
      uint32_t o[4];
#pragma unroll
      for (int k = 0; k < 8; k += 2) {
        float a0 = b[k], a1 = b[k + 1];
#pragma unroll
        for (int j = 0; j < TAPS; ++j) {
          a0 = fmaf(wv[k][j], win[j][k], a0);
          a1 = fmaf(wv[k + 1][j], win[j][k + 1], a1);
        }
        o[k / 2] = pack_bf16x2(rc_silu_bf16(a0), rc_silu_bf16(a1));
      }
      *reinterpret_cast<uint4*>(u + r * ldu + c) = make_uint4(o[0], o[1], o[2], o[3]);
#pragma unroll
      for (int j = 0; j < TAPS - 1; ++j)
#pragma unroll
        for (int k = 0; k < 8; ++k) win[j][k] = win[j + 1][k];
    }
  }
}

// ---------------------------------------------------------------- preparation
// One warp per (chunk, head). w_off: Mamba-2 -1 (the weight is the step size), delta the column of beta.
__global__ void __launch_bounds__(128)
rec_prep_kernel(const __nv_bfloat16* __restrict__ p, long long ldp, int dt_off, int w_off, int row0, const int* __restrict__ chunk_row,
                const int* __restrict__ chunk_rows, int heads, long long rows, const __nv_bfloat16* __restrict__ A_log,
                const __nv_bfloat16* __restrict__ dt_bias, float* __restrict__ cum, float* __restrict__ wt) {
  const int h = blockIdx.y * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (h >= heads) return;
  const int first = chunk_row[blockIdx.x], n = chunk_rows[blockIdx.x];
  const float A = -expf(__bfloat162float(A_log[h])) * RC_LOG2E, bias = __bfloat162float(dt_bias[h]);
  float run = 0.f, part[4];
#pragma unroll
  for (int k = 0; k < 4; ++k) {
    const int r = lane * 4 + k;
    if (r < n) {
      const __nv_bfloat16* pr = p + (row0 + first + r) * ldp;
      const float sp = rc_softplus(__bfloat162float(pr[dt_off + h]) + bias);
      run += A * sp;
      wt[h * rows + first + r] = w_off < 0 ? sp : 1.f / (1.f + expf(-__bfloat162float(pr[w_off + h])));
    }
    part[k] = run;
  }
  float inc = run;
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const float up = __shfl_up_sync(0xffffffffu, inc, o);
    if (lane >= o) inc += up;
  }
  float before = __shfl_up_sync(0xffffffffu, inc, 1);
  if (lane == 0) before = 0.f;
#pragma unroll
  for (int k = 0; k < 4; ++k)
    if (lane * 4 + k < n) cum[h * rows + first + lane * 4 + k] = before + part[k];
}

// One warp per (row, group, q or k).
__global__ void __launch_bounds__(256)
rec_unit_kernel(const __nv_bfloat16* __restrict__ u, long long ldu, int row0, int groups, int dim, int q_col, int k_col, long long rows, float qscale,
                float unit_eps, float* __restrict__ unit) {
  const int i = blockIdx.y * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (i >= 2 * groups) return;
  const long long r = blockIdx.x;
  const bool is_q = i < groups;
  const __nv_bfloat16* x = u + (row0 + r) * ldu + (is_q ? q_col + i * dim : k_col + (i - groups) * dim);
  float ss = 0.f;
  for (int d = lane * 8; d < dim; d += 256) {
    float v[8];
    unpack8(*reinterpret_cast<const uint4*>(x + d), v);
#pragma unroll
    for (int k = 0; k < 8; ++k) ss += v[k] * v[k];
  }
  ss = warp_sum(ss);
  if (lane == 0) unit[i * rows + r] = (is_q ? qscale : 1.f) / sqrtf(ss + unit_eps);
}

// ---------------------------------------------------------------- operand tiles
// One atom [128 rows x 64 columns] of u, zeros past `rows` rows and `dim` columns. `fetch` and `store` are apart so that a caller can have
// several atoms in flight.
constexpr int RC_FILL = RT_C * 8 / RC_THREADS;
struct AtomTile {
  uint4 raw[RC_FILL];
  __device__ __forceinline__ void fetch(const __nv_bfloat16* base, long long ld, int rows, int dim0, int dim) {
#pragma unroll
    for (int n = 0; n < RC_FILL; ++n) {
      const int i = threadIdx.x + n * RC_THREADS, r = i >> 3, d = dim0 + (i & 7) * 8;
      raw[n] = r < rows && d < dim ? *reinterpret_cast<const uint4*>(base + r * ld + d) : make_uint4(0, 0, 0, 0);
    }
  }
  __device__ __forceinline__ void store(uint8_t* hi) const {
#pragma unroll
    for (int n = 0; n < RC_FILL; ++n) {
      const int i = threadIdx.x + n * RC_THREADS;
      *reinterpret_cast<uint4*>(hi + rt_sw(i >> 3, i & 7)) = raw[n];
    }
  }
  __device__ __forceinline__ void store_scaled(uint8_t* hi, uint8_t* lo, const float* scale) const {
#pragma unroll
    for (int n = 0; n < RC_FILL; ++n) {
      const int i = threadIdx.x + n * RC_THREADS;
      float v[8];
      unpack8(raw[n], v);
      const float f = scale[i >> 3];
#pragma unroll
      for (int k = 0; k < 8; ++k) v[k] *= f;
      store_split(hi, lo, rt_sw(i >> 3, i & 7), v);
    }
  }
};

// ---------------------------------------------------------------- Mamba-2: sums of the chunks
__global__ void __launch_bounds__(RC_THREADS, 1)
ssd_state_kernel(const __grid_constant__ CUtensorMap tmap_v, RecTiles p, int atoms_v, int tmem_cols) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t *k_hi = smem, *k_lo = smem + 2 * RT_ATOM, *v_s = smem + 4 * RT_ATOM;
  float* weight = reinterpret_cast<float*>(v_s + atoms_v * RT_ATOM);
  uint64_t* bars = reinterpret_cast<uint64_t*>(weight + RT_C);
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 2);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int chunk = blockIdx.x, head = blockIdx.y;
  const int first = p.chunk_row[chunk], rows = p.chunk_rows[chunk];
  if (threadIdx.x == 0) {
    mbar_init(smem_u32(bars), 1);
    mbar_init(smem_u32(bars + 1), 1);
    *abort_flag = 0;
    mbar_fence_init();
    fence_proxy_async();
    mbar_arrive_expect_tx(smem_u32(bars), atoms_v * RT_ATOM);
    for (int a = 0; a < atoms_v; ++a)
      tma_load_2d(smem_u32(v_s + a * RT_ATOM), &tmap_v, smem_u32(bars), p.v_col + head * p.vdim + a * 64, p.row0 + first);
  }
  if (warp == 1) {
    tmem_alloc(smem_u32(tmem_slot), tmem_cols);
    tmem_relinquish();
  }
  const float* cum = p.cum + head * p.rows + first;
  if (threadIdx.x < RT_C)
    weight[threadIdx.x] = threadIdx.x < rows ? exp2f(cum[rows - 1] - cum[threadIdx.x]) * p.wt[head * p.rows + first + threadIdx.x] : 0.f;
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *tmem_slot;
  const int quarter = warp & 3, side = warp >> 2;
  const uint32_t idesc = make_idesc_bf16(128, (p.vdim + 15) / 16 * 16, true, true);
  const __nv_bfloat16* kb = p.u + (p.row0 + first) * p.ldu + p.k_col + head / p.per_group * p.dim;
  float* out = p.start + (static_cast<long long>(chunk) * p.heads + head) * p.dim * p.vdim;
  for (int d0 = 0, m = 0; d0 < p.dim; d0 += 128, ++m) {
    AtomTile f[2];
#pragma unroll
    for (int a = 0; a < 2; ++a) f[a].fetch(kb, p.ldu, rows, d0 + a * 64, p.dim);
#pragma unroll
    for (int a = 0; a < 2; ++a) f[a].store_scaled(k_hi + a * RT_ATOM, k_lo + a * RT_ATOM, weight);
    fence_proxy_async();
    tc_fence_before();
    __syncthreads();
    if (threadIdx.x == 0) {
      mbar_wait(smem_u32(bars), 0, abort_flag, p.status, RLB_ERR_WAIT_FULL);
      tc_fence_after();
      for (int part = 0; part < 2; ++part) {
        const uint32_t k = smem_u32(part ? k_lo : k_hi);
        for (int kk = 0; kk < RT_C / 16; ++kk)
          umma_f16(tmem, make_smem_desc_sw128(k + kk * 2048, RT_ATOM, 1024), make_smem_desc_sw128(smem_u32(v_s) + kk * 2048, RT_ATOM, 1024), idesc,
                   (part | kk) != 0 ? 1u : 0u);
      }
      umma_commit(smem_u32(bars + 1));
    }
    mbar_wait(smem_u32(bars + 1), m & 1, abort_flag, p.status, RLB_ERR_WAIT_TMEM_FULL);
    __syncwarp();
    tc_fence_after();
    const int d = d0 + quarter * 32 + lane;
    for (int c = side * 32; c < p.vdim; c += RC_THREADS / 4) {
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

// Start states of the chunks in the place of their sums; the sequence's state row advances.
__global__ void __launch_bounds__(256)
ssd_scan_kernel(RecTiles p, const int* __restrict__ piece_chunk, const int* __restrict__ positions, const long long* __restrict__ state_rows,
                float* __restrict__ state, long long num_states) {
  const int piece = blockIdx.y, head = blockIdx.z, elems = p.dim * p.vdim;
  const int e = (blockIdx.x * blockDim.x + threadIdx.x) * 4;
  const long long sr = state_rows[piece];
  if (sr < 0 || sr >= num_states) {
    if (threadIdx.x == 0 && p.status) atomicCAS(p.status, 0, RLB_ERR_BOUNDS);
    return;
  }
  if (e >= elems) return;
  const int c0 = piece_chunk[piece], c1 = piece_chunk[piece + 1];
  float4* sp = reinterpret_cast<float4*>(state + (sr * p.heads + head) * static_cast<long long>(elems) + e);
  float4 s = make_float4(0.f, 0.f, 0.f, 0.f);
  if (positions[p.row0 + p.chunk_row[c0]] != 0) s = *sp;
  const long long step = static_cast<long long>(p.heads) * elems;
  float* q = p.start + (static_cast<long long>(c0) * p.heads + head) * elems + e;
  constexpr int AHEAD = 8;
  for (int c = c0; c < c1; c += AHEAD, q += AHEAD * step) {
    float4 add[AHEAD];
    float f[AHEAD];
#pragma unroll
    for (int k = 0; k < AHEAD; ++k)
      if (c + k < c1) {
        add[k] = *reinterpret_cast<const float4*>(q + k * step);
        f[k] = exp2f(p.cum[head * p.rows + p.chunk_row[c + k] + p.chunk_rows[c + k] - 1]);
      }
#pragma unroll
    for (int k = 0; k < AHEAD; ++k)
      if (c + k < c1) {
        *reinterpret_cast<float4*>(q + k * step) = s;
        s = make_float4(fmaf(s.x, f[k], add[k].x), fmaf(s.y, f[k], add[k].y), fmaf(s.z, f[k], add[k].z), fmaf(s.w, f[k], add[k].w));
      }
  }
  *sp = s;
}

// ---------------------------------------------------------------- delta rule: A, its inverse, W, V', decayed keys
constexpr int WY_LD = 132, WY_TMP = 64 * 68;     // row stride of A in floats; scratch of the block products

// out[2 rows][4 cols] = sum over k in [k0, k1) of a[r][k] b[k][c..c+3]; k0, k1 multiples of 4
__device__ __forceinline__ void small_tile(const float* a, int lda, const float* b, int ldb, int k0, int k1, float (&o)[2][4]) {
  for (int k = k0; k < k1; k += 4) {
    const float4 a0 = *reinterpret_cast<const float4*>(a + k), a1 = *reinterpret_cast<const float4*>(a + lda + k);
    const float av[2][4] = {{a0.x, a0.y, a0.z, a0.w}, {a1.x, a1.y, a1.z, a1.w}};
#pragma unroll
    for (int q = 0; q < 4; ++q) {
      const float4 bv = *reinterpret_cast<const float4*>(b + (k + q) * ldb);
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        o[r][0] = fmaf(av[r][q], bv.x, o[r][0]);
        o[r][1] = fmaf(av[r][q], bv.y, o[r][1]);
        o[r][2] = fmaf(av[r][q], bv.z, o[r][2]);
        o[r][3] = fmaf(av[r][q], bv.w, o[r][3]);
      }
    }
  }
}

__global__ void __launch_bounds__(RC_THREADS, 1)
delta_wy_kernel(const __grid_constant__ CUtensorMap tmap_v, RecTiles p, int atoms_v) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t *k_hi = smem, *k_lo = smem + 2 * RT_ATOM;
  uint8_t *t_hi = smem + 4 * RT_ATOM, *t_lo = smem + 6 * RT_ATOM;       // T over A once A has been read
  float* A = reinterpret_cast<float*>(t_hi);                             // [128][WY_LD]
  uint8_t* v_s = t_hi + 68 * 1024;
  float* tmp = reinterpret_cast<float*>(v_s + atoms_v * RT_ATOM);
  float *cum = tmp + WY_TMP, *wt = cum + RT_C, *uk = wt + RT_C, *f1 = uk + RT_C, *f2 = f1 + RT_C;
  uint64_t* bars = reinterpret_cast<uint64_t*>(f2 + RT_C);
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 2);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int chunk = blockIdx.x, head = blockIdx.y, group = head / p.per_group, groups = p.heads / p.per_group;
  const int first = p.chunk_row[chunk], rows = p.chunk_rows[chunk];
  if (tid == 0) {
    mbar_init(smem_u32(bars), 1);
    mbar_init(smem_u32(bars + 1), 1);
    *abort_flag = 0;
    mbar_fence_init();
    fence_proxy_async();
    mbar_arrive_expect_tx(smem_u32(bars), atoms_v * RT_ATOM);
    for (int a = 0; a < atoms_v; ++a)
      tma_load_2d(smem_u32(v_s + a * RT_ATOM), &tmap_v, smem_u32(bars), p.v_col + head * p.vdim + a * 64, p.row0 + first);
  }
  if (warp == 1) {
    tmem_alloc(smem_u32(tmem_slot), 256);
    tmem_relinquish();
  }
  AtomTile f[2];
  const __nv_bfloat16* kb = p.u + (p.row0 + first) * p.ldu + p.k_col + group * p.dim;
#pragma unroll
  for (int a = 0; a < 2; ++a) f[a].fetch(kb, p.ldu, rows, a * 64, p.dim);
  if (tid < RT_C) {
    const bool live = tid < rows;
    const long long at = head * p.rows + first;
    const float c = live ? p.cum[at + tid] : 0.f, k = live ? p.unit[(groups + group) * p.rows + first + tid] : 0.f;
    cum[tid] = c;
    wt[tid] = live ? p.wt[at + tid] : 0.f;
    uk[tid] = k;
    f1[tid] = k * exp2f(c);                                             // key times the decay from the chunk's start
    f2[tid] = live ? k * exp2f(p.cum[at + rows - 1] - c) : 0.f;         // ... to the chunk's end
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *tmem_slot;
#pragma unroll
  for (int a = 0; a < 2; ++a) f[a].store_scaled(k_hi + a * RT_ATOM, k_lo + a * RT_ATOM, uk);
  fence_proxy_async();
  __syncthreads();
  if (tid == 0) {      // K K^T
    constexpr uint32_t idesc = make_idesc_bf16(RT_C, RT_C, false, false);
    const int steps = (p.dim + 15) / 16;
    for (int part = 0; part < 3; ++part) {
      const uint32_t a = smem_u32(part == 2 ? k_lo : k_hi), b = smem_u32(part == 1 ? k_lo : k_hi);
      for (int kk = 0; kk < steps; ++kk) {
        const uint32_t o = (kk >> 2) * RT_ATOM + (kk & 3) * 32;
        umma_f16(tmem, make_smem_desc_sw128(a + o, 16, 1024), make_smem_desc_sw128(b + o, 16, 1024), idesc, (part | kk) != 0 ? 1u : 0u);
      }
    }
    umma_commit(smem_u32(bars + 1));
  }
  mbar_wait(smem_u32(bars + 1), 0, abort_flag, p.status, RLB_ERR_WAIT_TMEM_FULL);
  __syncwarp();
  tc_fence_after();
  const int quarter = warp & 3, side = warp >> 2, i = quarter * 32 + lane;
  const uint32_t lane_addr = static_cast<uint32_t>(quarter * 32) << 16;
  {
    uint32_t r[32];
    tmem_ld_32x32b_x32(tmem + lane_addr + side * 32, r);
    tmem_ld_wait();
    const float ci = cum[i], wi = wt[i];
#pragma unroll
    for (int q = 0; q < 8; ++q) {
      float v[4];
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        const int j = side * 32 + q * 4 + k;
        v[k] = j < i && i < rows ? wi * exp2f(ci - cum[j]) * __uint_as_float(r[q * 4 + k]) : 0.f;
      }
      *reinterpret_cast<float4*>(A + i * WY_LD + side * 32 + q * 4) = make_float4(v[0], v[1], v[2], v[3]);
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp < 8) {      // inverses of the 16 x 16 blocks on the diagonal of I + A: lane c solves for column c
    float* B = A + warp * 16 * WY_LD + warp * 16;
    float x[16];
#pragma unroll
    for (int r = 0; r < 16; ++r) {
      float v = r == (lane & 15) ? 1.f : 0.f;
#pragma unroll
      for (int j = 0; j < r; ++j) v = fmaf(-B[r * WY_LD + j], x[j], v);
      x[r] = v;
    }
    __syncwarp();
    if (lane < 16) {
#pragma unroll
      for (int r = 0; r < 16; ++r) B[r * WY_LD + lane] = x[r];
    }
  }
  __syncthreads();
  // [T11 0; L21 T22] -> [T11 0; -T22 L21 T11  T22] for pairs of neighbouring blocks of n rows
#pragma unroll 1
  for (int n = 16; n < RT_C; n *= 2) {
    const int quads = n / 4, per = quads * (n / 2), tile = tid % per, pair = tid / per, base = pair * 2 * n;
    const int r = tile / quads * 2, c = tile % quads * 4;
    const bool live = pair < RT_C / (2 * n);
    float* L21 = A + (base + n) * WY_LD + base;
    float* X = tmp + pair * n * (n + 4);
    if (live) {
      float o[2][4] = {};
      small_tile(L21 + r * WY_LD, WY_LD, A + base * WY_LD + base + c, WY_LD, c, n, o);                 // T11[k][c] = 0 for k < c
#pragma unroll
      for (int q = 0; q < 2; ++q) *reinterpret_cast<float4*>(X + (r + q) * (n + 4) + c) = make_float4(o[q][0], o[q][1], o[q][2], o[q][3]);
    }
    __syncthreads();
    if (live) {
      float o[2][4] = {};
      small_tile(A + (base + n + r) * WY_LD + base + n, WY_LD, X + c, n + 4, 0, (r + 2 + 3) / 4 * 4, o);   // T22[r][k] = 0 for k > r
#pragma unroll
      for (int q = 0; q < 2; ++q) *reinterpret_cast<float4*>(L21 + (r + q) * WY_LD + c) = make_float4(-o[q][0], -o[q][1], -o[q][2], -o[q][3]);
    }
    __syncthreads();
  }
  {      // T diag(w) as operand tiles in the place of T; keys times the decay from the chunk's start; decayed keys to memory
    float t[4][8];
#pragma unroll
    for (int n = 0; n < 4; ++n) {
      const int q = tid + n * RC_THREADS, r = q >> 4, c = (q & 15) * 8;
      const float4 a = *reinterpret_cast<const float4*>(A + r * WY_LD + c), b = *reinterpret_cast<const float4*>(A + r * WY_LD + c + 4);
      const float v[8] = {a.x, a.y, a.z, a.w, b.x, b.y, b.z, b.w};
#pragma unroll
      for (int k = 0; k < 8; ++k) t[n][k] = c + k <= r ? v[k] * wt[c + k] : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int n = 0; n < 4; ++n) {
      const int q = tid + n * RC_THREADS, r = q >> 4, piece = q & 15;
      store_split(t_hi, t_lo, (piece >> 3) * RT_ATOM + rt_sw(r, piece & 7), t[n]);
    }
    const long long kt = (static_cast<long long>(chunk) * p.heads + head) * RT_C * RT_C;
#pragma unroll
    for (int a = 0; a < 2; ++a) {
      f[a].store_scaled(k_hi + a * RT_ATOM, k_lo + a * RT_ATOM, f1);
#pragma unroll
      for (int n = 0; n < RC_FILL; ++n) {
        const int q = tid + n * RC_THREADS, r = q >> 3, d = a * 64 + (q & 7) * 8;
        float v[8];
        unpack8(f[a].raw[n], v);
#pragma unroll
        for (int k = 0; k < 8; ++k) v[k] *= f2[r];
        uint4 hi, lo;
        split8(v, hi, lo);
        *reinterpret_cast<uint4*>(p.kt_hi + kt + r * RT_C + d) = hi;
        *reinterpret_cast<uint4*>(p.kt_lo + kt + r * RT_C + d) = lo;
      }
    }
  }
  fence_proxy_async();
  tc_fence_before();
  __syncthreads();
  const int dcols = (p.dim + 15) / 16 * 16, vcols = (p.vdim + 15) / 16 * 16;
  if (tid == 0) {
    mbar_wait(smem_u32(bars), 0, abort_flag, p.status, RLB_ERR_WAIT_FULL);
    tc_fence_after();
    const uint32_t idesc_w = make_idesc_bf16(RT_C, dcols, false, true), idesc_v = make_idesc_bf16(RT_C, vcols, false, true);
    for (int part = 0; part < 3; ++part) {
      const uint32_t t = smem_u32(part == 2 ? t_lo : t_hi), k = smem_u32(part == 1 ? k_lo : k_hi);
      for (int kk = 0; kk < RT_C / 16; ++kk) {
        const uint64_t td = make_smem_desc_sw128(t + (kk >> 2) * RT_ATOM + (kk & 3) * 32, 16, 1024);
        umma_f16(tmem, td, make_smem_desc_sw128(k + kk * 2048, RT_ATOM, 1024), idesc_w, (part | kk) != 0 ? 1u : 0u);
        if (part != 1) umma_f16(tmem + RT_C, td, make_smem_desc_sw128(smem_u32(v_s) + kk * 2048, RT_ATOM, 1024), idesc_v, (part | kk) != 0 ? 1u : 0u);
      }
    }
    umma_commit(smem_u32(bars + 1));
  }
  mbar_wait(smem_u32(bars + 1), 1, abort_flag, p.status, RLB_ERR_WAIT_TMEM_FULL);
  __syncwarp();
  tc_fence_after();
  const long long tile = (static_cast<long long>(chunk) * p.heads + head) * RT_C + i;
  {
    uint32_t r[32];
    const int c = side * 32;
    tmem_ld_32x32b_x32(tmem + lane_addr + c, r);
    tmem_ld_wait();
#pragma unroll
    for (int q = 0; q < 4; ++q) {
      float v[8];
#pragma unroll
      for (int k = 0; k < 8; ++k) v[k] = c + q * 8 + k < p.dim ? __uint_as_float(r[q * 8 + k]) : 0.f;
      uint4 hi, lo;
      split8(v, hi, lo);
      *reinterpret_cast<uint4*>(p.w_hi + tile * RT_C + c + q * 8) = hi;
      *reinterpret_cast<uint4*>(p.w_lo + tile * RT_C + c + q * 8) = lo;
    }
    tmem_ld_32x32b_x32(tmem + RT_C + lane_addr + c, r);
    tmem_ld_wait();
#pragma unroll
    for (int q = 0; q < 8; ++q)
      if (c + q * 4 < p.vdim)
        *reinterpret_cast<float4*>(p.u0 + tile * p.vdim + c + q * 4) =
            make_float4(__uint_as_float(r[q * 4]), __uint_as_float(r[q * 4 + 1]), __uint_as_float(r[q * 4 + 2]), __uint_as_float(r[q * 4 + 3]));
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem, 256);
  }
}

// ---------------------------------------------------------------- delta rule: chunk after chunk
// VB value columns per CTA. High and low parts of the state (and of the writes) stand side by side as one operand of 2 VB columns, so that
// hi * [hi | lo] is one product; the epilogue adds the two halves.
constexpr int DS_THREADS = 192;
template <int VB>
__global__ void __launch_bounds__(DS_THREADS, 1)
delta_scan_kernel(const __grid_constant__ CUtensorMap tmap_whi, const __grid_constant__ CUtensorMap tmap_wlo, const __grid_constant__ CUtensorMap tmap_khi,
                  const __grid_constant__ CUtensorMap tmap_klo, RecTiles p, const int* __restrict__ piece_chunk, const int* __restrict__ positions,
                  const long long* __restrict__ state_rows, float* __restrict__ state, long long num_states) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t *w_s = smem, *k_s = smem + 4 * RT_ATOM;                 // each [hi: 2 atoms | lo: 2 atoms]
  constexpr int ATOMS = VB / 32, PIECES = VB / 8;                 // atoms and 16-byte pieces per part of the state and write operands
  uint8_t *s_s = smem + 8 * RT_ATOM, *u_s = s_s + ATOMS * RT_ATOM;
  auto hi_at = [](int row, int q) { return rt_sw(row, q); };
  auto lo_at = [](int row, int q) { return VB == 64 ? RT_ATOM + rt_sw(row, q) : rt_sw(row, q + 4); };
  uint64_t* bars = reinterpret_cast<uint64_t*>(u_s + ATOMS * RT_ATOM);
  uint64_t *w_full = bars, *w_empty = bars + 1, *k_full = bars + 2, *k_empty = bars + 3, *acc1 = bars + 4, *acc2 = bars + 5, *s_ready = bars + 6,
           *u_ready = bars + 7;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 8);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int v0 = blockIdx.x * VB, head = blockIdx.y, piece = blockIdx.z;
  const long long sr = state_rows[piece];
  if (sr < 0 || sr >= num_states) {      // uniform
    if (threadIdx.x == 0 && p.status) atomicCAS(p.status, 0, RLB_ERR_BOUNDS);
    return;
  }
  if (threadIdx.x == 0) {
    for (int b = 0; b < 6; ++b) mbar_init(smem_u32(bars + b), 1);
    mbar_init(smem_u32(s_ready), 128);
    mbar_init(smem_u32(u_ready), 128);
    *abort_flag = 0;
    mbar_fence_init();
    fence_proxy_async();
  }
  if (warp == 1) {
    tmem_alloc(smem_u32(tmem_slot), 4 * VB);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *tmem_slot;
  const int c0 = piece_chunk[piece], c1 = piece_chunk[piece + 1];
  const int atoms_d = (p.dim + 63) / 64;
  if (warp == 0) {
    if (lane == 0) {
      for (int c = c0; c < c1; ++c) {
        const uint32_t ph = (c - c0) & 1;
        const int row = (c * p.heads + head) * RT_C;
        if (!mbar_wait(smem_u32(w_empty), ph ^ 1, abort_flag, p.status, RLB_ERR_WAIT_EMPTY)) break;
        mbar_arrive_expect_tx(smem_u32(w_full), 2 * atoms_d * RT_ATOM);
        for (int a = 0; a < atoms_d; ++a) {
          tma_load_2d(smem_u32(w_s + a * RT_ATOM), &tmap_whi, smem_u32(w_full), a * 64, row);
          tma_load_2d(smem_u32(w_s + (2 + a) * RT_ATOM), &tmap_wlo, smem_u32(w_full), a * 64, row);
        }
        if (!mbar_wait(smem_u32(k_empty), ph ^ 1, abort_flag, p.status, RLB_ERR_WAIT_EMPTY)) break;
        mbar_arrive_expect_tx(smem_u32(k_full), 4 * RT_ATOM);
        for (int a = 0; a < 2; ++a) {
          tma_load_2d(smem_u32(k_s + a * RT_ATOM), &tmap_khi, smem_u32(k_full), a * 64, row);
          tma_load_2d(smem_u32(k_s + (2 + a) * RT_ATOM), &tmap_klo, smem_u32(k_full), a * 64, row);
        }
      }
    }
  } else if (warp == 1) {
    if (lane == 0) {
      constexpr uint32_t idesc_w2 = make_idesc_bf16(RT_C, 2 * VB, false, true), idesc_w1 = make_idesc_bf16(RT_C, VB, false, true);
      constexpr uint32_t idesc_k2 = make_idesc_bf16(RT_C, 2 * VB, true, true), idesc_k1 = make_idesc_bf16(RT_C, VB, true, true);
      const int steps = (p.dim + 15) / 16;
      for (int c = c0; c < c1; ++c) {
        const uint32_t ph = (c - c0) & 1;
        if (!mbar_wait(smem_u32(w_full), ph, abort_flag, p.status, RLB_ERR_WAIT_FULL)) break;
        if (!mbar_wait(smem_u32(s_ready), ph, abort_flag, p.status, RLB_ERR_WAIT_FLAG)) break;
        tc_fence_after();
        for (int part = 0; part < 2; ++part) {      // W S: hi [hi | lo], then lo hi
          const uint32_t w = smem_u32(w_s + part * 2 * RT_ATOM);
          for (int kk = 0; kk < steps; ++kk)
            umma_f16(tmem, make_smem_desc_sw128(w + (kk >> 2) * RT_ATOM + (kk & 3) * 32, 16, 1024), make_smem_desc_sw128(smem_u32(s_s) + kk * 2048, RT_ATOM, 1024),
                     part ? idesc_w1 : idesc_w2, (part | kk) != 0 ? 1u : 0u);
        }
        umma_commit(smem_u32(w_empty));
        umma_commit(smem_u32(acc1));
        if (!mbar_wait(smem_u32(k_full), ph, abort_flag, p.status, RLB_ERR_WAIT_FULL)) break;
        if (!mbar_wait(smem_u32(u_ready), ph, abort_flag, p.status, RLB_ERR_WAIT_FLAG)) break;
        tc_fence_after();
        for (int part = 0; part < 2; ++part) {      // K^T U
          const uint32_t k = smem_u32(k_s + part * 2 * RT_ATOM);
          for (int kk = 0; kk < RT_C / 16; ++kk)
            umma_f16(tmem + 2 * VB, make_smem_desc_sw128(k + kk * 2048, RT_ATOM, 1024), make_smem_desc_sw128(smem_u32(u_s) + kk * 2048, RT_ATOM, 1024),
                     part ? idesc_k1 : idesc_k2, (part | kk) != 0 ? 1u : 0u);
        }
        umma_commit(smem_u32(k_empty));
        umma_commit(smem_u32(acc2));
      }
    }
  } else {
    const int quarter = warp & 3, row = quarter * 32 + lane;
    const uint32_t lane_addr = static_cast<uint32_t>(quarter * 32) << 16;
    const bool mine = row < p.dim;
    float* st = state + ((sr * p.heads + head) * p.dim + row) * static_cast<long long>(p.vdim) + v0;
    float S[VB];
    const bool fresh = positions[p.row0 + p.chunk_row[c0]] == 0;
#pragma unroll
    for (int q = 0; q < VB / 4; ++q) {
      float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
      if (mine && !fresh && v0 + q * 4 < p.vdim) v = *reinterpret_cast<const float4*>(st + q * 4);
      S[q * 4] = v.x; S[q * 4 + 1] = v.y; S[q * 4 + 2] = v.z; S[q * 4 + 3] = v.w;
    }
    bool ok = true;
    float4 u[VB / 4];
    auto fetch = [&](int c) {      // the row's part of V' of chunk c
      const float* up = p.u0 + ((static_cast<long long>(c) * p.heads + head) * RT_C + row) * p.vdim + v0;
#pragma unroll
      for (int q = 0; q < VB / 4; ++q) u[q] = v0 + q * 4 < p.vdim ? *reinterpret_cast<const float4*>(up + q * 4) : make_float4(0.f, 0.f, 0.f, 0.f);
    };
    fetch(c0);
    for (int c = c0; c < c1; ++c) {
      const uint32_t ph = (c - c0) & 1;
      const long long tile = static_cast<long long>(c) * p.heads + head;
      const int first = p.chunk_row[c], rows = p.chunk_rows[c];
      const float f = exp2f(p.cum[head * p.rows + first + rows - 1]);
      // the state as operand (the products that read the tiles before have completed), the chunk's start state for the outputs
#pragma unroll
      for (int q = 0; q < VB / 8; ++q) {
        const float v[8] = {S[q * 8], S[q * 8 + 1], S[q * 8 + 2], S[q * 8 + 3], S[q * 8 + 4], S[q * 8 + 5], S[q * 8 + 6], S[q * 8 + 7]};
        uint4 hi, lo;
        split8(v, hi, lo);
        *reinterpret_cast<uint4*>(s_s + hi_at(row, q)) = hi;
        *reinterpret_cast<uint4*>(s_s + lo_at(row, q)) = lo;
      }
      fence_proxy_async();
      mbar_arrive(smem_u32(s_ready));
      if (!mbar_wait(smem_u32(acc1), ph, abort_flag, p.status, RLB_ERR_WAIT_TMEM_FULL)) {
        ok = false;
        break;
      }
      tc_fence_after();
#pragma unroll
      for (int half = 0; half < ATOMS; ++half) {
        uint32_t r[32], r2[32];
        tmem_ld_32x32b_x32(tmem + lane_addr + half * 32, r);
        tmem_ld_32x32b_x32(tmem + VB + lane_addr + half * 32, r2);
        tmem_ld_wait();
#pragma unroll
        for (int k = 0; k < 32; ++k) r[k] = __float_as_uint(__uint_as_float(r[k]) + __uint_as_float(r2[k]));
#pragma unroll
        for (int q = 0; q < 4; ++q) {
          const float4 a = u[half * 8 + q * 2], b = u[half * 8 + q * 2 + 1];
          const float v[8] = {a.x - __uint_as_float(r[q * 8]),     a.y - __uint_as_float(r[q * 8 + 1]), a.z - __uint_as_float(r[q * 8 + 2]),
                              a.w - __uint_as_float(r[q * 8 + 3]), b.x - __uint_as_float(r[q * 8 + 4]), b.y - __uint_as_float(r[q * 8 + 5]),
                              b.z - __uint_as_float(r[q * 8 + 6]), b.w - __uint_as_float(r[q * 8 + 7])};
          uint4 hi, lo;
          split8(v, hi, lo);
          *reinterpret_cast<uint4*>(u_s + hi_at(row, half * 4 + q)) = hi;
          *reinterpret_cast<uint4*>(u_s + lo_at(row, half * 4 + q)) = lo;
        }
      }
      fence_proxy_async();
      tc_fence_before();
      mbar_arrive(smem_u32(u_ready));
      // under the second product: the next chunk's V', the chunk's start state and its writes (the warp's own rows, line by line)
      if (c + 1 < c1) fetch(c + 1);
      if (mine) {
        float* so = p.start + (tile * p.dim + row) * p.vdim + v0;
#pragma unroll
        for (int q = 0; q < VB / 4; ++q)
          if (v0 + q * 4 < p.vdim) *reinterpret_cast<float4*>(so + q * 4) = make_float4(S[q * 4], S[q * 4 + 1], S[q * 4 + 2], S[q * 4 + 3]);
      }
      __syncwarp();
#pragma unroll
      for (int q = 0; q < PIECES; ++q) {
        const int r = quarter * 32 + q * (32 / PIECES) + lane / PIECES, piece = lane % PIECES;
        if (r < rows && v0 + piece * 8 < p.vdim) {
          const long long g = (first + r) * static_cast<long long>(p.heads * p.vdim) + head * p.vdim + v0 + piece * 8;
          *reinterpret_cast<uint4*>(p.uu_hi + g) = *reinterpret_cast<const uint4*>(u_s + hi_at(r, piece));
          *reinterpret_cast<uint4*>(p.uu_lo + g) = *reinterpret_cast<const uint4*>(u_s + lo_at(r, piece));
        }
      }
      __syncwarp();
      if (!mbar_wait(smem_u32(acc2), ph, abort_flag, p.status, RLB_ERR_WAIT_TMEM_FULL)) {
        ok = false;
        break;
      }
      tc_fence_after();
#pragma unroll
      for (int half = 0; half < ATOMS; ++half) {
        uint32_t r[32], r2[32];
        tmem_ld_32x32b_x32(tmem + 2 * VB + lane_addr + half * 32, r);
        tmem_ld_32x32b_x32(tmem + 3 * VB + lane_addr + half * 32, r2);
        tmem_ld_wait();
#pragma unroll
        for (int k = 0; k < 32; ++k) S[half * 32 + k] = fmaf(S[half * 32 + k], f, __uint_as_float(r[k]) + __uint_as_float(r2[k]));
      }
      tc_fence_before();
    }
    if (ok && mine) {
#pragma unroll
      for (int q = 0; q < VB / 4; ++q)
        if (v0 + q * 4 < p.vdim) *reinterpret_cast<float4*>(st + q * 4) = make_float4(S[q * 4], S[q * 4 + 1], S[q * 4 + 2], S[q * 4 + 3]);
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem, 4 * VB);
  }
}

// ---------------------------------------------------------------- outputs
template <bool DELTA>
__global__ void __launch_bounds__(RC_THREADS, 1)
rec_out_kernel(const __grid_constant__ CUtensorMap tmap_v, const __grid_constant__ CUtensorMap tmap_vlo, RecTiles p, int atoms_v, int tmem_cols) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t *q_hi = smem, *q_lo = smem + RT_ATOM, *k_hi = smem + 2 * RT_ATOM, *k_lo = smem + 3 * RT_ATOM;
  uint8_t *w_hi = smem, *w_lo = smem + 2 * RT_ATOM;      // decayed weights [128 x 128], over the queries and keys once those have been read
  uint8_t* s_hi = smem + 4 * RT_ATOM;                    // 64 state rows x vdim
  uint8_t* s_lo = s_hi + atoms_v * RT_SATOM;
  uint8_t* v_s = s_lo + atoms_v * RT_SATOM;
  uint8_t* v_lo = v_s + atoms_v * RT_ATOM;               // (delta)
  float* cum = reinterpret_cast<float*>(v_lo + (DELTA ? atoms_v * RT_ATOM : 0));
  float *wt = cum + RT_C, *uq = wt + RT_C, *uk = uq + RT_C, *ssq = uk + RT_C;      // ssq [column groups][128]
  uint64_t* bars = reinterpret_cast<uint64_t*>(ssq + RC_THREADS);
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 2);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int chunk = blockIdx.x, head = blockIdx.y, group = head / p.per_group, groups = p.heads / p.per_group;
  const int first = p.chunk_row[chunk], rows = p.chunk_rows[chunk];
  if (tid == 0) {
    mbar_init(smem_u32(bars), 1);
    mbar_init(smem_u32(bars + 1), 1);
    *abort_flag = 0;
    mbar_fence_init();
    fence_proxy_async();
    mbar_arrive_expect_tx(smem_u32(bars), (DELTA ? 2 : 1) * atoms_v * RT_ATOM);
    for (int a = 0; a < atoms_v; ++a) {
      const int x = (DELTA ? 0 : p.v_col) + head * p.vdim + a * 64, row = (DELTA ? 0 : p.row0) + first;
      tma_load_2d(smem_u32(v_s + a * RT_ATOM), &tmap_v, smem_u32(bars), x, row);
      if (DELTA) tma_load_2d(smem_u32(v_lo + a * RT_ATOM), &tmap_vlo, smem_u32(bars), x, row);
    }
  }
  if (warp == 1) {
    tmem_alloc(smem_u32(tmem_slot), tmem_cols);
    tmem_relinquish();
  }
  if (tid < RT_C) {
    const bool live = tid < rows;
    cum[tid] = live ? p.cum[head * p.rows + first + tid] : 0.f;
    if (DELTA) {
      uq[tid] = live ? p.unit[group * p.rows + first + tid] : 0.f;
      uk[tid] = live ? p.unit[(groups + group) * p.rows + first + tid] : 0.f;
    } else {
      wt[tid] = live ? p.wt[head * p.rows + first + tid] : 0.f;
    }
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_s = *tmem_slot, tmem_o = tmem_s + RT_C;
  const int vcols = (p.vdim + 15) / 16 * 16;
  const uint32_t idesc_s = make_idesc_bf16(RT_C, RT_C, false, false), idesc_o = make_idesc_bf16(RT_C, vcols, false, true);
  const float* S0 = p.start + (static_cast<long long>(chunk) * p.heads + head) * p.dim * p.vdim;
  const __nv_bfloat16* ub = p.u + (p.row0 + first) * p.ldu + group * p.dim;
  int done = 0;      // commits waited for
  for (int d0 = 0; d0 < p.dim; d0 += 64) {
    AtomTile fq, fk;      // the loads of queries, keys and start state are in flight together
    fq.fetch(ub + p.q_col, p.ldu, rows, d0, p.dim);
    fk.fetch(ub + p.k_col, p.ldu, rows, d0, p.dim);
    const int pieces = atoms_v * 8;      // 8-column pieces of a state row
    float4 sx[4], sy[4];
#pragma unroll
    for (int n = 0; n < 4; ++n) {        // 64 rows x at most 32 pieces
      const int i = tid + n * RC_THREADS, r = i / pieces, v0 = (i % pieces) * 8;
      sx[n] = sy[n] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (i < 64 * pieces && d0 + r < p.dim && v0 < p.vdim) {
        sx[n] = *reinterpret_cast<const float4*>(S0 + static_cast<long long>(d0 + r) * p.vdim + v0);
        sy[n] = *reinterpret_cast<const float4*>(S0 + static_cast<long long>(d0 + r) * p.vdim + v0 + 4);
      }
    }
    if (d0 > 0) {      // the previous products have read the stage
      mbar_wait(smem_u32(bars + 1), done & 1, abort_flag, p.status, RLB_ERR_WAIT_EMPTY);
      ++done;
      __syncthreads();
    }
    if (DELTA) {
      fq.store_scaled(q_hi, q_lo, uq);
      fk.store_scaled(k_hi, k_lo, uk);
    } else {
      fq.store(q_hi);
      fk.store(k_hi);
    }
#pragma unroll
    for (int n = 0; n < 4; ++n) {
      const int i = tid + n * RC_THREADS, r = i / pieces, g = i % pieces;
      if (i < 64 * pieces) {
        const float v[8] = {sx[n].x, sx[n].y, sx[n].z, sx[n].w, sy[n].x, sy[n].y, sy[n].z, sy[n].w};
        store_split(s_hi, s_lo, (g >> 3) * RT_SATOM + rt_sw(r, g & 7), v);
      }
    }
    fence_proxy_async();
    tc_fence_before();
    __syncthreads();
    if (tid == 0) {
      tc_fence_after();
      const int steps = min(4, (p.dim - d0 + 15) / 16);
      for (int part = 0; part < (DELTA ? 3 : 2); ++part) {     // hi hi, hi lo, lo hi (exact queries and keys: hi hi, and hi lo for the state)
        const uint32_t q = smem_u32(part == 2 ? q_lo : q_hi), k = smem_u32(part == 1 ? k_lo : k_hi), s = smem_u32(part == 1 ? s_lo : s_hi);
        for (int kk = 0; kk < steps; ++kk) {
          const uint32_t acc = (d0 | part | kk) != 0 ? 1u : 0u;
          const uint64_t qd = make_smem_desc_sw128(q + kk * 32, 16, 1024);
          if (DELTA || part == 0) umma_f16(tmem_s, qd, make_smem_desc_sw128(k + kk * 32, 16, 1024), idesc_s, acc);
          umma_f16(tmem_o, qd, make_smem_desc_sw128(s + kk * 2048, RT_SATOM, 1024), idesc_o, acc);
        }
      }
      umma_commit(smem_u32(bars + 1));
    }
  }
  mbar_wait(smem_u32(bars + 1), done & 1, abort_flag, p.status, RLB_ERR_WAIT_TMEM_FULL);
  ++done;
  __syncwarp();
  tc_fence_after();
  // groups of four warps share the rows and split the columns
  const int quarter = warp & 3, side = warp >> 2, i = quarter * 32 + lane;
  const uint32_t lane_addr = static_cast<uint32_t>(quarter * 32) << 16;
  const float ci = cum[i];
  for (int c = side * 32; c < RT_C; c += RC_THREADS / 4) {
    uint32_t r[32];
    tmem_ld_32x32b_x32(tmem_s + lane_addr + c, r);
    tmem_ld_wait();
#pragma unroll
    for (int q = 0; q < 4; ++q) {
      float v[8];
#pragma unroll
      for (int k = 0; k < 8; ++k) {
        const int j = c + q * 8 + k;
        v[k] = j <= i && i < rows ? __uint_as_float(r[q * 8 + k]) * exp2f(ci - cum[j]) * (DELTA ? 1.f : wt[j]) : 0.f;
      }
      store_split(w_hi, w_lo, (c >> 6) * RT_ATOM + rt_sw(i, ((c & 63) >> 3) + q), v);
    }
  }
  const float fi = exp2f(ci);
  for (int c = side * 32; c < vcols; c += RC_THREADS / 4) {     // start-state term: row i is 2^c_i times what stands in O
    uint32_t r[16];
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      if (c + h * 16 < vcols) {
        tmem_ld_32x32b_x16(tmem_o + lane_addr + c + h * 16, r);
        tmem_ld_wait();
#pragma unroll
        for (int k = 0; k < 16; ++k) r[k] = __float_as_uint(__uint_as_float(r[k]) * fi);
        tmem_st_32x32b_x16(tmem_o + lane_addr + c + h * 16, r);
      }
    }
  }
  tmem_st_wait();
  fence_proxy_async();
  tc_fence_before();
  __syncthreads();
  if (tid == 0) {
    mbar_wait(smem_u32(bars), 0, abort_flag, p.status, RLB_ERR_WAIT_FULL);
    tc_fence_after();
    for (int part = 0; part < (DELTA ? 3 : 2); ++part) {      // delta: hi hi, lo hi, hi lo
      const uint32_t w = smem_u32(part == 1 ? w_lo : w_hi), v = smem_u32(DELTA && part == 2 ? v_lo : v_s);
      for (int kk = 0; kk < RT_C / 16; ++kk)
        umma_f16(tmem_o, make_smem_desc_sw128(w + (kk >> 2) * RT_ATOM + (kk & 3) * 32, 16, 1024), make_smem_desc_sw128(v + kk * 2048, RT_ATOM, 1024), idesc_o, 1u);
    }
    umma_commit(smem_u32(bars + 1));
  }
  mbar_wait(smem_u32(bars + 1), done & 1, abort_flag, p.status, RLB_ERR_WAIT_TMEM_FULL);
  __syncwarp();
  tc_fence_after();
  float rstd = 1.f;
  if (DELTA) {
    float ss = 0.f;
    for (int c = side * 32; c < p.vdim; c += RC_THREADS / 4) {
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
    for (int g = 0; g < RC_THREADS / 128; ++g) ss += ssq[g * RT_C + i];
    rstd = 1.f / sqrtf(ss / static_cast<float>(p.vdim) + p.eps);
  }
  const long long row = p.row0 + first + i;
  const float Dh = DELTA ? 0.f : __bfloat162float(p.D[head]);
  for (int c = side * 32; c < p.vdim; c += RC_THREADS / 4) {
    uint32_t r[32];
    tmem_ld_32x32b_x32(tmem_o + lane_addr + c, r);
    tmem_ld_wait();
    if (i < rows) {
#pragma unroll
      for (int q = 0; q < 4; ++q) {
        const int v0 = c + q * 8;
        if (v0 < p.vdim) {
          float g[8], w[8];
          unpack8(*reinterpret_cast<const uint4*>(p.p + row * p.ldp + p.gate_off + head * p.vdim + v0), g);
          unpack8(*reinterpret_cast<const uint4*>(DELTA ? p.norm + v0 : p.u + row * p.ldu + p.v_col + head * p.vdim + v0), w);
          uint32_t o[4];
#pragma unroll
          for (int k = 0; k < 8; ++k) {
            const float acc = __uint_as_float(r[q * 8 + k]);
            g[k] = (DELTA ? acc * rstd * w[k] : fmaf(Dh, w[k], acc)) * rc_silu_bf16(g[k]);
          }
#pragma unroll
          for (int k = 0; k < 4; ++k) o[k] = pack_bf16x2(g[2 * k], g[2 * k + 1]);
          *reinterpret_cast<uint4*>(p.y + row * p.ldy + head * p.vdim + v0) = make_uint4(o[0], o[1], o[2], o[3]);
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
// One token per row. The convolution of the CTA's channels happens here: the ring slot of this position is the one no CTA reads, so the CTA
// that owns a channel (the first head of a group, for shared ones) writes it meanwhile.
struct RecStep {
  const __nv_bfloat16* p;
  long long ldp;
  int conv_off, channels, taps;
  const __nv_bfloat16* w;
  const __nv_bfloat16* bias;
  __nv_bfloat16* ring;
  const int* positions;
  const long long* state_rows;
  float* state;
  long long num_states;
  int heads, groups, dim, vdim;
  int gate_off, a_off, b_off;      // columns: gate, decay (dt), beta
  const __nv_bfloat16* A_log;
  const __nv_bfloat16* dt_bias;
  const __nv_bfloat16* D;          // Mamba-2
  const __nv_bfloat16* norm;       // delta
  float unit_eps, eps;
  __nv_bfloat16* y;
  long long ldy;
  int* status;
};

// A channel's inputs in registers (up to four taps), so that a thread has the loads of several channels in flight.
constexpr int SC_TAPS = 4;
struct StepChannel {
  __nv_bfloat16 in, past[SC_TAPS - 1];
  float w[SC_TAPS], b;
  __device__ __forceinline__ void fetch(const RecStep& s, long long row, long long sr, int pos, int c) {
    in = s.p[row * s.ldp + s.conv_off + c];
    b = s.bias ? __bfloat162float(s.bias[c]) : 0.f;
    const __nv_bfloat16* ring = s.ring + sr * s.taps * s.channels + c;
    const __nv_bfloat16* wc = s.w + static_cast<long long>(c + 1) * s.taps - 1;      // the current token's tap
    w[0] = __bfloat162float(*wc);
#pragma unroll
    for (int back = 1; back < SC_TAPS; ++back) {
      const bool live = back < s.taps && back <= pos;
      past[back - 1] = live ? ring[static_cast<long long>((pos - back) % s.taps) * s.channels] : __float2bfloat16(0.f);
      w[back] = live ? __bfloat162float(wc[-back]) : 0.f;
    }
  }
  // The convolved and activated value, rounded as the portions' convolution leaves it.
  __device__ __forceinline__ float finish(const RecStep& s, long long sr, int pos, int c, bool owner) const {
    float v = b;
    __nv_bfloat16* ring = s.ring + sr * s.taps * s.channels + c;
    for (int back = s.taps - 1; back >= SC_TAPS; --back)
      if (back <= pos)
        v = fmaf(__bfloat162float(s.w[static_cast<long long>(c + 1) * s.taps - 1 - back]),
                 __bfloat162float(ring[static_cast<long long>((pos - back) % s.taps) * s.channels]), v);
#pragma unroll
    for (int back = SC_TAPS - 1; back > 0; --back) v = fmaf(w[back], __bfloat162float(past[back - 1]), v);
    v = fmaf(w[0], __bfloat162float(in), v);
    if (owner) ring[static_cast<long long>(pos % s.taps) * s.channels] = in;
    return __bfloat162float(__float2bfloat16(rc_silu(v)));
  }
};
// out[i] = channel(i) for i < n; `channel` and `owner` name the convolved channel and whether this CTA keeps its ring. Two channels per
// thread in flight.
template <typename Channel, typename Owner, typename Store>
__device__ __forceinline__ void step_convolve(const RecStep& s, long long row, long long sr, int pos, int n, Channel channel, Owner owner, Store store) {
  const int step = blockDim.x;
  for (int i = threadIdx.x; i < n; i += 2 * step) {
    StepChannel a, b;
    const bool two = i + step < n;
    const int ca = channel(i), cb = two ? channel(i + step) : ca;
    a.fetch(s, row, sr, pos, ca);
    if (two) b.fetch(s, row, sr, pos, cb);
    store(i, a.finish(s, sr, pos, ca, owner(i)));
    if (two) store(i + step, b.finish(s, sr, pos, cb, owner(i + step)));
  }
}

__global__ void __launch_bounds__(256) mamba2_step_kernel(RecStep s) {
  extern __shared__ float sm[];
  float *x = sm, *B = x + s.vdim, *C = B + s.dim;
  float4* part = reinterpret_cast<float4*>(C + s.dim);      // [256] (dim and vdim are multiples of 8)
  const int row = blockIdx.x, head = blockIdx.y, tid = threadIdx.x, group = head / (s.heads / s.groups);
  pdl_sync();
  const long long sr = s.state_rows[row];
  if (sr < 0 || sr >= s.num_states) {
    if (tid == 0 && s.status) atomicCAS(s.status, 0, RLB_ERR_BOUNDS);
    return;
  }
  const int pos = s.positions[row], inner = s.heads * s.vdim;
  const bool first = head % (s.heads / s.groups) == 0;
  const float dt_in = __bfloat162float(s.p[row * s.ldp + s.a_off + head]), dt_b = __bfloat162float(s.dt_bias[head]), A_log = __bfloat162float(s.A_log[head]);
  step_convolve(s, row, sr, pos, s.vdim + 2 * s.dim,
                [&](int i) {
                  return i < s.vdim ? head * s.vdim + i
                                    : (i < s.vdim + s.dim ? inner + group * s.dim + i - s.vdim : inner + (s.groups + group) * s.dim + i - s.vdim - s.dim);
                },
                [&](int i) { return i < s.vdim || first; }, [&](int i, float v) { sm[i] = v; });
  const float dt = rc_softplus(dt_in + dt_b), dec = expf(-expf(A_log) * dt);
  __syncthreads();
  const int c4 = s.vdim / 4, slices = 256 / c4, slice = tid / c4, col = tid % c4;
  if (slice < slices) {
    const float4 v = reinterpret_cast<const float4*>(x)[col];
    float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
    float4* S = reinterpret_cast<float4*>(s.state + (sr * s.heads + head) * static_cast<long long>(s.dim) * s.vdim) + col;
    constexpr int U = 8;
    for (int i0 = slice; i0 < s.dim; i0 += U * slices) {
      float4 a[U];
#pragma unroll
      for (int q = 0; q < U; ++q) {
        const int i = i0 + q * slices;
        a[q] = i < s.dim && pos != 0 ? S[static_cast<long long>(i) * c4] : make_float4(0.f, 0.f, 0.f, 0.f);
      }
#pragma unroll
      for (int q = 0; q < U; ++q) {
        const int i = i0 + q * slices;
        if (i < s.dim) {
          const float b = dt * B[i], c = C[i];
          a[q] = make_float4(fmaf(dec, a[q].x, b * v.x), fmaf(dec, a[q].y, b * v.y), fmaf(dec, a[q].z, b * v.z), fmaf(dec, a[q].w, b * v.w));
          S[static_cast<long long>(i) * c4] = a[q];
          acc.x = fmaf(a[q].x, c, acc.x);
          acc.y = fmaf(a[q].y, c, acc.y);
          acc.z = fmaf(a[q].z, c, acc.z);
          acc.w = fmaf(a[q].w, c, acc.w);
        }
      }
    }
    part[tid] = acc;
  }
  __syncthreads();
  if (tid < c4) {
    float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int j = 0; j < slices; ++j) {
      const float4 t = part[j * c4 + tid];
      o.x += t.x; o.y += t.y; o.z += t.z; o.w += t.w;
    }
    const float4 v = reinterpret_cast<const float4*>(x)[tid];
    const float D = __bfloat162float(s.D[head]);
    const uint2 raw = *reinterpret_cast<const uint2*>(s.p + row * s.ldp + s.gate_off + head * s.vdim + tid * 4);
    const float2 z0 = unpack_bf16x2(raw.x), z1 = unpack_bf16x2(raw.y);
    *reinterpret_cast<uint2*>(s.y + row * s.ldy + head * s.vdim + tid * 4) =
        make_uint2(pack_bf16x2(fmaf(D, v.x, o.x) * rc_silu(z0.x), fmaf(D, v.y, o.y) * rc_silu(z0.y)),
                   pack_bf16x2(fmaf(D, v.z, o.z) * rc_silu(z1.x), fmaf(D, v.w, o.w) * rc_silu(z1.y)));
  }
}

// The head's state is contiguous (at most 64 KB): one bulk copy brings it to shared memory while the convolution runs, the read-out and the
// write work there, one bulk copy takes it back. The state's last writer stands far enough back on the stream for the copy to start before
// the dependency wait: a kernel may start once its predecessor has seen all work before it complete.
constexpr int DD_THREADS = 256;
__global__ void __launch_bounds__(DD_THREADS, 3) delta_step_kernel(RecStep s) {
  extern __shared__ __align__(16) float sm[];
  __shared__ float red[32];
  __shared__ __align__(8) uint64_t bar;
  __shared__ int abort_flag;
  float4* S = reinterpret_cast<float4*>(sm);                // [dim][vdim / 4]
  float *q = sm + s.dim * s.vdim, *k = q + s.dim, *v = k + s.dim;      // v: the value, then what is written
  float4* part = reinterpret_cast<float4*>(v + s.vdim);     // [2][DD_THREADS]
  const int row = blockIdx.x, head = blockIdx.y, tid = threadIdx.x, per = s.heads / s.groups, group = head / per, n = s.groups * s.dim;
  const long long sr = s.state_rows[row];
  const bool good = sr >= 0 && sr < s.num_states;
  float* state = s.state + ((good ? sr : 0) * s.heads + head) * static_cast<long long>(s.dim) * s.vdim;
  const uint32_t bytes = s.dim * s.vdim * 4;
  if (tid == 0) {
    mbar_init(smem_u32(&bar), 1);
    abort_flag = 0;
    mbar_fence_init();
    fence_proxy_async();
    if (good) {
      mbar_arrive_expect_tx(smem_u32(&bar), bytes);
      asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];" ::"r"(smem_u32(sm)), "l"(state), "r"(bytes),
                   "r"(smem_u32(&bar))
                   : "memory");
    }
  }
  pdl_sync();
  if (!good) {      // uniform
    if (tid == 0 && s.status) atomicCAS(s.status, 0, RLB_ERR_BOUNDS);
    return;
  }
  const int pos = s.positions[row];
  const float beta_in = __bfloat162float(s.p[row * s.ldp + s.b_off + head]), dt_in = __bfloat162float(s.p[row * s.ldp + s.a_off + head]);
  const float dt_b = __bfloat162float(s.dt_bias[head]), A_log = __bfloat162float(s.A_log[head]);
  const bool first = head % per == 0;
  step_convolve(s, row, sr, pos, 2 * s.dim + s.vdim,
                [&](int i) { return i < s.dim ? group * s.dim + i : (i < 2 * s.dim ? n + group * s.dim + i - s.dim : 2 * n + head * s.vdim + i - 2 * s.dim); },
                [&](int i) { return i >= 2 * s.dim || first; }, [&](int i, float x) { q[i] = x; });
  __syncthreads();      // (also: the barrier has been initialised)
  float qq = 0.f, kk = 0.f, qk = 0.f;      // every warp for itself
  for (int i = tid & 31; i < s.dim; i += 32) {
    const float qv = q[i], kv = k[i];
    qq += qv * qv;
    kk += kv * kv;
    qk += qv * kv;
  }
  qq = warp_sum(qq);
  kk = warp_sum(kk);
  qk = warp_sum(qk);
  const float qf = 1.f / (sqrtf(qq + s.unit_eps) * sqrtf(static_cast<float>(s.dim))), kf = 1.f / sqrtf(kk + s.unit_eps);
  const float beta = 1.f / (1.f + expf(-beta_in)), dec = expf(-expf(A_log) * rc_softplus(dt_in + dt_b));
  const int c4 = s.vdim / 4, slices = DD_THREADS / c4, slice = tid / c4, col = tid % c4;
  const bool live = slice < slices;
  const bool ok = mbar_wait(smem_u32(&bar), 0, &abort_flag, s.status, RLB_ERR_WAIT_FULL);
  float4 sk = make_float4(0.f, 0.f, 0.f, 0.f), sq = sk;
  if (live && pos != 0) {
#pragma unroll 4
    for (int i = slice; i < s.dim; i += slices) {
      const float4 t = S[i * c4 + col];
      const float kv = k[i], qv = q[i];
      sk.x = fmaf(t.x, kv, sk.x); sk.y = fmaf(t.y, kv, sk.y); sk.z = fmaf(t.z, kv, sk.z); sk.w = fmaf(t.w, kv, sk.w);
      sq.x = fmaf(t.x, qv, sq.x); sq.y = fmaf(t.y, qv, sq.y); sq.z = fmaf(t.z, qv, sq.z); sq.w = fmaf(t.w, qv, sq.w);
    }
  }
  part[tid] = sk;
  part[DD_THREADS + tid] = sq;
  __syncthreads();
  float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
  if (tid < c4) {
    float4 t = o;
    for (int j = 0; j < slices; ++j) {
      const float4 x = part[j * c4 + tid], y = part[DD_THREADS + j * c4 + tid];
      t.x += x.x; t.y += x.y; t.z += x.z; t.w += x.w;
      o.x += y.x; o.y += y.y; o.z += y.z; o.w += y.w;
    }
    float4 w = reinterpret_cast<float4*>(v)[tid];
    const float d = dec * kf;
    w = make_float4(beta * (w.x - d * t.x), beta * (w.y - d * t.y), beta * (w.z - d * t.z), beta * (w.w - d * t.w));
    const float f = dec * qf, g = qk * qf * kf;      // S'^T q = decay S^T q + (k . q) u
    o = make_float4(fmaf(g, w.x, f * o.x), fmaf(g, w.y, f * o.y), fmaf(g, w.z, f * o.z), fmaf(g, w.w, f * o.w));
    reinterpret_cast<float4*>(v)[tid] = make_float4(w.x * kf, w.y * kf, w.z * kf, w.w * kf);
  }
  __syncthreads();
  if (live) {
    const float4 w = reinterpret_cast<const float4*>(v)[col];
#pragma unroll 4
    for (int i = slice; i < s.dim; i += slices) {
      const float4 t = pos != 0 ? S[i * c4 + col] : make_float4(0.f, 0.f, 0.f, 0.f);
      const float kv = k[i];
      S[i * c4 + col] = make_float4(fmaf(dec, t.x, kv * w.x), fmaf(dec, t.y, kv * w.y), fmaf(dec, t.z, kv * w.z), fmaf(dec, t.w, kv * w.w));
    }
  }
  fence_proxy_async();
  __syncthreads();
  if (tid == 0 && ok) {
    asm volatile("cp.async.bulk.global.shared::cta.bulk_group [%0], [%1], %2;" ::"l"(state), "r"(smem_u32(sm)), "r"(bytes) : "memory");
    tma_store_commit();
  }
  const float ss = block_sum(o.x * o.x + o.y * o.y + o.z * o.z + o.w * o.w, red);
  if (tid < c4) {
    const float rstd = 1.f / sqrtf(ss / static_cast<float>(s.vdim) + s.eps);
    const uint2 raw = *reinterpret_cast<const uint2*>(s.p + row * s.ldp + s.gate_off + head * s.vdim + tid * 4);
    const uint2 wr = *reinterpret_cast<const uint2*>(s.norm + tid * 4);
    const float2 g0 = unpack_bf16x2(raw.x), g1 = unpack_bf16x2(raw.y), w0 = unpack_bf16x2(wr.x), w1 = unpack_bf16x2(wr.y);
    *reinterpret_cast<uint2*>(s.y + row * s.ldy + head * s.vdim + tid * 4) =
        make_uint2(pack_bf16x2(o.x * rstd * w0.x * rc_silu(g0.x), o.y * rstd * w0.y * rc_silu(g0.y)),
                   pack_bf16x2(o.z * rstd * w1.x * rc_silu(g1.x), o.w * rstd * w1.y * rc_silu(g1.y)));
  }
  if (tid == 0) tma_store_wait<0>();
}

int set_smem(const void* kernel, int bytes, int* configured) {
  if (bytes <= *configured) return 0;
  const cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, bytes);
  if (e != cudaSuccess) return static_cast<int>(e);
  *configured = bytes;
  return 0;
}

struct RecArgs {      // what both kinds of mixer pass (mirrored in ops/sequence_ops.py)
  const void *p, *u, *conv_w, *conv_bias, *A_log, *dt_bias, *D, *norm;
  void *y, *ring;
  const int *positions, *piece_chunk, *chunk_row, *chunk_rows;
  const long long* state_rows;      // of the singles or of the portions
  float *state, *cum, *wt, *unit, *start, *u0;
  void *w_hi, *w_lo, *kt_hi, *kt_lo, *uu_hi, *uu_lo;
  int* status;
  long long ldp, ldu, ldy, num_states, rows;      // rows: all rows of u, p, y
  int delta, heads, groups, dim, vdim, taps, channels, conv_off, gate_off, a_off, b_off, row0, pieces, chunks;
  float unit_eps, eps;
};
}  // namespace

// Shapes the chunked and the single-step kernels take.
RLB_API int rlb_rec_supported(int delta, int dim, int vdim) {
  return dim > 0 && vdim > 0 && dim % 8 == 0 && vdim % 8 == 0 && vdim <= (delta ? 128 : 256) && dim <= (delta ? 128 : 1024);
}

// Convolution of rows [0, rows) by runs, 8 channels per thread: channels, row strides multiples of 8; taps 2 .. 4; row_off and row_state per row.
RLB_API int rlb_conv_runs(const void* x, long long ldx, void* u, long long ldu, long long rows, int channels, int taps, const void* w, const void* bias,
                          const void* ring, const int* positions, const int* row_off, const long long* row_state, long long num_states, int* status,
                          void* stream) {
  if (rows <= 0) return 0;
  if (taps < 2 || taps > 4 || channels % 8 || ldx % 8 || ldu % 8 || !row_off || !row_state) return -2;
  if ((reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(u) | reinterpret_cast<uintptr_t>(ring) | reinterpret_cast<uintptr_t>(w) |
       reinterpret_cast<uintptr_t>(bias)) & 15)
    return -3;
  const dim3 grid(static_cast<unsigned>((rows + CV_RUN - 1) / CV_RUN), (channels / 8 + 127) / 128);
  auto k = taps == 2 ? conv_runs_kernel<2> : (taps == 3 ? conv_runs_kernel<3> : conv_runs_kernel<4>);
  k<<<grid, 128, 0, static_cast<cudaStream_t>(stream)>>>(static_cast<const __nv_bfloat16*>(x), ldx, static_cast<__nv_bfloat16*>(u), ldu, rows, channels,
      static_cast<const __nv_bfloat16*>(w), static_cast<const __nv_bfloat16*>(bias), static_cast<const __nv_bfloat16*>(ring), positions, row_off, row_state,
      num_states, status);
  return static_cast<int>(cudaGetLastError());
}

// Rows [0, pieces) of p: one token each of as many sequences, convolution included.
RLB_API int rlb_rec_step(const RecArgs* a, void* stream) {
  if (a->pieces <= 0) return 0;
  if (!rlb_rec_supported(a->delta, a->dim, a->vdim) || a->heads > 65535 || a->heads % a->groups || a->ldp % 4 || a->ldy % 4 || a->gate_off % 4) return -2;
  if ((reinterpret_cast<uintptr_t>(a->p) | reinterpret_cast<uintptr_t>(a->y) | reinterpret_cast<uintptr_t>(a->state) | reinterpret_cast<uintptr_t>(a->norm)) & 7)
    return -3;
  RecStep s{static_cast<const __nv_bfloat16*>(a->p), a->ldp, a->conv_off, a->channels, a->taps, static_cast<const __nv_bfloat16*>(a->conv_w),
            static_cast<const __nv_bfloat16*>(a->conv_bias), static_cast<__nv_bfloat16*>(a->ring), a->positions, a->state_rows, a->state, a->num_states,
            a->heads, a->groups, a->dim, a->vdim, a->gate_off, a->a_off, a->b_off, static_cast<const __nv_bfloat16*>(a->A_log),
            static_cast<const __nv_bfloat16*>(a->dt_bias), static_cast<const __nv_bfloat16*>(a->D), static_cast<const __nv_bfloat16*>(a->norm), a->unit_eps,
            a->eps, static_cast<__nv_bfloat16*>(a->y), a->ldy, a->status};
  const dim3 grid(a->pieces, a->heads), block(256);
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const int vec = a->vdim + 2 * a->dim;
  if (!a->delta) return static_cast<int>(rlb_launch_pdl(mamba2_step_kernel, grid, block, sizeof(float) * vec + sizeof(float4) * 256, st, s));
  if (reinterpret_cast<uintptr_t>(a->state) & 15) return -3;
  const int sm = static_cast<int>(sizeof(float)) * (a->dim * a->vdim + vec) + static_cast<int>(sizeof(float4)) * 2 * DD_THREADS;
  static int conf = 0;
  const int rc = set_smem(reinterpret_cast<const void*>(delta_step_kernel), sm, &conf);
  if (rc) return rc;
  return static_cast<int>(rlb_launch_pdl(delta_step_kernel, grid, dim3(DD_THREADS), sm, st, s));
}

// Portions: rows [row0, rows) of u, p, y in chunks of at most 128 rows (chunk_row counts from row0); piece i owns chunks [piece_chunk[i],
// piece_chunk[i + 1]) and state row state_rows[i]. Scratch (R = rows - row0, N = chunks * heads): cum, wt [heads, R], start [N, dim, vdim]; delta:
// unit [2, groups, R], w_*, kt_* [N * 128, 128], u0 [N * 128, vdim], uu_* [R, heads * vdim].
RLB_API int rlb_rec_portions(const RecArgs* a, void* stream) {
  if (a->pieces <= 0 || a->chunks <= 0) return 0;
  if (!rlb_rec_supported(a->delta, a->dim, a->vdim) || a->heads > 65535 || a->pieces > 65535 || a->heads % a->groups) return -2;
  if (a->ldp % 8 || a->ldu % 8 || a->ldy % 8 || a->gate_off % 8) return -2;
  if ((reinterpret_cast<uintptr_t>(a->p) | reinterpret_cast<uintptr_t>(a->u) | reinterpret_cast<uintptr_t>(a->y) | reinterpret_cast<uintptr_t>(a->start) |
       reinterpret_cast<uintptr_t>(a->norm)) & 15)
    return -3;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const long long R = a->rows - a->row0;
  const int inner = a->heads * a->vdim, n = a->groups * a->dim;
  RecTiles t{};
  t.u = static_cast<const __nv_bfloat16*>(a->u);
  t.ldu = a->ldu;
  t.p = static_cast<const __nv_bfloat16*>(a->p);
  t.ldp = a->ldp;
  t.y = static_cast<__nv_bfloat16*>(a->y);
  t.ldy = a->ldy;
  t.heads = a->heads;
  t.per_group = a->heads / a->groups;
  t.dim = a->dim;
  t.vdim = a->vdim;
  t.q_col = a->delta ? 0 : inner + n;      // delta: [q | k | v], Mamba-2: [x | B | C]
  t.k_col = a->delta ? n : inner;
  t.v_col = a->delta ? 2 * n : 0;
  t.gate_off = a->gate_off;
  t.row0 = a->row0;
  t.rows = R;
  t.chunk_row = a->chunk_row;
  t.chunk_rows = a->chunk_rows;
  t.cum = a->cum;
  t.wt = a->wt;
  t.unit = a->unit;
  t.eps = a->eps;
  t.D = static_cast<const __nv_bfloat16*>(a->D);
  t.norm = static_cast<const __nv_bfloat16*>(a->norm);
  t.start = a->start;
  t.w_hi = static_cast<__nv_bfloat16*>(a->w_hi);
  t.w_lo = static_cast<__nv_bfloat16*>(a->w_lo);
  t.kt_hi = static_cast<__nv_bfloat16*>(a->kt_hi);
  t.kt_lo = static_cast<__nv_bfloat16*>(a->kt_lo);
  t.u0 = a->u0;
  t.uu_hi = static_cast<__nv_bfloat16*>(a->uu_hi);
  t.uu_lo = static_cast<__nv_bfloat16*>(a->uu_lo);
  t.status = a->status;
  rec_prep_kernel<<<dim3(a->chunks, (a->heads + 3) / 4), 128, 0, st>>>(t.p, a->ldp, a->a_off, a->delta ? a->b_off : -1, a->row0, a->chunk_row, a->chunk_rows,
      a->heads, R, static_cast<const __nv_bfloat16*>(a->A_log), static_cast<const __nv_bfloat16*>(a->dt_bias), a->cum, a->wt);
  const int av = (a->vdim + 63) / 64, vpad = (a->vdim + 31) / 32 * 32;
  const dim3 grid(a->chunks, a->heads);
  CUtensorMap tv;
  int rc = rlb_make_tmap_2d(&tv, a->u, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, a->channels, a->rows, a->ldu * 2, 64, RT_C, CU_TENSOR_MAP_SWIZZLE_128B);
  if (rc) return -100 - rc;
  const int smem_out = 4 * RT_ATOM + 2 * av * RT_SATOM + (a->delta ? 2 : 1) * av * RT_ATOM + (4 * RT_C + RC_THREADS) * 4 + 64 + 1024;
  const int cols_out = vpad <= 128 ? 256 : 512;
  static int conf_state = 0, conf_out[2] = {0, 0}, conf_wy = 0, conf_scan[2] = {0, 0};
  if (!a->delta) {
    const int smem_state = (4 + av) * RT_ATOM + RT_C * 4 + 64 + 1024;
    if ((rc = set_smem(reinterpret_cast<const void*>(ssd_state_kernel), smem_state, &conf_state))) return rc;
    if ((rc = set_smem(reinterpret_cast<const void*>(rec_out_kernel<false>), smem_out, &conf_out[0]))) return rc;
    ssd_state_kernel<<<grid, RC_THREADS, smem_state, st>>>(tv, t, av, vpad <= 32 ? 32 : (vpad <= 64 ? 64 : (vpad <= 128 ? 128 : 256)));
    ssd_scan_kernel<<<dim3((a->dim * a->vdim / 4 + 255) / 256, a->pieces, a->heads), 256, 0, st>>>(t, a->piece_chunk, a->positions, a->state_rows, a->state,
                                                                                                   a->num_states);
    rec_out_kernel<false><<<grid, RC_THREADS, smem_out, st>>>(tv, tv, t, av, cols_out);
    return static_cast<int>(cudaGetLastError());
  }
  if (!a->unit || !a->u0 || !a->w_hi || !a->w_lo || !a->kt_hi || !a->kt_lo || !a->uu_hi || !a->uu_lo) return -2;
  if (static_cast<long long>(a->chunks) * a->heads * RT_C > 0x7fffffffll) return -2;
  rec_unit_kernel<<<dim3(static_cast<unsigned>(R), (2 * a->groups + 7) / 8), 256, 0, st>>>(t.u, a->ldu, a->row0, a->groups, a->dim, t.q_col, t.k_col, R,
      1.f / sqrtf(static_cast<float>(a->dim)), a->unit_eps, a->unit);
  CUtensorMap tm[6];
  const void* src[6] = {a->w_hi, a->w_lo, a->kt_hi, a->kt_lo, a->uu_hi, a->uu_lo};
  for (int m = 0; m < 6; ++m) {
    const uint64_t inner_cols = m < 4 ? RT_C : inner, outer = m < 4 ? static_cast<uint64_t>(a->chunks) * a->heads * RT_C : R;
    rc = rlb_make_tmap_2d(&tm[m], src[m], CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, inner_cols, outer, inner_cols * 2, 64, RT_C, CU_TENSOR_MAP_SWIZZLE_128B);
    if (rc) return -100 - rc;
  }
  const int smem_wy = 4 * RT_ATOM + 68 * 1024 + av * RT_ATOM + (WY_TMP + 5 * RT_C) * 4 + 64 + 1024;
  const bool narrow = static_cast<long long>(a->pieces) * a->heads * ((a->vdim + 63) / 64) <= 74;      // few chains: more, narrower CTAs
  const int vb = narrow ? 32 : 64, smem_scan = (8 + vb / 16) * RT_ATOM + 128 + 1024;
  auto scan = narrow ? delta_scan_kernel<32> : delta_scan_kernel<64>;
  if ((rc = set_smem(reinterpret_cast<const void*>(delta_wy_kernel), smem_wy, &conf_wy))) return rc;
  if ((rc = set_smem(reinterpret_cast<const void*>(scan), smem_scan, &conf_scan[narrow]))) return rc;
  if ((rc = set_smem(reinterpret_cast<const void*>(rec_out_kernel<true>), smem_out, &conf_out[1]))) return rc;
  delta_wy_kernel<<<grid, RC_THREADS, smem_wy, st>>>(tv, t, av);
  scan<<<dim3((a->vdim + vb - 1) / vb, a->heads, a->pieces), DS_THREADS, smem_scan, st>>>(tm[0], tm[1], tm[2], tm[3], t, a->piece_chunk,
      a->positions, a->state_rows, a->state, a->num_states);
  rec_out_kernel<true><<<grid, RC_THREADS, smem_out, st>>>(tm[4], tm[5], t, av, cols_out);
  return static_cast<int>(cudaGetLastError());
}
