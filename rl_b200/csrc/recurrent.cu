// Recurrent mixers with a short convolution (Mamba2LayerMixer, DeltaMixer) one token after another, for every size and for bf16 and fp32
// models. The chunked and single-step forms for bf16 are in recurrent_tiles.cu.
//
// State of a sequence: the last inputs of the convolution, a ring [taps, channels] indexed by position % taps in the model's type, and
// S [heads, dim, vdim] in fp32. A piece that starts at position 0 starts from zeros, whatever its rows held before.
//
// This file is compiled without fast math.
#include "recurrent.cuh"

#include <math.h>

namespace {
using namespace rlb;

// u[t, c] = silu(sum_j w[c, j] x[t - taps + 1 + j, c] (+ bias)). row_off: rows of the same piece before this row (null: none).
template <typename T>
__global__ void __launch_bounds__(256)
conv_rows_kernel(const T* __restrict__ x, long long ldx, T* __restrict__ u, long long ldu, int channels, int taps, const T* __restrict__ w,
                 const T* __restrict__ bias, const T* __restrict__ ring, const int* __restrict__ positions, const int* __restrict__ row_off,
                 const long long* __restrict__ row_state, long long num_states, int* status) {
  const long long row = blockIdx.x;
  const int c = blockIdx.y * 256 + threadIdx.x;
  if (c >= channels) return;
  long long sr = row_state[row];
  if (sr < 0 || sr >= num_states) {
    if (c == 0 && status) atomicCAS(status, 0, RLB_ERR_BOUNDS);
    sr = 0;
  }
  const int pos = positions[row], off = row_off ? row_off[row] : 0;
  float v = bias ? rc_ld(bias + c) : 0.f;
  for (int j = 0; j < taps; ++j) {
    const int back = taps - 1 - j;
    if (back > pos) continue;
    const float in = back <= off ? rc_ld(x + (row - back) * ldx + c) : rc_ld(ring + (sr * taps + (pos - back) % taps) * channels + c);
    v = fmaf(rc_ld(w + static_cast<long long>(c) * taps + j), in, v);
  }
  rc_st(u + row * ldu + c, v / (1.f + expf(-v)));
}

// The last taps - 1 inputs of every piece into its ring.
template <typename T>
__global__ void __launch_bounds__(256)
conv_state_kernel(const T* __restrict__ x, long long ldx, int row0, const int* __restrict__ cu, int channels, int taps, T* __restrict__ ring,
                  const int* __restrict__ positions, const long long* __restrict__ state_rows, long long num_states) {
  const int c = blockIdx.y * 256 + threadIdx.x;
  const long long sr = state_rows[blockIdx.x];
  if (c >= channels || sr < 0 || sr >= num_states) return;
  const int begin = row0 + (cu ? cu[blockIdx.x] : static_cast<int>(blockIdx.x)), end = row0 + (cu ? cu[blockIdx.x + 1] : static_cast<int>(blockIdx.x) + 1);
  for (int t = max(begin, end - taps + 1); t < end; ++t) ring[(sr * taps + positions[t] % taps) * channels + c] = x[static_cast<long long>(t) * ldx + c];
}

// One CTA per (piece, head): S <- a S + dt B x^T, y = S^T C + D x, times silu(z).
template <typename T>
__global__ void __launch_bounds__(256)
mamba2_rows_kernel(const T* __restrict__ u, long long ldu, const T* __restrict__ p, long long ldp, T* __restrict__ y, long long ldy, int z_off, int dt_off,
                   int heads, int groups, int dim, int vdim, int row0, const int* __restrict__ cu, const int* __restrict__ positions,
                   const long long* __restrict__ state_rows, float* __restrict__ state, long long num_states, const T* __restrict__ A_log,
                   const T* __restrict__ dt_bias, const T* __restrict__ D, int* status) {
  extern __shared__ float sm[];
  float* B = sm;                 // [dim], times dt
  float* C = B + dim;            // [dim]
  float* part = C + dim;         // [256]
  const int seq = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, g = h / (heads / groups);
  const int begin = cu ? cu[seq] : seq, end = cu ? cu[seq + 1] : seq + 1;
  const long long sr = state_rows[seq];
  if (sr < 0 || sr >= num_states) {
    if (tid == 0 && status) atomicCAS(status, 0, RLB_ERR_BOUNDS);
    return;
  }
  float* S = state + (sr * heads + h) * static_cast<long long>(dim) * vdim;
  const float A = -expf(rc_ld(A_log + h)), bias = rc_ld(dt_bias + h), Dh = rc_ld(D + h);
  const int inner = heads * vdim;
  const int slices = vdim >= 256 ? 1 : 256 / vdim, slice = vdim >= 256 ? 0 : tid / vdim;
  for (int t = begin; t < end; ++t) {
    const long long r = row0 + t;
    const bool fresh = positions[r] == 0;
    const float dt = rc_softplus(rc_ld(p + r * ldp + dt_off + h) + bias);
    const float dec = expf(A * dt);
    for (int i = tid; i < dim; i += 256) {
      B[i] = dt * rc_ld(u + r * ldu + inner + g * dim + i);
      C[i] = rc_ld(u + r * ldu + inner + (groups + g) * dim + i);
    }
    __syncthreads();
    auto out = [&](int v, float acc, float xv) {
      const float z = rc_ld(p + r * ldp + z_off + h * vdim + v);
      rc_st(y + r * ldy + h * vdim + v, fmaf(Dh, xv, acc) * (z / (1.f + expf(-z))));
    };
    if (slice < slices) {
      for (int v = vdim >= 256 ? tid : tid % vdim; v < vdim; v += 256) {
        const float xv = rc_ld(u + r * ldu + h * vdim + v);
        float acc = 0.f;
        for (int i = slice; i < dim; i += slices) {
          float* sp = S + static_cast<long long>(i) * vdim + v;
          const float nv = fresh ? B[i] * xv : fmaf(dec, *sp, B[i] * xv);
          *sp = nv;
          acc = fmaf(nv, C[i], acc);
        }
        if (slices > 1) {
          part[tid] = acc;
          break;
        }
        out(v, acc, xv);
      }
    }
    __syncthreads();
    if (slices > 1 && tid < vdim) {
      float acc = 0.f;
      for (int j = 0; j < slices; ++j) acc += part[j * vdim + tid];
      out(tid, acc, rc_ld(u + r * ldu + h * vdim + tid));
    }
  }
}

// One CTA per (piece, head): unit q and k; S <- g S; w = beta (v - S^T k); S <- S + k w^T; o = S^T q; RMS norm, weight, SiLU gate.
template <typename T>
__global__ void __launch_bounds__(256)
delta_rows_kernel(const T* __restrict__ u, long long ldu, const T* __restrict__ p, long long ldp, T* __restrict__ y, long long ldy, int g_off, int b_off,
                  int a_off, int heads, int kv_heads, int dim, int vdim, int row0, const int* __restrict__ cu, const int* __restrict__ positions,
                  const long long* __restrict__ state_rows, float* __restrict__ state, long long num_states, const T* __restrict__ A_log,
                  const T* __restrict__ dt_bias, const T* __restrict__ norm, float unit_eps, float eps, int* status) {
  extern __shared__ float sm[];
  __shared__ float red[32];
  float* q = sm;                 // [dim]
  float* k = q + dim;            // [dim]
  float* w = k + dim;            // [vdim] what is written; then the outputs
  float* part = w + vdim;        // [256]
  const int seq = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, g = h / (heads / kv_heads), n = kv_heads * dim;
  const int begin = cu ? cu[seq] : seq, end = cu ? cu[seq + 1] : seq + 1;
  const long long sr = state_rows[seq];
  if (sr < 0 || sr >= num_states) {
    if (tid == 0 && status) atomicCAS(status, 0, RLB_ERR_BOUNDS);
    return;
  }
  float* S = state + (sr * heads + h) * static_cast<long long>(dim) * vdim;
  const float A = -expf(rc_ld(A_log + h)), bias = rc_ld(dt_bias + h), qscale = 1.f / sqrtf(static_cast<float>(dim));
  const int slices = vdim >= 256 ? 1 : 256 / vdim, slice = vdim >= 256 ? 0 : tid / vdim, v0 = vdim >= 256 ? tid : tid % vdim;
  for (int t = begin; t < end; ++t) {
    const long long r = row0 + t;
    const bool fresh = positions[r] == 0;
    const T* ur = u + r * ldu;
    float qq = 0.f, kk = 0.f;
    for (int i = tid; i < dim; i += 256) {
      q[i] = rc_ld(ur + g * dim + i);
      k[i] = rc_ld(ur + n + g * dim + i);
      qq += q[i] * q[i];
      kk += k[i] * k[i];
    }
    qq = block_sum(qq, red);
    kk = block_sum(kk, red);
    const float qf = qscale / sqrtf(qq + unit_eps), kf = 1.f / sqrtf(kk + unit_eps);
    for (int i = tid; i < dim; i += 256) {
      q[i] *= qf;
      k[i] *= kf;
    }
    const float beta = 1.f / (1.f + expf(-rc_ld(p + r * ldp + b_off + h)));
    const float dec = fresh ? 0.f : expf(A * rc_softplus(rc_ld(p + r * ldp + a_off + h) + bias));
    __syncthreads();
    // what stands under k, after the decay
    if (slice < slices) {
      for (int v = v0; v < vdim; v += 256) {
        float acc = 0.f;
        if (!fresh)
          for (int i = slice; i < dim; i += slices) acc = fmaf(S[static_cast<long long>(i) * vdim + v], k[i], acc);
        if (slices > 1) {
          part[tid] = acc;
          break;
        }
        w[v] = beta * (rc_ld(ur + 2 * n + h * vdim + v) - dec * acc);
      }
    }
    __syncthreads();
    if (slices > 1 && tid < vdim) {
      float acc = 0.f;
      for (int j = 0; j < slices; ++j) acc += part[j * vdim + tid];
      w[tid] = beta * (rc_ld(ur + 2 * n + h * vdim + tid) - dec * acc);
    }
    __syncthreads();
    if (slice < slices) {
      for (int v = v0; v < vdim; v += 256) {
        const float wv = w[v];
        float acc = 0.f;
        for (int i = slice; i < dim; i += slices) {
          float* sp = S + static_cast<long long>(i) * vdim + v;
          const float nv = fresh ? k[i] * wv : fmaf(dec, *sp, k[i] * wv);
          *sp = nv;
          acc = fmaf(nv, q[i], acc);
        }
        if (slices > 1) {
          part[tid] = acc;
          break;
        }
        w[v] = acc;           // (this thread alone reads w[v])
      }
    }
    __syncthreads();
    if (slices > 1 && tid < vdim) {
      float acc = 0.f;
      for (int j = 0; j < slices; ++j) acc += part[j * vdim + tid];
      w[tid] = acc;
    }
    float ss = 0.f;
    for (int v = tid; v < vdim; v += 256) ss += w[v] * w[v];
    ss = block_sum(ss, red);
    const float rstd = 1.f / sqrtf(ss / static_cast<float>(vdim) + eps);
    for (int v = tid; v < vdim; v += 256) {
      const float gt = rc_ld(p + r * ldp + g_off + h * vdim + v);
      rc_st(y + r * ldy + h * vdim + v, w[v] * rstd * rc_ld(norm + v) * (gt / (1.f + expf(-gt))));
    }
    __syncthreads();
  }
}
}  // namespace

// Convolution of rows [0, rows) of x (columns [0, channels) from x on) into u; ring [states, taps, channels].
RLB_API int rlb_conv_rows(const void* x, int f32, long long ldx, void* u, long long ldu, long long rows, int channels, int taps, const void* w,
                          const void* bias, const void* ring, const int* positions, const int* row_off, const long long* row_state,
                          long long num_states, int* status, void* stream) {
  if (rows <= 0) return 0;
  if (taps < 1 || channels < 1) return -2;
  const dim3 grid(static_cast<unsigned>(rows), (channels + 255) / 256);
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (f32)
    conv_rows_kernel<float><<<grid, 256, 0, s>>>(static_cast<const float*>(x), ldx, static_cast<float*>(u), ldu, channels, taps, static_cast<const float*>(w),
        static_cast<const float*>(bias), static_cast<const float*>(ring), positions, row_off, row_state, num_states, status);
  else
    conv_rows_kernel<__nv_bfloat16><<<grid, 256, 0, s>>>(static_cast<const __nv_bfloat16*>(x), ldx, static_cast<__nv_bfloat16*>(u), ldu, channels, taps,
        static_cast<const __nv_bfloat16*>(w), static_cast<const __nv_bfloat16*>(bias), static_cast<const __nv_bfloat16*>(ring), positions, row_off,
        row_state, num_states, status);
  return static_cast<int>(cudaGetLastError());
}

// `cu` (offsets of the pieces, counted from row0) null: piece i is the single row row0 + i. After rlb_conv_rows of the same rows.
RLB_API int rlb_conv_state(const void* x, int f32, long long ldx, int row0, int pieces, const int* cu, int channels, int taps, void* ring,
                           const int* positions, const long long* state_rows, long long num_states, void* stream) {
  if (pieces <= 0) return 0;
  const dim3 grid(pieces, (channels + 255) / 256);
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (f32)
    conv_state_kernel<float><<<grid, 256, 0, s>>>(static_cast<const float*>(x), ldx, row0, cu, channels, taps, static_cast<float*>(ring), positions,
                                                  state_rows, num_states);
  else
    conv_state_kernel<__nv_bfloat16><<<grid, 256, 0, s>>>(static_cast<const __nv_bfloat16*>(x), ldx, row0, cu, channels, taps,
                                                          static_cast<__nv_bfloat16*>(ring), positions, state_rows, num_states);
  return static_cast<int>(cudaGetLastError());
}

RLB_API int rlb_mamba2_rows(const void* u, int f32, long long ldu, const void* p, long long ldp, void* y, long long ldy, int z_off, int dt_off, int heads,
                            int groups, int dim, int vdim, int row0, int pieces, const int* cu, const int* positions, const long long* state_rows,
                            float* state, long long num_states, const void* A_log, const void* dt_bias, const void* D, int* status, void* stream) {
  if (pieces <= 0) return 0;
  if (heads > 65535 || groups < 1 || heads % groups) return -2;
  const size_t sm = sizeof(float) * (2 * dim + 256);
  if (sm > 48 * 1024) return -2;
  const dim3 grid(pieces, heads);
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (f32)
    mamba2_rows_kernel<float><<<grid, 256, sm, s>>>(static_cast<const float*>(u), ldu, static_cast<const float*>(p), ldp, static_cast<float*>(y), ldy, z_off,
        dt_off, heads, groups, dim, vdim, row0, cu, positions, state_rows, state, num_states, static_cast<const float*>(A_log),
        static_cast<const float*>(dt_bias), static_cast<const float*>(D), status);
  else
    mamba2_rows_kernel<__nv_bfloat16><<<grid, 256, sm, s>>>(static_cast<const __nv_bfloat16*>(u), ldu, static_cast<const __nv_bfloat16*>(p), ldp,
        static_cast<__nv_bfloat16*>(y), ldy, z_off, dt_off, heads, groups, dim, vdim, row0, cu, positions, state_rows, state, num_states,
        static_cast<const __nv_bfloat16*>(A_log), static_cast<const __nv_bfloat16*>(dt_bias), static_cast<const __nv_bfloat16*>(D), status);
  return static_cast<int>(cudaGetLastError());
}

RLB_API int rlb_delta_rows(const void* u, int f32, long long ldu, const void* p, long long ldp, void* y, long long ldy, int g_off, int b_off, int a_off,
                           int heads, int kv_heads, int dim, int vdim, int row0, int pieces, const int* cu, const int* positions,
                           const long long* state_rows, float* state, long long num_states, const void* A_log, const void* dt_bias, const void* norm,
                           float unit_eps, float eps, int* status, void* stream) {
  if (pieces <= 0) return 0;
  if (heads > 65535 || kv_heads < 1 || heads % kv_heads) return -2;
  const size_t sm = sizeof(float) * (2 * dim + vdim + 256);
  if (sm > 48 * 1024) return -2;
  const dim3 grid(pieces, heads);
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (f32)
    delta_rows_kernel<float><<<grid, 256, sm, s>>>(static_cast<const float*>(u), ldu, static_cast<const float*>(p), ldp, static_cast<float*>(y), ldy, g_off,
        b_off, a_off, heads, kv_heads, dim, vdim, row0, cu, positions, state_rows, state, num_states, static_cast<const float*>(A_log),
        static_cast<const float*>(dt_bias), static_cast<const float*>(norm), unit_eps, eps, status);
  else
    delta_rows_kernel<__nv_bfloat16><<<grid, 256, sm, s>>>(static_cast<const __nv_bfloat16*>(u), ldu, static_cast<const __nv_bfloat16*>(p), ldp,
        static_cast<__nv_bfloat16*>(y), ldy, g_off, b_off, a_off, heads, kv_heads, dim, vdim, row0, cu, positions, state_rows, state, num_states,
        static_cast<const __nv_bfloat16*>(A_log), static_cast<const __nv_bfloat16*>(dt_bias), static_cast<const __nv_bfloat16*>(norm), unit_eps, eps, status);
  return static_cast<int>(cudaGetLastError());
}
