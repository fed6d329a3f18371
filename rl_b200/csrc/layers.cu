// Row kernels of post-norm and pre-norm layers (models/post_norm.py, models/pre_norm.py), for every size and for bf16 and fp32 models: the step that norms a sublayer's
// output and joins it to the residual stream, the polynomial activation of normed powers, the router with group-limited choice, the placement of the
// tokens' copies in per-expert row ranges, and the soft cap of the logits.
//
//   add_normed   x += m * rms(y) * w * ls (norms behind the sublayer) or x += y (pre-norm layers) on the fp32 stream, and what the next sublayer reads: x
//                itself in the model's type, or its RMS norm. y is a product's output or the weighted sum of a token's expert rows (combined here, never
//                stored), with rows of a shared unit and of the sublayer's own input added, each times a factor per row.
//   shift_rows   the same (or the start of the stream from the embedding tables), and behind the norm the blend with the token before: h + (h' - h) s,
//                for few rows. A CTA computes the row in front of its own again, so that the rows need no order among the CTAs; the stream is
//                written to a second buffer for that. Sequences continue from a state row [d] per place, see ShiftArgs.
//   blend_rows   the norm and the blend alone, for many rows: the first pass has left the stream and its rows' reciprocal root mean squares.
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
  const float* x;          // [rows, d]
  const void* y;           // [rows, ldy], or the experts' rows when copy_row is set
  long long ldy;
  const int* copy_row;     // [rows, k] row of each of a token's copies in y (out of [0, y_rows): skipped)
  const float* weight;     // [rows, k] (null: 1)
  int k, y_rows;
  int* counts;             // the experts' counts [experts], set to zero for the next layer
  int experts;
  const void* w;           // norm weight of the sublayer (null: its output joins as it is)
  const void* ls;          // [d] layer scale (null: ones)
  const void* next_w;      // weight of the next norm (null: h is x)
  void* h;                 // [rows, d]
  float* x_out;            // [rows, d]; x itself, except in shift_rows
  float* rstd;             // [rows] reciprocal root mean square of the new stream, in place of h (null: h)
  int d;
  float mult, eps;
  const void* also;        // [rows, ld_also] or null: added to the sublayer's output
  long long ld_also;
  const float* also_f;     // [rows] factor of those rows (null: 1)
  const void* own;         // [rows, ld_own] or null: the sublayer's input, added times own_f [rows]
  long long ld_own;
  const float* own_f;
};

// Columns (threadIdx.x + i * THREADS) * 4 of the sublayer's output of one row; KEEP groups of four columns per thread. EXPERTS: copy_row is set.
template <typename T, int THREADS, int KEEP, bool EXPERTS>
__device__ __forceinline__ void sublayer_row(const AddNormed& a, long long row, float4 (&v)[KEEP]) {
  const T *Y = static_cast<const T*>(a.y), *also = static_cast<const T*>(a.also), *own = static_cast<const T*>(a.own);
#pragma unroll
  for (int i = 0; i < KEEP; ++i) {
    const int c = (threadIdx.x + i * THREADS) * 4;
    v[i] = !EXPERTS && c < a.d ? ld4(Y + row * a.ldy + c) : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  auto add = [&](const T* p, float f) {
#pragma unroll
    for (int i = 0; i < KEEP; ++i) {
      const int c = (threadIdx.x + i * THREADS) * 4;
      const float4 t = c < a.d ? ld4(p + c) : make_float4(0.f, 0.f, 0.f, 0.f);
      v[i].x = fmaf(f, t.x, v[i].x); v[i].y = fmaf(f, t.y, v[i].y); v[i].z = fmaf(f, t.z, v[i].z); v[i].w = fmaf(f, t.w, v[i].w);
    }
  };
  if (also) add(also + row * a.ld_also, a.also_f ? a.also_f[row] : 1.f);
  if (own) {
    const float f = a.own_f[row];
    if (f != 0.f) add(own + row * a.ld_own, f);
  }
  if (!EXPERTS) return;
  constexpr int AHEAD = KEEP <= 2 ? 4 : 2;      // copies in flight
  for (int j0 = 0; j0 < a.k; j0 += AHEAD) {
    float4 e[AHEAD][KEEP];
    float wt[AHEAD];
#pragma unroll
    for (int j = 0; j < AHEAD; ++j) {
      const int r = j0 + j < a.k ? a.copy_row[row * a.k + j0 + j] : -1;
      const bool live = r >= 0 && r < a.y_rows;
      wt[j] = live ? (a.weight ? a.weight[row * a.k + j0 + j] : 1.f) : 0.f;
#pragma unroll
      for (int i = 0; i < KEEP; ++i) {
        const int c = (threadIdx.x + i * THREADS) * 4;
        e[j][i] = live && c < a.d ? ld4(Y + r * a.ldy + c) : make_float4(0.f, 0.f, 0.f, 0.f);
      }
    }
#pragma unroll
    for (int j = 0; j < AHEAD; ++j)
#pragma unroll
      for (int i = 0; i < KEEP; ++i) {
        v[i].x = fmaf(wt[j], e[j][i].x, v[i].x);
        v[i].y = fmaf(wt[j], e[j][i].y, v[i].y);
        v[i].z = fmaf(wt[j], e[j][i].z, v[i].z);
        v[i].w = fmaf(wt[j], e[j][i].w, v[i].w);
      }
  }
}

// xv <- xv + f v (w) (ls), f = mult / rms(v) where the sublayer's output is normed
template <typename T, int THREADS, int KEEP>
__device__ __forceinline__ void join_row(const AddNormed& a, const float4 (&v)[KEEP], float4 (&xv)[KEEP], float* red) {
  const T *w = static_cast<const T*>(a.w), *ls = static_cast<const T*>(a.ls);
  float f = a.mult;
  if (w) {
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < KEEP; ++i) ss += v[i].x * v[i].x + v[i].y * v[i].y + v[i].z * v[i].z + v[i].w * v[i].w;
    ss = block_sum(ss, red);
    f = a.mult / sqrtf(ss / static_cast<float>(a.d) + a.eps);
  }
  auto add = [&](auto weight) {
#pragma unroll
    for (int i = 0; i < KEEP; ++i) {
      const int c = (threadIdx.x + i * THREADS) * 4;
      if (c >= a.d) continue;
      const float4 wv = weight(c);
      xv[i].x = fmaf(v[i].x * f, wv.x, xv[i].x);
      xv[i].y = fmaf(v[i].y * f, wv.y, xv[i].y);
      xv[i].z = fmaf(v[i].z * f, wv.z, xv[i].z);
      xv[i].w = fmaf(v[i].w * f, wv.w, xv[i].w);
    }
  };
  if (w && ls) {
    add([&](int c) {
      const float4 x = ld4(w + c), y = ld4(ls + c);
      return make_float4(x.x * y.x, x.y * y.y, x.z * y.z, x.w * y.w);
    });
  } else if (w || ls) {
    add([&](int c) { return ld4((w ? w : ls) + c); });
  } else {
    add([](int) { return make_float4(1.f, 1.f, 1.f, 1.f); });
  }
}

// One column of the sublayer's output, for any size.
template <typename T>
__device__ __forceinline__ float sublayer_value(const AddNormed& a, long long row, int c) {
  const T *Y = static_cast<const T*>(a.y), *also = static_cast<const T*>(a.also), *own = static_cast<const T*>(a.own);
  float v = also ? (a.also_f ? a.also_f[row] : 1.f) * ldv(also + row * a.ld_also + c) : 0.f;
  if (own) v = fmaf(a.own_f[row], ldv(own + row * a.ld_own + c), v);
  if (!a.copy_row) return v + ldv(Y + row * a.ldy + c);
  for (int j = 0; j < a.k; ++j) {
    const int r = a.copy_row[row * a.k + j];
    if (r >= 0 && r < a.y_rows) v = fmaf(a.weight ? a.weight[row * a.k + j] : 1.f, ldv(Y + r * a.ldy + c), v);
  }
  return v;
}
template <typename T>
__device__ __forceinline__ float join_value(const AddNormed& a, long long row, int c, float f) {
  const T *w = static_cast<const T*>(a.w), *ls = static_cast<const T*>(a.ls);
  return fmaf(sublayer_value<T>(a, row, c) * f, (w ? ldv(w + c) : 1.f) * (ls ? ldv(ls + c) : 1.f), a.x[row * a.d + c]);
}
template <typename T, int THREADS>
__device__ __forceinline__ float join_factor(const AddNormed& a, long long row, float* red) {
  if (!a.w) return a.mult;
  float ss = 0.f;
  for (int c = threadIdx.x; c < a.d; c += THREADS) {
    const float v = sublayer_value<T>(a, row, c);
    ss += v * v;
  }
  return a.mult / sqrtf(block_sum(ss, red) / static_cast<float>(a.d) + a.eps);
}

// d a multiple of 4, at most 4 * AN_KEEP * THREADS: AN_KEEP groups of four columns stay in a thread's registers.
template <typename T, int THREADS, int AN_KEEP, bool EXPERTS>
__global__ void __launch_bounds__(THREADS, THREADS * AN_KEEP <= 512 ? 1024 / THREADS : (THREADS * AN_KEEP <= 1024 ? 768 / THREADS : 1)) add_normed_kernel(AddNormed a) {
  __shared__ float red[32];
  pdl_sync();
  const long long row = blockIdx.x;
  if (row == 0 && a.counts)
    for (int e = threadIdx.x; e < a.experts; e += THREADS) a.counts[e] = 0;
  float* x = a.x_out + row * a.d;
  T* h = static_cast<T*>(a.h) + row * a.d;
  const T* nw = static_cast<const T*>(a.next_w);
  float4 v[AN_KEEP], xv[AN_KEEP];
#pragma unroll
  for (int i = 0; i < AN_KEEP; ++i) {
    const int c = (threadIdx.x + i * THREADS) * 4;
    xv[i] = c < a.d ? ld4(a.x + row * a.d + c) : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  sublayer_row<T, THREADS, AN_KEEP, EXPERTS>(a, row, v);
  join_row<T, THREADS, AN_KEEP>(a, v, xv, red);
  float s2 = 0.f;
#pragma unroll
  for (int i = 0; i < AN_KEEP; ++i) {
    const int c = (threadIdx.x + i * THREADS) * 4;
    if (c >= a.d) continue;
    st4(x + c, xv[i]);
    if (!nw && !a.rstd) st4(h + c, xv[i]);
    s2 += xv[i].x * xv[i].x + xv[i].y * xv[i].y + xv[i].z * xv[i].z + xv[i].w * xv[i].w;
  }
  if (!nw && !a.rstd) return;
  s2 = block_sum(s2, red);
  const float g = 1.f / sqrtf(s2 / static_cast<float>(a.d) + a.eps);
  if (a.rstd) {
    if (threadIdx.x == 0) a.rstd[row] = g;
    return;
  }
#pragma unroll
  for (int i = 0; i < AN_KEEP; ++i) {
    const int c = (threadIdx.x + i * THREADS) * 4;
    if (c >= a.d) continue;
    const float4 wv = ld4(nw + c);
    st4(h + c, make_float4(xv[i].x * g * wv.x, xv[i].y * g * wv.y, xv[i].z * g * wv.z, xv[i].w * g * wv.w));
  }
}

// Any size.
template <typename T>
__global__ void __launch_bounds__(256) add_normed_any_kernel(AddNormed a) {
  __shared__ float red[32];
  pdl_sync();
  const long long row = blockIdx.x;
  if (row == 0 && a.counts)
    for (int e = threadIdx.x; e < a.experts; e += 256) a.counts[e] = 0;
  float* x = a.x_out + row * a.d;
  T* h = static_cast<T*>(a.h) + row * a.d;
  const T* nw = static_cast<const T*>(a.next_w);
  const float f = join_factor<T, 256>(a, row, red);
  float s2 = 0.f;
  for (int c = threadIdx.x; c < a.d; c += 256) {
    const float v = join_value<T>(a, row, c, f);
    x[c] = v;
    if (!nw) st1(h + c, v);
    s2 += v * v;
  }
  if (!nw) return;
  s2 = block_sum(s2, red);
  const float g = 1.f / sqrtf(s2 / static_cast<float>(a.d) + a.eps);
  for (int c = threadIdx.x; c < a.d; c += 256) st1(h + c, x[c] * g * ldv(nw + c));
}

// ---------------------------------------------------------------- blend with the token before
// The start of the residual stream: x = table[id] * scale, and a row of the pair table: number (id before * mul_prev + id * mul_cur) mod buckets,
// row `buckets` for a sequence's first token.
struct StartArgs {
  const int* ids;          // [rows]
  const void* table;       // [vocab, d]
  int vocab;
  float scale;
  const void* pairs;       // [buckets + 1, d] (null: none)
  int buckets;
  long long mul_prev, mul_cur;
  int* token;              // [states] last token of every sequence
  int* token_next;
};

// Rows [0, n_single) are one token each of as many sequences, portions follow. The state of a sequence's first row in the batch is read from
// `state`; single rows leave theirs there, portions in `next` (another CTA may still have to read their old one), from where commit_states moves it.
struct ShiftArgs {
  const void* s;           // [d] (null: no blend, and no state of it)
  const int* positions;    // [rows]
  const int* row_off;      // [rows] rows of the same piece in front (null: all rows are single)
  const long long* row_state;   // [rows] state row
  long long num_states, ld_state;
  float* state;            // [states, ld_state], this place's columns
  float* next;
  long long rows;
  int n_single;
  int* status;
};

__device__ __forceinline__ bool last_of_piece(const ShiftArgs& s, long long row) { return !s.row_off || row + 1 == s.rows || s.row_off[row + 1] == 0; }
// Where the last row of a piece leaves its normed stream (null: another row).
__device__ __forceinline__ float* leaves(const ShiftArgs& s, long long row, long long st) {
  return s.s && last_of_piece(s, row) ? (row < s.n_single ? s.state : s.next) + st * s.ld_state : nullptr;
}
__device__ __forceinline__ long long state_row(const ShiftArgs& s, long long row) {
  const long long r = s.row_state[row];
  if (r >= 0 && r < s.num_states) return r;
  if (threadIdx.x == 0 && s.status) atomicCAS(s.status, 0, RLB_ERR_BOUNDS);
  return 0;
}
// Offsets of a row's entries in the two tables (pair offset -1: no pair table).
__device__ __forceinline__ void start_rows(const StartArgs& e, const ShiftArgs& s, long long row, int d, long long& tok, long long& pair) {
  auto valid = [&](int id) {
    if (id >= 0 && id < e.vocab) return id;
    if (threadIdx.x == 0 && s.status) atomicCAS(s.status, 0, RLB_ERR_BOUNDS);
    return 0;
  };
  const int id = valid(e.ids[row]);
  tok = static_cast<long long>(id) * d;
  pair = -1;
  if (!e.pairs) return;
  long long b = e.buckets;
  if (s.positions[row] > 0) {
    const int before = s.row_off && s.row_off[row] > 0 ? valid(e.ids[row - 1]) : e.token[state_row(s, row)];
    b = (before * e.mul_prev + id * e.mul_cur) % e.buckets;
    if (b < 0) b += e.buckets;
  }
  pair = b * d;
}

template <typename T, int THREADS, int KEEP, bool START>
__global__ void __launch_bounds__(THREADS, 1) shift_rows_kernel(AddNormed a, ShiftArgs s, StartArgs e) {
  __shared__ float red[32];
  pdl_sync();
  const long long row = blockIdx.x;
  if (!START && row == 0 && a.counts)
    for (int i = threadIdx.x; i < a.experts; i += THREADS) a.counts[i] = 0;
  const T *nw = static_cast<const T*>(a.next_w), *sw = static_cast<const T*>(s.s), *table = static_cast<const T*>(e.table), *pairs = static_cast<const T*>(e.pairs);
  const long long st = state_row(s, row);
  const bool first = !s.row_off || s.row_off[row] == 0, fresh = first && s.positions[row] == 0;
  const bool again = sw && !first;                       // the row in front is computed again
  float* keep = leaves(s, row, st);
  const float* from = s.state + st * s.ld_state;
  if (a.d % 4 == 0 && a.d <= KEEP * 4 * THREADS) {
    float4 prev[KEEP];
#pragma unroll
    for (int i = 0; i < KEEP; ++i) {
      const int c = (threadIdx.x + i * THREADS) * 4;
      prev[i] = sw && first && !fresh && c < a.d ? ld4(from + c) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    for (long long r = row - (again ? 1 : 0); r <= row; ++r) {
      float4 v[KEEP], xv[KEEP];
      if (START) {
        long long tok, pair;
        start_rows(e, s, r, a.d, tok, pair);
#pragma unroll
        for (int i = 0; i < KEEP; ++i) {
          const int c = (threadIdx.x + i * THREADS) * 4;
          if (c >= a.d) continue;
          v[i] = ld4(table + tok + c);
          xv[i] = pair >= 0 ? ld4(pairs + pair + c) : make_float4(0.f, 0.f, 0.f, 0.f);
          xv[i] = make_float4(fmaf(v[i].x, e.scale, xv[i].x), fmaf(v[i].y, e.scale, xv[i].y), fmaf(v[i].z, e.scale, xv[i].z), fmaf(v[i].w, e.scale, xv[i].w));
        }
      } else {
#pragma unroll
        for (int i = 0; i < KEEP; ++i) {
          const int c = (threadIdx.x + i * THREADS) * 4;
          if (c < a.d) xv[i] = ld4(a.x + r * a.d + c);
        }
        if (a.copy_row) sublayer_row<T, THREADS, KEEP, true>(a, r, v);
        else sublayer_row<T, THREADS, KEEP, false>(a, r, v);
        join_row<T, THREADS, KEEP>(a, v, xv, red);
      }
      const bool mine = r == row;
      float s2 = 0.f;
#pragma unroll
      for (int i = 0; i < KEEP; ++i) {
        const int c = (threadIdx.x + i * THREADS) * 4;
        if (c >= a.d) continue;
        if (mine) st4(a.x_out + row * a.d + c, xv[i]);
        s2 += xv[i].x * xv[i].x + xv[i].y * xv[i].y + xv[i].z * xv[i].z + xv[i].w * xv[i].w;
      }
      s2 = block_sum(s2, red);
      const float g = 1.f / sqrtf(s2 / static_cast<float>(a.d) + a.eps);
#pragma unroll
      for (int i = 0; i < KEEP; ++i) {
        const int c = (threadIdx.x + i * THREADS) * 4;
        if (c >= a.d) continue;
        const float4 wv = ld4(nw + c), b = prev[i];
        const float4 h = make_float4(xv[i].x * g * wv.x, xv[i].y * g * wv.y, xv[i].z * g * wv.z, xv[i].w * g * wv.w);
        prev[i] = h;
        if (!mine) continue;
        const float4 f = sw ? ld4(sw + c) : make_float4(0.f, 0.f, 0.f, 0.f);
        st4(static_cast<T*>(a.h) + row * a.d + c, make_float4(fmaf(b.x - h.x, f.x, h.x), fmaf(b.y - h.y, f.y, h.y), fmaf(b.z - h.z, f.z, h.z), fmaf(b.w - h.w, f.w, h.w)));
        if (keep) st4(keep + c, h);
      }
    }
  } else {                                               // any size
    float f[2] = {0.f, 0.f}, g[2] = {0.f, 0.f};
    long long tok[2] = {0, 0}, pair[2] = {-1, -1};
    auto value = [&](int q, int c) {                     // stream of row `row - q`
      if (START) return fmaf(ldv(table + tok[q] + c), e.scale, pair[q] >= 0 ? ldv(pairs + pair[q] + c) : 0.f);
      return join_value<T>(a, row - q, c, f[q]);
    };
    for (int q = 0; q < (again ? 2 : 1); ++q) {
      if (START) start_rows(e, s, row - q, a.d, tok[q], pair[q]);
      else f[q] = join_factor<T, THREADS>(a, row - q, red);
      float s2 = 0.f;
      for (int c = threadIdx.x; c < a.d; c += THREADS) {
        const float v = value(q, c);
        s2 += v * v;
      }
      g[q] = 1.f / sqrtf(block_sum(s2, red) / static_cast<float>(a.d) + a.eps);
    }
    for (int c = threadIdx.x; c < a.d; c += THREADS) {
      const float v = value(0, c), n = ldv(nw + c), h = v * g[0] * n;
      const float b = !sw || fresh ? 0.f : (first ? from[c] : value(1, c) * g[1] * n);
      a.x_out[row * a.d + c] = v;
      st1(static_cast<T*>(a.h) + row * a.d + c, fmaf(b - h, sw ? ldv(sw + c) : 0.f, h));
      if (keep) keep[c] = h;
    }
  }
  if (START && e.token && last_of_piece(s, row)) {
    __syncthreads();                                     // (everyone has read the old one)
    if (threadIdx.x == 0) (row < s.n_single ? e.token : e.token_next)[st] = e.ids[row];
  }
}

// The start of the stream alone: x and rstd.
template <typename T, int THREADS, int KEEP>
__global__ void __launch_bounds__(THREADS) start_rows_kernel(AddNormed a, ShiftArgs s, StartArgs e) {
  __shared__ float red[32];
  pdl_sync();
  const long long row = blockIdx.x;
  const T *table = static_cast<const T*>(e.table), *pairs = static_cast<const T*>(e.pairs);
  long long tok, pair;
  start_rows(e, s, row, a.d, tok, pair);
  float4 v[KEEP], w[KEEP];
#pragma unroll
  for (int i = 0; i < KEEP; ++i) {
    const int c = (threadIdx.x + i * THREADS) * 4;
    v[i] = w[i] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (c >= a.d) continue;
    v[i] = ld4(table + tok + c);
    if (pair >= 0) w[i] = ld4(pairs + pair + c);
  }
  float s2 = 0.f;
#pragma unroll
  for (int i = 0; i < KEEP; ++i) {
    const int c = (threadIdx.x + i * THREADS) * 4;
    const float4 x = make_float4(fmaf(v[i].x, e.scale, w[i].x), fmaf(v[i].y, e.scale, w[i].y), fmaf(v[i].z, e.scale, w[i].z), fmaf(v[i].w, e.scale, w[i].w));
    if (c < a.d) st4(a.x_out + row * a.d + c, x);
    s2 += x.x * x.x + x.y * x.y + x.z * x.z + x.w * x.w;
  }
  s2 = block_sum(s2, red);      // (everyone has read the old token)
  if (threadIdx.x) return;
  a.rstd[row] = 1.f / sqrtf(s2 / static_cast<float>(a.d) + a.eps);
  if (e.token && last_of_piece(s, row)) (row < s.n_single ? e.token : e.token_next)[state_row(s, row)] = e.ids[row];
}

// h = n + (n' - n) * s with n = x * rstd * nw of the row and n' that of the token before. A thread walks BR_RUN rows of its four columns.
constexpr int BR_THREADS = 128, BR_RUN = 8;
template <typename T>
__global__ void __launch_bounds__(BR_THREADS) blend_rows_kernel(const float* __restrict__ x, const float* __restrict__ rstd, const T* __restrict__ nw, T* __restrict__ h,
                                                                int d, ShiftArgs s) {
  const int c = (blockIdx.y * BR_THREADS + threadIdx.x) * 4;
  const long long row0 = static_cast<long long>(blockIdx.x) * BR_RUN;
  pdl_sync();
  if (c >= d) return;
  const float4 wv = ld4(nw + c), f = ld4(static_cast<const T*>(s.s) + c);
  float4 xv[BR_RUN + 1];
#pragma unroll
  for (int i = 0; i <= BR_RUN; ++i) {
    const long long r = row0 - 1 + i;
    xv[i] = r >= 0 && r < s.rows ? ld4(x + r * d + c) : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  auto normed = [&](float4 v, long long r) {
    const float g = rstd[r];
    return make_float4(v.x * g * wv.x, v.y * g * wv.y, v.z * g * wv.z, v.w * g * wv.w);
  };
  float4 prev = row0 > 0 ? normed(xv[0], row0 - 1) : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
  for (int i = 0; i < BR_RUN; ++i) {
    const long long row = row0 + i;
    if (row >= s.rows) break;
    const float4 n = normed(xv[i + 1], row);
    const bool first = !s.row_off || s.row_off[row] == 0;
    long long st = 0;
    if (first || last_of_piece(s, row)) st = state_row(s, row);
    if (first) prev = s.positions[row] > 0 ? ld4(s.state + st * s.ld_state + c) : make_float4(0.f, 0.f, 0.f, 0.f);
    st4(h + row * d + c, make_float4(fmaf(prev.x - n.x, f.x, n.x), fmaf(prev.y - n.y, f.y, n.y), fmaf(prev.z - n.z, f.z, n.z), fmaf(prev.w - n.w, f.w, n.w)));
    if (float* keep = leaves(s, row, st)) st4(keep + c, n);
    prev = n;
  }
}

// state[r] = next[r] for the state rows of the portions (blockIdx.y), and the same for their last tokens.
__global__ void __launch_bounds__(256)
commit_states_kernel(float* __restrict__ state, const float* __restrict__ next, long long width, int* token, const int* token_next, const long long* rows,
                     long long num_states, int* status) {
  const long long r = rows[blockIdx.y];
  if (r < 0 || r >= num_states) {
    if (threadIdx.x == 0 && status) atomicCAS(status, 0, RLB_ERR_BOUNDS);
    return;
  }
  for (long long c = static_cast<long long>(blockIdx.x) * 256 + threadIdx.x; c < width; c += static_cast<long long>(gridDim.x) * 256)
    state[r * width + c] = next[r * width + c];
  if (token && blockIdx.x == 0 && threadIdx.x == 0) token[r] = token_next[r];
}

// ---------------------------------------------------------------- polynomial activation
// z <- c0 z / rms(z) + c1 z^2 / rms(z^2) + c2 z^3 / rms(z^3) + c3 along each row, in place: a cubic polynomial per row. One CTA per row.
template <int THREADS, int KEEP>
__global__ void __launch_bounds__(THREADS) poly_norm_kernel(__nv_bfloat16* __restrict__ z, long long ld, const __nv_bfloat16* __restrict__ coef, int n, float eps) {
  __shared__ float red[3][32];
  pdl_sync();
  __nv_bfloat16* p = z + blockIdx.x * ld;
  uint4 raw[KEEP];
#pragma unroll
  for (int i = 0; i < KEEP; ++i) {
    const int c = (threadIdx.x + i * THREADS) * 8;
    raw[i] = c < n ? *reinterpret_cast<const uint4*>(p + c) : make_uint4(0, 0, 0, 0);
  }
  float s1 = 0.f, s2 = 0.f, s3 = 0.f;
#pragma unroll
  for (int i = 0; i < KEEP; ++i) {
    const uint32_t r[4] = {raw[i].x, raw[i].y, raw[i].z, raw[i].w};
#pragma unroll
    for (int q = 0; q < 4; ++q) {
      const float2 f = unpack_bf16x2(r[q]);
      const float a = f.x * f.x, b = f.y * f.y, a2 = a * a, b2 = b * b;
      s1 += a + b;
      s2 += a2 + b2;
      s3 = fmaf(a2, a, fmaf(b2, b, s3));
    }
  }
  s1 = warp_sum(s1), s2 = warp_sum(s2), s3 = warp_sum(s3);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (lane == 0) red[0][warp] = s1, red[1][warp] = s2, red[2][warp] = s3;
  __syncthreads();
  float k[3];
#pragma unroll
  for (int q = 0; q < 3; ++q) k[q] = __bfloat162float(coef[q]) / sqrtf(warp_sum(lane < THREADS / 32 ? red[q][lane] : 0.f) / static_cast<float>(n) + eps);
  const float c3 = __bfloat162float(coef[3]);
#pragma unroll
  for (int i = 0; i < KEEP; ++i) {
    const int c = (threadIdx.x + i * THREADS) * 8;
    if (c >= n) continue;
    uint32_t r[4] = {raw[i].x, raw[i].y, raw[i].z, raw[i].w};
#pragma unroll
    for (int q = 0; q < 4; ++q) {
      const float2 f = unpack_bf16x2(r[q]);
      r[q] = pack_bf16x2(fmaf(fmaf(fmaf(k[2], f.x, k[1]), f.x, k[0]), f.x, c3), fmaf(fmaf(fmaf(k[2], f.y, k[1]), f.y, k[0]), f.y, c3));
    }
    *reinterpret_cast<uint4*>(p + c) = make_uint4(r[0], r[1], r[2], r[3]);
  }
}
template <typename T>
__global__ void __launch_bounds__(256) poly_norm_any_kernel(T* __restrict__ z, long long ld, const T* __restrict__ coef, int n, float eps) {
  __shared__ float red[32];
  pdl_sync();
  T* p = z + blockIdx.x * ld;
  float s[3] = {0.f, 0.f, 0.f};
  for (int c = threadIdx.x; c < n; c += 256) {
    const float v = ldv(p + c), v2 = v * v;
    s[0] += v2;
    s[1] = fmaf(v2, v2, s[1]);
    s[2] = fmaf(v2 * v2, v2, s[2]);
  }
  float k[3];
  for (int q = 0; q < 3; ++q) k[q] = ldv(coef + q) / sqrtf(block_sum(s[q], red) / static_cast<float>(n) + eps);
  const float c3 = ldv(coef + 3);
  for (int c = threadIdx.x; c < n; c += 256) {
    const float v = ldv(p + c);
    st1(p + c, fmaf(fmaf(fmaf(k[2], v, k[1]), v, k[0]), v, c3));
  }
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

struct RouterArgs {
  const float* logits;         // [T, ld]: E outputs, behind them the shared unit's gate
  long long ld;
  int T, E;
  const float* correction;     // [E] (null: none)
  int groups, keep, k;
  int softmax;                 // scores are a soft-max over the E outputs, else sigmoids
  float scale;                 // of the weights
  int experts;                 // outputs from here on stand for the token's own row
  float *w, *own_f, *gate;     // [T, k]; [T] sum of the weights of the token's own row (null: no such outputs); [T] sigmoid of the gate (null: none)
  int *idx, *rank, *counts;
};

__global__ void __launch_bounds__(MC_WARPS * 32) moe_choose_kernel(RouterArgs a) {
  extern __shared__ float sm[];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int t = blockIdx.x * MC_WARPS + warp, E = a.E, groups = a.groups, keep = a.keep, k = a.k;
  pdl_sync();
  if (t >= a.T) return;
  float* s = sm + warp * (2 * E + groups);
  float* c = s + E;
  float* gs = c + E;
  const float* z = a.logits + static_cast<long long>(t) * a.ld;
  if (a.softmax) {
    float mx = -INFINITY, sum = 0.f;
    for (int e = lane; e < E; e += 32) mx = fmaxf(mx, z[e]);
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
    for (int e = lane; e < E; e += 32) {
      s[e] = expf(z[e] - mx);
      sum += s[e];
    }
    sum = warp_sum(sum);
    for (int e = lane; e < E; e += 32) {
      s[e] /= sum;
      c[e] = a.correction ? s[e] + a.correction[e] : s[e];
    }
  } else {
    for (int e = lane; e < E; e += 32) {
      const float v = 1.f / (1.f + expf(-z[e]));
      s[e] = v;
      c[e] = a.correction ? v + a.correction[e] : v;
    }
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
  const bool own = lane < k && isel >= a.experts;
  if (lane < k) {
    const long long o = static_cast<long long>(t) * k + lane;
    wsel *= a.scale;
    a.w[o] = wsel;
    a.idx[o] = isel;
    a.rank[o] = own ? 0 : atomicAdd(a.counts + isel, 1);
  }
  if (a.own_f) {
    const float f = warp_sum(own ? wsel : 0.f);
    if (lane == 0) a.own_f[t] = f;
  }
  if (a.gate && lane == 0) a.gate[t] = 1.f / (1.f + expf(-z[E]));
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
    int row = e < E ? row0[e] * 128 + rank[c] : -1;      // (outputs behind the experts have no rows)
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

// What a join adds to the stream, see AddNormed; `x_out` may be x itself (rlb_add_normed) or must not overlap it (rlb_shift_rows).
struct RlbJoin {
  const float* x;
  const void* y;
  const int* copy_row;
  const float* weight;
  int* counts;
  const void *w, *ls, *next_w, *also, *own;
  const float *also_f, *own_f;
  void* h;
  float *x_out, *rstd;
  long long ldy, ld_also, ld_own, rows;
  int f32, k, y_rows, experts, d;
  float mult, eps;
};
// Blend with the token before and, with ids, the start of the stream in place of a join; see ShiftArgs and StartArgs.
struct RlbShift {
  const void* s;
  const int *positions, *row_off;
  const long long* row_state;
  float *state, *next;
  const int* ids;
  const void *table, *pairs;
  int *token, *token_next;
  int* status;
  long long num_states, ld_state, mul_prev, mul_cur;
  int n_single, vocab, buckets;
  float scale;
};

namespace {
int join_args(const RlbJoin& j, AddNormed& a) {
  if (j.d % 4 == 0 && ((j.y && j.ldy % 4) || (j.also && j.ld_also % 4) || (j.own && j.ld_own % 4))) return -2;
  if (j.own && !j.own_f) return -2;
  if (j.rstd && (j.d % 4 || j.d > 4096)) return -2;
  a = AddNormed{j.x, j.y, j.ldy, j.copy_row, j.weight, j.k, j.y_rows, j.counts, j.experts, j.w, j.ls, j.next_w, j.h, j.x_out, j.rstd, j.d, j.mult, j.eps,
                j.also, j.ld_also, j.also_f, j.own, j.ld_own, j.own_f};
  return 0;
}
}  // namespace

// x [rows, d] fp32 += mult * rms(y) * w * ls (w null: mult * y * ls); h [rows, d] = x, or rms(x) * next_w. With copy_row [rows, k]: y of a row is the
// sum of its k weighted (weight null: plain) rows of y [y_rows, ldy], and counts [experts] are set to zero. also, own: added to y times their factors.
// rstd [rows] (d a multiple of 4, at most 4096): written in place of h, for rlb_blend_rows.
RLB_API int rlb_add_normed(const RlbJoin* j, void* stream) {
  if (j->rows <= 0) return 0;
  AddNormed a;
  if (int rc = join_args(*j, a)) return rc;
  const long long rows = j->rows;
  const int d = j->d;
  const dim3 grid(static_cast<unsigned>(rows));
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  auto go = [&](auto kernel, int threads) { return static_cast<int>(rlb_launch_pdl(kernel, grid, dim3(threads), 0, s, a)); };
#define RLB_ADD(T, THREADS, KEEP) (a.copy_row ? go(add_normed_kernel<T, THREADS, KEEP, true>, THREADS) : go(add_normed_kernel<T, THREADS, KEEP, false>, THREADS))
  if (d % 4 || d > 8192) return j->f32 ? go(add_normed_any_kernel<float>, 256) : go(add_normed_any_kernel<__nv_bfloat16>, 256);
  if (j->f32) return d <= 4096 ? RLB_ADD(float, 256, 4) : RLB_ADD(float, 256, 8);
  if (rows < 148 * 4 && d > 1024)       // few rows: more threads per row
    return d <= 2048 ? RLB_ADD(__nv_bfloat16, 512, 1) : (d <= 4096 ? RLB_ADD(__nv_bfloat16, 512, 2) : RLB_ADD(__nv_bfloat16, 512, 4));
  return d <= 1024 ? RLB_ADD(__nv_bfloat16, 256, 1) : (d <= 2048 ? RLB_ADD(__nv_bfloat16, 256, 2) : (d <= 4096 ? RLB_ADD(__nv_bfloat16, 256, 4)
                                                                                                                : RLB_ADD(__nv_bfloat16, 256, 8)));
#undef RLB_ADD
}

// rlb_add_normed into x_out, or with ids the embedding, and h = n + (n' - n) * s with n = rms(x) * next_w and n' that of the sequence's token
// before (s null, with ids only: h = n). With ids and rstd only the stream and the reciprocal root mean squares are written.
RLB_API int rlb_shift_rows(const RlbJoin* j, const RlbShift* t, void* stream) {
  if (j->rows <= 0) return 0;
  AddNormed a;
  if (int rc = join_args(*j, a)) return rc;
  const bool start = t->ids != nullptr;
  if (!j->next_w || (!t->s && !start) || (t->s && (!t->state || !t->next)) || j->x == j->x_out) return -2;
  if (start && t->pairs && (t->buckets < 1 || !t->token || !t->token_next)) return -2;
  if (j->d % 4 == 0 && t->ld_state % 4) return -2;
  const long long rows = j->rows;
  const int d = j->d;
  ShiftArgs s{t->s, t->positions, t->row_off, t->row_state, t->num_states, t->ld_state, t->state, t->next, rows, t->n_single, t->status};
  StartArgs e{t->ids, t->table, t->vocab, t->scale, t->pairs, t->buckets, t->mul_prev, t->mul_cur, t->token, t->token_next};
  const dim3 grid(static_cast<unsigned>(rows));
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  auto go = [&](auto kernel, int threads) { return static_cast<int>(rlb_launch_pdl(kernel, grid, dim3(threads), 0, st, a, s, e)); };
#define RLB_SHIFT(T, THREADS, KEEP) (start ? go(shift_rows_kernel<T, THREADS, KEEP, true>, THREADS) : go(shift_rows_kernel<T, THREADS, KEEP, false>, THREADS))
  if (a.rstd) {
    if (!start) return -2;
    if (j->f32) return go(start_rows_kernel<float, 256, 4>, 256);
    return d <= 1024 ? go(start_rows_kernel<__nv_bfloat16, 128, 2>, 128) : (d <= 2048 ? go(start_rows_kernel<__nv_bfloat16, 256, 2>, 256)
                                                                                        : go(start_rows_kernel<__nv_bfloat16, 256, 4>, 256));
  }
  if (j->f32) return RLB_SHIFT(float, 256, 4);
  if (rows < 148 * 4 && d > 1024) return d <= 2048 ? RLB_SHIFT(__nv_bfloat16, 512, 1) : (d <= 4096 ? RLB_SHIFT(__nv_bfloat16, 512, 2) : RLB_SHIFT(__nv_bfloat16, 512, 4));
  return d <= 1024 ? RLB_SHIFT(__nv_bfloat16, 256, 1) : (d <= 2048 ? RLB_SHIFT(__nv_bfloat16, 256, 2) : (d <= 4096 ? RLB_SHIFT(__nv_bfloat16, 256, 4)
                                                                                                                : RLB_SHIFT(__nv_bfloat16, 512, 4)));
#undef RLB_SHIFT
}

// h [rows, d] = n + (n' - n) * t->s with n = x * rstd * nw; d a multiple of 4.
RLB_API int rlb_blend_rows(const float* x, const float* rstd, const void* nw, void* h, int f32, long long rows, int d, const RlbShift* t, void* stream) {
  if (rows <= 0) return 0;
  if (d % 4 || t->ld_state % 4 || !t->s || !t->state || !t->next) return -2;
  ShiftArgs s{t->s, t->positions, t->row_off, t->row_state, t->num_states, t->ld_state, t->state, t->next, rows, t->n_single, t->status};
  const dim3 grid(static_cast<unsigned>((rows + BR_RUN - 1) / BR_RUN), (d / 4 + BR_THREADS - 1) / BR_THREADS);
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (f32) return static_cast<int>(rlb_launch_pdl(blend_rows_kernel<float>, grid, dim3(BR_THREADS), 0, st, x, rstd, static_cast<const float*>(nw), static_cast<float*>(h), d, s));
  return static_cast<int>(rlb_launch_pdl(blend_rows_kernel<__nv_bfloat16>, grid, dim3(BR_THREADS), 0, st, x, rstd, static_cast<const __nv_bfloat16*>(nw),
                                         static_cast<__nv_bfloat16*>(h), d, s));
}

// state [num_states, width] and token [num_states] (null: none) of the state rows `rows` [n] take over what the step left in the second buffers.
RLB_API int rlb_commit_states(float* state, const float* next, long long width, int* token, const int* token_next, const long long* rows, int n,
                              long long num_states, int* status, void* stream) {
  if (n <= 0) return 0;
  if (n > 65535) return -2;
  const long long want = (width + 255) / 256;
  commit_states_kernel<<<dim3(static_cast<unsigned>(want < 64 ? (want > 0 ? want : 1) : 64), n), 256, 0, static_cast<cudaStream_t>(stream)>>>(
      state, next, width, token, token_next, rows, num_states, status);
  return static_cast<int>(cudaGetLastError());
}

// z [rows, ld], n columns: c0 z / rms(z) + c1 z^2 / rms(z^2) + c2 z^3 / rms(z^3) + c3 in place; coef [4].
RLB_API int rlb_poly_norm_rows(void* z, long long ld, int f32, const void* coef, long long rows, int n, float eps, void* stream) {
  if (rows <= 0) return 0;
  const dim3 grid(static_cast<unsigned>(rows));
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (f32)
    return static_cast<int>(rlb_launch_pdl(poly_norm_any_kernel<float>, grid, dim3(256), 0, s, static_cast<float*>(z), ld, static_cast<const float*>(coef), n, eps));
  auto* zp = static_cast<__nv_bfloat16*>(z);
  auto* cp = static_cast<const __nv_bfloat16*>(coef);
  if (n % 8 == 0 && ld % 8 == 0 && n <= 32768 && !(reinterpret_cast<uintptr_t>(z) & 15)) {
    const bool few = rows < 148 * 4;
    auto go = [&](auto kernel, int threads) { return static_cast<int>(rlb_launch_pdl(kernel, grid, dim3(threads), 0, s, zp, ld, cp, n, eps)); };
    if (n <= 1024) return go(poly_norm_kernel<128, 1>, 128);
    if (n <= 2048) return go(poly_norm_kernel<256, 1>, 256);
    if (n <= 4096) return few ? go(poly_norm_kernel<512, 1>, 512) : go(poly_norm_kernel<256, 2>, 256);
    if (n <= 8192) return few ? go(poly_norm_kernel<1024, 1>, 1024) : go(poly_norm_kernel<256, 4>, 256);
    if (n <= 16384) return few ? go(poly_norm_kernel<1024, 2>, 1024) : go(poly_norm_kernel<512, 4>, 512);
    return go(poly_norm_kernel<1024, 4>, 1024);
  }
  return static_cast<int>(rlb_launch_pdl(poly_norm_any_kernel<__nv_bfloat16>, grid, dim3(256), 0, s, zp, ld, cp, n, eps));
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

// Scores sigmoid(logits [T, E]) or their soft-max, choice by score + correction (null: none) among the `keep` best of `groups` groups, weights the
// scores times `scale`. counts [experts] (zero before the call) receives the experts' copies, rank each copy's number among them; outputs
// [experts, E) stand for the token itself: own_f receives their weights' sum. gate: sigmoid of logits column E.
RLB_API int rlb_moe_choose(const float* logits, long long ld, int T, int E, const float* correction, int groups, int keep, int k, int softmax, float scale,
                           int experts, float* out_w, int* out_idx, int* out_rank, int* counts, float* own_f, float* gate, void* stream) {
  if (T <= 0) return 0;
  if (E < 1 || E > MP_MAX_E || k < 1 || k > 32 || k > E || groups < 1 || E % groups || keep < 1 || keep > groups) return -2;
  if (experts > E || (experts < E && !own_f) || (gate && ld <= E)) return -2;
  const size_t smem = sizeof(float) * MC_WARPS * (2 * E + groups);
  const RouterArgs a{logits, ld, T, E, correction, groups, keep, k, softmax, scale, experts, out_w, own_f, gate, out_idx, out_rank, counts};
  return static_cast<int>(rlb_launch_pdl(moe_choose_kernel, dim3((T + MC_WARPS - 1) / MC_WARPS), dim3(MC_WARPS * 32), smem, static_cast<cudaStream_t>(stream), a));
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
