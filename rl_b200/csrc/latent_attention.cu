// Prompt portions of latent attention on the 5th-generation tensor cores (tcgen05 + TMEM + TMA), bf16 in / fp32 accumulate.
//
// The portion's context (cached tokens and its own) is gathered from the latent pages once per layer (`latent_gather_kernel`) and
// decompressed by one GEMM into per-head keys and values [tokens, heads * dim | heads * vdim]; the key part that all heads share is
// read from the gathered latent rows themselves, so it is never copied per head. One CTA per (128-row query tile, head), two CTAs per
// SM:
//   warp 0      TMA producer: Q once (unrotated and rotated parts are separate groups of 64-column swizzle atoms), then K / V tiles of
//               64 keys. K and V have one buffer and one pair of barriers each: the next K tile streams in as soon as the QK product
//               has read the current one, i.e. under the softmax and the PV product, the next V tile under the next QK and softmax
//   warp 1      tcgen05.mma issuer: S = Q K^T over dim + rot_dim in 16-wide steps, O += P V
//   warps 2..5  softmax, one thread per query row, stale-maximum rescaling; the epilogue normalises and, where the output columns hold
//               gates, multiplies by sigmoid(gate). With sigmoid weights (SIG) there is no maximum and no sum: every visible key weighs
//               sigmoid(score + a number per head), O only accumulates
// The same kernel serves grouped-query attention (rlb_flash_gqa): no rotated source of its own (the rotation is in the queries and keys), several
// query heads per key / value head, keys and values read from column ranges of one matrix, a gate or none.
// Query rows stand at the end of their context: row r of a portion of n tokens in a context of c sees keys up to c - n + r. With chunks of C
// positions (the context then begins at a chunk's border) row i sees keys from i - i % C on, and a tile starts where its first row's chunk does.
// With a window of W and the first K tokens kept it sees keys j with i - j < W or j < K: a tile visits the kept tokens' tiles and those from its
// first row's window on. The context may leave out whole tiles between the two (`skip` positions per portion).
#include "common.cuh"

#include <math.h>

namespace {
using namespace rlb;

constexpr int LA_BQ = 128, LA_BKV = 64;
constexpr int LA_Q_ATOM = LA_BQ * 128, LA_KV_ATOM = LA_BKV * 128, LA_P_BYTES = LA_BQ * 128;
constexpr int LA_THREADS = 192;
constexpr float LA_LOG2E = 1.4426950408889634f;
constexpr float LA_RESCALE = 8.0f;   // log2 units a row maximum may grow before O is rescaled

__device__ __forceinline__ void la_tmem_st_x32(uint32_t taddr, const uint32_t (&r)[32]) {
  asm volatile(
      "tcgen05.st.sync.aligned.32x32b.x32.b32 [%0], "
      "{%1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15, %16, "
      "%17, %18, %19, %20, %21, %22, %23, %24, %25, %26, %27, %28, %29, %30, %31, %32};"
      :
      : "r"(taddr), "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]), "r"(r[8]),
        "r"(r[9]), "r"(r[10]), "r"(r[11]), "r"(r[12]), "r"(r[13]), "r"(r[14]), "r"(r[15]), "r"(r[16]), "r"(r[17]),
        "r"(r[18]), "r"(r[19]), "r"(r[20]), "r"(r[21]), "r"(r[22]), "r"(r[23]), "r"(r[24]), "r"(r[25]), "r"(r[26]),
        "r"(r[27]), "r"(r[28]), "r"(r[29]), "r"(r[30]), "r"(r[31])
      : "memory");
}

struct FlashLatentParams {
  const int* cu_q;      // [portions + 1] row offsets, counted from row0
  const int* cu_ctx;    // [portions + 1] offsets into the gathered context
  int portions, row0;
  int heads, dim, rot_dim, vdim, rank;
  int q_off, mix_off;
  int atoms_n, atoms_r, atoms_v;   // 64-column swizzle atoms of the unrotated / rotated query and of the value
  int vcols;                       // columns of the PV product: vdim rounded up to 16
  int tmem_cols;
  float scale_log2;
  __nv_bfloat16* p;                // output rows (gated: the gates stand there)
  long long ldp;
  int* status;
  int per_kv;                      // query heads per key / value head
  int k_col, v_col;                // first key / value column of kv head 0
  int ctx_row0;                    // row of the key / value matrix that cu_ctx counts from
  int gated;
  int chunk;                       // > 0: keys of the row's own chunk only
  int window, keep;                // window > 0: keys nearer than that, or among the first `keep` tokens
  const int* skip;                 // [portions] positions left out of the context behind the kept tokens' tiles (null: none)
  const __nv_bfloat16* offset;     // [heads] added to the scaled scores (sigmoid weights)
};

// 1 / (1 + 2^x_i) for four x (above 30 they count as 30): one reciprocal serves all of them.
__device__ __forceinline__ void la_sigmoid4(float (&x)[4]) {
  float d[4];
#pragma unroll
  for (int i = 0; i < 4; ++i) d[i] = 1.f + exp2f(fminf(x[i], 30.f));
  const float ab = d[0] * d[1], cd = d[2] * d[3], r = __fdividef(1.f, ab * cd), rab = r * cd, rcd = r * ab;
  x[0] = rab * d[1];
  x[1] = rab * d[0];
  x[2] = rcd * d[3];
  x[3] = rcd * d[2];
}

template <bool SIG>
__global__ void __launch_bounds__(LA_THREADS, 2)
flash_latent_kernel(const __grid_constant__ CUtensorMap tmap_q, const __grid_constant__ CUtensorMap tmap_kv,
                    const __grid_constant__ CUtensorMap tmap_lat, FlashLatentParams p) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  const int atoms_q = p.atoms_n + p.atoms_r;
  uint8_t* q_s = smem;
  uint8_t* k_s = q_s + atoms_q * LA_Q_ATOM;
  uint8_t* v_s = k_s + atoms_q * LA_KV_ATOM;
  uint8_t* p_s = v_s + p.atoms_v * LA_KV_ATOM;
  uint64_t* bars = reinterpret_cast<uint64_t*>(p_s + LA_P_BYTES);
  uint64_t *q_full = bars, *k_full = bars + 1, *v_full = bars + 2, *k_empty = bars + 3, *v_empty = bars + 4, *s_full = bars + 5, *p_full = bars + 6;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 7);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  int* info = reinterpret_cast<int*>(tmem_slot + 2);   // first query row, portion rows, tile, first context row, context rows, valid, skip

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int head = blockIdx.y;
  if (threadIdx.x == 0) {
    // tiles are walked from the last (which sees most keys) to the first
    int tile = gridDim.x - 1 - blockIdx.x, s = 0, n = 0;
    for (; s < p.portions; ++s) {
      n = (p.cu_q[s + 1] - p.cu_q[s] + LA_BQ - 1) / LA_BQ;
      if (tile < n) break;
      tile -= n;
    }
    info[5] = s < p.portions;
    if (s < p.portions) {
      info[0] = p.cu_q[s];
      info[1] = p.cu_q[s + 1] - p.cu_q[s];
      info[2] = tile;
      info[3] = p.cu_ctx[s];
      info[4] = p.cu_ctx[s + 1] - p.cu_ctx[s];
      info[6] = p.skip ? p.skip[s] : 0;
    }
    for (int i = 0; i < 6; ++i) mbar_init(smem_u32(bars + i), 1);
    mbar_init(smem_u32(p_full), 128);
    *abort_flag = 0;
    mbar_fence_init();
    fence_proxy_async();
  }
  __syncthreads();
  if (!info[5]) return;   // uniform, before any TMEM allocation
  if (warp == 1) {
    tmem_alloc(smem_u32(tmem_slot), p.tmem_cols);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_s = *tmem_slot, tmem_o = tmem_s + 64;
  const int q_row0 = p.row0 + info[0], n_q = info[1], q0 = info[2] * LA_BQ, c_row0 = p.ctx_row0 + info[3], n_ctx = info[4];
  const int q_rows = min(LA_BQ, n_q - q0);
  const int skip = info[6];
  const int shift = n_ctx - n_q + skip;                              // query row i of the portion sees keys <= shift + i
  // tiles of 64 context rows: the kept tokens' (`sinks` of them, when tiles that no row sees follow), then all from first_tile on
  const int lo0 = p.chunk > 0 ? (shift + q0) / p.chunk * p.chunk : (p.window > 0 ? max(0, shift + q0 - p.window + 1) : 0);
  const int kept_tiles = p.window > 0 ? (p.keep + LA_BKV - 1) / LA_BKV : 0;
  int first_tile = max(0, lo0 - skip) / LA_BKV, sinks = kept_tiles;
  if (first_tile <= kept_tiles) {
    sinks = 0;
    if (kept_tiles > 0) first_tile = 0;
  }
  const int n_kv = sinks + (shift - skip + q0 + q_rows + LA_BKV - 1) / LA_BKV - first_tile;
  auto tile_of = [&](int j) { return j < sinks ? j : first_tile + j - sinks; };

  if (warp == 0) {
    if (lane == 0) {
      prefetch_tmap(&tmap_q);
      prefetch_tmap(&tmap_kv);
      prefetch_tmap(&tmap_lat);
      const int qx = p.q_off + head * (p.dim + p.rot_dim);
      mbar_arrive_expect_tx(smem_u32(q_full), atoms_q * LA_Q_ATOM);
      for (int a = 0; a < atoms_q; ++a)
        tma_load_2d(smem_u32(q_s + a * LA_Q_ATOM), &tmap_q, smem_u32(q_full), a < p.atoms_n ? qx + a * 64 : qx + p.dim + (a - p.atoms_n) * 64, q_row0 + q0);
      for (int j = 0; j < n_kv; ++j) {
        const uint32_t ph = j & 1;
        const int row = c_row0 + tile_of(j) * LA_BKV;
        if (!mbar_wait(smem_u32(k_empty), ph ^ 1, abort_flag, p.status, RLB_ERR_WAIT_EMPTY)) break;
        mbar_arrive_expect_tx(smem_u32(k_full), atoms_q * LA_KV_ATOM);
        for (int a = 0; a < p.atoms_n; ++a) tma_load_2d(smem_u32(k_s + a * LA_KV_ATOM), &tmap_kv, smem_u32(k_full), p.k_col + head / p.per_kv * p.dim + a * 64, row);
        for (int a = 0; a < p.atoms_r; ++a)
          tma_load_2d(smem_u32(k_s + (p.atoms_n + a) * LA_KV_ATOM), &tmap_lat, smem_u32(k_full), p.rank + a * 64, row);
        if (!mbar_wait(smem_u32(v_empty), ph ^ 1, abort_flag, p.status, RLB_ERR_WAIT_EMPTY)) break;
        mbar_arrive_expect_tx(smem_u32(v_full), p.atoms_v * LA_KV_ATOM);
        for (int a = 0; a < p.atoms_v; ++a)
          tma_load_2d(smem_u32(v_s + a * LA_KV_ATOM), &tmap_kv, smem_u32(v_full), p.v_col + head / p.per_kv * p.vdim + a * 64, row);
      }
    }
  } else if (warp == 1) {
    if (lane == 0) {
      constexpr uint32_t idesc_s = make_idesc_bf16(LA_BQ, LA_BKV, false, false);
      const uint32_t idesc_o = make_idesc_bf16(LA_BQ, p.vcols, false, true);
      const int steps_n = p.dim / 16, steps_r = (p.rot_dim + 15) / 16;
      // S = Q K^T: the unrotated steps, then the rotated ones (key columns past the rotated part hold zeros)
      auto issue_s = [&](int j) -> bool {
        if (!mbar_wait(smem_u32(k_full), j & 1, abort_flag, p.status, RLB_ERR_WAIT_FULL)) return false;
        tc_fence_after();
        for (int kk = 0; kk < steps_n + steps_r; ++kk) {
          const int a = kk < steps_n ? kk / 4 : p.atoms_n + (kk - steps_n) / 4, o = kk < steps_n ? kk % 4 : (kk - steps_n) % 4;
          umma_f16(tmem_s, make_smem_desc_sw128(smem_u32(q_s + a * LA_Q_ATOM) + o * 32, 16, 1024),
                   make_smem_desc_sw128(smem_u32(k_s + a * LA_KV_ATOM) + o * 32, 16, 1024), idesc_s, kk != 0 ? 1u : 0u);
        }
        umma_commit(smem_u32(k_empty));
        umma_commit(smem_u32(s_full));
        return true;
      };
      bool ok = mbar_wait(smem_u32(q_full), 0, abort_flag, p.status, RLB_ERR_WAIT_FULL);
      for (int j = 0; j < n_kv && ok; ++j) {
        if (!issue_s(j)) break;
        if (!mbar_wait(smem_u32(p_full), j & 1, abort_flag, p.status, RLB_ERR_WAIT_FLAG)) break;
        if (!mbar_wait(smem_u32(v_full), j & 1, abort_flag, p.status, RLB_ERR_WAIT_FULL)) break;
        tc_fence_after();
#pragma unroll
        for (int kk = 0; kk < LA_BKV / 16; ++kk)
          umma_f16(tmem_o, make_smem_desc_sw128(smem_u32(p_s) + kk * 32, 16, 1024),
                   make_smem_desc_sw128(smem_u32(v_s) + kk * (16 * 128), LA_KV_ATOM, 1024), idesc_o, (j | kk) != 0 ? 1u : 0u);
        umma_commit(smem_u32(v_empty));    // also tells the softmax warps that O and P may be touched
      }
    }
  } else {
    const int quarter = warp & 3, r = quarter * 32 + lane;
    const uint32_t lane_addr = static_cast<uint32_t>(quarter * 32) << 16;
    const int qi = shift + q0 + r;      // last key this row sees
    // first key behind the kept ones: of this row, of the last row
    const int lo = p.chunk > 0 ? qi - qi % p.chunk : (p.window > 0 ? max(0, qi - p.window + 1) : 0), last = shift + q0 + LA_BQ - 1;
    const int lo_last = p.chunk > 0 ? last / p.chunk * p.chunk : (p.window > 0 ? max(0, last - p.window + 1) : 0);
    const float off = SIG ? __bfloat162float(p.offset[head]) * LA_LOG2E : 0.f;
    float m_ref = -INFINITY, l = 0.f;
    bool ok = true;
    for (int j = 0; j < n_kv; ++j) {
      if (!mbar_wait(smem_u32(s_full), j & 1, abort_flag, p.status, RLB_ERR_WAIT_TMEM_FULL)) {
        ok = false;
        break;
      }
      tc_fence_after();
      uint32_t s0[32], s1[32];
      tmem_ld_32x32b_x32(tmem_s + lane_addr, s0);
      tmem_ld_32x32b_x32(tmem_s + lane_addr + 32, s1);
      tmem_ld_wait();
      const int tile = tile_of(j), k0 = tile * LA_BKV + (tile >= kept_tiles ? skip : 0);
      const bool edge = k0 + LA_BKV - 1 > shift + q0 || (k0 < lo_last && k0 + LA_BKV > p.keep);
      uint32_t pk[32];
      if constexpr (SIG) {
#pragma unroll
        for (int i = 0; i < 32; i += 4) {
          float a[4], b[4];
#pragma unroll
          for (int q = 0; q < 4; ++q) {
            a[q] = -fmaf(__uint_as_float(s0[i + q]), p.scale_log2, off);
            b[q] = -fmaf(__uint_as_float(s1[i + q]), p.scale_log2, off);
          }
          la_sigmoid4(a);
          la_sigmoid4(b);
          if (edge) {
#pragma unroll
            for (int q = 0; q < 4; ++q) {
              const int ka = k0 + i + q, kb = ka + 32;
              if (ka > qi || (ka < lo && ka >= p.keep)) a[q] = 0.f;
              if (kb > qi || (kb < lo && kb >= p.keep)) b[q] = 0.f;
            }
          }
          pk[i / 2] = pack_bf16x2(a[0], a[1]);
          pk[i / 2 + 1] = pack_bf16x2(a[2], a[3]);
          pk[16 + i / 2] = pack_bf16x2(b[0], b[1]);
          pk[16 + i / 2 + 1] = pack_bf16x2(b[2], b[3]);
        }
        if (j > 0 && !mbar_wait(smem_u32(v_empty), (j - 1) & 1, abort_flag, p.status, RLB_ERR_WAIT_TMEM_EMPTY)) {
          ok = false;
          break;
        }
      } else {
        float mx = -INFINITY;
#pragma unroll
        for (int i = 0; i < 32; ++i) {
          float a = __uint_as_float(s0[i]) * p.scale_log2, b = __uint_as_float(s1[i]) * p.scale_log2;
          if (edge) {
            if (k0 + i > qi || (k0 + i < lo && k0 + i >= p.keep)) a = -INFINITY;
            if (k0 + 32 + i > qi || (k0 + 32 + i < lo && k0 + 32 + i >= p.keep)) b = -INFINITY;
          }
          s0[i] = __float_as_uint(a);
          s1[i] = __float_as_uint(b);
          mx = fmaxf(mx, fmaxf(a, b));
        }
        float factor = 1.f;
        bool need = false;
        if (mx > m_ref + LA_RESCALE || m_ref == -INFINITY) {
          const float m_new = fmaxf(mx, m_ref);
          if (m_new != -INFINITY) {
            factor = m_ref == -INFINITY ? 0.f : exp2f(m_ref - m_new);
            need = m_ref != -INFINITY;
            m_ref = m_new;
          }
        }
        l *= factor;
        float rowsum = 0.f;
        const float mr = m_ref == -INFINITY ? 0.f : m_ref;
#pragma unroll
        for (int i = 0; i < 16; ++i) {
          const float e0 = exp2f(__uint_as_float(s0[2 * i]) - mr), e1 = exp2f(__uint_as_float(s0[2 * i + 1]) - mr);
          const float f0 = exp2f(__uint_as_float(s1[2 * i]) - mr), f1 = exp2f(__uint_as_float(s1[2 * i + 1]) - mr);
          rowsum += (e0 + e1) + (f0 + f1);
          pk[i] = pack_bf16x2(e0, e1);
          pk[16 + i] = pack_bf16x2(f0, f1);
        }
        l += rowsum;
        if (j > 0) {
          if (!mbar_wait(smem_u32(v_empty), (j - 1) & 1, abort_flag, p.status, RLB_ERR_WAIT_TMEM_EMPTY)) {
            ok = false;
            break;
          }
          tc_fence_after();
        }
        if (__any_sync(0xffffffffu, need)) {
          for (int c = 0; c < p.vcols; c += 32) {   // (the last 32 columns may reach past vcols: allocated, never read as output)
            uint32_t o[32];
            tmem_ld_32x32b_x32(tmem_o + lane_addr + c, o);
            tmem_ld_wait();
#pragma unroll
            for (int i = 0; i < 32; ++i) o[i] = __float_as_uint(__uint_as_float(o[i]) * factor);
            la_tmem_st_x32(tmem_o + lane_addr + c, o);
          }
          tmem_st_wait();
        }
      }
#pragma unroll
      for (int c = 0; c < 8; ++c)
        *reinterpret_cast<uint4*>(p_s + r * 128 + ((c ^ (r & 7)) << 4)) = make_uint4(pk[4 * c], pk[4 * c + 1], pk[4 * c + 2], pk[4 * c + 3]);
      fence_proxy_async();
      tc_fence_before();
      mbar_arrive(smem_u32(p_full));
    }
    if (ok && mbar_wait(smem_u32(v_empty), (n_kv - 1) & 1, abort_flag, p.status, RLB_ERR_WAIT_TMEM_EMPTY)) {
      tc_fence_after();
      const float inv_l = SIG ? 1.f : (l > 0.f ? 1.f / l : 0.f);
      __nv_bfloat16* dst = p.p + static_cast<long long>(q_row0 + q0 + r) * p.ldp + p.mix_off + head * p.vdim;
      for (int c = 0; c < p.vdim; c += 32) {
        uint32_t o[32];
        tmem_ld_32x32b_x32(tmem_o + lane_addr + c, o);
        tmem_ld_wait();
        if (r < q_rows) {
#pragma unroll
          for (int q = 0; q < 4; ++q) {
            if (c + q * 8 < p.vdim) {
              uint4 g = make_uint4(0, 0, 0, 0);
              uint32_t* gw = reinterpret_cast<uint32_t*>(&g);
              if (!p.gated) {
#pragma unroll
                for (int w = 0; w < 4; ++w)
                  gw[w] = pack_bf16x2(__uint_as_float(o[q * 8 + 2 * w]) * inv_l, __uint_as_float(o[q * 8 + 2 * w + 1]) * inv_l);
                *reinterpret_cast<uint4*>(dst + c + q * 8) = g;
                continue;
              }
              g = *reinterpret_cast<uint4*>(dst + c + q * 8);
#pragma unroll
              for (int w = 0; w < 4; ++w) {
                const float2 gf = unpack_bf16x2(gw[w]);
                gw[w] = pack_bf16x2(__uint_as_float(o[q * 8 + 2 * w]) * inv_l / (1.f + __expf(-gf.x)),
                                    __uint_as_float(o[q * 8 + 2 * w + 1]) * inv_l / (1.f + __expf(-gf.y)));
              }
              *reinterpret_cast<uint4*>(dst + c + q * 8) = g;
            }
          }
        }
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem_s, p.tmem_cols);
  }
}

// out[i] = cache row slots[i]; rows of `vecs` 16-byte pieces
__global__ void latent_gather_kernel(const uint4* __restrict__ cache, const long long* __restrict__ slots, uint4* __restrict__ out, long long n,
                                     int vecs, long long num_slots, int* status) {
  for (long long i = static_cast<long long>(blockIdx.x) * blockDim.x + threadIdx.x; i < n * vecs; i += static_cast<long long>(gridDim.x) * blockDim.x) {
    const long long t = i / vecs;
    const long long s = slots[t];
    if (s < 0 || s >= num_slots) {
      if (status) atomicCAS(status, 0, RLB_ERR_BOUNDS);
      out[i] = make_uint4(0, 0, 0, 0);
      continue;
    }
    out[i] = cache[s * vecs + (i - t * vecs)];
  }
}

int launch_flash(const CUtensorMap& tq, const CUtensorMap& tkv, const CUtensorMap& tl, const FlashLatentParams& f, int max_tiles, cudaStream_t stream) {
  const int smem = (f.atoms_n + f.atoms_r) * (LA_Q_ATOM + LA_KV_ATOM) + f.atoms_v * LA_KV_ATOM + LA_P_BYTES + 256 + 1024;
  static int configured[2] = {0, 0};
  const bool sig = f.offset != nullptr;
  auto kernel = sig ? flash_latent_kernel<true> : flash_latent_kernel<false>;
  if (smem > configured[sig]) {
    cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e != cudaSuccess) return static_cast<int>(e);
    configured[sig] = smem;
  }
  kernel<<<dim3(max_tiles, f.heads), LA_THREADS, smem, stream>>>(tq, tkv, tl, f);
  return static_cast<int>(cudaGetLastError());
}
}  // namespace

RLB_API int rlb_latent_gather(const void* cache, const long long* slots, void* out, long long n, int width, long long num_slots, int* status,
                              void* stream) {
  if (n <= 0) return 0;
  if (width % 8) return -2;
  const long long want = (n * (width / 8) + 255) / 256;
  latent_gather_kernel<<<static_cast<unsigned>(want < 148 * 16 ? want : 148 * 16), 256, 0, static_cast<cudaStream_t>(stream)>>>(
      static_cast<const uint4*>(cache), slots, static_cast<uint4*>(out), n, width / 8, num_slots, status);
  return static_cast<int>(cudaGetLastError());
}

// Shapes the kernel takes: dim a multiple of 16, rot_dim, vdim and rank of 8, at most 256 query columns (in 64-column groups, rotated
// and unrotated apart) and 256 value columns.
RLB_API int rlb_flash_latent_supported(int dim, int rot_dim, int vdim, int rank) {
  const int an = (dim + 63) / 64, ar = (rot_dim + 63) / 64, av = (vdim + 63) / 64;
  return dim > 0 && dim % 16 == 0 && rot_dim % 8 == 0 && vdim % 8 == 0 && rank % 8 == 0 && an + ar <= 4 && av <= 4 && vdim > 0;
}

// q [rows, q_width] (bf16, row stride ldq): prepared queries from column q_off; the portions are rows [row0, row0 + cu_q[portions]). kv [ctx_rows,
// heads * (dim + vdim)]: decompressed keys and values of the gathered context, lat [ctx_rows, width]: its latent rows. out (row stride ldo, may be
// the rows of q): head outputs from column mix_off, gated by what stands there when `gated`. max_tiles >= number of 128-row tiles.
RLB_API int rlb_flash_latent(const void* q, long long rows, long long ldq, int q_width, int row0, const void* kv, const void* lat, long long ctx_rows,
                             int width, const int* cu_q, const int* cu_ctx, int portions, int heads, int dim, int rot_dim, int vdim, int rank,
                             int q_off, void* out, long long ldo, int mix_off, int gated, float scale, int max_tiles, int* status, void* stream) {
  if (portions <= 0 || rows <= 0 || max_tiles <= 0) return 0;
  if (!rlb_flash_latent_supported(dim, rot_dim, vdim, rank)) return -2;
  if (ldq % 8 || ldo % 8 || width % 8 || q_off % 8 || mix_off % 8 || (dim + rot_dim) % 8 || heads > 65535) return -2;
  if ((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(out) | reinterpret_cast<uintptr_t>(kv) | reinterpret_cast<uintptr_t>(lat)) & 15) return -3;
  FlashLatentParams f{};
  f.cu_q = cu_q;
  f.cu_ctx = cu_ctx;
  f.portions = portions;
  f.row0 = row0;
  f.heads = heads;
  f.dim = dim;
  f.rot_dim = rot_dim;
  f.vdim = vdim;
  f.rank = rank;
  f.q_off = q_off;
  f.mix_off = mix_off;
  f.atoms_n = (dim + 63) / 64;
  f.atoms_r = (rot_dim + 63) / 64;
  f.atoms_v = (vdim + 63) / 64;
  f.vcols = (vdim + 15) / 16 * 16;
  f.tmem_cols = 64 + (vdim + 31) / 32 * 32 <= 128 ? 128 : (64 + (vdim + 31) / 32 * 32 <= 256 ? 256 : 512);
  f.scale_log2 = scale * LA_LOG2E;
  f.p = static_cast<__nv_bfloat16*>(out);
  f.ldp = ldo;
  f.status = status;
  f.per_kv = 1;
  f.k_col = 0;
  f.v_col = heads * dim;
  f.ctx_row0 = 0;
  f.gated = gated;
  const long long kvw = static_cast<long long>(heads) * (dim + vdim);
  CUtensorMap tq, tkv, tl;
  int rc = rlb_make_tmap_2d(&tq, q, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, q_width, rows, ldq * 2, 64, LA_BQ, CU_TENSOR_MAP_SWIZZLE_128B);
  if (rc) return -100 - rc;
  rc = rlb_make_tmap_2d(&tkv, kv, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, kvw, ctx_rows, kvw * 2, 64, LA_BKV, CU_TENSOR_MAP_SWIZZLE_128B);
  if (rc) return -100 - rc;
  rc = rlb_make_tmap_2d(&tl, lat, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, width, ctx_rows, static_cast<uint64_t>(width) * 2, 64, LA_BKV,
                        CU_TENSOR_MAP_SWIZZLE_128B);
  if (rc) return -100 - rc;
  return launch_flash(tq, tkv, tl, f, max_tiles, static_cast<cudaStream_t>(stream));
}

// Grouped-query attention of prompt portions. p: projected rows with normed and rotated queries at q_off; the portions are its rows
// [row0, row0 + cu_q[portions]). Keys of kv head g: columns [k_col + g * dim, + dim) of kv [kv_rows, kv_width], values [v_col + g * vdim, + vdim);
// row ctx_row0 + cu_ctx[i] is the first of portion i's context (kv may be p itself), with chunk > 0 the first of a chunk. window > 0: keys
// j with i - j < window or j < keep; skip [portions] (null: zeros; multiples of 64): positions that portion i's context leaves out behind its first
// ceil(keep / 64) * 64 rows. offset [heads] (bf16; null: soft-max): the weights are sigmoid(score + offset), unnormalised. y (row stride ldy, may be
// the rows of p): head outputs, with `gated` multiplied by sigmoid of what stands there. dim a multiple of 16, vdim of 8.
RLB_API int rlb_flash_gqa(void* p, long long rows, long long ldp, int in_width, int row0, const void* kv, long long kv_rows, long long ldkv, int kv_width,
                          int ctx_row0, int k_col, int v_col, const int* cu_q, const int* cu_ctx, int portions, int heads, int kv_heads, int dim, int vdim,
                          int q_off, int chunk, int window, int keep, const int* skip, const void* offset, int gated, float scale, int max_tiles, void* y, long long ldy,
                          int* status, void* stream) {
  if (portions <= 0 || rows <= 0 || max_tiles <= 0) return 0;
  if (!rlb_flash_latent_supported(dim, 0, vdim, 8) || kv_heads < 1 || heads % kv_heads || (chunk > 0 && window > 0) || (skip && window <= 0)) return -2;
  if (ldp % 8 || ldkv % 8 || ldy % 8 || q_off % 8 || k_col % 8 || v_col % 8 || heads > 65535) return -2;
  if ((reinterpret_cast<uintptr_t>(p) | reinterpret_cast<uintptr_t>(kv) | reinterpret_cast<uintptr_t>(y)) & 15) return -3;
  FlashLatentParams f{};
  f.cu_q = cu_q;
  f.cu_ctx = cu_ctx;
  f.portions = portions;
  f.row0 = row0;
  f.heads = heads;
  f.dim = dim;
  f.vdim = vdim;
  f.q_off = q_off;
  f.atoms_n = (dim + 63) / 64;
  f.atoms_v = (vdim + 63) / 64;
  f.vcols = (vdim + 15) / 16 * 16;
  f.tmem_cols = 64 + (vdim + 31) / 32 * 32 <= 128 ? 128 : (64 + (vdim + 31) / 32 * 32 <= 256 ? 256 : 512);
  f.scale_log2 = scale * LA_LOG2E;
  f.p = static_cast<__nv_bfloat16*>(y);
  f.ldp = ldy;
  f.status = status;
  f.per_kv = heads / kv_heads;
  f.k_col = k_col;
  f.v_col = v_col;
  f.ctx_row0 = ctx_row0;
  f.chunk = chunk;
  f.window = window;
  f.keep = window > 0 ? keep : 0;
  f.skip = skip;
  f.offset = static_cast<const __nv_bfloat16*>(offset);
  f.gated = gated;
  CUtensorMap tq, tkv;
  int rc = rlb_make_tmap_2d(&tq, p, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, in_width, rows, ldp * 2, 64, LA_BQ, CU_TENSOR_MAP_SWIZZLE_128B);
  if (rc) return -100 - rc;
  rc = rlb_make_tmap_2d(&tkv, kv, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, kv_width, kv_rows, ldkv * 2, 64, LA_BKV, CU_TENSOR_MAP_SWIZZLE_128B);
  if (rc) return -100 - rc;
  return launch_flash(tq, tkv, tkv, f, max_tiles, static_cast<cudaStream_t>(stream));
}
