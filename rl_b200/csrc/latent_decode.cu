// Decode form of latent attention on the tensor cores (tcgen05 + TMEM + TMA), bf16 in / fp32 accumulate. Every row is one query token
// with its own page table. Keys and values are never decompressed: all heads of a row read the same cached latent rows.
//
//   heads GEMM   q_lat[t, h, :] = q[t, h, :dim] W_uk[h]         the unrotated query carried into the latent space (W_uk read MN-major)
//   attention    S^T[64 tokens, HN heads] = L Q^T                one CTA per (row, group of HN heads, split of the context); the tile of
//                O^T[128 dims, HN] (x rank / 128) += L^T P        latent rows is both K and V: it is fetched once
//   combine      joins the splits
//   heads GEMM   y[t, h, :] = o[t, h, :] W_uv[h]^T * sigmoid(gate), written over the gate columns of the projected rows
//
// The attention kernel streams latent tiles of 64 tokens as 16 KB slots (two 64-column groups) through a ring that holds at least
// two tiles: the scores of tile i + 1 are computed under the softmax of tile i, and the PV product gives slots back one by one, so
// the stream from memory never stops. The score product is issued with 128 rows; rows 64.. read the neighbouring slot and their
// results are ignored (the instruction's cost is hidden under the stream). The narrow MMAs are bound by the issuing thread, so
// every descriptor is a precomputed base plus a constant. O stays in TMEM over all tiles; it is rescaled only when a running
// maximum grew by more than 2^8.
#include "common.cuh"

#include <math.h>

namespace {
using namespace rlb;

// ---------------------------------------------------------------------------------------------------- per-head GEMM
constexpr int HG_T = 128, HG_K = 64;      // rows of A per tile, reduction step
template <int BN, int STAGES>
struct HgCfg {
  static constexpr int STAGE = (HG_T + BN) * HG_K * 2;
  static constexpr int SMEM = STAGES * STAGE + 256 + 1024;
  static constexpr int TMEM = BN < 32 ? 32 : BN;
};
constexpr int HG_THREADS = 192;

struct HeadsGemm {
  int M, N, K;            // rows, columns and reduction length per head
  int a_off, a_head;      // first A column of head h: a_off + h * a_head
  int b_row0, b_head;     // first B row of head h: b_row0 + h * b_head
  __nv_bfloat16* out;
  long long ldo;
  int o_off, o_head;
  int gate;               // out = acc * sigmoid(out) instead of out = acc
  int* status;
};

template <bool B_MN, int BN, int STAGES>
__global__ void __launch_bounds__(HG_THREADS, 1)
gemm_heads_kernel(const __grid_constant__ CUtensorMap tmap_a, const __grid_constant__ CUtensorMap tmap_b, HeadsGemm g) {
  static_assert(!B_MN || BN == 128, "the MN-major operand is fetched as two 64-column boxes");
  constexpr int HG_STAGES = STAGES, HG_STAGE = HgCfg<BN, STAGES>::STAGE;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint64_t* full = reinterpret_cast<uint64_t*>(smem + HG_STAGES * HG_STAGE);
  uint64_t* empty = full + HG_STAGES;
  uint64_t* acc_bar = empty + HG_STAGES;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(acc_bar + 1);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (threadIdx.x == 0) {
    for (int s = 0; s < HG_STAGES; ++s) {
      mbar_init(smem_u32(full + s), 1);
      mbar_init(smem_u32(empty + s), 1);
    }
    mbar_init(smem_u32(acc_bar), 1);
    *abort_flag = 0;
    mbar_fence_init();
    fence_proxy_async();
    prefetch_tmap(&tmap_a);
    prefetch_tmap(&tmap_b);
  }
  if (warp == 1) {
    tmem_alloc(smem_u32(tmem_slot), HgCfg<BN, STAGES>::TMEM);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  pdl_sync();
  const uint32_t tmem = *tmem_slot;
  const int n0 = blockIdx.x * BN, m0 = blockIdx.y * HG_T, head = blockIdx.z;
  const int num_k = (g.K + HG_K - 1) / HG_K;

  if (warp == 0) {
    if (lane == 0) {
      for (int kb = 0; kb < num_k; ++kb) {
        const int s = kb % HG_STAGES;
        if (!mbar_wait(smem_u32(empty + s), ((kb / HG_STAGES) & 1) ^ 1, abort_flag, g.status, RLB_ERR_WAIT_EMPTY)) break;
        const uint32_t bar = smem_u32(full + s), a = smem_u32(smem + s * HG_STAGE), b = a + HG_T * HG_K * 2;
        mbar_arrive_expect_tx(bar, HG_STAGE);
        tma_load_2d(a, &tmap_a, bar, g.a_off + head * g.a_head + kb * HG_K, m0);
        const int brow = g.b_row0 + head * g.b_head;
        if (B_MN) {
          tma_load_2d(b, &tmap_b, bar, n0, brow + kb * HG_K);
          tma_load_2d(b + HG_K * 128, &tmap_b, bar, n0 + 64, brow + kb * HG_K);
        } else {
          tma_load_2d(b, &tmap_b, bar, kb * HG_K, brow + n0);
        }
      }
    }
  } else if (warp == 1) {
    if (lane == 0) {
      constexpr uint32_t idesc = make_idesc_bf16(HG_T, BN, false, B_MN);
      bool ok = true;
      for (int kb = 0; kb < num_k; ++kb) {
        const int s = kb % HG_STAGES;
        if (!mbar_wait(smem_u32(full + s), (kb / HG_STAGES) & 1, abort_flag, g.status, RLB_ERR_WAIT_FULL)) {
          ok = false;
          break;
        }
        tc_fence_after();
        const uint32_t a = smem_u32(smem + s * HG_STAGE), b = a + HG_T * HG_K * 2;
        const uint64_t ad = make_smem_desc_sw128(a, 16, 1024), bd = B_MN ? make_smem_desc_sw128(b, HG_K * 128, 1024) : make_smem_desc_sw128(b, 16, 1024);
        constexpr uint32_t bstep = (B_MN ? 16 * 128 : 32) >> 4;
        const int steps = min(HG_K / 16, (g.K - kb * HG_K + 15) / 16);   // columns past K belong to the next head
        for (int kk = 0; kk < steps; ++kk) umma_f16(tmem, ad + kk * 2, bd + kk * bstep, idesc, (kb | kk) != 0 ? 1u : 0u);
        umma_commit(smem_u32(empty + s));
      }
      if (ok) umma_commit(smem_u32(acc_bar));
    }
  } else {
    const int quarter = warp & 3, row = m0 + quarter * 32 + lane;
    if (mbar_wait(smem_u32(acc_bar), 0, abort_flag, g.status, RLB_ERR_WAIT_TMEM_FULL)) {
      tc_fence_after();
      __nv_bfloat16* o = g.out + static_cast<long long>(row) * g.ldo + g.o_off + static_cast<long long>(head) * g.o_head + n0;
      for (int c = 0; c < BN && n0 + c < g.N; c += 32) {
        uint32_t r[32];
        tmem_ld_32x32b_x32(tmem + (static_cast<uint32_t>(quarter * 32) << 16) + c, r);
        tmem_ld_wait();
        if (row >= g.M) continue;
#pragma unroll
        for (int q = 0; q < 4; ++q) {
          if (n0 + c + q * 8 < g.N) {     // N is a multiple of 8
            uint4 v;
            uint32_t* vw = reinterpret_cast<uint32_t*>(&v);
            if (g.gate) {
              v = *reinterpret_cast<const uint4*>(o + c + q * 8);
#pragma unroll
              for (int w = 0; w < 4; ++w) {
                const float2 gf = unpack_bf16x2(vw[w]);
                vw[w] = pack_bf16x2(__uint_as_float(r[q * 8 + 2 * w]) / (1.f + __expf(-gf.x)), __uint_as_float(r[q * 8 + 2 * w + 1]) / (1.f + __expf(-gf.y)));
              }
            } else {
#pragma unroll
              for (int w = 0; w < 4; ++w) vw[w] = pack_bf16x2(__uint_as_float(r[q * 8 + 2 * w]), __uint_as_float(r[q * 8 + 2 * w + 1]));
            }
            *reinterpret_cast<uint4*>(o + c + q * 8) = v;
          }
        }
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem, HgCfg<BN, STAGES>::TMEM);
  }
}

// ---------------------------------------------------------------------------------------------------- attention
constexpr int LD_TOK = 64;
constexpr int LD_CHUNK = LD_TOK * 128;       // 64 tokens x 64 columns
constexpr int LD_SLOT = 2 * LD_CHUNK;        // 16 KB
constexpr int LD_MAX_SLOTS = 12;
constexpr int LD_THREADS = 192;
constexpr float LD_LOG2E = 1.4426950408889634f;
constexpr float LD_RESCALE = 8.0f;

struct LdParams {
  const int* block_table;
  int bt_stride;
  const int* seq_lens;
  int heads, rank, block_size;
  int chunks;         // 64-column groups of a latent row
  int pairs;          // 128-dim output tiles
  int slots_tile;     // ring slots of one tile: ceil(chunks / 2)
  int slots;          // ring size
  int tmem_cols;
  float scale_log2;
  int num_splits;
  float* part_o;      // [rows, heads, splits, rank]
  float* part_ml;     // [rows, heads, splits, 2]
  __nv_bfloat16* out; // [rows, heads * rank]
  int* status;
};

__device__ __forceinline__ void ld_bar_sync() { asm volatile("bar.sync 1, 128;" ::: "memory"); }
__device__ __forceinline__ uint32_t ld_sw128(int row, int c) { return row * 128 + (((c >> 3) ^ (row & 7)) << 4) + ((c * 2) & 15); }

// Butterfly over the warp that reduces N values per lane at once: after log2(N) exchanges each lane holds one value's partial
// result, the rest of the exchanges complete it. Returns the reduced value `lane / (32 / N)`.
template <int N, typename Op>
__device__ __forceinline__ float warp_reduce_many(float (&v)[N], int lane, Op op) {
  int n = N, off = 16;
#pragma unroll
  for (int step = 0; step < 5; ++step, off >>= 1) {
    if (n > 1) {
      n >>= 1;
      const bool up = lane & off;
#pragma unroll
      for (int k = 0; k < N / 2; ++k) {
        if (k < n) {
          const float keep = up ? v[k + n] : v[k], send = up ? v[k] : v[k + n];
          v[k] = op(keep, __shfl_xor_sync(0xffffffffu, send, off));
        }
      }
    } else {
      v[0] = op(v[0], __shfl_xor_sync(0xffffffffu, v[0], off));
    }
  }
  return v[0];
}

__device__ __forceinline__ void ld_tmem_ld16(uint32_t addr, uint32_t* r) { tmem_ld_32x32b_x16(addr, *reinterpret_cast<uint32_t(*)[16]>(r)); }
__device__ __forceinline__ void ld_tmem_st16(uint32_t addr, uint32_t* r) { tmem_st_32x32b_x16(addr, *reinterpret_cast<uint32_t(*)[16]>(r)); }

template <int HN>
__global__ void __launch_bounds__(LD_THREADS, 1)
latent_decode_kernel(const __grid_constant__ CUtensorMap tmap_lat, const __grid_constant__ CUtensorMap tmap_q, LdParams p) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  constexpr int QP = HN * 128;     // one 64-column group of Q or of P^T
  uint8_t* ring = smem;
  uint8_t* q_sm = ring + p.slots * LD_SLOT;
  uint8_t* p_sm = q_sm + p.chunks * QP;
  float* red = reinterpret_cast<float*>(p_sm + QP);        // [4][HN]
  uint64_t* bars = reinterpret_cast<uint64_t*>(red + 4 * HN);
  uint64_t *full = bars, *empty = bars + LD_MAX_SLOTS, *q_full = bars + 2 * LD_MAX_SLOTS;
  uint64_t *s_full = q_full + 1, *s_empty = q_full + 2, *p_ready = q_full + 3, *o_done = q_full + 4;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(q_full + 5);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (threadIdx.x == 0) {
    for (int s = 0; s < 2 * LD_MAX_SLOTS + 2; ++s) mbar_init(smem_u32(bars + s), 1);
    mbar_init(smem_u32(s_empty), 4);
    mbar_init(smem_u32(p_ready), 128);
    mbar_init(smem_u32(o_done), 1);
    *abort_flag = 0;
    mbar_fence_init();
    fence_proxy_async();
    prefetch_tmap(&tmap_lat);
    prefetch_tmap(&tmap_q);
  }
  if (warp == 1) {
    tmem_alloc(smem_u32(tmem_slot), p.tmem_cols);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  pdl_sync();
  const uint32_t tmem_s = *tmem_slot, tmem_o = tmem_s + HN;

  const int row = blockIdx.x, h0 = blockIdx.y * HN, split = blockIdx.z;
  const int bs = p.block_size;
  const int len = min(p.seq_lens[row], p.bt_stride * bs);
  const int per_split = ((len + p.num_splits - 1) / p.num_splits + LD_TOK - 1) / LD_TOK * LD_TOK;
  const int t_begin = split * per_split, t_end = min(len, t_begin + per_split);
  const int n_tiles = t_end > t_begin ? (t_end - t_begin + LD_TOK - 1) / LD_TOK : 0;

  if (warp == 0) {
    if (lane == 0 && n_tiles > 0) {
      mbar_arrive_expect_tx(smem_u32(q_full), p.chunks * QP);
      for (int c = 0; c < p.chunks; ++c) tma_load_2d(smem_u32(q_sm + c * QP), &tmap_q, smem_u32(q_full), c * 64, row * p.heads + h0);
      const int* bt = p.block_table + static_cast<long long>(row) * p.bt_stride;
      const int box = bs < LD_TOK ? bs : LD_TOK, nbox = LD_TOK / box;
      int slot = 0;
      uint32_t phase = 0;
      bool ok = true;
      for (int i = 0; i < n_tiles && ok; ++i) {
        const int t0 = t_begin + i * LD_TOK;
        for (int j = 0; j < p.slots_tile; ++j) {
          if (!mbar_wait(smem_u32(empty + slot), phase ^ 1, abort_flag, p.status, RLB_ERR_WAIT_EMPTY)) {
            ok = false;
            break;
          }
          const int nch = min(2, p.chunks - 2 * j);
          const uint32_t bar = smem_u32(full + slot), dst = smem_u32(ring + slot * LD_SLOT);
          mbar_arrive_expect_tx(bar, nch * LD_CHUNK);
          for (int b = 0; b < nbox; ++b) {
            // tokens past the end read pages of valid (if unrelated) content; their scores are masked before the softmax
            const int t = t0 + b * box;
            const int crow = bt[min(t / bs, p.bt_stride - 1)] * bs + t % bs;
            for (int c = 0; c < nch; ++c) tma_load_2d(dst + c * LD_CHUNK + b * box * 128, &tmap_lat, bar, (2 * j + c) * 64, crow);
          }
          if (++slot == p.slots) {
            slot = 0;
            phase ^= 1;
          }
        }
      }
    }
  } else if (warp == 1) {
    if (lane == 0 && n_tiles > 0) {
      constexpr uint32_t idesc_qk = make_idesc_bf16(128, HN, false, false);
      constexpr uint32_t idesc_pv = make_idesc_bf16(128, HN, true, false);
      const uint64_t k_desc = make_smem_desc_sw128(smem_u32(ring), 16, 1024), v_desc = make_smem_desc_sw128(smem_u32(ring), LD_CHUNK, 1024);
      const uint64_t q_desc = make_smem_desc_sw128(smem_u32(q_sm), 16, 1024), p_desc = make_smem_desc_sw128(smem_u32(p_sm), 16, 1024);
      int qk_slot = 0, pv_slot = 0;
      uint32_t qk_phase = 0;
      auto issue_qk = [&](int i) -> bool {
        if (!mbar_wait(smem_u32(s_empty), (i & 1) ^ 1, abort_flag, p.status, RLB_ERR_WAIT_TMEM_EMPTY)) return false;
        uint64_t qd = q_desc;
        for (int j = 0; j < p.slots_tile; ++j) {
          if (!mbar_wait(smem_u32(full + qk_slot), qk_phase, abort_flag, p.status, RLB_ERR_WAIT_FULL)) return false;
          tc_fence_after();
          const uint64_t kd = k_desc + static_cast<uint32_t>(qk_slot * (LD_SLOT >> 4));
          const bool two = 2 * j + 1 < p.chunks;
#pragma unroll
          for (int kk = 0; kk < 4; ++kk) umma_f16(tmem_s, kd + kk * 2, qd + kk * 2, idesc_qk, (j | kk) != 0 ? 1u : 0u);
          if (two) {
#pragma unroll
            for (int kk = 0; kk < 4; ++kk) umma_f16(tmem_s, kd + (LD_CHUNK >> 4) + kk * 2, qd + (QP >> 4) + kk * 2, idesc_qk, 1u);
          }
          qd += 2 * (QP >> 4);
          if (j >= p.pairs) umma_commit(smem_u32(empty + qk_slot));    // holds only the rotated key part
          if (++qk_slot == p.slots) {
            qk_slot = 0;
            qk_phase ^= 1;
          }
        }
        umma_commit(smem_u32(s_full));
        return true;
      };
      bool ok = mbar_wait(smem_u32(q_full), 0, abort_flag, p.status, RLB_ERR_WAIT_FULL);
      if (ok) ok = issue_qk(0);
      for (int i = 0; i < n_tiles && ok; ++i) {
        if (i + 1 < n_tiles && !issue_qk(i + 1)) break;     // under the softmax of tile i
        if (!mbar_wait(smem_u32(p_ready), i & 1, abort_flag, p.status, RLB_ERR_WAIT_FLAG)) break;
        tc_fence_after();
        for (int j = 0; j < p.slots_tile; ++j) {
          if (j < p.pairs) {
            const uint64_t vd = v_desc + static_cast<uint32_t>(pv_slot * (LD_SLOT >> 4));
#pragma unroll
            for (int kk = 0; kk < LD_TOK / 16; ++kk) umma_f16(tmem_o + j * HN, vd + kk * 128, p_desc + kk * 2, idesc_pv, (i | kk) != 0 ? 1u : 0u);
            umma_commit(smem_u32(empty + pv_slot));
          }
          if (++pv_slot == p.slots) pv_slot = 0;
        }
        umma_commit(smem_u32(o_done));
      }
    }
  } else {
    const int quarter = warp & 3, r = quarter * 32 + lane;
    const uint32_t lane_addr = static_cast<uint32_t>(quarter * 32) << 16;
    float m_ref[HN], l[HN];
#pragma unroll
    for (int g = 0; g < HN; ++g) {
      m_ref[g] = -INFINITY;
      l[g] = 0.f;
    }
    bool ok = true;
    for (int i = 0; i < n_tiles; ++i) {
      const uint32_t ph = i & 1;
      // a wait that ran out clears `ok` but leaves no loop early: every warp passes the same named barriers
      ok = ok && mbar_wait(smem_u32(s_full), ph, abort_flag, p.status, RLB_ERR_WAIT_TMEM_FULL);
      tc_fence_after();
      uint32_t sr[HN];
#pragma unroll
      for (int c = 0; c < HN; c += 16) ld_tmem_ld16(tmem_s + lane_addr + c, sr + c);
      tmem_ld_wait();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(smem_u32(s_empty));
      const bool valid = r < LD_TOK && t_begin + i * LD_TOK + r < t_end;
      float s[HN], mx[HN];
#pragma unroll
      for (int g = 0; g < HN; ++g) mx[g] = s[g] = valid ? __uint_as_float(sr[g]) * p.scale_log2 : -INFINITY;
      const float wm = warp_reduce_many<HN>(mx, lane, [](float a, float b) { return fmaxf(a, b); });
      if (lane % (32 / HN) == 0) red[quarter * HN + lane / (32 / HN)] = wm;
      ld_bar_sync();
      float f[HN];
      bool need = false;
#pragma unroll
      for (int g = 0; g < HN; ++g) {
        const float mt = fmaxf(fmaxf(red[g], red[HN + g]), fmaxf(red[2 * HN + g], red[3 * HN + g]));
        f[g] = 1.f;
        if (mt > m_ref[g] + LD_RESCALE || m_ref[g] == -INFINITY) {
          f[g] = m_ref[g] == -INFINITY ? 0.f : exp2f(m_ref[g] - mt);
          need = true;
          m_ref[g] = mt;
        }
        s[g] = s[g] == -INFINITY ? 0.f : exp2f(s[g] - m_ref[g]);
        l[g] = l[g] * f[g] + s[g];
      }
      if (i > 0) {
        ok = ok && mbar_wait(smem_u32(o_done), (i - 1) & 1, abort_flag, p.status, RLB_ERR_WAIT_TMEM_EMPTY);
        tc_fence_after();
        if (need) {     // the same decision in every thread: the maxima are shared
          for (int j = 0; j < p.pairs; ++j) {
#pragma unroll
            for (int c = 0; c < HN; c += 16) {
              uint32_t o[16];
              ld_tmem_ld16(tmem_o + lane_addr + j * HN + c, o);
              tmem_ld_wait();
#pragma unroll
              for (int g = 0; g < 16; ++g) o[g] = __float_as_uint(__uint_as_float(o[g]) * f[c + g]);
              ld_tmem_st16(tmem_o + lane_addr + j * HN + c, o);
            }
          }
          tmem_st_wait();
        }
      }
      if (r < LD_TOK) {
#pragma unroll
        for (int g = 0; g < HN; ++g) *reinterpret_cast<__nv_bfloat16*>(p_sm + ld_sw128(g, r)) = __float2bfloat16(s[g]);
      }
      fence_proxy_async();
      tc_fence_before();
      ld_bar_sync();      // the maxima of this tile have been read by everyone before the next tile overwrites them
      mbar_arrive(smem_u32(p_ready));
    }
    if (ok && n_tiles > 0) ok = mbar_wait(smem_u32(o_done), (n_tiles - 1) & 1, abort_flag, p.status, RLB_ERR_WAIT_TMEM_EMPTY);
    tc_fence_after();
    float lw[HN];
#pragma unroll
    for (int g = 0; g < HN; ++g) lw[g] = l[g];
    const float ws = warp_reduce_many<HN>(lw, lane, [](float a, float b) { return a + b; });
    if (lane % (32 / HN) == 0) red[quarter * HN + lane / (32 / HN)] = ws;
    ld_bar_sync();
#pragma unroll
    for (int g = 0; g < HN; ++g) l[g] = (red[g] + red[HN + g]) + (red[2 * HN + g] + red[3 * HN + g]);
    for (int j = 0; j < p.pairs; ++j) {
      uint32_t o[HN];
#pragma unroll
      for (int c = 0; c < HN; c += 16) ld_tmem_ld16(tmem_o + lane_addr + j * HN + c, o + c);
      tmem_ld_wait();
      const int d = j * 128 + r;
      if (d >= p.rank) continue;
#pragma unroll
      for (int g = 0; g < HN; ++g) {
        if (h0 + g >= p.heads) continue;
        const float v = (ok && n_tiles > 0) ? __uint_as_float(o[g]) : 0.f;
        const long long rh = static_cast<long long>(row) * p.heads + h0 + g;
        if (p.num_splits == 1)
          p.out[rh * p.rank + d] = __float2bfloat16(l[g] > 0.f ? v / l[g] : 0.f);
        else
          p.part_o[(rh * p.num_splits + split) * p.rank + d] = v;
      }
    }
    if (p.num_splits > 1 && r == 0) {
#pragma unroll
      for (int g = 0; g < HN; ++g) {
        if (h0 + g >= p.heads) continue;
        const long long i = ((static_cast<long long>(row) * p.heads + h0 + g) * p.num_splits + split) * 2;
        p.part_ml[i] = m_ref[g];
        p.part_ml[i + 1] = l[g];
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

__global__ void __launch_bounds__(128)
latent_combine_kernel(const float* __restrict__ part_o, const float* __restrict__ part_ml, int num_splits, int rank, __nv_bfloat16* __restrict__ out) {
  __shared__ float w[32];
  pdl_sync();
  const long long rh = blockIdx.x;
  if (threadIdx.x < 32) {     // num_splits <= 32: one lane per split
    const int s = threadIdx.x;
    const float m = s < num_splits ? part_ml[(rh * num_splits + s) * 2] : -INFINITY;
    const float l = s < num_splits ? part_ml[(rh * num_splits + s) * 2 + 1] : 0.f;
    const float mm = warp_max(m);
    const float f = m == -INFINITY ? 0.f : exp2f(m - mm);
    const float ll = warp_sum(l * f);
    w[s] = ll > 0.f ? f / ll : 0.f;
  }
  __syncthreads();
  const float4* src = reinterpret_cast<const float4*>(part_o + rh * num_splits * rank);
  const int n4 = rank / 4;
  for (int d = threadIdx.x; d < n4; d += 128) {
    float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 8
    for (int s = 0; s < num_splits; ++s) {
      const float4 v = src[s * n4 + d];
      acc.x = fmaf(v.x, w[s], acc.x);
      acc.y = fmaf(v.y, w[s], acc.y);
      acc.z = fmaf(v.z, w[s], acc.z);
      acc.w = fmaf(v.w, w[s], acc.w);
    }
    *reinterpret_cast<uint2*>(out + rh * rank + d * 4) = make_uint2(pack_bf16x2(acc.x, acc.y), pack_bf16x2(acc.z, acc.w));
  }
}

template <int HN>
int launch_latent_decode(const CUtensorMap& tl, const CUtensorMap& tq, LdParams p, int rows, cudaStream_t s) {
  // behind the ring: queries, weights, reductions, barriers, and at least the 8 KB that the score product may read past the last slot
  const int fixed = LD_CHUNK + p.chunks * HN * 128 + HN * 128 + 4 * HN * 4 + (2 * LD_MAX_SLOTS + 6) * 8 + 1024;
  int slots = (227 * 1024 - fixed) / LD_SLOT;
  if (slots > LD_MAX_SLOTS) slots = LD_MAX_SLOTS;
  if (p.slots_tile * 4 < slots) slots = p.slots_tile * 4;
  if (slots < 2 * p.slots_tile) return -2;      // the scores run one tile ahead of the PV product
  p.slots = slots;
  const int cols = (1 + p.pairs) * HN;
  p.tmem_cols = cols <= 32 ? 32 : (cols <= 64 ? 64 : (cols <= 128 ? 128 : (cols <= 256 ? 256 : 512)));
  const int smem = slots * LD_SLOT + fixed;
  static int configured = 0;
  if (smem > configured) {
    cudaError_t e = cudaFuncSetAttribute(latent_decode_kernel<HN>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e != cudaSuccess) return static_cast<int>(e);
    configured = smem;
  }
  return static_cast<int>(rlb_launch_pdl(latent_decode_kernel<HN>, dim3(rows, (p.heads + HN - 1) / HN, p.num_splits), dim3(LD_THREADS), smem, s, tl, tq, p));
}
}  // namespace

// Shapes the decode kernels take: dim a multiple of 16, rot_dim, vdim, rank of 8, rank at most 512 and a latent row of at most 640.
RLB_API int rlb_latent_decode_supported(int dim, int rot_dim, int vdim, int rank, int width, int block_size) {
  return dim > 0 && dim % 16 == 0 && rot_dim % 8 == 0 && vdim > 0 && vdim % 8 == 0 && rank % 8 == 0 && rank <= 512 && width % 8 == 0 && width <= 640 &&
         (block_size == 16 || block_size == 32 || block_size == 64 || (block_size > 0 && block_size % 128 == 0));
}

// q_lat [rows, heads, width] (bf16): columns [rank, width) hold the rotated query part (zero padded) already; columns [0, rank) are
// computed here. o_lat [rows, heads * rank] is scratch. part_o / part_ml: scratch for num_splits > 1. Only rows [0, rows) of p.
RLB_API int rlb_latent_decode(void* p, int rows, long long ldp, int in_width, int q_off, int mix_off, int heads, int dim, int rot_dim, int vdim,
                              int rank, int width, int block_size, int num_blocks, const void* cache, const int* block_table, int bt_stride,
                              const int* seq_lens, const void* kv_up, float scale, void* q_lat, void* o_lat, int num_splits, float* part_o,
                              float* part_ml, int* status, void* stream) {
  if (rows <= 0) return 0;
  if (!rlb_latent_decode_supported(dim, rot_dim, vdim, rank, width, block_size) || heads > 65535 || num_splits < 1 || num_splits > 32) return -2;
  if (ldp % 8 || q_off % 8 || mix_off % 8 || (dim + rot_dim) % 8 || (num_splits > 1 && (!part_o || !part_ml))) return -2;
  if ((reinterpret_cast<uintptr_t>(p) | reinterpret_cast<uintptr_t>(cache) | reinterpret_cast<uintptr_t>(kv_up) | reinterpret_cast<uintptr_t>(q_lat) |
       reinterpret_cast<uintptr_t>(o_lat)) & 15)
    return -3;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  static bool configured = false;
  if (!configured) {
    cudaError_t e = cudaFuncSetAttribute(gemm_heads_kernel<true, 128, 4>, cudaFuncAttributeMaxDynamicSharedMemorySize, HgCfg<128, 4>::SMEM);
    if (e == cudaSuccess) e = cudaFuncSetAttribute(gemm_heads_kernel<false, 32, 8>, cudaFuncAttributeMaxDynamicSharedMemorySize, HgCfg<32, 8>::SMEM);
    if (e != cudaSuccess) return static_cast<int>(e);
    configured = true;
  }
  const auto BF = CU_TENSOR_MAP_DATA_TYPE_BFLOAT16;
  const auto SW = CU_TENSOR_MAP_SWIZZLE_128B;
  CUtensorMap ta, tb, tl, tq;
  int rc = rlb_make_tmap_2d(&ta, p, BF, 2, in_width, rows, ldp * 2, HG_K, HG_T, SW);
  if (!rc) rc = rlb_make_tmap_2d(&tb, kv_up, BF, 2, rank, static_cast<uint64_t>(heads) * (dim + vdim), static_cast<uint64_t>(rank) * 2, 64, HG_K, SW);
  if (rc) return -100 - rc;
  HeadsGemm g{rows, rank, dim, q_off, dim + rot_dim, 0, dim, static_cast<__nv_bfloat16*>(q_lat), static_cast<long long>(heads) * width, 0, width, 0, status};
  cudaError_t e = rlb_launch_pdl(gemm_heads_kernel<true, 128, 4>, dim3((rank + 127) / 128, (rows + HG_T - 1) / HG_T, heads), dim3(HG_THREADS), HgCfg<128, 4>::SMEM, s, ta, tb, g);
  if (e != cudaSuccess) return static_cast<int>(e);

  LdParams d{};
  d.block_table = block_table;
  d.bt_stride = bt_stride;
  d.seq_lens = seq_lens;
  d.heads = heads;
  d.rank = rank;
  d.block_size = block_size;
  d.chunks = (width + 63) / 64;
  d.pairs = (rank + 127) / 128;
  d.slots_tile = (d.chunks + 1) / 2;
  d.scale_log2 = scale * LD_LOG2E;
  d.num_splits = num_splits;
  d.part_o = part_o;
  d.part_ml = part_ml;
  d.out = static_cast<__nv_bfloat16*>(o_lat);
  d.status = status;
  const int hn = heads > 16 ? 32 : 16;
  rc = rlb_make_tmap_2d(&tl, cache, BF, 2, width, static_cast<uint64_t>(num_blocks) * block_size, static_cast<uint64_t>(width) * 2, 64,
                        block_size < LD_TOK ? block_size : LD_TOK, SW);
  if (!rc) rc = rlb_make_tmap_2d(&tq, q_lat, BF, 2, width, static_cast<uint64_t>(rows) * heads, static_cast<uint64_t>(width) * 2, 64, hn, SW);
  if (rc) return -100 - rc;
  rc = hn == 32 ? launch_latent_decode<32>(tl, tq, d, rows, s) : launch_latent_decode<16>(tl, tq, d, rows, s);
  if (rc) return rc;
  if (num_splits > 1) {
    e = rlb_launch_pdl(latent_combine_kernel, dim3(static_cast<unsigned>(rows) * heads), dim3(128), 0, s, part_o, part_ml, num_splits, rank,
                       static_cast<__nv_bfloat16*>(o_lat));
    if (e != cudaSuccess) return static_cast<int>(e);
  }
  rc = rlb_make_tmap_2d(&ta, o_lat, BF, 2, static_cast<uint64_t>(heads) * rank, rows, static_cast<uint64_t>(heads) * rank * 2, HG_K, HG_T, SW);
  if (!rc) rc = rlb_make_tmap_2d(&tb, kv_up, BF, 2, rank, static_cast<uint64_t>(heads) * (dim + vdim), static_cast<uint64_t>(rank) * 2, HG_K, 32, SW);
  if (rc) return -100 - rc;
  HeadsGemm u{rows, vdim, rank, 0, rank, heads * dim, vdim, static_cast<__nv_bfloat16*>(p), ldp, mix_off, vdim, 1, status};
  e = rlb_launch_pdl(gemm_heads_kernel<false, 32, 8>, dim3((vdim + 31) / 32, (rows + HG_T - 1) / HG_T, heads), dim3(HG_THREADS), HgCfg<32, 8>::SMEM, s, ta, tb, u);
  return static_cast<int>(e);
}
