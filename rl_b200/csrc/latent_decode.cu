// Decode form of latent attention, bf16 in / fp32 accumulate. Every row is one query token with its own page table. Keys and values are
// never decompressed: all heads of a row read the same cached latent rows.
//
//   heads GEMM   q_lat[t, h, :] = q[t, h, :dim] W_uk[h]         the unrotated query carried into the latent space (tcgen05, W_uk MN-major)
//   attention    one CTA per (row, group of HN heads, split of the context): a tile of 64 latent rows is both K and V and is fetched once,
//                by TMA, into a ring of 64-column chunks
//   combine      joins the splits
//   heads GEMM   y[t, h, :] = o[t, h, :] W_uv[h]^T (tcgen05), times sigmoid(gate) where the output columns hold gates
//
// The attention products have 16 or 32 rows (heads) only. A tcgen05.mma with 128 latent rows on the M side and 16 heads on the N side
// occupies its pipe for about 120 cycles (measured: the issuing thread is held that long per instruction, although the tensor pipe is
// active for 32), which makes the 52 instructions of a 64-token tile take twice the time its 72 KB take to arrive. m16n8k16 warp
// MMAs fit 16 heads exactly, keep the queries and the output in registers, and leave the kernel bound by the stream.
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
constexpr int LD_TOK = 64;                   // tokens per tile
constexpr int LD_CHUNK = LD_TOK * 128;       // 64 tokens x 64 columns: 8 KB, 128-byte swizzle
constexpr int LD_MAX_RING = 24;              // chunks in the ring
constexpr int LD_HALF = 5;                   // 64-column groups of a latent row that one half of the warps multiplies (rows up to 640)
constexpr int LD_WARPS = 8;
constexpr int LD_THREADS = 32 * LD_WARPS + 128;
constexpr int LD_REGS_LOAD = 24, LD_REGS_COMPUTE = 240;   // per thread after the split; 384 threads are launched with 168 each
static_assert(128 * LD_REGS_LOAD + 256 * LD_REGS_COMPUTE <= LD_THREADS * 168, "the split exceeds what the block was launched with");
constexpr int LD_PSTRIDE = LD_TOK + 8;       // weights: 144-byte rows, free of bank conflicts
constexpr int LD_SSTRIDE = LD_TOK + 4;       // partial scores (fp32)
constexpr float LD_LOG2E = 1.4426950408889634f;

struct LdParams {
  const int* block_table;
  int bt_stride;
  const int* seq_lens;
  int heads, rank, width, block_size;
  int chunks;         // 64-column groups of a latent row
  int ring;           // chunk slots
  float scale_log2;
  int num_splits;
  const __nv_bfloat16* q;   // [rows, heads, width]
  float* part_o;      // [rows, heads, splits, rank]
  float* part_ml;     // [rows, heads, splits, 2]
  __nv_bfloat16* out; // [rows, heads * rank]
  int* status;
};

__device__ __forceinline__ void ld_bar_sync() { asm volatile("bar.sync 1, 256;" ::: "memory"); }
__device__ __forceinline__ void ldsm_x4(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void ldsm_x4_trans(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(addr)
               : "memory");
}
__device__ __forceinline__ void mma_16x8x16(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
               : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

// HN heads (16 or 32) of one row against one split of its context. Two warpgroups compute; the third one's first thread requests the
// chunks by TMA (a request waits for the queue whenever memory is the limit, so it must not stand in a computing warp's way) and gives
// its registers to the others.
//   scores   warp = (head group of 16, token group, half of the latent row): its queries stay in registers as A fragments, the two
//            halves' partial scores meet in shared memory
//   softmax  256 / HN threads per head, running maximum and sum in registers
//   PV       warp w owns output columns 64 w .. 64 w + 63 of all heads in registers
template <int HN>
__global__ void __launch_bounds__(LD_THREADS, 1)
latent_decode_kernel(const __grid_constant__ CUtensorMap tmap_lat, LdParams p) {
  constexpr int HG = HN / 16, TG = 4 / HG, TW = LD_TOK / TG;   // head groups, token groups, tokens per group
  constexpr int PER = 256 / HN, TPT = LD_TOK / PER;            // softmax threads per head, tokens per thread
  extern __shared__ uint8_t smem_raw[];
  uint8_t* ring = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  float* sred = reinterpret_cast<float*>(ring + p.ring * LD_CHUNK);                          // [2][HN][LD_SSTRIDE]
  __nv_bfloat16* pw = reinterpret_cast<__nv_bfloat16*>(sred + 2 * HN * LD_SSTRIDE);           // [HN][LD_PSTRIDE]
  float* fac = reinterpret_cast<float*>(pw + HN * LD_PSTRIDE);                                // [HN] rescale factors, at the end 1 / sum
  uint64_t* full = reinterpret_cast<uint64_t*>(fac + HN);
  uint64_t* tile_done = full + LD_MAX_RING;      // [2], tiles alternate
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tile_done + 2);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (threadIdx.x == 0) {
    for (int s = 0; s < LD_MAX_RING; ++s) mbar_init(smem_u32(full + s), 1);
    for (int s = 0; s < 2; ++s) mbar_init(smem_u32(tile_done + s), LD_WARPS);
    *abort_flag = 0;
    mbar_fence_init();
    fence_proxy_async();
    prefetch_tmap(&tmap_lat);
  }
  __syncthreads();
  pdl_sync();

  const int row = blockIdx.x, h0 = blockIdx.y * HN, split = blockIdx.z;
  const int bs = p.block_size;
  const int len = min(p.seq_lens[row], p.bt_stride * bs);
  const int per_split = ((len + p.num_splits - 1) / p.num_splits + LD_TOK - 1) / LD_TOK * LD_TOK;
  const int t_begin = split * per_split, t_end = min(len, t_begin + per_split);
  const int n_tiles = t_end > t_begin ? (t_end - t_begin + LD_TOK - 1) / LD_TOK : 0;

  if (warp >= LD_WARPS) {
    asm volatile("setmaxnreg.dec.sync.aligned.u32 %0;" ::"n"(LD_REGS_LOAD));
    if (warp == LD_WARPS && lane == 0) {
      const int* bt = p.block_table + static_cast<long long>(row) * p.bt_stride;
      const int box = bs < LD_TOK ? bs : LD_TOK, nbox = LD_TOK / box;
      int slot = 0, free_chunks = p.ring, freed = 0;      // tiles that have been given back
      bool ok = true;
      for (int i = 0; i < n_tiles && ok; ++i) {
        int crow[4];
#pragma unroll
        for (int b = 0; b < 4; ++b) {
          // tokens past the end read pages of valid (if unrelated) content; their scores are masked before the softmax
          const int t = t_begin + i * LD_TOK + b * box;
          crow[b] = b < nbox ? bt[min(t / bs, p.bt_stride - 1)] * bs + t % bs : 0;
        }
        for (int c = 0; c < p.chunks; ++c) {
          if (free_chunks == 0) {
            if (!mbar_wait(smem_u32(tile_done + (freed & 1)), (freed >> 1) & 1, abort_flag, p.status, RLB_ERR_WAIT_EMPTY)) {
              ok = false;
              break;
            }
            ++freed;
            free_chunks = p.chunks;
          }
          --free_chunks;
          const uint32_t bar = smem_u32(full + slot), dst = smem_u32(ring + slot * LD_CHUNK);
          mbar_arrive_expect_tx(bar, LD_CHUNK);
#pragma unroll
          for (int b = 0; b < 4; ++b)
            if (b < nbox) tma_load_2d(dst + b * box * 128, &tmap_lat, bar, c * 64, crow[b]);
          if (++slot == p.ring) slot = 0;
        }
      }
    }
    return;
  }
  asm volatile("setmaxnreg.inc.sync.aligned.u32 %0;" ::"n"(LD_REGS_COMPUTE));

  const int kh = warp & 1, tg = (warp >> 1) % TG, hg = (warp >> 1) / TG;
  const int c_begin = kh ? (p.chunks + 1) / 2 : 0, c_end = kh ? p.chunks : (p.chunks + 1) / 2;
  // query fragments of this warp's heads and half of the row
  uint32_t qf[LD_HALF * 4][4];
  {
    const int r0 = h0 + hg * 16 + (lane >> 2);
#pragma unroll
    for (int k = 0; k < LD_HALF * 4; ++k) {
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int h = r0 + (e & 1) * 8, col = c_begin * 64 + k * 16 + (lane & 3) * 2 + (e >> 1) * 8;
        qf[k][e] = (h < p.heads && col < p.width && k < (c_end - c_begin) * 4)
                       ? *reinterpret_cast<const uint32_t*>(p.q + (static_cast<long long>(row) * p.heads + h) * p.width + col)
                       : 0u;
      }
    }
  }
  float o[HG][8][4];
#pragma unroll
  for (int g = 0; g < HG; ++g)
#pragma unroll
    for (int n = 0; n < 8; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) o[g][n][e] = 0.f;
  const int sh = threadIdx.x / PER, st0 = (threadIdx.x % PER) * TPT;     // softmax: this thread's head and first token
  float m_run = -INFINITY, l_run = 0.f;
  const bool owns = warp * 64 < p.rank;
  const uint32_t p_addr = smem_u32(pw);
  int base = 0;             // ring slot of the tile's first chunk
  uint32_t phase = 0;       // its phase
  bool ok = true;

  for (int i = 0; i < n_tiles; ++i) {
    // ---- scores. A wait that ran out clears `ok` but leaves no loop early: every warp passes the same barriers.
    float s[TW / 8][4];
#pragma unroll
    for (int n = 0; n < TW / 8; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) s[n][e] = 0.f;
#pragma unroll
    for (int cc = 0; cc < LD_HALF; ++cc) {
      if (c_begin + cc < c_end) {
        int slot = base + c_begin + cc;
        const bool wrap = slot >= p.ring;
        if (wrap) slot -= p.ring;
        ok = ok && mbar_wait(smem_u32(full + slot), phase ^ (wrap ? 1u : 0u), abort_flag, p.status, RLB_ERR_WAIT_FULL);
        __syncwarp();
        const uint32_t chunk = smem_u32(ring + slot * LD_CHUNK);
#pragma unroll
        for (int kk = 0; kk < 4; ++kk) {
#pragma unroll
          for (int t = 0; t < TW / 16; ++t) {
            const int tok = tg * TW + t * 16 + (lane & 7) + ((lane >> 4) << 3), piece = 2 * kk + ((lane >> 3) & 1);
            uint32_t b[4];
            ldsm_x4(chunk + tok * 128 + ((piece ^ (tok & 7)) << 4), b);
            mma_16x8x16(s[2 * t], qf[cc * 4 + kk], b[0], b[1]);
            mma_16x8x16(s[2 * t + 1], qf[cc * 4 + kk], b[2], b[3]);
          }
        }
      }
    }
    {
      float* dst = sred + (kh * HN + hg * 16 + (lane >> 2)) * LD_SSTRIDE + tg * TW + (lane & 3) * 2;
#pragma unroll
      for (int n = 0; n < TW / 8; ++n) {
        *reinterpret_cast<float2*>(dst + n * 8) = make_float2(s[n][0], s[n][1]);
        *reinterpret_cast<float2*>(dst + 8 * LD_SSTRIDE + n * 8) = make_float2(s[n][2], s[n][3]);
      }
    }
    ld_bar_sync();
    // ---- softmax
    {
      float v[TPT];
      float mx = -INFINITY;
#pragma unroll
      for (int k = 0; k < TPT; k += 4) {
        const float4 a = *reinterpret_cast<const float4*>(sred + sh * LD_SSTRIDE + st0 + k), b = *reinterpret_cast<const float4*>(sred + (HN + sh) * LD_SSTRIDE + st0 + k);
        const float t[4] = {a.x + b.x, a.y + b.y, a.z + b.z, a.w + b.w};
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          v[k + e] = t_begin + i * LD_TOK + st0 + k + e < t_end ? t[e] * p.scale_log2 : -INFINITY;
          mx = fmaxf(mx, v[k + e]);
        }
      }
#pragma unroll
      for (int off = PER / 2; off > 0; off >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, off));
      const float mn = fmaxf(m_run, mx);       // finite: every tile holds a valid token
      const float f = m_run == -INFINITY ? 0.f : exp2f(m_run - mn);
      m_run = mn;
      float sum = 0.f;
#pragma unroll
      for (int k = 0; k < TPT; k += 2) {
        const float a = exp2f(v[k] - mn), b = exp2f(v[k + 1] - mn);
        sum += a + b;
        *reinterpret_cast<uint32_t*>(pw + sh * LD_PSTRIDE + st0 + k) = pack_bf16x2(a, b);
      }
      l_run = l_run * f + sum;                 // this thread's tokens; joined at the end
      if (threadIdx.x % PER == 0) fac[sh] = f;
    }
    ld_bar_sync();
    // ---- PV
    if (owns) {
      int slot = base + warp;
      if (slot >= p.ring) slot -= p.ring;
      const uint32_t chunk = smem_u32(ring + slot * LD_CHUNK);     // (its scores have been read, so it is there)
#pragma unroll
      for (int g = 0; g < HG; ++g) {
        const float f0 = fac[g * 16 + (lane >> 2)], f1 = fac[g * 16 + (lane >> 2) + 8];
#pragma unroll
        for (int n = 0; n < 8; ++n) {
          o[g][n][0] *= f0;
          o[g][n][1] *= f0;
          o[g][n][2] *= f1;
          o[g][n][3] *= f1;
        }
      }
#pragma unroll
      for (int ks = 0; ks < LD_TOK / 16; ++ks) {
        uint32_t a[HG][4];
#pragma unroll
        for (int g = 0; g < HG; ++g)
          ldsm_x4(p_addr + ((g * 16 + (lane & 15)) * LD_PSTRIDE + ks * 16 + (lane >> 4) * 8) * 2, a[g]);
        const int tok = ks * 16 + (lane & 15);
#pragma unroll
        for (int n2 = 0; n2 < 4; ++n2) {
          uint32_t b[4];
          ldsm_x4_trans(chunk + tok * 128 + (((n2 * 2 + (lane >> 4)) ^ (tok & 7)) << 4), b);
#pragma unroll
          for (int g = 0; g < HG; ++g) {
            mma_16x8x16(o[g][2 * n2], a[g], b[0], b[1]);
            mma_16x8x16(o[g][2 * n2 + 1], a[g], b[2], b[3]);
          }
        }
      }
    }
    __syncwarp();
    if (lane == 0) mbar_arrive(smem_u32(tile_done + (i & 1)));
    base += p.chunks;
    if (base >= p.ring) {
      base -= p.ring;
      phase ^= 1;
    }
  }
#pragma unroll
  for (int off = PER / 2; off > 0; off >>= 1) l_run += __shfl_xor_sync(0xffffffffu, l_run, off);
  ld_bar_sync();            // the last factors have been read
  if (threadIdx.x % PER == 0) {
    fac[sh] = p.num_splits > 1 ? 1.f : ((ok && l_run > 0.f) ? 1.f / l_run : 0.f);
    if (p.num_splits > 1 && h0 + sh < p.heads) {
      const long long k = ((static_cast<long long>(row) * p.heads + h0 + sh) * p.num_splits + split) * 2;
      p.part_ml[k] = m_run;
      p.part_ml[k + 1] = l_run;
    }
  }
  ld_bar_sync();
  if (!owns) return;
#pragma unroll
  for (int g = 0; g < HG; ++g) {
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int hl = g * 16 + half * 8 + (lane >> 2);
      if (h0 + hl >= p.heads) continue;
      const float f = fac[hl];
      const long long rh = static_cast<long long>(row) * p.heads + h0 + hl;
#pragma unroll
      for (int n = 0; n < 8; ++n) {
        const int d = warp * 64 + n * 8 + (lane & 3) * 2;
        if (d >= p.rank) continue;
        const float a = o[g][n][half * 2] * f, b = o[g][n][half * 2 + 1] * f;
        if (p.num_splits == 1)
          *reinterpret_cast<uint32_t*>(p.out + rh * p.rank + d) = pack_bf16x2(a, b);
        else
          *reinterpret_cast<float2*>(p.part_o + (rh * p.num_splits + split) * p.rank + d) = make_float2(a, b);
      }
    }
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
int launch_latent_decode(const CUtensorMap& tl, LdParams p, int rows, cudaStream_t s) {
  const int fixed = 2 * HN * LD_SSTRIDE * 4 + HN * LD_PSTRIDE * 2 + HN * 4 + (LD_MAX_RING + 2) * 8 + 16 + 1024;
  p.ring = (227 * 1024 - fixed) / LD_CHUNK;
  if (p.ring > LD_MAX_RING) p.ring = LD_MAX_RING;
  if (p.ring > 3 * p.chunks) p.ring = 3 * p.chunks;
  if (p.ring < p.chunks || p.chunks > 2 * LD_HALF) return -2;
  const int smem = p.ring * LD_CHUNK + fixed;
  static int configured = 0;
  if (smem > configured) {
    cudaError_t e = cudaFuncSetAttribute(latent_decode_kernel<HN>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e != cudaSuccess) return static_cast<int>(e);
    configured = smem;
  }
  return static_cast<int>(rlb_launch_pdl(latent_decode_kernel<HN>, dim3(rows, (p.heads + HN - 1) / HN, p.num_splits), dim3(LD_THREADS), smem, s, tl, p));
}
}  // namespace

// Shapes the decode kernels take: dim a multiple of 16, rot_dim, vdim, rank of 8, rank at most 512 and a latent row of at most 640.
RLB_API int rlb_latent_decode_supported(int dim, int rot_dim, int vdim, int rank, int width, int block_size) {
  return dim > 0 && dim % 16 == 0 && rot_dim % 8 == 0 && vdim > 0 && vdim % 8 == 0 && rank % 8 == 0 && rank <= 512 && width % 8 == 0 && width <= 640 &&
         (block_size == 16 || block_size == 32 || block_size == 64 || (block_size > 0 && block_size % 128 == 0));
}

// q_lat [rows, heads, width] (bf16): columns [rank, width) hold the rotated query part (zero padded) already; columns [0, rank) are
// computed here from the queries q [rows, q_width]. o_lat [rows, heads * rank] is scratch. part_o / part_ml: scratch for num_splits > 1. out (may
// be the rows of q): head outputs from column mix_off, gated by what stands there when `gated`.
RLB_API int rlb_latent_decode(const void* q, int rows, long long ldq, int q_width, int q_off, void* out, long long ldo, int mix_off, int gated, int heads, int dim, int rot_dim, int vdim,
                              int rank, int width, int block_size, int num_blocks, const void* cache, const int* block_table, int bt_stride,
                              const int* seq_lens, const void* kv_up, float scale, void* q_lat, void* o_lat, int num_splits, float* part_o,
                              float* part_ml, int* status, void* stream) {
  if (rows <= 0) return 0;
  if (!rlb_latent_decode_supported(dim, rot_dim, vdim, rank, width, block_size) || heads > 65535 || num_splits < 1 || num_splits > 32) return -2;
  if (ldq % 8 || ldo % 8 || q_off % 8 || mix_off % 8 || (dim + rot_dim) % 8 || (num_splits > 1 && (!part_o || !part_ml))) return -2;
  if ((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(out) | reinterpret_cast<uintptr_t>(cache) | reinterpret_cast<uintptr_t>(kv_up) | reinterpret_cast<uintptr_t>(q_lat) |
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
  CUtensorMap ta, tb, tl;
  int rc = rlb_make_tmap_2d(&ta, q, BF, 2, q_width, rows, ldq * 2, HG_K, HG_T, SW);
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
  d.width = width;
  d.chunks = (width + 63) / 64;
  d.q = static_cast<const __nv_bfloat16*>(q_lat);
  d.scale_log2 = scale * LD_LOG2E;
  d.num_splits = num_splits;
  d.part_o = part_o;
  d.part_ml = part_ml;
  d.out = static_cast<__nv_bfloat16*>(o_lat);
  d.status = status;
  const int hn = heads > 16 ? 32 : 16;
  rc = rlb_make_tmap_2d(&tl, cache, BF, 2, width, static_cast<uint64_t>(num_blocks) * block_size, static_cast<uint64_t>(width) * 2, 64,
                        block_size < LD_TOK ? block_size : LD_TOK, SW);
  if (rc) return -100 - rc;
  rc = hn == 32 ? launch_latent_decode<32>(tl, d, rows, s) : launch_latent_decode<16>(tl, d, rows, s);
  if (rc) return rc;
  if (num_splits > 1) {
    e = rlb_launch_pdl(latent_combine_kernel, dim3(static_cast<unsigned>(rows) * heads), dim3(128), 0, s, part_o, part_ml, num_splits, rank,
                       static_cast<__nv_bfloat16*>(o_lat));
    if (e != cudaSuccess) return static_cast<int>(e);
  }
  rc = rlb_make_tmap_2d(&ta, o_lat, BF, 2, static_cast<uint64_t>(heads) * rank, rows, static_cast<uint64_t>(heads) * rank * 2, HG_K, HG_T, SW);
  if (!rc) rc = rlb_make_tmap_2d(&tb, kv_up, BF, 2, rank, static_cast<uint64_t>(heads) * (dim + vdim), static_cast<uint64_t>(rank) * 2, HG_K, 32, SW);
  if (rc) return -100 - rc;
  HeadsGemm u{rows, vdim, rank, 0, rank, heads * dim, vdim, static_cast<__nv_bfloat16*>(out), ldo, mix_off, vdim, gated, status};
  e = rlb_launch_pdl(gemm_heads_kernel<false, 32, 8>, dim3((vdim + 31) / 32, (rows + HG_T - 1) / HG_T, heads), dim3(HG_THREADS), HgCfg<32, 8>::SMEM, s, ta, tb, u);
  return static_cast<int>(e);
}
