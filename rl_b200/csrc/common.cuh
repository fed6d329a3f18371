// Shared device helpers for the sm_100a kernels: mbarrier, TMA, tcgen05/TMEM PTX wrappers,
// bounded waits and small numeric utilities.
//
// Every wait in this library is bounded: a wait that runs out records a code in a global
// status word and returns false, so that the kernel can release what it holds (TMEM) and
// return with the CUDA context still usable.
#pragma once

#include <cuda.h>
#include <cuda_bf16.h>
#include <cuda_fp8.h>
#include <cuda_runtime.h>
#include <stdint.h>

#define RLB_API extern "C" __attribute__((visibility("default")))

// Status codes written to the status word by kernels whose wait ran out.
enum RlbStatus : int {
  RLB_OK = 0,
  RLB_ERR_WAIT_FULL = 1,        // consumer waited for a TMA-filled stage
  RLB_ERR_WAIT_EMPTY = 2,       // producer waited for a free stage
  RLB_ERR_WAIT_TMEM_FULL = 3,   // epilogue waited for an accumulator
  RLB_ERR_WAIT_TMEM_EMPTY = 4,  // MMA warp waited for a drained accumulator
  RLB_ERR_WAIT_FLAG = 5,        // wait on a flag written by another CTA or GPU
  RLB_ERR_BAD_ARG = 6,
  RLB_ERR_WAIT_PEER = 7,        // wait on a peer GPU's signal
  RLB_ERR_BOUNDS = 8,           // a build with -DRLB_DEBUG_BOUNDS saw an index outside its buffer (the access was skipped)
};

namespace rlb {

constexpr unsigned long long kWaitLimitNs = 2000000000ull;  // 2 s

__device__ __forceinline__ uint32_t smem_u32(const void* p) {
  return static_cast<uint32_t>(__cvta_generic_to_shared(p));
}

__device__ __forceinline__ unsigned long long globaltimer_ns() {
  unsigned long long t;
  asm volatile("mov.u64 %0, %%globaltimer;" : "=l"(t));
  return t;
}

__device__ __forceinline__ bool elect_one() {
  uint32_t pred = 0;
  asm volatile(
      "{\n\t"
      ".reg .pred p;\n\t"
      "elect.sync _|p, 0xffffffff;\n\t"
      "selp.u32 %0, 1, 0, p;\n\t"
      "}\n"
      : "=r"(pred));
  return pred != 0;
}

// ---------------------------------------------------------------- mbarrier
__device__ __forceinline__ void mbar_init(uint32_t bar, uint32_t count) {
  asm volatile("mbarrier.init.shared::cta.b64 [%0], %1;" ::"r"(bar), "r"(count) : "memory");
}
__device__ __forceinline__ void mbar_fence_init() {
  asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
}
__device__ __forceinline__ void fence_proxy_async() {
  asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
}
__device__ __forceinline__ void mbar_arrive_expect_tx(uint32_t bar, uint32_t bytes) {
  asm volatile("mbarrier.arrive.expect_tx.shared::cta.b64 _, [%0], %1;" ::"r"(bar), "r"(bytes)
               : "memory");
}
__device__ __forceinline__ void mbar_arrive(uint32_t bar) {
  asm volatile("mbarrier.arrive.shared::cta.b64 _, [%0];" ::"r"(bar) : "memory");
}
__device__ __forceinline__ uint32_t mbar_try_wait(uint32_t bar, uint32_t parity) {
  uint32_t done;
  asm volatile(
      "{\n\t"
      ".reg .pred p;\n\t"
      "mbarrier.try_wait.parity.shared::cta.b64 p, [%1], %2;\n\t"
      "selp.u32 %0, 1, 0, p;\n\t"
      "}\n"
      : "=r"(done)
      : "r"(bar), "r"(parity)
      : "memory");
  return done;
}

// Bounded wait. `abort_flag` is a shared-memory word that any role of the CTA sets when its own
// wait ran out, so that the others stop early instead of each waiting out the full limit.
__device__ __forceinline__ bool mbar_wait(uint32_t bar, uint32_t parity, volatile int* abort_flag,
                                          int* status, int code, unsigned long long limit_ns = kWaitLimitNs) {
  if (mbar_try_wait(bar, parity)) return true;
  const unsigned long long t0 = globaltimer_ns();
  uint32_t polls = 0;
  while (true) {
    if (mbar_try_wait(bar, parity)) return true;
    if (((++polls) & 255u) == 0u) {
      if (*abort_flag) return false;
      if (globaltimer_ns() - t0 > limit_ns) {
        *abort_flag = 1;
        if (status) atomicCAS(status, 0, code);
        return false;
      }
    }
  }
}

// ---------------------------------------------------------------- TMA (no cluster multicast anywhere)
__device__ __forceinline__ void tma_load_2d(uint32_t dst, const CUtensorMap* map, uint32_t bar, int c0,
                                            int c1) {
  asm volatile(
      "cp.async.bulk.tensor.2d.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%3, %4}], "
      "[%2];"
      :
      : "r"(dst), "l"(map), "r"(bar), "r"(c0), "r"(c1)
      : "memory");
}
__device__ __forceinline__ void tma_load_3d(uint32_t dst, const CUtensorMap* map, uint32_t bar, int c0,
                                            int c1, int c2) {
  asm volatile(
      "cp.async.bulk.tensor.3d.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%3, %4, "
      "%5}], [%2];"
      :
      : "r"(dst), "l"(map), "r"(bar), "r"(c0), "r"(c1), "r"(c2)
      : "memory");
}
__device__ __forceinline__ void tma_store_2d(const CUtensorMap* map, uint32_t src, int c0, int c1) {
  asm volatile("cp.async.bulk.tensor.2d.global.shared::cta.bulk_group [%0, {%2, %3}], [%1];"
               :
               : "l"(map), "r"(src), "r"(c0), "r"(c1)
               : "memory");
}
__device__ __forceinline__ void tma_store_commit() { asm volatile("cp.async.bulk.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void tma_store_wait_read() {
  asm volatile("cp.async.bulk.wait_group.read %0;" ::"n"(N) : "memory");
}
template <int N>
__device__ __forceinline__ void tma_store_wait() {
  asm volatile("cp.async.bulk.wait_group %0;" ::"n"(N) : "memory");
}
__device__ __forceinline__ void prefetch_tmap(const CUtensorMap* map) {
  asm volatile("prefetch.tensormap [%0];" ::"l"(map) : "memory");
}

// ---------------------------------------------------------------- tcgen05 / TMEM
__device__ __forceinline__ void tmem_alloc(uint32_t smem_dst, uint32_t ncols) {
  asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_dst),
               "r"(ncols)
               : "memory");
}
__device__ __forceinline__ void tmem_relinquish() {
  asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
}
__device__ __forceinline__ void tmem_dealloc(uint32_t taddr, uint32_t ncols) {
  asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(taddr), "r"(ncols) : "memory");
}
__device__ __forceinline__ void tc_fence_before() {
  asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
}
__device__ __forceinline__ void tc_fence_after() {
  asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
}
// D[tmem] (+)= A[smem] * B[smem]; one thread issues for the CTA.
__device__ __forceinline__ void umma_f16(uint32_t tmem_d, uint64_t desc_a, uint64_t desc_b, uint32_t idesc,
                                         uint32_t accumulate) {
  asm volatile(
      "{\n\t"
      ".reg .pred p;\n\t"
      "setp.ne.b32 p, %4, 0;\n\t"
      "tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, p;\n\t"
      "}\n"
      :
      : "r"(tmem_d), "l"(desc_a), "l"(desc_b), "r"(idesc), "r"(accumulate)
      : "memory");
}
// D[tmem] (+)= A[tmem] * B[smem]
__device__ __forceinline__ void umma_f16_ts(uint32_t tmem_d, uint32_t tmem_a, uint64_t desc_b, uint32_t idesc,
                                            uint32_t accumulate) {
  asm volatile(
      "{\n\t"
      ".reg .pred p;\n\t"
      "setp.ne.b32 p, %4, 0;\n\t"
      "tcgen05.mma.cta_group::1.kind::f16 [%0], [%1], %2, %3, p;\n\t"
      "}\n"
      :
      : "r"(tmem_d), "r"(tmem_a), "l"(desc_b), "r"(idesc), "r"(accumulate)
      : "memory");
}
// fp8 (e4m3/e5m2) operands, dense, no block scales.
__device__ __forceinline__ void umma_f8f6f4(uint32_t tmem_d, uint64_t desc_a, uint64_t desc_b, uint32_t idesc,
                                            uint32_t accumulate) {
  asm volatile(
      "{\n\t"
      ".reg .pred p;\n\t"
      "setp.ne.b32 p, %4, 0;\n\t"
      "tcgen05.mma.cta_group::1.kind::f8f6f4 [%0], %1, %2, %3, p;\n\t"
      "}\n"
      :
      : "r"(tmem_d), "l"(desc_a), "l"(desc_b), "r"(idesc), "r"(accumulate)
      : "memory");
}
// MXFP8: block scales (UE8M0, one per 32 along K) read from TMEM.
__device__ __forceinline__ void umma_mxf8(uint32_t tmem_d, uint64_t desc_a, uint64_t desc_b, uint32_t idesc,
                                          uint32_t accumulate, uint32_t tmem_sfa, uint32_t tmem_sfb) {
  asm volatile(
      "{\n\t"
      ".reg .pred p;\n\t"
      "setp.ne.b32 p, %4, 0;\n\t"
      "tcgen05.mma.cta_group::1.kind::mxf8f6f4.block_scale [%0], %1, %2, %3, [%5], [%6], p;\n\t"
      "}\n"
      :
      : "r"(tmem_d), "l"(desc_a), "l"(desc_b), "r"(idesc), "r"(accumulate), "r"(tmem_sfa), "r"(tmem_sfb)
      : "memory");
}
// smem -> TMEM copy of scale factors (32 lanes x 128 bits, replicated to the 4 lane quarters)
__device__ __forceinline__ void tmem_cp_32x128b_warpx4(uint32_t tmem_dst, uint64_t smem_desc) {
  asm volatile("tcgen05.cp.cta_group::1.32x128b.warpx4 [%0], %1;" ::"r"(tmem_dst), "l"(smem_desc) : "memory");
}
// mbarrier arrives once all tcgen05 ops issued so far by this thread have completed.
__device__ __forceinline__ void umma_commit(uint32_t bar) {
  asm volatile("tcgen05.commit.cta_group::1.mbarrier::arrive::one.shared::cluster.b64 [%0];" ::"r"(bar)
               : "memory");
}
__device__ __forceinline__ void tmem_ld_wait() { asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory"); }
__device__ __forceinline__ void tmem_st_wait() { asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory"); }

// Each thread of the warp reads 32 consecutive fp32 columns of its own TMEM lane.
__device__ __forceinline__ void tmem_ld_32x32b_x32(uint32_t taddr, uint32_t (&r)[32]) {
  asm volatile(
      "tcgen05.ld.sync.aligned.32x32b.x32.b32 "
      "{%0, %1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15, "
      "%16, %17, %18, %19, %20, %21, %22, %23, %24, %25, %26, %27, %28, %29, %30, %31}, [%32];"
      : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]),
        "=r"(r[8]), "=r"(r[9]), "=r"(r[10]), "=r"(r[11]), "=r"(r[12]), "=r"(r[13]), "=r"(r[14]), "=r"(r[15]),
        "=r"(r[16]), "=r"(r[17]), "=r"(r[18]), "=r"(r[19]), "=r"(r[20]), "=r"(r[21]), "=r"(r[22]), "=r"(r[23]),
        "=r"(r[24]), "=r"(r[25]), "=r"(r[26]), "=r"(r[27]), "=r"(r[28]), "=r"(r[29]), "=r"(r[30]), "=r"(r[31])
      : "r"(taddr)
      : "memory");
}
__device__ __forceinline__ void tmem_ld_32x32b_x16(uint32_t taddr, uint32_t (&r)[16]) {
  asm volatile(
      "tcgen05.ld.sync.aligned.32x32b.x16.b32 "
      "{%0, %1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15}, [%16];"
      : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]),
        "=r"(r[8]), "=r"(r[9]), "=r"(r[10]), "=r"(r[11]), "=r"(r[12]), "=r"(r[13]), "=r"(r[14]), "=r"(r[15])
      : "r"(taddr)
      : "memory");
}
__device__ __forceinline__ void tmem_st_32x32b_x16(uint32_t taddr, const uint32_t (&r)[16]) {
  asm volatile(
      "tcgen05.st.sync.aligned.32x32b.x16.b32 [%0], "
      "{%1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15, %16};"
      :
      : "r"(taddr), "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]),
        "r"(r[8]), "r"(r[9]), "r"(r[10]), "r"(r[11]), "r"(r[12]), "r"(r[13]), "r"(r[14]), "r"(r[15])
      : "memory");
}

// ---------------------------------------------------------------- UMMA descriptors
// Shared-memory matrix descriptor, 128-byte swizzle, sm_100 version field set.
//   K-major tile:  rows of 128 B (64 bf16), 8-row groups `sbo` bytes apart (1024 for a dense tile).
//   MN-major tile: k-rows of 128 B (64 elements along M/N); 8-k groups `sbo` bytes apart, further
//                  64-element column groups `lbo` bytes apart.
__device__ __forceinline__ uint64_t make_smem_desc_sw128(uint32_t smem_addr, uint32_t lbo_bytes,
                                                          uint32_t sbo_bytes) {
  uint64_t d = 0;
  d |= static_cast<uint64_t>((smem_addr & 0x3FFFFu) >> 4);
  d |= static_cast<uint64_t>((lbo_bytes >> 4) & 0x3FFFu) << 16;
  d |= static_cast<uint64_t>((sbo_bytes >> 4) & 0x3FFFu) << 32;
  d |= 1ull << 46;  // descriptor version for sm_100
  d |= 2ull << 61;  // SWIZZLE_128B
  return d;
}
// No-swizzle descriptor (used for scale-factor copies).
__device__ __forceinline__ uint64_t make_smem_desc_noswz(uint32_t smem_addr, uint32_t lbo_bytes,
                                                          uint32_t sbo_bytes) {
  uint64_t d = 0;
  d |= static_cast<uint64_t>((smem_addr & 0x3FFFFu) >> 4);
  d |= static_cast<uint64_t>((lbo_bytes >> 4) & 0x3FFFu) << 16;
  d |= static_cast<uint64_t>((sbo_bytes >> 4) & 0x3FFFu) << 32;
  d |= 1ull << 46;
  return d;
}
// Instruction descriptor for kind::f16 with bf16 operands and fp32 accumulation.
__host__ __device__ constexpr uint32_t make_idesc_bf16(int m, int n, bool a_mn_major, bool b_mn_major) {
  return (1u << 4)                                   // D format fp32
         | (1u << 7)                                 // A bf16
         | (1u << 10)                                // B bf16
         | (static_cast<uint32_t>(a_mn_major) << 15)
         | (static_cast<uint32_t>(b_mn_major) << 16)
         | (static_cast<uint32_t>(n >> 3) << 17)
         | (static_cast<uint32_t>(m >> 4) << 24);
}
// kind::f8f6f4 / mxf8f6f4 with e4m3 operands (format code 0), fp32 accumulation.
__host__ __device__ constexpr uint32_t make_idesc_e4m3(int m, int n) {
  return (1u << 4) | (static_cast<uint32_t>(n >> 3) << 17) | (static_cast<uint32_t>(m >> 4) << 24);
}
__host__ __device__ constexpr uint32_t make_idesc_mxf8_e4m3(int m, int n) {
  return (1u << 23)  // scale format UE8M0
         | (static_cast<uint32_t>(n >> 3) << 17) | (static_cast<uint32_t>(m >> 4) << 24);
}

// ---------------------------------------------------------------- programmatic dependent launch
// A kernel launched with rlb_launch_pdl may begin while its predecessor on the stream is still draining. It must run
// pdl_wait() before its first access to global memory (the wait returns once the predecessor has completed and its
// writes are visible); what stands before the wait (barrier init, TMEM allocation, descriptor prefetch) overlaps the
// predecessor's tail. pdl_trigger() after the wait lets the successor start the same way. Both are no-ops in a kernel
// that was launched without the attribute.
__device__ __forceinline__ void pdl_wait() { asm volatile("griddepcontrol.wait;" ::: "memory"); }
__device__ __forceinline__ void pdl_trigger() { asm volatile("griddepcontrol.launch_dependents;" ::: "memory"); }
__device__ __forceinline__ void pdl_sync() {
  pdl_wait();
  pdl_trigger();
}

// ---------------------------------------------------------------- numerics
__device__ __forceinline__ uint32_t pack_bf16x2(float lo, float hi) {
  __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
  return *reinterpret_cast<uint32_t*>(&v);
}
__device__ __forceinline__ float2 unpack_bf16x2(uint32_t v) {
  __nv_bfloat162 b = *reinterpret_cast<__nv_bfloat162*>(&v);
  return __bfloat1622float2(b);
}
__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}
__device__ __forceinline__ float warp_max(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, o));
  return v;
}
// tanh that keeps its relative accuracy near zero whatever math mode the file is compiled with: the odd Taylor series below 1/4
// (remainder under 1e-8 relative), 1 - 2 / (1 + exp(2|x|)) above.
__device__ __forceinline__ float tanh_acc(float x) {
  const float a = fabsf(x);
  if (a < 0.25f) {
    const float q = x * x;
    return x * (1.f + q * (-1.f / 3.f + q * (2.f / 15.f + q * (-17.f / 315.f + q * (62.f / 2835.f)))));
  }
  return copysignf(1.f - 2.f / (1.f + expf(2.f * a)), x);
}

// What follows a product in a layer-list model. LIN_GLU, LIN_SILU: columns 2i and 2i + 1 are gate and up of a gated unit (clamped, or silu
// without limits), the output has N / 2 columns. LIN_GELU_MUL: gelu_tanh times a table row chosen by the row's token. LIN_CAP: scale, then soft cap (cap > 0).
enum RlbLinearAct : int { LIN_NONE = 0, LIN_GLU = 1, LIN_GELU_MUL = 2, LIN_CAP = 3, LIN_SILU = 4 };
struct LinearEpi {
  const void* bias;      // [N] in the weights' type, or null: added to the product
  int act;
  float limit;           // LIN_GLU
  float scale, cap;      // LIN_CAP
  const void* table;     // LIN_GELU_MUL: [vocab, ld_table] in the weights' type, columns [table_off, table_off + table_cols)
  long long ld_table;
  int table_off, table_cols, vocab;
  const void* ids;       // [rows] int32 or int64
  int ids64;
  const float* row_scale;   // [rows] or null: the product's rows are multiplied by it first
};
__device__ __forceinline__ float clamped_glu(float g, float u, float limit) {
  g = fminf(g, limit);
  u = fminf(fmaxf(u, -limit), limit);
  return g / (1.f + expf(-1.702f * g)) * (u + 1.f);
}
__device__ __forceinline__ float gated_unit(int act, float g, float u, float limit) { return act == LIN_SILU ? g / (1.f + expf(-g)) * u : clamped_glu(g, u, limit); }
__host__ __device__ inline bool lin_gated(int act) { return act == LIN_GLU || act == LIN_SILU; }
__device__ __forceinline__ float gelu_tanh_acc(float z) { return 0.5f * z * (1.f + tanh_acc(0.7978845608028654f * (z + 0.044715f * z * z * z))); }
__device__ __forceinline__ float soft_cap(float z, float scale, float cap) {
  z *= scale;
  return cap > 0.f ? cap * tanh_acc(z / cap) : z;
}
__device__ __forceinline__ long long lin_token(const LinearEpi& e, long long row) {
  const long long id = e.ids64 ? static_cast<const long long*>(e.ids)[row] : static_cast<const int*>(e.ids)[row];
  return id < 0 || id >= e.vocab ? 0 : id;      // (the embedding reports bad ids)
}

// Epilogue of the products of layer-list models. With `x`: the fp32 residual stream x[row, col] += acc (+ e) (+ step) is
// updated in place and the output is the dynamic-tanh norm w * tanh(alpha x) + b of the new value. Without: the output is acc after
// `lin`, squared ReLU on columns >= act_from.
struct LayerEpilogue {
  float* x;
  long long ldx;             // row stride of x and e
  const float* e;
  const __nv_bfloat16* step;
  const __nv_bfloat16* alpha;
  const __nv_bfloat16* nw;
  const __nv_bfloat16* nb;
  int act_from;
  LinearEpi lin;
};
// Four consecutive columns of one row (col a multiple of 4). Gated units: the two outputs are in .x and .y.
__device__ __forceinline__ float4 layer_epilogue4(const LayerEpilogue& le, float4 v, long long row, int col, float alpha) {
  if (le.lin.bias) {
    const uint2 bv = *reinterpret_cast<const uint2*>(static_cast<const __nv_bfloat16*>(le.lin.bias) + col);
    const float2 b0 = unpack_bf16x2(bv.x), b1 = unpack_bf16x2(bv.y);
    v.x += b0.x; v.y += b0.y; v.z += b1.x; v.w += b1.y;
  }
  if (le.x) {
    float4* xp = reinterpret_cast<float4*>(le.x + row * le.ldx + col);
    const float4 old = *xp;
    v.x += old.x; v.y += old.y; v.z += old.z; v.w += old.w;
    if (le.e) {
      const float4 ev = *reinterpret_cast<const float4*>(le.e + row * le.ldx + col);
      v.x += ev.x; v.y += ev.y; v.z += ev.z; v.w += ev.w;
    }
    if (le.step) {
      const uint2 sv = *reinterpret_cast<const uint2*>(le.step + col);
      const float2 s0 = unpack_bf16x2(sv.x), s1 = unpack_bf16x2(sv.y);
      v.x += s0.x; v.y += s0.y; v.z += s1.x; v.w += s1.y;
    }
    *xp = v;
    const uint2 wv = *reinterpret_cast<const uint2*>(le.nw + col), bv = *reinterpret_cast<const uint2*>(le.nb + col);
    const float2 w0 = unpack_bf16x2(wv.x), w1 = unpack_bf16x2(wv.y), b0 = unpack_bf16x2(bv.x), b1 = unpack_bf16x2(bv.y);
    v.x = tanh_acc(alpha * v.x) * w0.x + b0.x;
    v.y = tanh_acc(alpha * v.y) * w0.y + b0.y;
    v.z = tanh_acc(alpha * v.z) * w1.x + b1.x;
    v.w = tanh_acc(alpha * v.w) * w1.y + b1.y;
  } else if (lin_gated(le.lin.act)) {
    v.x = gated_unit(le.lin.act, v.x, v.y, le.lin.limit);
    v.y = gated_unit(le.lin.act, v.z, v.w, le.lin.limit);
  } else if (le.lin.act == LIN_GELU_MUL) {
    const __nv_bfloat16* t = static_cast<const __nv_bfloat16*>(le.lin.table) + lin_token(le.lin, row) * le.lin.ld_table + le.lin.table_off;
    float* f = reinterpret_cast<float*>(&v);
#pragma unroll
    for (int i = 0; i < 4; ++i) f[i] = col + i < le.lin.table_cols ? gelu_tanh_acc(f[i]) * __bfloat162float(t[col + i]) : 0.f;
  } else if (le.lin.act == LIN_CAP) {
    v.x = soft_cap(v.x, le.lin.scale, le.lin.cap); v.y = soft_cap(v.y, le.lin.scale, le.lin.cap);
    v.z = soft_cap(v.z, le.lin.scale, le.lin.cap); v.w = soft_cap(v.w, le.lin.scale, le.lin.cap);
  } else if (col >= le.act_from) {   // act_from is a multiple of 8
    v.x = fmaxf(v.x, 0.f); v.y = fmaxf(v.y, 0.f); v.z = fmaxf(v.z, 0.f); v.w = fmaxf(v.w, 0.f);
    v.x *= v.x; v.y *= v.y; v.z *= v.z; v.w *= v.w;
  }
  return v;
}

// Block-wide sum; `red` is shared scratch of >= 32 floats. All threads get the result.
__device__ __forceinline__ float block_sum(float v, float* red) {
  const int lane = threadIdx.x & 31, w = threadIdx.x >> 5, nw = (blockDim.x + 31) >> 5;
  v = warp_sum(v);
  __syncthreads();
  if (lane == 0) red[w] = v;
  __syncthreads();
  float r = (lane < nw) ? red[lane] : 0.f;
  r = warp_sum(r);
  return r;
}
__device__ __forceinline__ float block_max(float v, float* red) {
  const int lane = threadIdx.x & 31, w = threadIdx.x >> 5, nw = (blockDim.x + 31) >> 5;
  v = warp_max(v);
  __syncthreads();
  if (lane == 0) red[w] = v;
  __syncthreads();
  float r = (lane < nw) ? red[lane] : -INFINITY;
  r = warp_max(r);
  return r;
}

}  // namespace rlb

// A product and what follows it: out = epilogue(a w^T), for rlb_linear_rows (any size, bf16 or fp32), rlb_linear_tiled and
// rlb_linear_skinny (bf16 shapes that TMA can address) and rlb_linear_grouped. Grouped: 128-row tile t of `a` belongs to expert
// tile_expert[t] (-1: unused) whose weight is w + expert * N * ldw; rlb_linear_rows may read row r of `a` from a_rows[r] (-1: zeros). row_scale
// [M] (rlb_linear_grouped and rlb_linear_rows): row r of the product is multiplied by row_scale[r] before anything else.
struct RlbLinear {
  const void* a;
  const void* w;
  void* out;
  const void* bias;
  const void* table;
  const void* ids;
  const int* tile_expert;
  const int* a_rows;
  int* status;
  const float* row_scale;
  long long lda, ldw, ldo, ld_table;
  int M, N, K, in_f32, out_f32, act, table_off, table_cols, vocab, ids64, experts, num_a_rows;
  float limit, scale, cap;
};
inline rlb::LinearEpi rlb_linear_epi(const RlbLinear& l) {
  return rlb::LinearEpi{l.bias, l.act, l.limit, l.scale, l.cap, l.table, l.ld_table, l.table_off, l.table_cols, l.vocab, l.ids, l.ids64, l.row_scale};
}

// ---------------------------------------------------------------- host helpers
typedef CUresult (*RlbEncodeTiledFn)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*,
                                     const cuuint64_t*, const cuuint32_t*, const cuuint32_t*,
                                     CUtensorMapInterleave, CUtensorMapSwizzle, CUtensorMapL2promotion,
                                     CUtensorMapFloatOOBfill);
// Resolves cuTensorMapEncodeTiled through the runtime, so that the library needs no link to libcuda.
RlbEncodeTiledFn rlb_get_encode_tiled();
// 2-D row-major tensor map: `inner` contiguous elements per row, `outer` rows, row pitch in bytes.
// Returns 0 on success.
int rlb_make_tmap_2d(CUtensorMap* map, const void* base, CUtensorMapDataType dtype, int elem_bytes,
                     uint64_t inner, uint64_t outer, uint64_t pitch_bytes, uint32_t box_inner,
                     uint32_t box_outer, CUtensorMapSwizzle swizzle);

// Whether kernels that support it are launched with programmatic stream serialization (RLB_PDL=0 turns it off).
bool rlb_pdl_enabled();
// Launches `kernel` so that it may overlap the tail of its predecessor (see pdl_wait). `extra` attributes (a cluster
// dimension, for instance) are passed through.
template <typename... KArgs, typename... Args>
inline cudaError_t rlb_launch_pdl(void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem, cudaStream_t stream,
                                  Args&&... args) {
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = grid;
  cfg.blockDim = block;
  cfg.dynamicSmemBytes = smem;
  cfg.stream = stream;
  cudaLaunchAttribute attr[1];
  attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[0].val.programmaticStreamSerializationAllowed = 1;
  cfg.attrs = attr;
  cfg.numAttrs = rlb_pdl_enabled() ? 1 : 0;
  return cudaLaunchKernelEx(&cfg, kernel, static_cast<KArgs>(args)...);
}
