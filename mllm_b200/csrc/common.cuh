// Shared device/host helpers for the sm_100a kernels of mllm_b200.
//
// Thin inline-PTX wrappers for the Blackwell primitives the kernels use:
// mbarrier (with bounded waits), TMA tiled loads (cp.async.bulk.tensor, never
// with cluster multicast), tcgen05 tensor-memory allocation / MMA / commit /
// load, proxy fences, and system-scope flag accesses for peer memory.
//
// Every wait in this file is bounded: after a fixed time it gives
// up and returns false so the calling kernel can record an error status and
// leave in an orderly way (free TMEM, let copies in flight land) instead of
// spinning forever on a shared GPU.
#pragma once

#include <cuda.h>
#include <cuda_bf16.h>
#include <cuda_fp16.h>
#include <cuda_fp8.h>
#include <cuda_runtime.h>
#include <stdint.h>

#include <type_traits>

namespace mb200 {

// ---------------------------------------------------------------------------
// status words written by kernels when a bounded wait runs out
// ---------------------------------------------------------------------------
enum KernelStatus : int {
  kStatusOk = 0,
  kStatusPipelineTimeout = 1,  // an intra-kernel mbarrier wait ran out
  kStatusPeerTimeout = 2,      // a flag written by another rank never arrived
  kStatusBadIndex = 3,         // a slot / page / expert index was out of range
};

// Waits are bounded by elapsed time, not by a poll count (how long one poll takes is up to the
// hardware): a few thousand polls without sleeping first, then polls separated by nanosleep until the
// budget on the global nanosecond timer is spent.
constexpr uint32_t kFastPolls = 2048;
constexpr uint64_t kPipelineWaitNs = 2000000000ull;  // waits between roles of one CTA: 2 s
constexpr uint64_t kPeerWaitNs = 8000000000ull;      // waits for another rank's flag: 8 s

__device__ __forceinline__ uint64_t global_ns() {
  uint64_t t;
  asm volatile("mov.u64 %0, %%globaltimer;" : "=l"(t));
  return t;
}

__device__ __forceinline__ uint32_t smem_u32(const void* p) {
  return static_cast<uint32_t>(__cvta_generic_to_shared(p));
}

__device__ __forceinline__ uint32_t lane_id() { return threadIdx.x & 31; }

__device__ __forceinline__ bool elect_one() {
  uint32_t pred = 0;
  asm volatile(
      "{\n\t.reg .pred P;\n\t.reg .b32 R;\n\t"
      "elect.sync R|P, 0xffffffff;\n\t"
      "selp.u32 %0, 1, 0, P;\n\t}"
      : "=r"(pred));
  return pred != 0;
}

// ---------------------------------------------------------------------------
// mbarrier
// ---------------------------------------------------------------------------
__device__ __forceinline__ void mbar_init(uint64_t* bar, uint32_t count) {
  asm volatile("mbarrier.init.shared::cta.b64 [%0], %1;" ::"r"(smem_u32(bar)), "r"(count));
}

__device__ __forceinline__ void fence_barrier_init() {
  asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
}

__device__ __forceinline__ void mbar_arrive(uint64_t* bar) {
  asm volatile("mbarrier.arrive.shared::cta.b64 _, [%0];" ::"r"(smem_u32(bar)) : "memory");
}

__device__ __forceinline__ void mbar_arrive_expect_tx(uint64_t* bar, uint32_t bytes) {
  asm volatile("mbarrier.arrive.expect_tx.shared::cta.b64 _, [%0], %1;" ::"r"(smem_u32(bar)), "r"(bytes)
               : "memory");
}

__device__ __forceinline__ bool mbar_try_wait(uint64_t* bar, uint32_t parity) {
  uint32_t done;
  asm volatile(
      "{\n\t.reg .pred P;\n\t"
      "mbarrier.try_wait.parity.shared::cta.b64 P, [%1], %2;\n\t"
      "selp.u32 %0, 1, 0, P;\n\t}"
      : "=r"(done)
      : "r"(smem_u32(bar)), "r"(parity)
      : "memory");
  return done != 0;
}

// Same, with an upper bound (ns) on how long the hardware may keep the thread suspended in the call.
__device__ __forceinline__ bool mbar_try_wait_hint(uint64_t* bar, uint32_t parity, uint32_t suspend_ns) {
  uint32_t done;
  asm volatile(
      "{\n\t.reg .pred P;\n\t"
      "mbarrier.try_wait.parity.shared::cta.b64 P, [%1], %2, %3;\n\t"
      "selp.u32 %0, 1, 0, P;\n\t}"
      : "=r"(done)
      : "r"(smem_u32(bar)), "r"(parity), "r"(suspend_ns)
      : "memory");
  return done != 0;
}

// Bounded wait. Returns false when the phase did not complete within kPipelineWaitNs, or as soon as
// *abort (a flag in shared memory that another role of the CTA sets when it gives up) is non-zero.
__device__ __forceinline__ bool mbar_wait(uint64_t* bar, uint32_t parity, const volatile int* abort = nullptr) {
  for (uint32_t i = 0; i < kFastPolls; ++i)
    if (mbar_try_wait(bar, parity)) return true;
  const uint64_t t0 = global_ns();
  for (uint32_t i = 0;; ++i) {
    if (mbar_try_wait_hint(bar, parity, 2000u)) return true;
    if ((i & 7u) == 7u) {
      if (abort != nullptr && *abort != 0) return false;
      if (global_ns() - t0 > kPipelineWaitNs) return false;
    }
    __nanosleep(32);
  }
}

// Bounded wait for warps that share their scheduler with working warps: backs off from the first
// failed poll so that the polling loop does not compete for issue slots.
__device__ __forceinline__ bool mbar_wait_relaxed(uint64_t* bar, uint32_t parity, uint32_t sleep_ns = 200) {
  if (mbar_try_wait(bar, parity)) return true;
  const uint64_t t0 = global_ns();
  for (uint32_t i = 0;; ++i) {
    __nanosleep(sleep_ns);
    if (mbar_try_wait_hint(bar, parity, 2000u)) return true;
    if ((i & 7u) == 7u && global_ns() - t0 > kPipelineWaitNs) return false;
  }
}

// ---------------------------------------------------------------------------
// fences between the generic proxy, the async proxy (TMA / tcgen05) and threads
// ---------------------------------------------------------------------------
__device__ __forceinline__ void fence_proxy_async_smem() {
  asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
}
__device__ __forceinline__ void fence_proxy_async_all() { asm volatile("fence.proxy.async;" ::: "memory"); }
__device__ __forceinline__ void tc_fence_before_sync() {
  asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
}
__device__ __forceinline__ void tc_fence_after_sync() {
  asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
}

// ---------------------------------------------------------------------------
// TMA: 2-D tiled load global -> shared, completion on an mbarrier.
// The x coordinate times the element size must be a multiple of 16 bytes.
// ---------------------------------------------------------------------------
__device__ __forceinline__ void tma_load_2d(void* smem_dst, const CUtensorMap* map, uint64_t* bar, int x, int y) {
  asm volatile(
      "cp.async.bulk.tensor.2d.shared::cluster.global.tile.mbarrier::complete_tx::bytes"
      " [%0], [%1, {%3, %4}], [%2];"
      ::"r"(smem_u32(smem_dst)), "l"(reinterpret_cast<uint64_t>(map)), "r"(smem_u32(bar)), "r"(x), "r"(y)
      : "memory");
}

__device__ __forceinline__ void tma_prefetch_desc(const CUtensorMap* map) {
  asm volatile("prefetch.tensormap [%0];" ::"l"(reinterpret_cast<uint64_t>(map)) : "memory");
}

// ---------------------------------------------------------------------------
// tcgen05: tensor memory and 5th-generation tensor-core MMA (single-CTA group)
// ---------------------------------------------------------------------------
// Whole-warp call. Writes the TMEM base address of `ncols` columns to *smem_out.
__device__ __forceinline__ void tmem_alloc(uint32_t* smem_out, uint32_t ncols) {
  asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(smem_out)),
               "r"(ncols)
               : "memory");
}
__device__ __forceinline__ void tmem_relinquish() {
  asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
}
__device__ __forceinline__ void tmem_dealloc(uint32_t taddr, uint32_t ncols) {
  asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(taddr), "r"(ncols) : "memory");
}

// Shared-memory matrix descriptor for a K-major operand tile stored as rows of
// 128 bytes with the 128-byte swizzle (what a TMA load with SWIZZLE_128B and a
// 128-byte inner box produces). Groups of 8 rows are 1024 bytes apart.
__device__ __forceinline__ uint64_t umma_desc_k_sw128(uint32_t smem_addr) {
  uint64_t d = 0;
  d |= static_cast<uint64_t>((smem_addr & 0x3FFFF) >> 4);  // start address, 16-byte units
  d |= static_cast<uint64_t>(1) << 16;                     // leading byte offset (unused with swizzle)
  d |= static_cast<uint64_t>(1024 >> 4) << 32;             // stride between 8-row groups
  d |= static_cast<uint64_t>(1) << 46;                     // descriptor version (sm_100)
  d |= static_cast<uint64_t>(2) << 61;                     // SWIZZLE_128B
  return d;
}

// MN-major operand (the contiguous direction is M or N, e.g. V in P*V): 128-byte
// swizzled rows of 64 16-bit elements along MN; `lbo` = byte stride between
// 64-element column blocks along MN, `sbo` = byte stride between groups of 8 K rows.
__device__ __forceinline__ uint64_t umma_desc_mn_sw128(uint32_t smem_addr, uint32_t lbo, uint32_t sbo) {
  uint64_t d = 0;
  d |= static_cast<uint64_t>((smem_addr & 0x3FFFF) >> 4);
  d |= static_cast<uint64_t>((lbo >> 4) & 0x3FFF) << 16;
  d |= static_cast<uint64_t>((sbo >> 4) & 0x3FFF) << 32;
  d |= static_cast<uint64_t>(1) << 46;
  d |= static_cast<uint64_t>(2) << 61;
  return d;
}

// Instruction descriptor. c_fmt: 1 = f32 accumulate, 2 = s32. ab_fmt: kind::f16 -> 0 f16,
// 1 bf16; kind::i8 -> 0 u8, 1 s8. *_mn_major: 0 = K-major operand, 1 = MN-major operand.
__host__ __device__ constexpr uint32_t umma_idesc(uint32_t m, uint32_t n, uint32_t c_fmt, uint32_t a_fmt,
                                                  uint32_t b_fmt, uint32_t a_mn_major = 0,
                                                  uint32_t b_mn_major = 0) {
  return (c_fmt << 4) | (a_fmt << 7) | (b_fmt << 10) | (a_mn_major << 15) | (b_mn_major << 16) |
         ((n >> 3) << 17) | ((m >> 4) << 24);
}

// D[tmem] (+)= A[smem] * B[smem]; issued by ONE thread.
__device__ __forceinline__ void umma_f16(uint32_t d_tmem, uint64_t a_desc, uint64_t b_desc, uint32_t idesc,
                                         uint32_t accumulate) {
  asm volatile(
      "{\n\t.reg .pred p;\n\t"
      "setp.ne.b32 p, %4, 0;\n\t"
      "tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, p;\n\t}"
      ::"r"(d_tmem), "l"(a_desc), "l"(b_desc), "r"(idesc), "r"(accumulate)
      : "memory");
}

__device__ __forceinline__ void umma_i8(uint32_t d_tmem, uint64_t a_desc, uint64_t b_desc, uint32_t idesc,
                                        uint32_t accumulate) {
  asm volatile(
      "{\n\t.reg .pred p;\n\t"
      "setp.ne.b32 p, %4, 0;\n\t"
      "tcgen05.mma.cta_group::1.kind::i8 [%0], %1, %2, %3, p;\n\t}"
      ::"r"(d_tmem), "l"(a_desc), "l"(b_desc), "r"(idesc), "r"(accumulate)
      : "memory");
}

// A operand from tensor memory (e.g. softmax probabilities), B from shared memory.
__device__ __forceinline__ void umma_f16_ts(uint32_t d_tmem, uint32_t a_tmem, uint64_t b_desc, uint32_t idesc,
                                            uint32_t accumulate) {
  asm volatile(
      "{\n\t.reg .pred p;\n\t"
      "setp.ne.b32 p, %4, 0;\n\t"
      "tcgen05.mma.cta_group::1.kind::f16 [%0], [%1], %2, %3, p;\n\t}"
      ::"r"(d_tmem), "r"(a_tmem), "l"(b_desc), "r"(idesc), "r"(accumulate)
      : "memory");
}

// All tcgen05 ops issued so far by this thread arrive on `bar` when they finish.
__device__ __forceinline__ void umma_commit(uint64_t* bar) {
  asm volatile("tcgen05.commit.cta_group::1.mbarrier::arrive::one.shared::cluster.b64 [%0];" ::"r"(smem_u32(bar))
               : "memory");
}

// Warp-collective: lane i of the warp reads TMEM lane (base_lane + i), 32 consecutive
// 32-bit columns starting at the column encoded in taddr.
__device__ __forceinline__ void tmem_ld_32x32(uint32_t taddr, uint32_t (&r)[32]) {
  asm volatile(
      "tcgen05.ld.sync.aligned.32x32b.x32.b32 "
      "{%0, %1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15, "
      "%16, %17, %18, %19, %20, %21, %22, %23, %24, %25, %26, %27, %28, %29, %30, %31}, [%32];"
      : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]),
        "=r"(r[8]), "=r"(r[9]), "=r"(r[10]), "=r"(r[11]), "=r"(r[12]), "=r"(r[13]), "=r"(r[14]), "=r"(r[15]),
        "=r"(r[16]), "=r"(r[17]), "=r"(r[18]), "=r"(r[19]), "=r"(r[20]), "=r"(r[21]), "=r"(r[22]),
        "=r"(r[23]), "=r"(r[24]), "=r"(r[25]), "=r"(r[26]), "=r"(r[27]), "=r"(r[28]), "=r"(r[29]),
        "=r"(r[30]), "=r"(r[31])
      : "r"(taddr)
      : "memory");
}

__device__ __forceinline__ void tmem_ld_32x16(uint32_t taddr, uint32_t (&r)[16]) {
  asm volatile(
      "tcgen05.ld.sync.aligned.32x32b.x16.b32 "
      "{%0, %1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15}, [%16];"
      : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]),
        "=r"(r[8]), "=r"(r[9]), "=r"(r[10]), "=r"(r[11]), "=r"(r[12]), "=r"(r[13]), "=r"(r[14]), "=r"(r[15])
      : "r"(taddr)
      : "memory");
}

__device__ __forceinline__ void tmem_st_32x32(uint32_t taddr, const uint32_t (&r)[32]) {
  asm volatile(
      "tcgen05.st.sync.aligned.32x32b.x32.b32 [%0], "
      "{%1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15, %16, "
      "%17, %18, %19, %20, %21, %22, %23, %24, %25, %26, %27, %28, %29, %30, %31, %32};"
      ::"r"(taddr), "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]),
        "r"(r[8]), "r"(r[9]), "r"(r[10]), "r"(r[11]), "r"(r[12]), "r"(r[13]), "r"(r[14]), "r"(r[15]),
        "r"(r[16]), "r"(r[17]), "r"(r[18]), "r"(r[19]), "r"(r[20]), "r"(r[21]), "r"(r[22]), "r"(r[23]),
        "r"(r[24]), "r"(r[25]), "r"(r[26]), "r"(r[27]), "r"(r[28]), "r"(r[29]), "r"(r[30]), "r"(r[31])
      : "memory");
}

__device__ __forceinline__ void tmem_st_32x16(uint32_t taddr, const uint32_t (&r)[16]) {
  asm volatile(
      "tcgen05.st.sync.aligned.32x32b.x16.b32 [%0], "
      "{%1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15, %16};"
      ::"r"(taddr), "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]),
        "r"(r[8]), "r"(r[9]), "r"(r[10]), "r"(r[11]), "r"(r[12]), "r"(r[13]), "r"(r[14]), "r"(r[15])
      : "memory");
}

__device__ __forceinline__ float fast_exp2(float x) {
  float y;
  asm volatile("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

__device__ __forceinline__ void tmem_ld_wait() { asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory"); }
__device__ __forceinline__ void tmem_st_wait() { asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory"); }

// ---------------------------------------------------------------------------
// flags in (peer) global memory, system scope
// ---------------------------------------------------------------------------
__device__ __forceinline__ void st_release_sys(uint32_t* p, uint32_t v) {
  asm volatile("st.release.sys.global.u32 [%0], %1;" ::"l"(p), "r"(v) : "memory");
}
__device__ __forceinline__ uint32_t ld_acquire_sys(const uint32_t* p) {
  uint32_t v;
  asm volatile("ld.acquire.sys.global.u32 %0, [%1];" : "=r"(v) : "l"(p) : "memory");
  return v;
}
__device__ __forceinline__ void red_add_release_sys(uint32_t* p, uint32_t v) {
  asm volatile("red.release.sys.global.add.u32 [%0], %1;" ::"l"(p), "r"(v) : "memory");
}
// Bounded spin until *p >= want. False when kPeerWaitNs (or `budget_ns`) went by first.  When `status`
// is given the wait also gives up as soon as that word is non-zero: once one wait of the process has
// run out (a peer is gone or far behind) the later ones return after a few hundred polls instead of
// spending their full budget each, so the host reaches its status check quickly.
__device__ __forceinline__ bool wait_flag_ge(const uint32_t* p, uint32_t want, const int* status = nullptr,
                                             uint64_t budget_ns = kPeerWaitNs) {
  for (uint32_t i = 0; i < 64; ++i)
    if (ld_acquire_sys(p) >= want) return true;
  const uint64_t t0 = global_ns();
  for (uint32_t i = 0;; ++i) {
    if (ld_acquire_sys(p) >= want) return true;
    __nanosleep(64);
    if ((i & 63u) == 63u) {
      if (status != nullptr && *reinterpret_cast<const volatile int*>(status) != 0) return false;
      if (global_ns() - t0 > budget_ns) return false;
    }
  }
}

// counters in shared memory that one role of a CTA bumps and another polls (cannot be lapped, unlike
// an mbarrier phase)
__device__ __forceinline__ void red_add_release_cta_smem(uint32_t* p, uint32_t v) {
  asm volatile("red.release.cta.shared::cta.add.u32 [%0], %1;" ::"r"(smem_u32(p)), "r"(v) : "memory");
}
__device__ __forceinline__ uint32_t ld_acquire_cta_smem(const uint32_t* p) {
  uint32_t v;
  asm volatile("ld.acquire.cta.shared::cta.u32 %0, [%1];" : "=r"(v) : "r"(smem_u32(p)) : "memory");
  return v;
}

// ---------------------------------------------------------------------------
// programmatic dependent launch: a kernel launched through launch_pdl() may start while the
// previous kernel in the stream is still draining; everything it does before pdl_wait() must
// not touch global memory written by earlier kernels (barrier set-up, tensor-memory allocation,
// descriptor prefetch are fine).  Both calls are no-ops for ordinary launches.
// ---------------------------------------------------------------------------
__device__ __forceinline__ void pdl_wait() { asm volatile("griddepcontrol.wait;" ::: "memory"); }
__device__ __forceinline__ void pdl_launch_dependents() {
  asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
}

// ---------------------------------------------------------------------------
// small numeric helpers
// ---------------------------------------------------------------------------
__device__ __forceinline__ uint32_t pack_bf16x2(float lo, float hi) {
  __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
  return *reinterpret_cast<uint32_t*>(&v);
}
// 8-bit KV cache formats (no scaling factors): 0 = the cache holds the activation dtype
constexpr int kKvSame = 0, kKvE4M3 = 1, kKvE5M2 = 2;
// two floats -> two fp8 bytes (lo in the low byte), round to nearest even, saturating at the format's largest value
__device__ __forceinline__ uint32_t pack_fp8x2(float lo, float hi, int fmt) {
  return static_cast<uint32_t>(__nv_cvt_float2_to_fp8x2(make_float2(lo, hi), __NV_SATFINITE, fmt == kKvE5M2 ? __NV_E5M2 : __NV_E4M3));
}
// two fp8 bytes (low 16 bits of `u`) -> two floats; every fp8 value is exact in fp16, bf16 and fp32
__device__ __forceinline__ float2 unpack_fp8x2(uint32_t u, int fmt) {
  const __half2_raw r = __nv_cvt_fp8x2_to_halfraw2(static_cast<__nv_fp8x2_storage_t>(u & 0xffffu), fmt == kKvE5M2 ? __NV_E5M2 : __NV_E4M3);
  return __half22float2(*reinterpret_cast<const __half2*>(&r));
}

__device__ __forceinline__ float2 unpack_bf16x2(uint32_t u) {
  __nv_bfloat162 v = *reinterpret_cast<__nv_bfloat162*>(&u);
  return __bfloat1622float2(v);
}

__device__ __forceinline__ float to_f32(__nv_bfloat16 v) { return __bfloat162float(v); }
__device__ __forceinline__ float to_f32(__half v) { return __half2float(v); }
__device__ __forceinline__ float to_f32(float v) { return v; }
template <typename T>
__device__ __forceinline__ T from_f32(float v);
template <>
__device__ __forceinline__ __nv_bfloat16 from_f32<__nv_bfloat16>(float v) {
  return __float2bfloat16_rn(v);
}
template <>
__device__ __forceinline__ __half from_f32<__half>(float v) {
  return __float2half_rn(v);
}
template <>
__device__ __forceinline__ float from_f32<float>(float v) {
  return v;
}

// tanh form of the GELU
__device__ __forceinline__ float gelu_tanh_f(float v) {
  const float k = 0.7978845608028654f;
  return 0.5f * v * (1.f + tanhf(k * (v + 0.044715f * v * v * v)));
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

// Activation of the gate half of a gated product whose result is rounded to 16 bits: SiLU, or (GELU) the tanh form of
// the GELU as v * sigmoid(2 sqrt(2 / pi) (v + 0.044715 v^3)), since 0.5 (1 + tanh(y)) = sigmoid(2 y).
template <bool GELU>
__device__ __forceinline__ float gate_act(float v) {
  if constexpr (GELU) return v / (1.f + __expf(-v * fmaf(0.07135481627f, fminf(v * v, 1e30f), 1.5957691216f)));
  return v / (1.f + __expf(-v));
}

// Gated unit with bounds: g = min(gate, limit), u = clamp(up, -limit, limit), g * sigmoid(1.702 g) * (u + 1)
__device__ __forceinline__ float clamped_gate(float gate, float up, float limit) {
  const float g = fminf(gate, limit), u = fminf(fmaxf(up, -limit), limit);
  return __fdividef(g, 1.f + __expf(-1.702f * g)) * (u + 1.f);
}

// run a statement with T bound to the 16-bit element type named by a DType value
#define MB200_DISPATCH_HALF(dt, ...)          \
  if ((dt) == ::mb200::kBF16) {               \
    using T = __nv_bfloat16;                  \
    __VA_ARGS__;                              \
  } else {                                    \
    using T = __half;                         \
    __VA_ARGS__;                              \
  }

// the same with fp32 as a third element type
#define MB200_DISPATCH_FLOAT(dt, ...)         \
  if ((dt) == ::mb200::kF32) {                \
    using T = float;                          \
    __VA_ARGS__;                              \
  } else                                      \
    MB200_DISPATCH_HALF(dt, __VA_ARGS__)

// Host side: raises `kernel`'s dynamic shared-memory limit to `bytes`, once per (kernel, device).
// cudaFuncSetAttribute acts on the current device only, so the record of what was set is kept per
// device; safe to call from several threads.
cudaError_t ensure_dynamic_smem(const void* kernel, int bytes);

// Host side, opt-in (MLLM_B200_MAX_CARVEOUT=1): asks, once per (kernel, device), for the largest shared-memory
// carve-out for `kernel`, so that every kernel of this library runs with the same split of the SM's L1 /
// shared-memory array.
void ensure_max_carveout(const void* kernel);

// Host side: launch with the programmatic-stream-serialization attribute (MLLM_B200_PDL=0 turns
// it off).  Works under stream capture: the dependency becomes a programmatic graph edge.
bool pdl_enabled();

template <typename... KArgs, typename... Args>
inline cudaError_t launch_pdl(void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem, cudaStream_t stream,
                              Args&&... args) {
  ensure_max_carveout(reinterpret_cast<const void*>(kernel));
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = grid;
  cfg.blockDim = block;
  cfg.dynamicSmemBytes = smem;
  cfg.stream = stream;
  cudaLaunchAttribute attr[1];
  attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[0].val.programmaticStreamSerializationAllowed = pdl_enabled() ? 1 : 0;
  cfg.attrs = attr;
  cfg.numAttrs = 1;
  return cudaLaunchKernelEx(&cfg, kernel, static_cast<KArgs>(args)...);
}

}  // namespace mb200
