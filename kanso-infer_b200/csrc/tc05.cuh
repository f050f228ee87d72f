// tcgen05 / TMEM wrappers and shared-memory matrix descriptors shared by the tensor-core GEMM
// kernels (inline PTX for sm_100a).
#pragma once
#include <cuda.h>  // CUtensorMap only; the encoder is looked up through the runtime

#include "common.cuh"

namespace kanso {

// ---- tcgen05 wrappers ----
__device__ __forceinline__ void tmem_alloc(uint32_t* dst_smem, uint32_t ncols) {
  asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(
                   smem_u32(dst_smem)),
               "r"(ncols)
               : "memory");
  asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
}
__device__ __forceinline__ void tmem_dealloc(uint32_t taddr, uint32_t ncols) {
  asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(taddr), "r"(ncols)
               : "memory");
}
__device__ __forceinline__ void tc_fence_before() {
  asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
}
__device__ __forceinline__ void tc_fence_after() {
  asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
}
__device__ __forceinline__ void fence_proxy_async_smem() {
  asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
}
__device__ __forceinline__ void tc_mma_f16(uint32_t d_tmem, uint64_t a_desc, uint64_t b_desc,
                                           uint32_t idesc, uint32_t accumulate) {
  asm volatile(
      "{\n.reg .pred p;\nsetp.ne.b32 p, %4, 0;\n"
      "tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, p;\n}\n" ::"r"(d_tmem),
      "l"(a_desc), "l"(b_desc), "r"(idesc), "r"(accumulate)
      : "memory");
}
// A 64-bit descriptor from its two words. Offsets between tiles of one CTA only ever change the
// start-address field in the low word (14 bits of address >> 4: shared memory ends below 256 KB).
__device__ __forceinline__ uint64_t tc_desc_join(uint32_t lo, uint32_t hi) {
  uint64_t d;
  asm("mov.b64 %0, {%1, %2};" : "=l"(d) : "r"(lo), "r"(hi));
  return d;
}
__device__ __forceinline__ void tc_commit(uint64_t* bar) {
  asm volatile("tcgen05.commit.cta_group::1.mbarrier::arrive::one.shared::cluster.b64 [%0];" ::"r"(
                   smem_u32(bar))
               : "memory");
}
// 32 lanes x 16 consecutive 32-bit columns of this warp's TMEM quarter
__device__ __forceinline__ void tmem_ld16(uint32_t taddr, uint32_t (&r)[16]) {
  asm volatile(
      "tcgen05.ld.sync.aligned.32x32b.x16.b32 {%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,"
      "%15}, [%16];"
      : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]),
        "=r"(r[7]), "=r"(r[8]), "=r"(r[9]), "=r"(r[10]), "=r"(r[11]), "=r"(r[12]), "=r"(r[13]),
        "=r"(r[14]), "=r"(r[15])
      : "r"(taddr)
      : "memory");
  asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
}

// ---- tensor-map copies into this CTA's shared memory ----
__device__ __forceinline__ void tma_load_2d(void* dst_smem, const CUtensorMap* map, int x, int y,
                                            uint64_t* bar) {
  asm volatile(
      "cp.async.bulk.tensor.2d.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, "
      "{%2, %3}], [%4];" ::"r"(smem_u32(dst_smem)),
      "l"(map), "r"(x), "r"(y), "r"(smem_u32(bar))
      : "memory");
}
__device__ __forceinline__ void tma_load_3d(void* dst_smem, const CUtensorMap* map, int x, int y,
                                            int z, uint64_t* bar) {
  asm volatile(
      "cp.async.bulk.tensor.3d.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, "
      "{%2, %3, %4}], [%5];" ::"r"(smem_u32(dst_smem)),
      "l"(map), "r"(x), "r"(y), "r"(z), "r"(smem_u32(bar))
      : "memory");
}

// Shared-memory matrix descriptor, K-major, no swizzle: core matrix = 8 rows x 16 bytes stored
// contiguously; lbo = bytes between core matrices adjacent in K, sbo = bytes between core
// matrices adjacent in the row (M/N) direction.
__device__ __forceinline__ uint64_t tc_smem_desc(uint32_t smem_addr, uint32_t lbo, uint32_t sbo) {
  uint64_t d = 0;
  d |= (uint64_t)((smem_addr >> 4) & 0x3FFF);
  d |= (uint64_t)((lbo >> 4) & 0x3FFF) << 16;
  d |= (uint64_t)((sbo >> 4) & 0x3FFF) << 32;
  d |= (uint64_t)1 << 46;  // descriptor version of this architecture
  return d;                // base offset 0, swizzle mode 0 (none)
}
// Instruction descriptor for kind::f16: f16 x f16 -> f32, both operands K-major.
__host__ __device__ inline uint32_t tc_idesc_f16(int m, int n) {
  uint32_t d = 0;
  d |= 1u << 4;                      // accumulator format f32
  d |= 0u << 7;                      // A format f16
  d |= 0u << 10;                     // B format f16
  d |= (uint32_t)(n >> 3) << 17;     // N / 8
  d |= (uint32_t)(m >> 4) << 24;     // M / 16
  return d;
}

// The same for tiles in the 128-byte swizzle as the copy engine writes them: rows of 128 bytes,
// groups of eight rows 1024 bytes apart, the tile on a 1024-byte boundary. A step of 32 bytes
// along K adds 2 to the low word.
__device__ __forceinline__ uint64_t tc_smem_desc_sw128(uint32_t smem_addr) {
  uint64_t d = 0;
  d |= (uint64_t)((smem_addr >> 4) & 0x3FFF);
  d |= (uint64_t)1 << 16;
  d |= (uint64_t)(1024 >> 4) << 32;
  d |= (uint64_t)1 << 46;
  d |= (uint64_t)2 << 61;  // 128-byte swizzle
  return d;
}
// bf16 x bf16 -> f32, both operands K-major.
__host__ __device__ inline uint32_t tc_idesc_bf16(int m, int n) {
  return tc_idesc_f16(m, n) | (1u << 7) | (1u << 10);
}

__device__ __forceinline__ void tmem_ld32(uint32_t taddr, uint32_t (&r)[32]) {
  asm volatile(
      "tcgen05.ld.sync.aligned.32x32b.x32.b32 {%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,"
      "%15,%16,%17,%18,%19,%20,%21,%22,%23,%24,%25,%26,%27,%28,%29,%30,%31}, [%32];"
      : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]),
        "=r"(r[7]), "=r"(r[8]), "=r"(r[9]), "=r"(r[10]), "=r"(r[11]), "=r"(r[12]), "=r"(r[13]),
        "=r"(r[14]), "=r"(r[15]), "=r"(r[16]), "=r"(r[17]), "=r"(r[18]), "=r"(r[19]), "=r"(r[20]),
        "=r"(r[21]), "=r"(r[22]), "=r"(r[23]), "=r"(r[24]), "=r"(r[25]), "=r"(r[26]), "=r"(r[27]),
        "=r"(r[28]), "=r"(r[29]), "=r"(r[30]), "=r"(r[31])
      : "r"(taddr)
      : "memory");
  asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
}
// The reverse of tmem_ld16.
__device__ __forceinline__ void tmem_st16(uint32_t taddr, const uint32_t (&r)[16]) {
  asm volatile(
      "tcgen05.st.sync.aligned.32x32b.x16.b32 [%16], {%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,"
      "%14,%15};" ::"r"(r[0]),
      "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]), "r"(r[8]),
      "r"(r[9]), "r"(r[10]), "r"(r[11]), "r"(r[12]), "r"(r[13]), "r"(r[14]), "r"(r[15]), "r"(taddr)
      : "memory");
  asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory");
}
// Bounded, and ends early when another role has given up.
__device__ __forceinline__ bool mbar_wait_abort(uint64_t* bar, uint32_t parity, volatile int* abort_flag) {
  for (uint32_t i = 0; i < (1u << 22); ++i) {
    if (mbar_try_wait(bar, parity)) return true;
    if ((i & 63u) == 63u && *abort_flag) break;
  }
  *abort_flag = 1;
  return false;
}

// N-major operand in the 128-byte swizzle: panels of 64 columns, `panel` bytes apart, of rows of
// 128 bytes (one per k), groups of eight rows 1024 bytes apart. 16 k further is 2048 bytes.
__device__ __forceinline__ uint64_t tc_smem_desc_nmajor(uint32_t addr, uint32_t panel) {
  uint64_t d = 0;
  d |= (uint64_t)((addr >> 4) & 0x3FFF);
  d |= (uint64_t)((panel >> 4) & 0x3FFF) << 16;
  d |= (uint64_t)(1024 >> 4) << 32;
  d |= (uint64_t)1 << 46;
  d |= (uint64_t)2 << 61;
  return d;
}

// One product over operands that lie in panels of 64 columns in the 128-byte swizzle: `steps` of
// 16 columns from the tiles at shared-memory addresses a and b on, panels a_panel and b_panel bytes
// apart. The issuing thread is alone with this: what it computes per instruction is one addition.
__device__ __forceinline__ void tc_mma_panels(uint32_t d_tmem, uint32_t a, uint32_t b,
                                              uint32_t a_panel, uint32_t b_panel, int steps,
                                              uint32_t idesc, uint32_t accumulate) {
  const uint64_t desc = tc_smem_desc_sw128(0);
  const uint32_t lo = (uint32_t)desc, hi = (uint32_t)(desc >> 32);
  uint32_t al = lo + (a >> 4), bl = lo + (b >> 4);
  for (; steps >= 4; steps -= 4) {
    tc_mma_f16(d_tmem, tc_desc_join(al, hi), tc_desc_join(bl, hi), idesc, accumulate);
#pragma unroll
    for (int j = 1; j < 4; ++j)
      tc_mma_f16(d_tmem, tc_desc_join(al + 2 * j, hi), tc_desc_join(bl + 2 * j, hi), idesc, 1);
    accumulate = 1;
    al += a_panel >> 4;
    bl += b_panel >> 4;
  }
  for (int j = 0; j < steps; ++j) {
    tc_mma_f16(d_tmem, tc_desc_join(al + 2 * j, hi), tc_desc_join(bl + 2 * j, hi), idesc,
               accumulate);
    accumulate = 1;
  }
}

}  // namespace kanso
