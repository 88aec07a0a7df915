// The 5th-generation tensor cores: shared-memory operand tiles, TMEM, and the instructions a block needs to run
// matrix products with accumulators (and, where wanted, the A operand) in TMEM. One-block form (cta_group::1) only.
//
// Operand tiles are bf16 with 128-byte rows of 64 elements and the 128-byte swizzle: element (row, e) of a tile sits in
// block e / 64 (blocks are rows * 128 bytes apart), row `row`, 16-byte chunk (e % 64 / 8) ^ (row % 8). The same bytes
// serve as
//   a K-major operand:  rows = M or N, elements along K     (scores: q and k rows)
//   an MN-major one:    rows = K, elements along M or N     (values: v rows)
#pragma once
#include "mma.cuh"
#include "ring.cuh"

namespace djv {

// byte offset of a 16-byte chunk in a tile of `rows` rows; chunk = e / 8
__device__ __forceinline__ uint32_t sw128_offset(int rows, int row, int chunk) {
  return (uint32_t)((chunk >> 3) * rows * 128 + row * 128 + (((chunk & 7) ^ (row & 7)) << 4));
}

// Shared-memory matrix descriptor, 128-byte swizzle: start address, leading and stride byte offsets (16-byte units),
// descriptor version 1 of this architecture, layout 2.
__device__ __forceinline__ uint64_t sw128_desc(uint32_t addr, uint32_t leading_bytes, uint32_t stride_bytes) {
  return (uint64_t)((addr >> 4) & 0x3fff) | (uint64_t)((leading_bytes >> 4) & 0x3fff) << 16 |
         (uint64_t)((stride_bytes >> 4) & 0x3fff) << 32 | 1ull << 46 | 2ull << 61;
}
// K-major: groups of 8 rows are 1024 bytes apart; step `k16` along K advances 32 bytes inside a 64-element block
__device__ __forceinline__ uint64_t desc_k_major(uint32_t tile, int rows, int k16) {
  return sw128_desc(tile + (uint32_t)(k16 >> 2) * rows * 128 + (k16 & 3) * 32, 16, 1024);
}
// MN-major: 64-element blocks are rows * 128 bytes apart, groups of 8 K rows 1024; step `k16` takes 16 rows
__device__ __forceinline__ uint64_t desc_mn_major(uint32_t tile, int rows, int k16) {
  return sw128_desc(tile + (uint32_t)k16 * 2048, (uint32_t)rows * 128, 1024);
}
// Instruction descriptor: fp32 accumulators, bf16 operands, M x N
__host__ __device__ constexpr uint32_t mma_idesc(int M, int N, bool a_mn_major, bool b_mn_major) {
  return 1u << 4 | 1u << 7 | 1u << 10 | (a_mn_major ? 1u << 15 : 0u) | (b_mn_major ? 1u << 16 : 0u) |
         (uint32_t)(N >> 3) << 17 | (uint32_t)(M >> 4) << 24;
}

// ---- TMEM allocation (whole warp) ----
__device__ __forceinline__ void tmem_alloc(uint32_t *smem_slot, uint32_t columns) {
  asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(smem_slot)),
               "r"(columns)
               : "memory");
  asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;");
}
__device__ __forceinline__ void tmem_dealloc(uint32_t addr, uint32_t columns) {
  asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(addr), "r"(columns) : "memory");
}

// ---- products (one thread) ----
__device__ __forceinline__ void mma_ss(uint32_t d, uint64_t a, uint64_t b, uint32_t idesc, bool accumulate) {
  asm volatile(
      "{\n"
      ".reg .pred p;\n"
      "setp.ne.b32 p, %4, 0;\n"
      "tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, p;\n"
      "}\n" ::"r"(d),
      "l"(a), "l"(b), "r"(idesc), "r"((uint32_t)accumulate)
      : "memory");
}
__device__ __forceinline__ void mma_ts(uint32_t d, uint32_t a_tmem, uint64_t b, uint32_t idesc, bool accumulate) {
  asm volatile(
      "{\n"
      ".reg .pred p;\n"
      "setp.ne.b32 p, %4, 0;\n"
      "tcgen05.mma.cta_group::1.kind::f16 [%0], [%1], %2, %3, p;\n"
      "}\n" ::"r"(d),
      "r"(a_tmem), "l"(b), "r"(idesc), "r"((uint32_t)accumulate)
      : "memory");
}
// one arrival on the barrier when every product issued so far by this thread is complete
__device__ __forceinline__ void mma_commit(uint64_t *bar) {
  asm volatile("tcgen05.commit.cta_group::1.mbarrier::arrive::one.shared::cluster.b64 [%0];" ::"r"(smem_u32(bar))
               : "memory");
}
// ordering of tcgen05 accesses around block barriers and mbarrier waits
__device__ __forceinline__ void tmem_fence_before() { asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory"); }
__device__ __forceinline__ void tmem_fence_after() { asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory"); }
__device__ __forceinline__ void tmem_wait_ld() { asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory"); }
__device__ __forceinline__ void tmem_wait_st() { asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory"); }

// ---- TMEM <-> registers (whole warp; a warp reaches lanes 32 * (warp % 4) .. + 31) ----
// 32 lanes x 32 columns: column c of this thread's lane in r[c]
__device__ __forceinline__ void tmem_ld32(uint32_t (&r)[32], uint32_t addr) {
  asm volatile(
      "tcgen05.ld.sync.aligned.32x32b.x32.b32 {%0, %1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15, "
      "%16, %17, %18, %19, %20, %21, %22, %23, %24, %25, %26, %27, %28, %29, %30, %31}, [%32];"
      : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]), "=r"(r[8]), "=r"(r[9]), "=r"(r[10]), "=r"(r[11]), "=r"(r[12]), "=r"(r[13]), "=r"(r[14]), "=r"(r[15]), "=r"(r[16]), "=r"(r[17]), "=r"(r[18]), "=r"(r[19]), "=r"(r[20]), "=r"(r[21]), "=r"(r[22]), "=r"(r[23]), "=r"(r[24]), "=r"(r[25]), "=r"(r[26]), "=r"(r[27]), "=r"(r[28]), "=r"(r[29]), "=r"(r[30]), "=r"(r[31])
      : "r"(addr));
}
// 32 lanes x 16 columns
__device__ __forceinline__ void tmem_ld16(uint32_t (&r)[16], uint32_t addr) {
  asm volatile(
      "tcgen05.ld.sync.aligned.32x32b.x16.b32 {%0, %1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15}, [%16];"
      : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]), "=r"(r[8]), "=r"(r[9]), "=r"(r[10]), "=r"(r[11]), "=r"(r[12]), "=r"(r[13]), "=r"(r[14]), "=r"(r[15])
      : "r"(addr));
}
// 32 lanes x 16 columns
__device__ __forceinline__ void tmem_st16(uint32_t addr, const uint32_t (&r)[16]) {
  asm volatile(
      "tcgen05.st.sync.aligned.32x32b.x16.b32 [%0], {%1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15, %16};" ::"r"(addr),
      "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]), "r"(r[8]), "r"(r[9]), "r"(r[10]), "r"(r[11]), "r"(r[12]), "r"(r[13]), "r"(r[14]), "r"(r[15])
      : "memory");
}
}  // namespace djv
