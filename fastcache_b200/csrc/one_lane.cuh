// Instructions issued by one lane of a warp that is converged otherwise: only the instruction is predicated, loops, addresses and
// descriptors stay warp-uniform.  (Inside a long divergent single-lane branch every TMA load and MMA
// costs hundreds of cycles of issue; a few MMAs in a row stand best in an `if (elect_one())` of their own.)
// `issue`: 1 on the issuing lane, 0 on the others.
#pragma once
#include "ptx.cuh"

namespace fc {

__device__ __forceinline__ void one_commit(uint64_t* bar, uint32_t issue) {
  asm volatile(
      "{\n\t.reg .pred q;\n\tsetp.ne.b32 q, %1, 0;\n\t"
      "@q tcgen05.commit.cta_group::1.mbarrier::arrive::one.shared::cluster.b64 [%0];\n\t}"
      ::"r"(smem_u32(bar)), "r"(issue)
      : "memory");
}
__device__ __forceinline__ void one_expect(uint64_t* bar, uint32_t bytes, uint32_t issue) {
  asm volatile(
      "{\n\t.reg .pred q;\n\tsetp.ne.b32 q, %2, 0;\n\t"
      "@q mbarrier.arrive.expect_tx.shared::cta.b64 _, [%0], %1;\n\t}"
      ::"r"(smem_u32(bar)), "r"(bytes), "r"(issue)
      : "memory");
}
__device__ __forceinline__ void one_load_2d(void* dst, const CUtensorMap* m, uint64_t* bar, int x, int y, uint32_t issue) {
  asm volatile(
      "{\n\t.reg .pred q;\n\tsetp.ne.b32 q, %5, 0;\n\t"
      "@q cp.async.bulk.tensor.2d.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%3, %4}], [%2];\n\t}"
      ::"r"(smem_u32(dst)), "l"(reinterpret_cast<uint64_t>(m)), "r"(smem_u32(bar)), "r"(x), "r"(y), "r"(issue)
      : "memory");
}
__device__ __forceinline__ void one_load_3d(void* dst, const CUtensorMap* m, uint64_t* bar, int x, int y, int z, uint32_t issue) {
  asm volatile(
      "{\n\t.reg .pred q;\n\tsetp.ne.b32 q, %6, 0;\n\t"
      "@q cp.async.bulk.tensor.3d.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%3, %4, %5}], [%2];\n\t}"
      ::"r"(smem_u32(dst)), "l"(reinterpret_cast<uint64_t>(m)), "r"(smem_u32(bar)), "r"(x), "r"(y), "r"(z), "r"(issue)
      : "memory");
}
// a wait by every lane, with one answer
__device__ __forceinline__ bool warp_wait(uint64_t* bar, uint32_t parity, uint32_t* status, uint32_t code) {
  return __all_sync(0xffffffffu, mbar_wait(bar, parity, status, code)) != 0;
}

}  // namespace fc
