// Two CTAs of a cluster that work on one tile (cta_group::2): addresses and barriers of the other CTA, tensor memory,
// copies counted on a barrier of either CTA, products of 256 rows.
#pragma once
#include "sm100_common.cuh"

namespace rb {

__device__ __forceinline__ uint32_t cluster_ctarank() {
  uint32_t r;
  asm volatile("mov.u32 %0, %%cluster_ctarank;" : "=r"(r));
  return r;
}
// shared::cluster address of the same shared-memory offset in CTA `rank` of this cluster
__device__ __forceinline__ uint32_t map_to_cta(uint32_t smem_addr, uint32_t rank) {
  uint32_t r;
  asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(r) : "r"(smem_addr), "r"(rank));
  return r;
}
__device__ __forceinline__ void cluster_sync_all() {
  asm volatile("barrier.cluster.arrive.release.aligned;\n\tbarrier.cluster.wait.acquire.aligned;" ::: "memory");
}
__device__ __forceinline__ void mbar_arrive_cluster(uint32_t cluster_addr) {
  asm volatile("mbarrier.arrive.release.cluster.shared::cluster.b64 _, [%0];" ::"r"(cluster_addr) : "memory");
}
// The same without ordering this CTA's other writes for the other CTA, which costs about a thousand cycles: for what lies in
// tensor memory, ordered by the tcgen05 fences on both sides.
__device__ __forceinline__ void mbar_arrive_tmem_pair(uint32_t cluster_addr) {
  asm volatile("mbarrier.arrive.shared::cluster.b64 _, [%0];" ::"r"(cluster_addr) : "memory");
}
__device__ __forceinline__ void st_cluster_u32(uint32_t cluster_addr, uint32_t v) {
  asm volatile("st.shared::cluster.u32 [%0], %1;" ::"r"(cluster_addr), "r"(v) : "memory");
}
// try_wait that also orders against writes released by a thread of the OTHER CTA of the pair
__device__ __forceinline__ bool mbar_try_wait_cluster(uint32_t bar, uint32_t parity) {
  uint32_t ok;
  asm volatile(
      "{\n\t.reg .pred P;\n\t"
      "mbarrier.try_wait.parity.acquire.cluster.shared::cta.b64 P, [%1], %2;\n\t"
      "selp.u32 %0, 1, 0, P;\n\t}\n"
      : "=r"(ok)
      : "r"(bar), "r"(parity)
      : "memory");
  return ok != 0;
}
__device__ __forceinline__ bool mbar_wait_cluster(uint32_t bar, uint32_t parity, volatile int* abort_flag,
                                                  int* status, int code) {
  if (mbar_try_wait_cluster(bar, parity)) return true;
  uint64_t t0 = globaltimer_ns();
  uint32_t spins = 0;
  while (true) {
    if (mbar_try_wait_cluster(bar, parity)) return true;
    if ((++spins & 0x3ff) == 0) {
      if (*abort_flag) return false;
      if (globaltimer_ns() - t0 > RB_WAIT_BUDGET_NS) {
        record_error(status, code);
        *abort_flag = 1;
        return false;
      }
    }
  }
}
__device__ __forceinline__ void tmem_alloc_2cta(uint32_t dst_smem, uint32_t ncols) {
  asm volatile("tcgen05.alloc.cta_group::2.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(dst_smem), "r"(ncols) : "memory");
}
__device__ __forceinline__ void tmem_relinquish_2cta() {
  asm volatile("tcgen05.relinquish_alloc_permit.cta_group::2.sync.aligned;" ::: "memory");
}
__device__ __forceinline__ void tmem_dealloc_2cta(uint32_t taddr, uint32_t ncols) {
  asm volatile("tcgen05.dealloc.cta_group::2.sync.aligned.b32 %0, %1;" ::"r"(taddr), "r"(ncols) : "memory");
}
// copy of one box into this CTA's shared memory; the bytes are counted on `bar_cluster_addr`, which
// may be a barrier of the other CTA of the pair
__device__ __forceinline__ void tma_load_2d_pair(uint32_t dst, const CUtensorMap* m, uint32_t bar_cluster_addr,
                                                 int x, int y) {
  asm volatile(
      "cp.async.bulk.tensor.2d.cta_group::2.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%3, "
      "%4}], [%2];" ::"r"(dst),
      "l"(reinterpret_cast<uint64_t>(m)), "r"(bar_cluster_addr), "r"(x), "r"(y)
      : "memory");
}
// whole warp, uniform arguments; one elected lane issues
__device__ __forceinline__ void umma_f16_pair_w(uint32_t tmem_d, uint64_t adesc, uint64_t bdesc, uint32_t idesc,
                                                uint32_t accumulate) {
  asm volatile(
      "{\n\t.reg .pred p, e;\n\telect.sync _|e, 0xffffffff;\n\tsetp.ne.b32 p, %4, 0;\n\t"
      "@e tcgen05.mma.cta_group::2.kind::f16 [%0], %1, %2, %3, {%5, %5, %5, %5, %5, %5, %5, %5}, p;\n\t}\n" ::"r"(tmem_d),
      "l"(adesc), "l"(bdesc), "r"(idesc), "r"(accumulate), "r"(0u)
      : "memory");
}
// the barrier (anywhere in the cluster) receives one arrival once every MMA issued so far is complete
__device__ __forceinline__ void umma_commit_pair_w(uint32_t bar_cluster_addr) {
  asm volatile(
      "{\n\t.reg .pred e;\n\telect.sync _|e, 0xffffffff;\n\t"
      "@e tcgen05.commit.cta_group::2.mbarrier::arrive::one.shared::cluster.b64 [%0];\n\t}\n" ::"r"(bar_cluster_addr)
      : "memory");
}
// three-dimensional form of tma_load_2d_pair
__device__ __forceinline__ void tma_load_3d_pair(uint32_t dst, const CUtensorMap* m, uint32_t bar_cluster_addr, int x, int y, int z) {
  asm volatile(
      "cp.async.bulk.tensor.3d.cta_group::2.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%3, "
      "%4, %5}], [%2];" ::"r"(dst),
      "l"(reinterpret_cast<uint64_t>(m)), "r"(bar_cluster_addr), "r"(x), "r"(y), "r"(z)
      : "memory");
}
// Four products of one accumulator whose operands advance by constants, as umma_f16_w4 and umma_f16_ts_w4 for one CTA.
template <int A_STEP, int B_STEP>
__device__ __forceinline__ void umma_f16_pair_w4(uint32_t tmem_d, uint64_t adesc, uint64_t bdesc, uint32_t idesc, uint32_t accumulate) {
  asm volatile(
      "{\n\t.reg .pred p, e, t;\n\t.reg .b64 a1, a2, a3, b1, b2, b3;\n\t"
      "elect.sync _|e, 0xffffffff;\n\tsetp.ne.b32 p, %4, 0;\n\tsetp.eq.u32 t, 0, 0;\n\t"
      "add.s64 a1, %1, %6;\n\tadd.s64 a2, %1, %7;\n\tadd.s64 a3, %1, %8;\n\t"
      "add.s64 b1, %2, %9;\n\tadd.s64 b2, %2, %10;\n\tadd.s64 b3, %2, %11;\n\t"
      "@e tcgen05.mma.cta_group::2.kind::f16 [%0], %1, %2, %3, {%5, %5, %5, %5, %5, %5, %5, %5}, p;\n\t"
      "@e tcgen05.mma.cta_group::2.kind::f16 [%0], a1, b1, %3, {%5, %5, %5, %5, %5, %5, %5, %5}, t;\n\t"
      "@e tcgen05.mma.cta_group::2.kind::f16 [%0], a2, b2, %3, {%5, %5, %5, %5, %5, %5, %5, %5}, t;\n\t"
      "@e tcgen05.mma.cta_group::2.kind::f16 [%0], a3, b3, %3, {%5, %5, %5, %5, %5, %5, %5, %5}, t;\n\t}\n" ::"r"(tmem_d),
      "l"(adesc), "l"(bdesc), "r"(idesc), "r"(accumulate), "r"(0u), "n"(A_STEP), "n"(2 * A_STEP), "n"(3 * A_STEP),
      "n"(B_STEP), "n"(2 * B_STEP), "n"(3 * B_STEP)
      : "memory");
}
template <int A_STEP, int B_STEP>
__device__ __forceinline__ void umma_f16_ts_pair_w4(uint32_t tmem_d, uint32_t tmem_a, uint64_t bdesc, uint32_t idesc, uint32_t accumulate) {
  asm volatile(
      "{\n\t.reg .pred p, e, t;\n\t.reg .b32 a1, a2, a3;\n\t.reg .b64 b1, b2, b3;\n\t"
      "elect.sync _|e, 0xffffffff;\n\tsetp.ne.b32 p, %4, 0;\n\tsetp.eq.u32 t, 0, 0;\n\t"
      "add.s32 a1, %1, %6;\n\tadd.s32 a2, %1, %7;\n\tadd.s32 a3, %1, %8;\n\t"
      "add.s64 b1, %2, %9;\n\tadd.s64 b2, %2, %10;\n\tadd.s64 b3, %2, %11;\n\t"
      "@e tcgen05.mma.cta_group::2.kind::f16 [%0], [%1], %2, %3, {%5, %5, %5, %5, %5, %5, %5, %5}, p;\n\t"
      "@e tcgen05.mma.cta_group::2.kind::f16 [%0], [a1], b1, %3, {%5, %5, %5, %5, %5, %5, %5, %5}, t;\n\t"
      "@e tcgen05.mma.cta_group::2.kind::f16 [%0], [a2], b2, %3, {%5, %5, %5, %5, %5, %5, %5, %5}, t;\n\t"
      "@e tcgen05.mma.cta_group::2.kind::f16 [%0], [a3], b3, %3, {%5, %5, %5, %5, %5, %5, %5, %5}, t;\n\t}\n" ::"r"(tmem_d),
      "r"(tmem_a), "l"(bdesc), "r"(idesc), "r"(accumulate), "r"(0u), "n"(A_STEP), "n"(2 * A_STEP), "n"(3 * A_STEP),
      "n"(B_STEP), "n"(2 * B_STEP), "n"(3 * B_STEP)
      : "memory");
}

}  // namespace rb
