// Warp-level tensor products (16-bit operands in registers, fp32 sums) and what feeds them: for tiles too small for
// tcgen05, or whose operands are made in registers from fp32 numbers.
#pragma once
#include "sm100_common.cuh"

namespace rb {

__device__ __forceinline__ void ldmatrix_x4(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void ldmatrix_x4_trans(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
// c [16 x 8] += a [16 x 16] b [16 x 8]
__device__ __forceinline__ void mma_bf16(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

// An fp32 number as the sum of two bf16 numbers (16 bits of mantissa): products of such pairs, hi hi + hi lo + lo hi, have a
// relative error near 2^-17.
struct SplitPair {
  uint32_t hi, lo;               // two numbers each
};
__device__ __forceinline__ SplitPair split2(float a, float b) {
  SplitPair s;
  s.hi = pack2<__nv_bfloat16>(a, b);
  const float2 h = unpack2<__nv_bfloat16>(s.hi);
  s.lo = pack2<__nv_bfloat16>(a - h.x, b - h.y);
  return s;
}

// 16 bytes global -> shared; !live: zeros
__device__ __forceinline__ void copy16(uint32_t dst, const void* src, bool live) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(live ? 16 : 0) : "memory");
}
__device__ __forceinline__ void copy_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void copy_wait() {
  asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory");
}

// Byte offset of 16-byte chunk c of row r in a tile whose rows have CHUNKS chunks (2, 4, or a multiple of 8), placed so that
// eight neighbouring rows' chunks c lie in different banks.
template <int CHUNKS>
__device__ __forceinline__ uint32_t tile_at(int r, int c) {
  if constexpr (CHUNKS == 2) return r * 32 + ((c ^ ((r >> 2) & 1)) << 4);
  else if constexpr (CHUNKS == 4) return r * 64 + ((c ^ ((r >> 1) & 3)) << 4);
  else return r * CHUNKS * 16 + ((c ^ (r & 7)) << 4);
}

}  // namespace rb
