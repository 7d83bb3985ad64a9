// Warp-level matrix products (mma.sync m16n8k16, bf16 operands, fp32 accumulators) for small tiles whose operands are
// made in registers between products: fragments, and the split of fp32 values into two bf16 terms that keeps a product
// with an exact bf16 operand at 16 bits of mantissa.
#pragma once

#include "tw_common.cuh"

namespace tw {

__device__ __forceinline__ void ldmatrix_x4(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldmatrix_x4_trans(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void mma_bf16(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
      : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// hi + lo = (x, y) to 16 bits of mantissa
__device__ __forceinline__ void split_bf16x2(float x, float y, uint32_t& hi, uint32_t& lo) {
  hi = pack_bf16x2(x, y);
  const float2 l = fma2(unpack_bf16x2(hi), make_float2(-1.f, -1.f), make_float2(x, y));
  lo = pack_bf16x2(l.x, l.y);
}

// Element offsets of a lane's row for ldmatrix.x4 out of a row-major tile with row stride `ld`:
// A operand [m][k], 16 x 16
__device__ __forceinline__ int frag_a(int lane, int ld) { return (lane & 15) * ld + (lane >> 4) * 8; }
// A operand stored [k][m] (use the .trans load)
__device__ __forceinline__ int frag_a_t(int lane, int ld) { return ((lane & 7) + (lane >> 4) * 8) * ld + ((lane >> 3) & 1) * 8; }
// B operand stored [n][k], two 8-column blocks: registers 0, 1 and 2, 3
__device__ __forceinline__ int frag_b(int lane, int ld) { return ((lane >> 4) * 8 + (lane & 7)) * ld + ((lane >> 3) & 1) * 8; }
// B operand stored [k][n] (use the .trans load), two 8-column blocks
__device__ __forceinline__ int frag_b_t(int lane, int ld) { return (lane & 15) * ld + (lane >> 4) * 8; }

// 16-byte asynchronous copy; `bytes` < 16 fills the rest with zeros.
__device__ __forceinline__ void cp_async16(void* dst, const void* src, int bytes) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(dst)), "l"(src), "r"(bytes) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

}  // namespace tw
