// Warp-level mma.sync m16n8k16 (bf16 in, f32 accumulate) with its ldmatrix loads, for tiles that are too small for a
// 128-row tcgen05 tile.  Fragment layout, g = lane / 4, c = lane % 4:
//   A (16 x 16)  a0 = (row g, k 2c, 2c+1), a1 = (row g + 8, same k), a2 = (row g, k 2c+8, 2c+9), a3 = (row g + 8, ...)
//   B (16 x 8)   b0 = (k 2c, 2c+1, col g), b1 = (k 2c+8, 2c+9, col g)
//   C (16 x 8)   c0, c1 = (row g, cols 2c, 2c+1), c2, c3 = (row g + 8, same cols)
// So the C fragments of two neighbouring 8-column tiles, packed to bf16 pairs, are the A fragment of a 16-deep product.
#pragma once

#include "common.cuh"

namespace teeny {

__device__ __forceinline__ void mma_bf16_16816(float (&d)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3,
                                               uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
      : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
      : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void ldsm_x4(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void ldsm_x4_trans(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// Soft-capped score in the log2 domain: log2(e) cap tanh(s scale / cap), through tanh(y) = 1 - 2 / (1 + exp(2 y)).  `two_y` =
// 2 log2(e) scale / cap, cap_l2 = log2(e) cap; absolute error about 1e-7 cap.
__device__ __forceinline__ float softcap_log2(float s, float two_y, float cap_l2) {
  float r;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(ex2(s * two_y) + 1.0f));
  return fmaf(-2.0f * cap_l2, r, cap_l2);
}
__device__ __forceinline__ float sigmoid_f(float x) { return 1.0f / (1.0f + expf(-x)); }

// Two f32 values as bf16 pairs: x = hi + lo up to 2^-17 of |x|.
__device__ __forceinline__ void split_bf16x2(float x, float y, uint32_t& hi, uint32_t& lo) {
  hi = pack_bf16x2(x, y);
  lo = pack_bf16x2(x - bf16_lo(hi), y - bf16_hi(hi));
}

}  // namespace teeny
