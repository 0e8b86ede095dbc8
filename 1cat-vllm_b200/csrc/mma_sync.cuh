// Warp-level bf16 products (mma.sync m16n8k16, fp32 accumulators) and the shared-memory fragment loads for them. Operand tiles are row-major with
// a pitch in elements whose byte size is 16 modulo 128 or so, so that the eight rows of a fragment fall into different bank groups.
// Operands that are 32-bit by definition enter as two bf16 planes, the rounded value and what rounding took from it (`split2`).
#pragma once
#include "common.cuh"

namespace oc {

__device__ __forceinline__ void ldsm_x4(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void ldsm_x4_t(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void mma16816(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ uint32_t pack2(float lo, float hi) {
  __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
  return *reinterpret_cast<uint32_t*>(&v);
}
// two neighbouring values as a rounded pair and the pair of remainders
__device__ __forceinline__ void split2(float a, float b, uint32_t& hi, uint32_t& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
  hi = *reinterpret_cast<const uint32_t*>(&h);
  const float2 f = __bfloat1622float2(h);
  lo = pack2(a - f.x, b - f.y);
}
// A fragment (16 x 16) of a tile stored [m][k]: element (m0 + i, k0 + j)
__device__ __forceinline__ uint32_t a_addr(uint32_t base, int pitch, int m0, int k0, int lane) {
  return base + (uint32_t)(((m0 + (lane & 7) + ((lane >> 3) & 1) * 8) * pitch + k0 + (lane >> 4) * 8) * 2);
}
// B fragments of two adjacent n tiles from a tile stored [n][k]: r0, r1 = tile n0; r2, r3 = tile n0 + 8
__device__ __forceinline__ uint32_t bnk_addr(uint32_t base, int pitch, int n0, int k0, int lane) {
  return base + (uint32_t)(((n0 + (lane & 7) + (lane >> 4) * 8) * pitch + k0 + ((lane >> 3) & 1) * 8) * 2);
}
// the same from a tile stored [k][n], loaded transposed
__device__ __forceinline__ uint32_t bkn_addr(uint32_t base, int pitch, int k0, int n0, int lane) {
  return base + (uint32_t)(((k0 + (lane & 7) + ((lane >> 3) & 1) * 8) * pitch + n0 + (lane >> 4) * 8) * 2);
}
// A fragment of X^T where X is stored [k][m], loaded transposed: element (m0 + i, k0 + j) = X[k0 + j][m0 + i]
__device__ __forceinline__ uint32_t at_addr(uint32_t base, int pitch, int m0, int k0, int lane) {
  return base + (uint32_t)(((k0 + (lane & 7) + (lane >> 4) * 8) * pitch + m0 + ((lane >> 3) & 1) * 8) * 2);
}
// 16 bytes global -> shared, asynchronously; `bytes` of them are read, the rest becomes zero
__device__ __forceinline__ void cp_async16(uint32_t dst, const void* src, int bytes) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(bytes) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

}  // namespace oc
