// Warp-level bfloat16 products (mma.sync m16n8k16, fp32 accumulators) for tiles too small or too
// entangled with fp32 arithmetic for tcgen05: fragment loads from row-major shared memory, the product,
// and the split of fp32 values into two bfloat16 terms.
#pragma once

#include <cuda_bf16.h>

#include "common.cuh"

namespace ctdk {

__device__ __forceinline__ void ldsm4(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(addr)
               : "memory");
}
__device__ __forceinline__ void ldsm4_trans(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(addr)
               : "memory");
}
// A fragment (16 rows m0.., 16 columns k0..) of a row-major [m][k] tile with row pitch ld.
__device__ __forceinline__ void ldsm_a(uint32_t (&r)[4], const __nv_bfloat16* s, int ld, int m0, int k0, int lane) {
  const int m = m0 + ((lane >> 3) & 1) * 8 + (lane & 7), k = k0 + (lane >> 4) * 8;
  ldsm4(r, smem_u32(s + m * ld + k));
}
// The same fragment of a tile stored [k][m].
__device__ __forceinline__ void ldsm_a_trans(uint32_t (&r)[4], const __nv_bfloat16* s, int ld, int m0, int k0, int lane) {
  const int k = k0 + (lane >> 4) * 8 + (lane & 7), m = m0 + ((lane >> 3) & 1) * 8;
  ldsm4_trans(r, smem_u32(s + k * ld + m));
}
// B fragments of two neighbouring column tiles (16 rows k0.., 16 columns n0..) of a tile stored [n][k]:
// r[0], r[1] for columns n0..n0+7, r[2], r[3] for the next eight.
__device__ __forceinline__ void ldsm_b(uint32_t (&r)[4], const __nv_bfloat16* s, int ld, int k0, int n0, int lane) {
  const int n = n0 + (lane >> 4) * 8 + (lane & 7), k = k0 + ((lane >> 3) & 1) * 8;
  ldsm4(r, smem_u32(s + n * ld + k));
}
// The same of a row-major [k][n] tile.
__device__ __forceinline__ void ldsm_b_trans(uint32_t (&r)[4], const __nv_bfloat16* s, int ld, int k0, int n0, int lane) {
  const int k = k0 + ((lane >> 3) & 1) * 8 + (lane & 7), n = n0 + (lane >> 4) * 8;
  ldsm4_trans(r, smem_u32(s + k * ld + n));
}
__device__ __forceinline__ void mma_bf16(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// (x, y) as packed bfloat16 pairs hi + lo with hi + lo within 2^-16 of the values.
__device__ __forceinline__ void split_bf16x2(float x, float y, uint32_t& hi, uint32_t& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
  const float2 f = __bfloat1622float2(h);
  const __nv_bfloat162 l = __floats2bfloat162_rn(x - f.x, y - f.y);
  hi = *reinterpret_cast<const uint32_t*>(&h);
  lo = *reinterpret_cast<const uint32_t*>(&l);
}
__device__ __forceinline__ void cp_async16(void* dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_async_wait() {
  asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory");
}
__device__ __forceinline__ void cp_async_wait_all() { cp_async_wait<0>(); }

}  // namespace ctdk
