// Matrix products on fp32 operands with tensor cores: every operand is the sum of two bf16 numbers, x = hi + lo (lo is the
// rounding error of hi), and a product keeps hi hi + hi lo + lo hi.  The dropped lo lo term is 2^-16 of the result, so the
// products of the chunked recurrences stay at 32-bit quality on tensor cores.
#pragma once
#include "common.cuh"

namespace b2 {

__device__ __forceinline__ void split_pair(float x0, float x1, uint32_t& hi, uint32_t& lo) {
  hi = pack_bf16x2(x0, x1);
  const float2 h = unpack_bf16x2(hi);
  lo = pack_bf16x2(x0 - h.x, x1 - h.y);
}

// D += A B for one m16n8k16 tile (A row-major, B column-major fragments)
__device__ __forceinline__ void mma_bf16(float (&d)[4], const uint32_t (&a)[4], const uint32_t (&b)[2]) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
      : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b[0]), "r"(b[1]));
}
struct FragA {
  uint32_t hi[4], lo[4];
};
struct FragB {
  uint32_t hi[2], lo[2];
};
__device__ __forceinline__ void mma_split(float (&d)[4], const FragA& a, const FragB& b) {
  mma_bf16(d, a.hi, b.hi);
  mma_bf16(d, a.hi, b.lo);
  mma_bf16(d, a.lo, b.hi);
}
// ---- split operands as two bf16 matrices (hi, lo), fragments by ldmatrix; ld in elements, rows 16-byte aligned -------------
__device__ __forceinline__ void ldsm_x4(const __nv_bfloat16* p, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(smem_u32(p))
               : "memory");
}
__device__ __forceinline__ void ldsm_x4_t(const __nv_bfloat16* p, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(smem_u32(p))
               : "memory");
}
// A fragment (m16 x k16) of a matrix stored [m][k] / [k][m]; `p` at the tile's first element
__device__ __forceinline__ void ldsm_a_mk(const __nv_bfloat16* p, int ld, int lane, uint32_t (&r)[4]) {
  ldsm_x4(p + (lane & 15) * ld + (lane >> 4) * 8, r);
}
__device__ __forceinline__ void ldsm_a_km(const __nv_bfloat16* p, int ld, int lane, uint32_t (&r)[4]) {
  ldsm_x4_t(p + ((lane & 7) + (lane >> 4) * 8) * ld + ((lane >> 3) & 1) * 8, r);
}
// B fragments of two neighbouring n8 tiles (k16 x n16), stored [n][k] / [k][n]: r[0..1] the first tile, r[2..3] the second
__device__ __forceinline__ void ldsm_b_nk(const __nv_bfloat16* p, int ld, int lane, uint32_t (&r)[4]) {
  ldsm_x4(p + ((lane & 7) + (lane >> 4) * 8) * ld + ((lane >> 3) & 1) * 8, r);
}
__device__ __forceinline__ void ldsm_b_kn(const __nv_bfloat16* p, int ld, int lane, uint32_t (&r)[4]) {
  ldsm_x4_t(p + (lane & 15) * ld + (lane >> 4) * 8, r);
}
// the two n8 tiles of `b` with the same A fragment
__device__ __forceinline__ void mma_n16(float (&d0)[4], float (&d1)[4], const uint32_t (&a)[4], const uint32_t (&b)[4]) {
  const uint32_t b0[2] = {b[0], b[1]}, b1[2] = {b[2], b[3]};
  mma_bf16(d0, a, b0);
  mma_bf16(d1, a, b1);
}
// eight fp32 values as eight hi and eight lo halves, 16 bytes each
__device__ __forceinline__ void store8_split(__nv_bfloat16* hi, __nv_bfloat16* lo, const float (&f)[8]) {
  uint4 h, l;
  split_pair(f[0], f[1], h.x, l.x);
  split_pair(f[2], f[3], h.y, l.y);
  split_pair(f[4], f[5], h.z, l.z);
  split_pair(f[6], f[7], h.w, l.w);
  *reinterpret_cast<uint4*>(hi) = h;
  *reinterpret_cast<uint4*>(lo) = l;
}

// Bulk copy global -> shared (16-byte aligned, a multiple of 16 bytes), completion on an mbarrier.
__device__ __forceinline__ void bulk_load(void* dst, const void* src, uint32_t bytes, uint64_t* bar) {
  asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];" ::"r"(smem_u32(dst)),
               "l"(src), "r"(bytes), "r"(smem_u32(bar))
               : "memory");
}

}  // namespace b2
