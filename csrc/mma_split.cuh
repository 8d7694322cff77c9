// Matrix products on fp32 operands with tensor cores: every operand is the sum of two bf16 numbers, x = hi + lo (lo is the
// rounding error of hi), and a product keeps hi hi + hi lo + lo hi.  The dropped lo lo term is 2^-16 of the result, so the
// products of the chunked recurrences stay at 32-bit quality while they run on mma.sync.
//
// In shared and global memory an operand element is one 32-bit word, hi in the low half and lo in the high half: the size of
// a float, and a fragment needs two byte permutes per pair of elements instead of a conversion.
#pragma once
#include "common.cuh"

namespace b2 {

__device__ __forceinline__ uint32_t split_word(float x) {
  const __nv_bfloat16 hi = __float2bfloat16(x);
  const __nv_bfloat16 lo = __float2bfloat16(x - __bfloat162float(hi));
  return static_cast<uint32_t>(__bfloat16_as_ushort(hi)) | (static_cast<uint32_t>(__bfloat16_as_ushort(lo)) << 16);
}
__device__ __forceinline__ uint32_t pair_hi(uint32_t w0, uint32_t w1) { return __byte_perm(w0, w1, 0x5410); }
__device__ __forceinline__ uint32_t pair_lo(uint32_t w0, uint32_t w1) { return __byte_perm(w0, w1, 0x7632); }
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
// B exact in bf16 (lo = 0)
__device__ __forceinline__ void mma_split_bx(float (&d)[4], const FragA& a, const uint32_t (&b)[2]) {
  mma_bf16(d, a.hi, b);
  mma_bf16(d, a.lo, b);
}

__device__ __forceinline__ void set_a(FragA& f, int i, uint2 w) {
  f.hi[i] = pair_hi(w.x, w.y);
  f.lo[i] = pair_lo(w.x, w.y);
}
// Fragments from word matrices.  g = lane / 4, q = lane % 4.  `p` points at element (first row, first k) of the tile.
// A stored [m][k] (ld = 8 mod 32 words: conflict-free 8-byte reads)
__device__ __forceinline__ FragA lda_mk(const uint32_t* p, int ld, int g, int q) {
  FragA f;
  set_a(f, 0, *reinterpret_cast<const uint2*>(p + g * ld + 2 * q));
  set_a(f, 1, *reinterpret_cast<const uint2*>(p + (g + 8) * ld + 2 * q));
  set_a(f, 2, *reinterpret_cast<const uint2*>(p + g * ld + 2 * q + 8));
  set_a(f, 3, *reinterpret_cast<const uint2*>(p + (g + 8) * ld + 2 * q + 8));
  return f;
}
// A stored [k][m] (ld = 4 mod 32 words: conflict-free 4-byte reads)
__device__ __forceinline__ FragA lda_km(const uint32_t* p, int ld, int g, int q) {
  FragA f;
  set_a(f, 0, make_uint2(p[(2 * q) * ld + g], p[(2 * q + 1) * ld + g]));
  set_a(f, 1, make_uint2(p[(2 * q) * ld + g + 8], p[(2 * q + 1) * ld + g + 8]));
  set_a(f, 2, make_uint2(p[(2 * q + 8) * ld + g], p[(2 * q + 9) * ld + g]));
  set_a(f, 3, make_uint2(p[(2 * q + 8) * ld + g + 8], p[(2 * q + 9) * ld + g + 8]));
  return f;
}
// B stored [n][k]
__device__ __forceinline__ FragB ldb_nk(const uint32_t* p, int ld, int g, int q) {
  FragB f;
  const uint2 a = *reinterpret_cast<const uint2*>(p + g * ld + 2 * q), b = *reinterpret_cast<const uint2*>(p + g * ld + 2 * q + 8);
  f.hi[0] = pair_hi(a.x, a.y); f.lo[0] = pair_lo(a.x, a.y);
  f.hi[1] = pair_hi(b.x, b.y); f.lo[1] = pair_lo(b.x, b.y);
  return f;
}
// B stored [k][n]
__device__ __forceinline__ FragB ldb_kn(const uint32_t* p, int ld, int g, int q) {
  FragB f;
  const uint32_t a = p[(2 * q) * ld + g], b = p[(2 * q + 1) * ld + g], c = p[(2 * q + 8) * ld + g], d = p[(2 * q + 9) * ld + g];
  f.hi[0] = pair_hi(a, b); f.lo[0] = pair_lo(a, b);
  f.hi[1] = pair_hi(c, d); f.lo[1] = pair_lo(c, d);
  return f;
}
// Two neighbouring n8 tiles of a plain bf16 matrix stored [k][n] (ld in elements, rows 16-byte aligned), 16 rows of k.
__device__ __forceinline__ void ldb_kn_bf16_x2(const __nv_bfloat16* p, int ld, int lane, uint32_t (&b0)[2], uint32_t (&b1)[2]) {
  const uint32_t addr = smem_u32(p + (lane & 15) * ld + (lane >> 4) * 8);
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(b0[0]), "=r"(b0[1]), "=r"(b1[0]), "=r"(b1[1])
               : "r"(addr)
               : "memory");
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

__device__ __forceinline__ void cp_async16(void* dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_async_wait() {
  asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory");
}

}  // namespace b2
