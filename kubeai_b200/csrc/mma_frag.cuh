// Warp-level tensor-core fragments (mma.sync m16n8k16, bf16 in, fp32 out) and the exact splitting of fp32 operands into
// bf16 terms, for the kernels whose tiles are too small or too private to a warp for tcgen05.
//
// Fragment layout, lane = 4 g + t:  A (16 x 16): a0 = (row g, k 2t, 2t+1), a1 = (row g+8, same k), a2 = (row g, k 2t+8, 2t+9),
// a3 = (row g+8, same).  B (16 x 8): b0 = (k 2t, 2t+1, column g), b1 = (k 2t+8, 2t+9, column g).  C (16 x 8): c0, c1 = (row g,
// columns 2t, 2t+1), c2, c3 = (row g+8, same columns).  Two neighbouring C tiles (columns n .. n+15) are, packed to bf16, the
// A fragment of a product that contracts over those columns.
#pragma once
#include <cuda_bf16.h>
#include <stdint.h>

namespace b200 {
namespace frag {

__device__ __forceinline__ uint32_t smem_addr(const void* p) { return static_cast<uint32_t>(__cvta_generic_to_shared(p)); }
__device__ __forceinline__ void ldsm_x4(uint32_t* r, uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldsm_x4_trans(uint32_t* r, uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void mma(float* c, const uint32_t* a, uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void cp_async16(uint32_t dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_async_wait_all() { asm volatile("cp.async.wait_all;" ::: "memory"); }

// Addresses a lane gives to ldsm_x4 on a row-major bf16 tile with leading dimension ld (elements):
// a_addr: rows r0 .. r0+15 as the rows of A, columns c0 .. c0+15 as k
// b_addr: rows r0 .. r0+15 as 16 columns of B (two 8-column tiles: registers 0, 1 and 2, 3), columns c0 .. c0+15 as k
// at_addr (transposing load): rows r0 .. r0+15 as k, columns c0 .. c0+15 as the rows of A
// bt_addr (transposing load): rows r0 .. r0+15 as k, columns c0 .. c0+15 as 16 columns of B (registers 0, 1 and 2, 3)
__device__ __forceinline__ uint32_t a_addr(const __nv_bfloat16* p, int ld, int r0, int c0, int lane) {
  return smem_addr(p + (r0 + (lane & 7) + 8 * ((lane >> 3) & 1)) * ld + c0 + 8 * (lane >> 4));
}
__device__ __forceinline__ uint32_t b_addr(const __nv_bfloat16* p, int ld, int r0, int c0, int lane) {
  return smem_addr(p + (r0 + (lane & 7) + 8 * (lane >> 4)) * ld + c0 + 8 * ((lane >> 3) & 1));
}
__device__ __forceinline__ uint32_t at_addr(const __nv_bfloat16* p, int ld, int r0, int c0, int lane) {
  return smem_addr(p + (r0 + (lane & 7) + 8 * (lane >> 4)) * ld + c0 + 8 * ((lane >> 3) & 1));
}
__device__ __forceinline__ uint32_t bt_addr(const __nv_bfloat16* p, int ld, int r0, int c0, int lane) {
  return smem_addr(p + (r0 + (lane & 7) + 8 * ((lane >> 3) & 1)) * ld + c0 + 8 * (lane >> 4));
}

__device__ __forceinline__ uint32_t pack(float lo, float hi) {
  const __nv_bfloat162 b = __floats2bfloat162_rn(lo, hi);
  return *reinterpret_cast<const uint32_t*>(&b);
}
__device__ __forceinline__ float low(uint32_t v) { return __uint_as_float(v << 16); }
__device__ __forceinline__ float high(uint32_t v) { return __uint_as_float(v & 0xffff0000u); }

// (x, y) = (t0 + t1 + t2) as three packed bf16 pairs: 24 bits of every number, so a product with an exact bf16 operand that
// accumulates all three terms carries an fp32 operand's full precision
__device__ __forceinline__ void split3(float x, float y, uint32_t* t0, uint32_t* t1, uint32_t* t2) {
  *t0 = pack(x, y);
  x -= low(*t0); y -= high(*t0);
  *t1 = pack(x, y);
  x -= low(*t1); y -= high(*t1);
  *t2 = pack(x, y);
}

}  // namespace frag
}  // namespace b200
