// Warp-level tensor-core helpers (ldmatrix, mma.sync m16n8k16 bf16 with fp32 accumulation, cp.async) for kernels whose tiles
// are too small or too interleaved with per-element work for a tcgen05 tile.
//
// Fragment coordinates: g = lane >> 2, t = lane & 3.  A (16 x 16): a0 (row g, columns 2t, 2t + 1), a1 (row g + 8), a2 (row g,
// columns + 8), a3 (row g + 8, columns + 8).  C (16 x 8): c0, c1 (row g, columns 2t, 2t + 1), c2, c3 (row g + 8).
#pragma once
#include "rb_common.cuh"

namespace rb {

__device__ __forceinline__ void wm_ldsm_x4(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void wm_ldsm_x4_t(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void wm_mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// Addresses for the operand fragments of a row-major bf16 matrix in shared memory (`pitch` in elements):
// A rows [r0, r0 + 16), columns [k0, k0 + 16)
__device__ __forceinline__ uint32_t wm_a(uint32_t base, int pitch, int r0, int k0, int lane) {
  return base + ((r0 + (lane & 15)) * pitch + k0 + (lane >> 4) * 8) * 2;
}
// A = transpose of rows [k0, k0 + 16), columns [r0, r0 + 16): for wm_ldsm_x4_t
__device__ __forceinline__ uint32_t wm_a_t(uint32_t base, int pitch, int r0, int k0, int lane) {
  return base + ((k0 + (lane & 7) + ((lane >> 4) & 1) * 8) * pitch + r0 + ((lane >> 3) & 1) * 8) * 2;
}
// B of two n-tiles from rows [n0, n0 + 16) (the n index), columns [k0, k0 + 16): registers 0, 1 and 2, 3
__device__ __forceinline__ uint32_t wm_b(uint32_t base, int pitch, int n0, int k0, int lane) {
  return base + ((n0 + (lane & 7) + ((lane >> 4) << 3)) * pitch + k0 + ((lane >> 3) & 1) * 8) * 2;
}
// B of two n-tiles from rows [k0, k0 + 16) (the k index), columns [n0, n0 + 16): for wm_ldsm_x4_t
__device__ __forceinline__ uint32_t wm_b_t(uint32_t base, int pitch, int n0, int k0, int lane) {
  return base + ((k0 + (lane & 7) + ((lane >> 3) & 1) * 8) * pitch + n0 + (lane >> 4) * 8) * 2;
}
// 16-byte asynchronous global -> shared copy; !ok writes zeros and reads nothing
__device__ __forceinline__ void wm_cp16(uint32_t dst, const void* src, bool ok) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(ok ? 16 : 0) : "memory");
}
__device__ __forceinline__ void wm_cp_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void wm_cp_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

__device__ __forceinline__ float wm_ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// v = hi + lo with both halves bf16: about 16 bits of v
__device__ __forceinline__ void wm_split(float a, float b, uint32_t& hi, uint32_t& lo) {
  hi = pack_bf16x2(a, b);
  const float2 h = unpack_bf16x2(hi);
  lo = pack_bf16x2(a - h.x, b - h.y);
}

}  // namespace rb
