// mma.sync building blocks for kernels whose tiles are row-major in shared memory with a padded row stride (an odd
// multiple of 16 bytes, which keeps ldmatrix free of bank conflicts): asynchronous copies with zero fill, fragment loads,
// the bf16 MMA, and the split of an fp32 value into two bf16 terms.
#pragma once
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

namespace pm {

__device__ __forceinline__ uint32_t ms_addr(const void* p) { return static_cast<uint32_t>(__cvta_generic_to_shared(p)); }

// 16 bytes global -> shared; with valid == false nothing is read and the destination is zeroed.
__device__ __forceinline__ void ms_cp16(uint32_t dst, const void* src, bool valid) {
  const int n = valid ? 16 : 0;
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(n) : "memory");
}
__device__ __forceinline__ void ms_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void ms_wait() {
  asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory");
}

// Bulk copy global -> shared of this CTA (16-byte aligned addresses, a multiple of 16 bytes); arrival is counted on `bar`.
__device__ __forceinline__ void ms_bulk_copy(uint32_t dst, const void* src, uint32_t bytes, uint64_t* bar) {
  asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];" ::"r"(dst), "l"(src),
               "r"(bytes), "r"(ms_addr(bar))
               : "memory");
}

__device__ __forceinline__ void ms_ldsm4(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(addr));
}
__device__ __forceinline__ void ms_ldsm4_t(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(addr));
}
__device__ __forceinline__ void ms_ldsm2(uint32_t addr, uint32_t& r0, uint32_t& r1) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x2.shared.b16 {%0,%1}, [%2];" : "=r"(r0), "=r"(r1) : "r"(addr));
}
__device__ __forceinline__ void ms_ldsm2_t(uint32_t addr, uint32_t& r0, uint32_t& r1) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x2.trans.shared.b16 {%0,%1}, [%2];" : "=r"(r0), "=r"(r1) : "r"(addr));
}
__device__ __forceinline__ void ms_mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

// Address this lane passes to ldmatrix for
//  * the 16 x 16 A operand at (r0, k0) of a tile stored [row][k]                                   (plain load)
//  * two 8-wide B operand tiles n0, n0 + 8 at k0 of a tile stored [n][k]                           (plain load)
//  * two 8-wide B operand tiles n0, n0 + 8 at k0 of a tile stored [k][n]                           (transposed load)
//  * the 16 x 16 A operand at (r0, k0) of a tile stored [k][row]                                   (transposed load)
__device__ __forceinline__ uint32_t ms_a_at(uint32_t tile, int ld, int r0, int k0, int lane) {
  return tile + static_cast<uint32_t>(((r0 + (lane & 15)) * ld + k0 + ((lane >> 4) << 3)) * 2);
}
__device__ __forceinline__ uint32_t ms_b_nt_at(uint32_t tile, int ld, int n0, int k0, int lane) {
  const int id = lane >> 3;
  return tile + static_cast<uint32_t>(((n0 + ((id >> 1) << 3) + (lane & 7)) * ld + k0 + ((id & 1) << 3)) * 2);
}
__device__ __forceinline__ uint32_t ms_b_nn_at(uint32_t tile, int ld, int k0, int n0, int lane) {
  const int id = lane >> 3;
  return tile + static_cast<uint32_t>(((k0 + ((id & 1) << 3) + (lane & 7)) * ld + n0 + ((id >> 1) << 3)) * 2);
}
__device__ __forceinline__ uint32_t ms_a_t_at(uint32_t tile, int ld, int k0, int r0, int lane) {
  const int id = lane >> 3;
  return tile + static_cast<uint32_t>(((k0 + ((id >> 1) << 3) + (lane & 7)) * ld + r0 + ((id & 1) << 3)) * 2);
}

// (a, b) -> bf16 pair of the rounded values and bf16 pair of what the rounding left (about 16 significant bits in all).
__device__ __forceinline__ void ms_split(float a, float b, uint32_t& hi, uint32_t& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
  const float2 f = __bfloat1622float2(h);
  const __nv_bfloat162 l = __floats2bfloat162_rn(a - f.x, b - f.y);
  hi = *reinterpret_cast<const uint32_t*>(&h);
  lo = *reinterpret_cast<const uint32_t*>(&l);
}

}  // namespace pm
