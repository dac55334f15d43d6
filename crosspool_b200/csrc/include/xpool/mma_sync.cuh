// Warp-level matrix fragments (mma.sync m16n8k16, bf16 inputs, fp32 sums) for recurrences whose state has to be scaled and
// split again between chunks, and asynchronous copies of their tiles.
//   A operand, rows x k:   lane holds rows g, g + 8 and columns 2 q, 2 q + 1 (+ 8) with g = lane / 4, q = lane % 4
//   accumulator:           lane holds rows g, g + 8 and columns 2 q, 2 q + 1
#pragma once

#include <cuda_bf16.h>
#include <stdint.h>

#include "xpool/sm100.cuh"

namespace xpool {
namespace frag {

__device__ __forceinline__ void ldsm4(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(addr));
}
__device__ __forceinline__ void ldsm4t(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(addr));
}
__device__ __forceinline__ void mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// (x, y) as a bf16 pair of packed values: hi + lo carries 16 mantissa bits
__device__ __forceinline__ void split2(float x, float y, uint32_t& hi, uint32_t& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
  const float2 f = __bfloat1622float2(h);
  const __nv_bfloat162 l = __floats2bfloat162_rn(x - f.x, y - f.y);
  hi = *reinterpret_cast<const uint32_t*>(&h);
  lo = *reinterpret_cast<const uint32_t*>(&l);
}
__device__ __forceinline__ float2 unpack2(uint32_t v) { return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&v)); }

// Byte offsets of a lane's ldmatrix row in tiles of `pitch` elements:
// A operand (or transposed accumulator source) from [rows][k]; four registers = one 16 x 16 block
__device__ __forceinline__ uint32_t a_lane(int lane, int pitch) { return ((lane & 15) * pitch + (lane >> 4) * 8) * 2; }
// B operand from [n][k]: registers 0, 1 = columns 0..7, registers 2, 3 = columns 8..15
__device__ __forceinline__ uint32_t b_lane(int lane, int pitch) { return (((lane & 7) + ((lane >> 4) << 3)) * pitch + ((lane >> 3) & 1) * 8) * 2; }
// B operand from [k][n], read transposed: registers as above
__device__ __forceinline__ uint32_t bt_lane(int lane, int pitch) { return (((lane & 7) + ((lane >> 3) & 1) * 8) * pitch + (lane >> 4) * 8) * 2; }
// A operand from [k][rows], read transposed
__device__ __forceinline__ uint32_t at_lane(int lane, int pitch) { return (((lane & 7) + (lane >> 4) * 8) * pitch + ((lane >> 3) & 1) * 8) * 2; }

// 16 bytes to shared memory; zeros when not ok
__device__ __forceinline__ void copy16(void* dst, const void* src, bool ok) {
  const int sz = ok ? 16 : 0;
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(sm100::smem_u32(dst)), "l"(src), "r"(sz));
}
__device__ __forceinline__ void copies_issued() { asm volatile("cp.async.commit_group;"); }
template <int kLeft>
__device__ __forceinline__ void copies_wait() {
  asm volatile("cp.async.wait_group %0;" ::"n"(kLeft) : "memory");
}

}  // namespace frag
}  // namespace xpool
