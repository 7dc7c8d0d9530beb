// Warp-level tensor-pipe helpers of the bf16 mixer kernels (mma.sync): operand loads from shared memory, 16-byte copies
// into it, and values split into a bf16 head and a bf16 remainder.
#pragma once
#include <cuda_bf16.h>
#include <stdint.h>

#include "ptx.cuh"

namespace tmb {

using bf16 = __nv_bfloat16;

__device__ __forceinline__ void mma16816(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
               : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ uint32_t pack(float lo, float hi) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(lo, hi);
  return *reinterpret_cast<const uint32_t*>(&h);
}
// What rounding to bf16 leaves behind.
__device__ __forceinline__ float rest(float v) { return v - __bfloat162float(__float2bfloat16_rn(v)); }

__device__ __forceinline__ void copy16(void* dst, const void* src, bool live) {   // 16 bytes, zero-filled unless live
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(dst)), "l"(src), "r"(live ? 16 : 0) : "memory");
}
__device__ __forceinline__ void copy_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void copy_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

// Operand tiles in shared memory are row-major with `pitch` elements per row, pitch = 16 n + 8: the eight rows of an
// ldmatrix tile then start in eight different bank groups.
__device__ __forceinline__ void load_a(uint32_t (&a)[4], const bf16* tile, int pitch, int row, int col, int lane) {
  ldmatrix_x4(a, smem_u32(tile + (row + (lane & 15)) * pitch + col + (lane >> 4) * 8));
}
// A = tile^T: tile holds [k][m]
__device__ __forceinline__ void load_a_transposed(uint32_t (&a)[4], const bf16* tile, int pitch, int k, int m, int lane) {
  ldmatrix_x4_trans(a, smem_u32(tile + (k + (lane & 7) + (lane >> 4) * 8) * pitch + m + ((lane >> 3) & 1) * 8));
}
// two n8 tiles of B, tile holds [n][k]
__device__ __forceinline__ void load_b(uint32_t (&b)[4], const bf16* tile, int pitch, int n, int k, int lane) {
  ldmatrix_x4(b, smem_u32(tile + (n + (lane & 7) + (lane >> 4) * 8) * pitch + k + ((lane >> 3) & 1) * 8));
}
// two n8 tiles of B, tile holds [k][n]
__device__ __forceinline__ void load_b_transposed(uint32_t (&b)[4], const bf16* tile, int pitch, int k, int n, int lane) {
  ldmatrix_x4_trans(b, smem_u32(tile + (k + (lane & 7) + ((lane >> 3) & 1) * 8) * pitch + n + (lane >> 4) * 8));
}

}  // namespace tmb
