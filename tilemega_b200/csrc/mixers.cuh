// Addressing, norm and rotary helpers shared by the mixer kernels of a ragged step.
#pragma once
#include "element.cuh"
#include "ops.h"
#include "ptx.cuh"

namespace tmb {

// Element offset of pool row `kv` (block * 16 + row in block) of one key/value head.
__device__ __forceinline__ size_t pool_offset(int kv, int group, int kv_heads, int pool_dim) {
  return ((size_t(kv / kRaggedBlock) * kv_heads + group) * kRaggedBlock + kv % kRaggedBlock) * pool_dim;
}

// Pool row of position j of the sequence that owns this block-table row.
__device__ __forceinline__ int key_row(const int* table, int j, const StepRows& r) {
  const int block = min(max(table[min(j / kRaggedBlock, r.max_blocks - 1)], 0), r.num_blocks - 1);
  return block * kRaggedBlock + j % kRaggedBlock;
}

// Entry d of a head after the rotation (rotate-half pairs d and d + half; entries behind them pass).
template <typename T> __device__ __forceinline__ float rotated(const T* head, int d, int half, const float2* angle) {
  if (d >= 2 * half) return to_f(head[d]);
  const int i = d < half ? d : d - half;
  const float u = to_f(head[i]), v = to_f(head[i + half]);
  const float2 cs = angle[i];
  return d < half ? u * cs.x - v * cs.y : v * cs.x + u * cs.y;
}

// The same for a head whose entries are first scaled: entry d by inv * weight[d] (weight null: not at all).
template <typename T>
__device__ __forceinline__ float normed_rotated(const T* head, const float* weight, float inv, int d, int half, const float2* angle) {
  if (!weight) return rotated(head, d, half, angle);
  if (d >= 2 * half) return to_f(head[d]) * inv * weight[d];
  const int i = d < half ? d : d - half;
  const float u = to_f(head[i]) * inv * weight[i], v = to_f(head[i + half]) * inv * weight[i + half];
  const float2 cs = angle[i];
  return d < half ? u * cs.x - v * cs.y : v * cs.x + u * cs.y;
}

// A thread's share of the squares of `count` consecutive elements, spread over `threads` threads.
template <typename T> __device__ __forceinline__ float square_sum(const T* at, int count, int threads) {
  float sq = 0.f;
  if (sizeof(T) == 2 && (reinterpret_cast<uintptr_t>(at) & 15) == 0 && count % 8 == 0) {
    for (int i = threadIdx.x; i < count / 8; i += threads) {
      float v[8];
      unpack8(reinterpret_cast<const uint4*>(at)[i], v);
#pragma unroll
      for (int j = 0; j < 8; ++j) sq = fmaf(v[j], v[j], sq);
    }
  } else {
    for (int i = threadIdx.x; i < count; i += threads) {
      const float v = to_f(at[i]);
      sq = fmaf(v, v, sq);
    }
  }
  return sq;
}
// 1 / rms of two vectors from every thread's shares of their squares; `part` holds one entry per warp.
template <int THREADS>
__device__ __forceinline__ float2 inverse_rms(float2 squares, int count_a, int count_b, float eps, float2* part) {
  squares.x = warp_sum(squares.x);
  squares.y = warp_sum(squares.y);
  if ((threadIdx.x & 31) == 0) part[threadIdx.x >> 5] = squares;
  __syncthreads();
  float2 sum = make_float2(0.f, 0.f);
#pragma unroll
  for (int w = 0; w < THREADS / 32; ++w) {
    sum.x += part[w].x;
    sum.y += part[w].y;
  }
  return make_float2(1.f / sqrtf(sum.x / float(count_a) + eps), 1.f / sqrtf(sum.y / float(count_b) + eps));
}

// A layer's values blended with those of another layer for the same rows, see AttentionArgs.
struct Blend {
  const float* by = nullptr;         // null: the layer's own as they are
  const void* from = nullptr;
  int stride = 0;
};
// Value i (of kv_heads x vdim) of a row; `own` points to the row's first.
template <typename T> __device__ __forceinline__ T blended(const Blend& b, const T* own, int row, int i) {
  if (!b.by) return own[i];
  const float f = *b.by;
  return from_f<T>((1.f - f) * to_f(own[i]) + f * to_f(static_cast<const T*>(b.from)[size_t(row) * b.stride + i]));
}

// Four neighbours, of which the first `count` are there (zeros behind them); `wide`: their address suits one load.
template <typename T> __device__ __forceinline__ void load_four(const T* at, int count, bool wide, float (&v)[4]) {
  if (wide && count >= 4) {
    if constexpr (sizeof(T) == 4) {
      const float4 q = *reinterpret_cast<const float4*>(at);
      v[0] = q.x, v[1] = q.y, v[2] = q.z, v[3] = q.w;
    } else {
      const uint2 w = *reinterpret_cast<const uint2*>(at);
      v[0] = bf_lo(w.x), v[1] = bf_hi(w.x), v[2] = bf_lo(w.y), v[3] = bf_hi(w.y);
    }
  } else {
#pragma unroll
    for (int i = 0; i < 4; ++i) v[i] = i < count ? to_f(at[i]) : 0.f;
  }
}

__device__ __forceinline__ float sigmoid(float v) { return 1.f / (1.f + expf(-v)); }

}  // namespace tmb
