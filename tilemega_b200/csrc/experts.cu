// Routing of a ragged step's rows to experts: router logits, the best experts of every row, and the assignments sorted
// by expert into the tiles the per-expert products run on. One kernel: its last CTA to finish sorts.
#include <cuda_bf16.h>

#include <algorithm>

#include "element.cuh"
#include "ops.h"
#include "ptx.cuh"
#include "tensor_map.h"

namespace tmb {
namespace {

constexpr int kFusedRows = 64;        // up to this many rows the router's product is part of the kernel
constexpr int kHeld = 8;              // router weights a lane loads before the dependency wait, in 16-byte pieces

template <typename T> __device__ __forceinline__ float dot16(const uint4& a, const uint4& b);
template <> __device__ __forceinline__ float dot16<__nv_bfloat16>(const uint4& a, const uint4& b) {
  float x[8], y[8], sum = 0.f;
  unpack8(a, x);
  unpack8(b, y);
#pragma unroll
  for (int i = 0; i < 8; ++i) sum = fmaf(x[i], y[i], sum);
  return sum;
}
template <> __device__ __forceinline__ float dot16<float>(const uint4& a, const uint4& b) {
  float sum = __uint_as_float(a.x) * __uint_as_float(b.x);
  sum = fmaf(__uint_as_float(a.y), __uint_as_float(b.y), sum);
  sum = fmaf(__uint_as_float(a.z), __uint_as_float(b.z), sum);
  return fmaf(__uint_as_float(a.w), __uint_as_float(b.w), sum);
}

// The warp's row: its `top` largest logits in falling order, the smaller index first where two are equal. Every turn
// takes the largest of those behind the one before it in that order.
__device__ __forceinline__ void choose(const RouteArgs& a, int row, int lane) {
  const float* z = a.logits + size_t(row) * a.experts;
  float before = INFINITY;
  int before_at = -1;
  for (int k = 0; k < a.top; ++k) {
    float best = -INFINITY;
    int at = 0x7fffffff;
    for (int e = lane; e < a.experts; e += 32) {
      const float v = __ldcg(z + e);
      if (v > before || (v == before && e <= before_at)) continue;
      if (v > best || at == 0x7fffffff) {
        best = v;
        at = e;
      }
    }
#pragma unroll
    for (int o = 16; o; o >>= 1) {
      const float v = __shfl_xor_sync(0xffffffffu, best, o);
      const int i = __shfl_xor_sync(0xffffffffu, at, o);
      if (v > best || (v == best && i < at)) {
        best = v;
        at = i;
      }
    }
    at = min(at, a.experts - 1);      // (logits that are not numbers: any expert, but a valid one)
    if (lane == 0) {
      a.choice[row * a.top + k] = at;
      a.score[row * a.top + k] = 1.f / (1.f + expf(-best));
    }
    before = best;
    before_at = at;
  }
}

// The step's assignments sorted by expert, by one CTA. `first` holds every expert's first slot, then its next free one.
__device__ __forceinline__ void sort_assignments(const RouteArgs& a, int* counts, int* first) {
  const int n = a.rows * a.top, threads = blockDim.x, lane = threadIdx.x & 31;
  for (int e = threadIdx.x; e < a.experts; e += threads) counts[e] = 0;
  __syncthreads();
  for (int i = threadIdx.x; i < n; i += threads) atomicAdd(&counts[__ldcg(a.choice + i)], 1);
  __syncthreads();
  if (threadIdx.x < 32) {
    int slots = 0, tiles = 0;
    for (int base = 0; base < a.experts; base += 32) {
      const int e = base + lane, count = e < a.experts ? counts[e] : 0, mine = (count + a.tile_rows - 1) / a.tile_rows;
      int slot_sum = count, tile_sum = mine;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const int s = __shfl_up_sync(0xffffffffu, slot_sum, o), t = __shfl_up_sync(0xffffffffu, tile_sum, o);
        if (lane >= o) {
          slot_sum += s;
          tile_sum += t;
        }
      }
      const int at = slots + slot_sum - count;
      if (e < a.experts) first[e] = at;
      for (int t = 0; t < mine; ++t)
        a.tiles[tiles + tile_sum - mine + t] = {e, at + t * a.tile_rows, min(count - t * a.tile_rows, a.tile_rows), 0};
      slots += __shfl_sync(0xffffffffu, slot_sum, 31);
      tiles += __shfl_sync(0xffffffffu, tile_sum, 31);
    }
    if (lane == 0) *a.tile_count = tiles;
  }
  __syncthreads();
  // (the order of an expert's slots is whatever the counters make it: every slot is computed by itself)
  for (int i = threadIdx.x; i < n; i += threads) {
    const int slot = atomicAdd(&first[__ldcg(a.choice + i)], 1);
    a.list[slot] = i;
    a.slot_score[slot] = __ldcg(a.score + i);
  }
}

// FUSED: a warp takes one expert and runs its router row over all rows; the last CTA chooses and sorts. Otherwise the
// logits are there and a warp takes one row; the last CTA sorts.
template <typename T, bool FUSED>
__global__ void __launch_bounds__(FUSED ? 256 : 1024) route(RouteArgs a) {
  __shared__ int counts[kMaxExperts], first[kMaxExperts];
  __shared__ unsigned last;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5;
  if constexpr (FUSED) {
    constexpr int N = 16 / sizeof(T);
    const int e = blockIdx.x * warps + warp, pieces = a.k_stride / N;
    const uint4* w = reinterpret_cast<const uint4*>(static_cast<const T*>(a.router) + size_t(min(e, a.experts - 1)) * a.k_stride);
    uint4 held[kHeld];
#pragma unroll
    for (int i = 0; i < kHeld; ++i) held[i] = lane + 32 * i < pieces ? w[lane + 32 * i] : make_uint4(0, 0, 0, 0);
    dependency_wait();
    allow_dependents();
    if (e < a.experts)
      for (int row = 0; row < a.rows; ++row) {
        const uint4* h = reinterpret_cast<const uint4*>(static_cast<const T*>(a.h) + size_t(row) * a.k_stride);
        float sum = 0.f;
#pragma unroll
        for (int i = 0; i < kHeld; ++i)
          if (lane + 32 * i < pieces) sum += dot16<T>(h[lane + 32 * i], held[i]);
        for (int i = lane + 32 * kHeld; i < pieces; i += 32) sum += dot16<T>(h[i], w[i]);
        sum = warp_sum(sum);
        if (lane == 0) a.logits[size_t(row) * a.experts + e] = sum;
      }
  } else {
    dependency_wait();
    allow_dependents();
    const int row = blockIdx.x * warps + warp;
    if (row < a.rows) choose(a, row, lane);
  }
  __syncthreads();
  if (threadIdx.x == 0) last = atom_acq_rel_add(a.count, 1u) == gridDim.x - 1 ? 1u : 0u;
  __syncthreads();
  if (!last) return;
  if (threadIdx.x == 0) *a.count = 0;   // for the next launch
  if constexpr (FUSED) {
    for (int row = warp; row < a.rows; row += warps) choose(a, row, lane);
    __syncthreads();
  }
  sort_assignments(a, counts, first);
}

template <typename T> int RouteAs(const Queue& q, const RouteArgs& a) {
  if (RouteFused(a.rows)) return int(Launch(route<T, true>, dim3(unsigned((a.experts + 7) / 8)), dim3(256), 0, q.stream, q.chained, a));
  return int(Launch(route<T, false>, dim3(unsigned((a.rows + 31) / 32)), dim3(1024), 0, q.stream, q.chained, a));
}

}  // namespace

bool RouteFused(int rows) { return rows <= kFusedRows; }

int Route(const Queue& q, const RouteArgs& a) {
  if (a.rows <= 0) return 0;
  if (a.experts > kMaxExperts || a.top > a.experts || a.tile_rows < 1 || a.k_stride % 8) return int(cudaErrorInvalidValue);
  return q.f32 ? RouteAs<float>(q, a) : RouteAs<__nv_bfloat16>(q, a);
}

}  // namespace tmb
