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

// Floats as unsigned integers of the same order.
__device__ __forceinline__ unsigned ordered(float v) {
  const unsigned u = __float_as_uint(v);
  return u & 0x80000000u ? ~u : u | 0x80000000u;
}

// The warp's row: its `top` largest logits in falling order, the smaller index first where two are equal. HELD: up to
// 32 * kMine experts, a lane keeps its own in registers and strikes out what was taken; otherwise every turn takes the
// largest of those behind the one before it in that order.
constexpr int kMine = 8;
template <bool HELD> __device__ __forceinline__ void choose(const RouteArgs& a, int row, int lane) {
  const float* z = a.logits + size_t(row) * (a.experts + a.extra);
  unsigned key[kMine];
  if (HELD)
#pragma unroll
    for (int i = 0; i < kMine; ++i) key[i] = lane + 32 * i < a.experts ? max(ordered(__ldcg(z + lane + 32 * i)), 1u) : 0u;   // 0: taken, or none
  unsigned before = 0xffffffffu;
  int before_at = -1, taken = 0;         // taken: the lane-th choice
  for (int k = 0; k < a.top; ++k) {
    unsigned best = 0u;
    int at = 0x7fffffff;
    if (HELD) {
#pragma unroll
      for (int i = 0; i < kMine; ++i)
        if (key[i] > best) {
          best = key[i];
          at = lane + 32 * i;
        }
    } else {
      for (int e = lane; e < a.experts; e += 32) {
        const unsigned v = max(ordered(__ldcg(z + e)), 1u);
        if (v > before || (v == before && e <= before_at)) continue;
        if (v > best) {
          best = v;
          at = e;
        }
      }
    }
    const unsigned high = __reduce_max_sync(0xffffffffu, best);
    at = __reduce_min_sync(0xffffffffu, best == high ? at : 0x7fffffff);
    if (HELD) {
#pragma unroll
      for (int i = 0; i < kMine; ++i)
        if (at == lane + 32 * i) key[i] = 0u;
    }
    before = high;
    before_at = at;
    if (lane == k) taken = min(at, a.experts - 1);
  }
  const float logit = lane < a.top ? __ldcg(z + taken) : -INFINITY;
  float score = 1.f / (1.f + expf(-logit));
  if (a.chosen) {
    const float e = expf(logit - warp_max(logit));
    score = e / warp_sum(e);
  }
  if (lane < a.top) {
    a.choice[row * a.top + lane] = taken;
    a.score[row * a.top + lane] = score;
  }
}
// The same where scores are not the logits' order: ranked by score + correction, from the best groups only. `line` holds the
// row's logits, then its ranks (shared memory where HELD, else a.ranks). One warp runs this once, so its loops stay short code.
template <bool HELD> __device__ __forceinline__ void choose_ranked(const RouteArgs& a, int row, int lane, float* line, const float* correction) {
  const float* z = a.logits + size_t(row) * (a.experts + a.extra);
  float high = -INFINITY, sum = 0.f;
#pragma unroll 4
  for (int e = lane; e < a.experts; e += 32) {
    const float v = __ldcg(z + e);
    line[e] = v;
    high = fmaxf(high, v);
  }
  if (a.softmax) {
    high = warp_max(high);
#pragma unroll 1
    for (int e = lane; e < a.experts; e += 32) sum += expf(line[e] - high);
    sum = warp_sum(sum);
  }
  auto score_of = [&](float logit) { return a.softmax ? expf(logit - high) / sum : 1.f / (1.f + expf(-logit)); };
#pragma unroll 1
  for (int e = lane; e < a.experts; e += 32) line[e] = score_of(line[e]) + (correction ? correction[e] : 0.f);
  __syncwarp();
  // the largest key behind (before, before_at) in falling order, the smaller index first where two are equal
  unsigned before = 0xffffffffu;
  int before_at = -1;
  auto next = [&](unsigned best, int at) {
    before = __reduce_max_sync(0xffffffffu, best);
    before_at = __reduce_min_sync(0xffffffffu, best == before ? at : 0x7fffffff);
  };
  auto behind = [&](unsigned v, int at) { return v < before || (v == before && at > before_at); };
  if (a.keep_groups < a.groups) {
    const int size = a.experts / a.groups;
    auto largest = [&](int g) {
      unsigned v = 1u;
#pragma unroll 4
      for (int e = g * size; e < (g + 1) * size; ++e) v = max(v, ordered(line[e]));
      return v;
    };
    const unsigned mine = lane < a.groups ? largest(lane) : 0u;
    auto rank_of = [&](int g) { return g == lane ? mine : largest(g); };
#pragma unroll 1
    for (int k = 0; k < a.keep_groups; ++k) {
      unsigned best = 0u;
      int at = 0x7fffffff;
#pragma unroll 1
      for (int g = lane; g < a.groups; g += 32) {
        const unsigned v = rank_of(g);
        if (behind(v, g) && v > best) {
          best = v;
          at = g;
        }
      }
      next(best, at);
    }
    __syncwarp();
#pragma unroll 1
    for (int g = lane; g < a.groups; g += 32)
      if (behind(rank_of(g), g))
        for (int e = g * size; e < (g + 1) * size; ++e) line[e] = -INFINITY;
    __syncwarp();
  }
  unsigned key[kMine];
  if (HELD)
#pragma unroll
    for (int i = 0; i < kMine; ++i) key[i] = lane + 32 * i < a.experts ? max(ordered(line[lane + 32 * i]), 1u) : 0u;
  before = 0xffffffffu;
  before_at = -1;
  int taken = 0;
#pragma unroll 1
  for (int k = 0; k < a.top; ++k) {
    unsigned best = 0u;
    int at = 0x7fffffff;
    if (HELD) {
#pragma unroll
      for (int i = 0; i < kMine; ++i)
        if (key[i] > best) {
          best = key[i];
          at = lane + 32 * i;
        }
    } else {
      for (int e = lane; e < a.experts; e += 32) {
        const unsigned v = max(ordered(line[e]), 1u);
        if (behind(v, e) && v > best) {
          best = v;
          at = e;
        }
      }
    }
    next(best, at);
    if (HELD) {
#pragma unroll
      for (int i = 0; i < kMine; ++i)
        if (before_at == lane + 32 * i) key[i] = 0u;
    }
    if (lane == k) taken = min(before_at, a.experts - 1);
  }
  const float score = lane < a.top ? score_of(__ldcg(z + taken)) : 0.f, total = warp_sum(score);
  if (lane < a.top) {
    a.choice[row * a.top + lane] = taken;
    a.score[row * a.top + lane] = a.weights ? score / (total + 1e-20f) : score;
  }
}
__device__ __forceinline__ void choose(const RouteArgs& a, int row, int lane, float* line, const float* correction) {
  const bool held = a.experts <= 32 * kMine;
  if (a.ranks) {
    if (held) choose_ranked<true>(a, row, lane, line, correction);
    else choose_ranked<false>(a, row, lane, a.ranks + size_t(row) * a.experts, correction);
  } else {
    if (held) choose<true>(a, row, lane);
    else choose<false>(a, row, lane);
  }
}

// The step's assignments sorted by expert, by one CTA. `first` holds every expert's first slot, then its next free one.
__device__ __forceinline__ void sort_assignments(const RouteArgs& a, int* counts, int* first) {
  constexpr int U = 8;                  // assignments a thread has in flight
  const int n = a.rows * a.top, threads = blockDim.x, lane = threadIdx.x & 31;
  int choice[U];
  auto load = [&](int base) {
#pragma unroll
    for (int u = 0; u < U; ++u) choice[u] = base + u * threads < n ? __ldcg(a.choice + base + u * threads) : -1;
  };
  load(threadIdx.x);
  for (int e = threadIdx.x; e < a.experts; e += threads) counts[e] = 0;
  __syncthreads();
  for (int base = threadIdx.x; base < n; base += U * threads) {
    if (base >= U * threads) load(base);
#pragma unroll
    for (int u = 0; u < U; ++u)
      if (choice[u] >= 0) atomicAdd(&counts[choice[u]], 1);
  }
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
  for (int base = threadIdx.x; base < n; base += U * threads) {
    if (n > U * threads) load(base);
    float score[U];
#pragma unroll
    for (int u = 0; u < U; ++u) score[u] = choice[u] >= 0 ? __ldcg(a.score + base + u * threads) : 0.f;
#pragma unroll
    for (int u = 0; u < U; ++u) {
      if (choice[u] < 0) continue;
      const int slot = atomicAdd(&first[choice[u]], 1);
      a.list[slot] = base + u * threads;
      a.slot_score[slot] = score[u];
    }
  }
}

// True for the CTA that arrives last of `of`; the counter is left at zero. Every thread takes part.
__device__ __forceinline__ bool arrives_last(unsigned* counter, unsigned of, unsigned* flag) {
  __syncthreads();
  if (threadIdx.x == 0) {
    *flag = atom_acq_rel_add(counter, 1u) == of - 1 ? 1u : 0u;
    if (*flag) *counter = 0;
  }
  __syncthreads();
  return *flag != 0;
}

// FUSED: blockIdx = (eight experts, eight rows); a warp runs its expert's router row over the rows, the last CTA of the
// rows chooses, a warp a row, and the last of all sorts. Otherwise the logits are there, a warp chooses for one row, and
// the last CTA sorts.
template <typename T, bool FUSED>
__global__ void __launch_bounds__(FUSED ? 256 : 1024) route(RouteArgs a) {
  __shared__ int counts[kMaxExperts], first[kMaxExperts];
  __shared__ unsigned last;
  __shared__ float ranks[FUSED ? 8 : 32][32 * kMine];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5, logits = a.experts + a.extra;
  // corrections wait in the table of slots, which is written behind their last use
  float* correction = a.correction ? reinterpret_cast<float*>(first) : nullptr;
  if (correction)
    for (int e = threadIdx.x; e < a.experts; e += blockDim.x) correction[e] = a.correction[e];
  if constexpr (FUSED) {
    constexpr int N = 16 / sizeof(T);
    const int e = blockIdx.x * 8 + warp, pieces = a.k_stride / N, row0 = blockIdx.y * 8, rows = min(8, a.rows - row0);
    const uint4* w = reinterpret_cast<const uint4*>(static_cast<const T*>(a.router) + size_t(min(e, logits - 1)) * a.k_stride);
    uint4 held[kHeld];
#pragma unroll
    for (int i = 0; i < kHeld; ++i) held[i] = lane + 32 * i < pieces ? w[lane + 32 * i] : make_uint4(0, 0, 0, 0);
    dependency_wait();
    allow_dependents();
    if (e < logits)
      for (int row = row0; row < row0 + rows; ++row) {
        const uint4* h = reinterpret_cast<const uint4*>(static_cast<const T*>(a.h) + size_t(row) * a.k_stride);
        uint4 x[kHeld];
#pragma unroll
        for (int i = 0; i < kHeld; ++i) x[i] = lane + 32 * i < pieces ? h[lane + 32 * i] : make_uint4(0, 0, 0, 0);
        float sum = 0.f;
#pragma unroll
        for (int i = 0; i < kHeld; ++i) sum += dot16<T>(x[i], held[i]);
        for (int i = lane + 32 * kHeld; i < pieces; i += 32) sum += dot16<T>(h[i], w[i]);
        sum = warp_sum(sum);
        if (lane == 0) a.logits[size_t(row) * logits + e] = sum;
      }
    if (!arrives_last(a.count + 1 + blockIdx.y, gridDim.x, &last)) return;
    if (warp < rows) choose(a, row0 + warp, lane, ranks[warp], correction);
    if (gridDim.y == 1) __syncthreads();
    else if (!arrives_last(a.count, gridDim.y, &last)) return;
  } else {
    dependency_wait();
    allow_dependents();
    const int row = blockIdx.x * warps + warp;
    if (correction) __syncthreads();
    if (row < a.rows) choose(a, row, lane, ranks[warp], correction);
    if (!arrives_last(a.count, gridDim.x, &last)) return;
  }
  sort_assignments(a, counts, first);
}

// out[slot] = h[list[slot] / top], 16 bytes a thread.
__global__ void __launch_bounds__(256) gather_rows(const uint4* h, const int* list, int top, uint4* out, int pieces) {
  dependency_wait();
  allow_dependents();
  const size_t slot = blockIdx.x;
  const uint4* from = h + size_t(list[slot] / top) * pieces;
  for (int i = threadIdx.x; i < pieces; i += 256) out[slot * pieces + i] = from[i];
}

template <typename T> int RouteAs(const Queue& q, const RouteArgs& a) {
  if (RouteFused(a.rows))
    return int(Launch(route<T, true>, dim3(unsigned((a.experts + a.extra + 7) / 8), unsigned((a.rows + 7) / 8)), dim3(256), 0, q.stream, q.chained, a));
  return int(Launch(route<T, false>, dim3(unsigned((a.rows + 31) / 32)), dim3(1024), 0, q.stream, q.chained, a));
}

}  // namespace

bool RouteFused(int rows) { return rows <= kFusedRows; }

int Route(const Queue& q, const RouteArgs& a) {
  if (a.rows <= 0) return 0;
  if (a.experts > kMaxExperts || a.top > a.experts || a.top > kMaxTop || a.tile_rows < 1 || a.k_stride % 8 ||
      (!a.ranks && (a.softmax || a.correction || a.keep_groups < a.groups)) || (a.chosen && a.ranks))
    return int(cudaErrorInvalidValue);
  return q.f32 ? RouteAs<float>(q, a) : RouteAs<__nv_bfloat16>(q, a);
}

int GatherRows(const Queue& q, const void* h, int k_stride, const ExpertSlots& slots, void* out) {
  if (q.f32 || slots.slots <= 0) return q.f32 ? int(cudaErrorInvalidValue) : 0;
  return int(Launch(gather_rows, dim3(unsigned(slots.slots)), dim3(256), 0, q.stream, q.chained, static_cast<const uint4*>(h), slots.list, slots.top,
                    static_cast<uint4*>(out), k_stride / 8));
}

}  // namespace tmb
