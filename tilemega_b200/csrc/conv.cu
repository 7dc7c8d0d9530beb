// The row operation in front of a layer with grouped norms and a short convolution over time, see ConvNormArgs: the side input
// of the layer before normed and added, the grouped norm, the convolution and its history, in one pass over the row.
#include <cuda_bf16.h>

#include <algorithm>

#include "element.cuh"
#include "ops.h"
#include "ptx.cuh"
#include "tensor_map.h"

namespace tmb {
namespace {

constexpr int kThreads = 512, kWarps = kThreads / 32;

// A CTA walks a tile of one entry's rows (SELECT: one chosen row), a thread always the same columns: N units of E, one kThreads
// units behind the other. It starts count - 1 rows before the tile, whose h it forms again (x is never written in place), so
// tiles do not wait for one another; the first tile reads the history and writes the new one, and tiles are at least count - 1
// rows long, so no other tile touches it. blockIdx = (tile, entry).
// HELD: up to four taps stay in registers.
constexpr int kHeldTaps = 4;
template <typename T, int E, int N, bool SELECT, bool HELD>
__global__ void __launch_bounds__(kThreads) conv_norm(StepRows r, ConvNormArgs a, int tile) {
  extern __shared__ __align__(16) float memory[];
  __shared__ float side_part[kWarps];
  const int units = a.width / E, lead = max(a.count - 1, 0), run = a.width / a.groups, run_units = run / E;
  const bool whole = run_units % 32 == 0;                 // a warp's units lie in one run: one partial sum for all of them
  const int per = whole ? run_units / 32 : run_units;     // partial sums of a run
  float* ring = memory;                                   // [lead][width]: h of the last positions
  float* partial = ring + size_t(lead) * a.width;
  float* inverse = partial + (whole ? units / 32 : units);
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  float weight[N][E], side_weight[N][E], held[HELD ? kHeldTaps : 1][N][E];
  auto each = [&](auto&& visit) {
#pragma unroll
    for (int n = 0; n < N; ++n)
      if (const int c = threadIdx.x + kThreads * n; c < units) visit(n, c);
  };
  auto load = [&](const float* at, int c, float (&v)[E]) {
    if constexpr (E == 4) {
      const float4 q = reinterpret_cast<const float4*>(at)[c];
      v[0] = q.x, v[1] = q.y, v[2] = q.z, v[3] = q.w;
    } else {
      v[0] = at[c];
    }
  };
  auto store = [&](float* at, int c, const float (&v)[E]) {
    if constexpr (E == 4) reinterpret_cast<float4*>(at)[c] = make_float4(v[0], v[1], v[2], v[3]);
    else at[c] = v[0];
  };
  auto store_elements = [&](void* at, size_t row, int c, const float (&v)[E]) {
    T* line = static_cast<T*>(at) + row * a.stride;
    if constexpr (E == 4) {
      alignas(16) T e[4] = {from_f<T>(v[0]), from_f<T>(v[1]), from_f<T>(v[2]), from_f<T>(v[3])};
      if (sizeof(T) == 2) reinterpret_cast<uint2*>(line)[c] = *reinterpret_cast<const uint2*>(e);
      else reinterpret_cast<uint4*>(line)[c] = *reinterpret_cast<const uint4*>(e);
    } else {
      line[c] = from_f<T>(v[0]);
    }
  };
  auto slot_of = [&](int position) { return ((position % lead) + lead) % lead; };
  each([&](int n, int c) {
    load(a.weight, c, weight[n]);
    if (a.side) load(a.side_weight, c, side_weight[n]);
    if constexpr (HELD) {                                 // held[j]: of j tokens before
#pragma unroll
      for (int j = 0; j < kHeldTaps; ++j)
        if (j < a.count) load(a.taps + size_t(lead - j) * a.width, c, held[j][n]);
    } else {
      for (int j = 0; j < a.count; ++j) asm volatile("prefetch.global.L2 [%0];" ::"l"(a.taps + size_t(j) * a.width + size_t(c) * E));
    }
  });
  Entry e{0, 0, 0, 0};
  int first = 0, end = 1;
  if constexpr (!SELECT) {
    e = r.entry[blockIdx.y];              // (tables and histories: written before the kernel this one depends on)
    first = blockIdx.x * tile;
    end = min(first + tile, e.rows);
    if (first >= e.rows) {
      dependency_wait();
      allow_dependents();
      return;
    }
    if (first == 0)
      for (int back = 1; back <= lead; ++back) {
        const int position = e.first_position - back;
        each([&](int, int c) {
          float v[E] = {};
          if (position >= 0) load(a.history + (size_t(e.slot) * lead + position % lead) * a.width, c, v);
          store(ring + size_t(slot_of(position)) * a.width, c, v);
        });
      }
  }
  dependency_wait();
  allow_dependents();

  float x[N][E], h[N][E], next_x[N][E], y[N][E];
  auto request = [&](int row) {            // one row ahead of its use
    each([&](int n, int c) {
      load(a.x + size_t(row) * a.width, c, next_x[n]);
      if (a.side) load(a.side + size_t(row) * a.width, c, y[n]);
    });
  };
  auto form = [&](int following) {         // x' and h of the row requested last
    float sq = 0.f;
#pragma unroll
    for (int n = 0; n < N; ++n)
#pragma unroll
      for (int i = 0; i < E; ++i) x[n][i] = next_x[n][i];
    if (a.side) {
      each([&](int n, int) {
#pragma unroll
        for (int i = 0; i < E; ++i) sq = fmaf(y[n][i], y[n][i], sq);
      });
      sq = warp_sum(sq);
      if (lane == 0) side_part[warp] = sq;
      __syncthreads();
      sq = 0.f;
#pragma unroll
      for (int w = 0; w < kWarps; ++w) sq += side_part[w];
      const float inv = 1.f / sqrtf(sq / float(a.width) + a.eps);
      each([&](int n, int) {
#pragma unroll
        for (int i = 0; i < E; ++i) x[n][i] = fmaf(a.gain, y[n][i] * inv * side_weight[n][i], x[n][i]);
      });
    }
    if (following >= 0) request(following);
#pragma unroll
    for (int n = 0; n < N; ++n) {
      const int c = threadIdx.x + kThreads * n;
      float v = 0.f;
      if (c < units)
#pragma unroll
        for (int i = 0; i < E; ++i) v = fmaf(x[n][i], x[n][i], v);
      if (whole) {                          // (warps are inside or outside as a whole)
        v = warp_sum(v);
        if (lane == 0 && c < units) partial[c / 32] = v;
      } else if (c < units) {
        partial[c] = v;
      }
    }
    __syncthreads();
    for (int g = warp; g < a.groups; g += kWarps) {
      float v = 0.f;
      for (int i = lane; i < per; i += 32) v += partial[g * per + i];
      v = warp_sum(v);
      if (lane == 0) inverse[g] = 1.f / sqrtf(v / float(run) + a.eps);
    }
    __syncthreads();
    each([&](int n, int c) {
      const float inv = inverse[c / run_units];
#pragma unroll
      for (int i = 0; i < E; ++i) h[n][i] = x[n][i] * inv * weight[n][i];
    });
  };
  if constexpr (SELECT) {
    request(a.select ? min(max(a.select[blockIdx.x], 0), a.limit - 1) : int(blockIdx.x));
    form(-1);
    each([&](int n, int c) { store_elements(a.normed, blockIdx.x, c, h[n]); });
  } else {
    const int start = max(0, first - lead);
    int at = lead ? slot_of(e.first_position + start) : 0;   // the row's place in the ring
    auto keep = [&]() {
      if (lead == 0) return;
      float* to = ring + size_t(at) * a.width;
      each([&](int n, int c) { store(to, c, h[n]); });
      at = at + 1 == lead ? 0 : at + 1;
    };
    request(e.first_row + start);
    for (int j = start; j < end; ++j) {
      const size_t row = size_t(e.first_row) + j;
      form(j + 1 < end ? int(row) + 1 : -1);
      if (j >= first) {
        each([&](int n, int c) {
          if (a.x_out) store(a.x_out + row * a.width, c, x[n]);
          store_elements(a.normed, row, c, h[n]);
          if (a.count == 0) return;
          float sum[E], by[E], old[E];
          if constexpr (HELD) {
#pragma unroll
            for (int i = 0; i < E; ++i) sum[i] = fmaf(held[0][n][i], h[n][i], h[n][i]);
#pragma unroll
            for (int back = 1; back < kHeldTaps; ++back) {
              if (back > lead) break;
              load(ring + size_t(at >= back ? at - back : at - back + lead) * a.width, c, old);
#pragma unroll
              for (int i = 0; i < E; ++i) sum[i] = fmaf(held[back][n][i], old[i], sum[i]);
            }
          } else {
            load(a.taps + size_t(lead) * a.width, c, by);
#pragma unroll
            for (int i = 0; i < E; ++i) sum[i] = fmaf(by[i], h[n][i], h[n][i]);
            for (int back = 1; back <= lead; ++back) {
              load(a.taps + size_t(lead - back) * a.width, c, by);
              load(ring + size_t(at >= back ? at - back : at - back + lead) * a.width, c, old);
#pragma unroll
              for (int i = 0; i < E; ++i) sum[i] = fmaf(by[i], old[i], sum[i]);
            }
          }
          store_elements(a.convolved, row, c, sum);
        });
      }
      keep();
    }
    if (first == 0 && lead > 0) {
      if (e.rows > tile) {
        at = slot_of(e.first_position + e.rows - lead);
        request(e.first_row + e.rows - lead);
        for (int j = e.rows - lead; j < e.rows; ++j) {
          form(j + 1 < e.rows ? e.first_row + j + 1 : -1);
          keep();
        }
      }
      for (int j = max(0, e.rows - lead); j < e.rows; ++j) {
        const int place = slot_of(e.first_position + j);
        each([&](int, int c) {
          float v[E];
          load(ring + size_t(place) * a.width, c, v);
          store(a.history + (size_t(e.slot) * lead + place) * a.width, c, v);
        });
      }
    }
  }
}

template <typename T, int E, int N> int ConvNormWith(const Queue& q, const StepRows& r, const ConvNormArgs& a) {
  const int lead = std::max(a.count - 1, 0), units = a.width / E;
  const size_t smem = (size_t(lead) * a.width + units + a.groups) * sizeof(float);
  if (a.select) return int(Launch(conv_norm<T, E, N, true, false>, dim3(unsigned(a.rows)), dim3(kThreads), smem, q.stream, q.chained, r, a, 1));
  const int tile = std::max({1, lead, std::min(8, (a.rows + 2 * q.sm_count - 1) / (2 * q.sm_count))});
  auto kernel = conv_norm<T, E, N, false, false>;
  if constexpr (N * E <= 8)
    if (a.count <= kHeldTaps) kernel = conv_norm<T, E, N, false, true>;
  return int(Launch(kernel, dim3(unsigned((r.longest + tile - 1) / tile), unsigned(r.entries)), dim3(kThreads), smem, q.stream, q.chained, r, a, tile));
}

template <typename T> int ConvNormAs(const Queue& q, const StepRows& r, const ConvNormArgs& a) {
  if (a.width % 4 == 0 && (a.width / a.groups) % 4 == 0)
    return a.width <= 4 * kThreads ? ConvNormWith<T, 4, 1>(q, r, a) : a.width <= 8 * kThreads ? ConvNormWith<T, 4, 2>(q, r, a) : ConvNormWith<T, 4, 4>(q, r, a);
  return a.width <= 4 * kThreads ? ConvNormWith<T, 1, 4>(q, r, a) : ConvNormWith<T, 1, 16>(q, r, a);
}

constexpr int kMostMemory = 226 * 1024;

template <typename T, int E, int N> cudaError_t Raise() {
  for (auto kernel : {conv_norm<T, E, N, false, false>, conv_norm<T, E, N, true, false>, conv_norm<T, E, N, false, (N * E <= 8)>}) {
    const cudaError_t err = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, kMostMemory);
    if (err != cudaSuccess) return err;
  }
  return cudaSuccess;
}
template <typename T> cudaError_t RaiseAll() {
  for (cudaError_t err : {Raise<T, 4, 1>(), Raise<T, 4, 2>(), Raise<T, 4, 4>(), Raise<T, 1, 4>(), Raise<T, 1, 16>()})
    if (err != cudaSuccess) return err;
  return cudaSuccess;
}

}  // namespace

int ConvNorm(const Queue& q, const StepRows& r, const ConvNormArgs& a) {
  if (a.rows <= 0) return 0;
  if (a.groups < 1 || a.width % a.groups || a.width > kMaxConvWidth || a.count < 0 || a.count > kMaxTaps || (a.select && a.count) ||
      (a.side && a.x_out == a.x) || (a.count > 1 && !a.history))
    return int(cudaErrorInvalidValue);
  return q.f32 ? ConvNormAs<float>(q, r, a) : ConvNormAs<__nv_bfloat16>(q, r, a);
}

int PrepareConv() {
  const cudaError_t err = RaiseAll<float>();
  return int(err == cudaSuccess ? RaiseAll<__nv_bfloat16>() : err);
}

}  // namespace tmb
