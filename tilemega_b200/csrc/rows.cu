// Row operations of a ragged step: embedding and row tables, RMS norm over the fp32 residual stream and of what is added
// to it, greedy sampling, and the hand-over of sampled tokens to the next step.
#include <cuda_bf16.h>

#include <type_traits>

#include "element.cuh"
#include "ops.h"
#include "ptx.cuh"
#include "tensor_map.h"

namespace tmb {
namespace {

// One CTA per row. The row's entry is found by bisection over the entries' first rows (ascending, no gaps).
template <typename T>
__global__ void __launch_bounds__(256) start_step(StepRows r, const int* tokens, const T* embed, float* x, int streams, T* copy,
                                                  int copy_stride, int width, int vocab, float scale) {
  const int row = blockIdx.x;
  dependency_wait();
  allow_dependents();
  int lo = 0, hi = r.entries - 1;
  while (lo < hi) {
    const int mid = (lo + hi + 1) / 2;
    if (r.entry[mid].first_row <= row) lo = mid;
    else hi = mid - 1;
  }
  const Entry e = r.entry[lo];
  if (threadIdx.x == 0) {
    const int position = min(max(e.first_position + row - e.first_row, 0), r.capacity - 1);
    const int* table = r.block_table + size_t(min(max(e.slot, 0), r.slots - 1)) * r.max_blocks;
    const int block = min(max(table[min(position / kRaggedBlock, r.max_blocks - 1)], 0), r.num_blocks - 1);
    r.row_entry[row] = lo;
    r.row_position[row] = position;
    r.row_kv[row] = block * kRaggedBlock + position % kRaggedBlock;
  }
  const int token = min(max(tokens[row], 0), vocab - 1);
#pragma unroll 8
  for (int i = threadIdx.x; i < width; i += 256) {
    const T value = embed[size_t(token) * width + i];
    for (int s = 0; s < streams; ++s) x[(size_t(row) * streams + s) * width + i] = to_f(value) * scale;
    if (copy) copy[size_t(row) * copy_stride + i] = value;
  }
}

template <typename T>
__global__ void __launch_bounds__(256) rms_norm(NormArgs a) {
  __shared__ float part[8];
  dependency_wait();
  allow_dependents();
  const int i = blockIdx.x;
  const int row = a.select ? min(max(a.select[i], 0), a.limit - 1) : i;
  float* x = a.x + size_t(row) * a.width;
  const T* again = nullptr;
  if (a.again) again = static_cast<const T*>(a.again) + size_t(min(max(a.tokens[row], 0), a.vocab - 1)) * a.width;
  float sq = 0.f;
  for (int c = threadIdx.x; c < a.width; c += 256) {
    float v = x[c];
    if (again) {
      v += to_f(again[c]);
      x[c] = v;
    }
    sq = fmaf(v, v, sq);
  }
  sq = warp_sum(sq);
  if ((threadIdx.x & 31) == 0) part[threadIdx.x >> 5] = sq;
  __syncthreads();
  sq = 0.f;
#pragma unroll
  for (int w = 0; w < 8; ++w) sq += part[w];
  const float inv = 1.f / sqrtf(sq / float(a.width) + a.eps);
  T* out = static_cast<T*>(a.out) + size_t(i) * a.out_stride;
  for (int c = threadIdx.x; c < a.width; c += 256) out[c] = from_f<T>(x[c] * inv * a.weight[c]);   // each thread re-reads its own columns
}

// The same for widths that are multiples of 4 up to 8192: one pass, the row in registers, the weights loaded before the
// dependency wait.
constexpr int kQuads = 4;
template <typename T>
__global__ void __launch_bounds__(512) rms_norm_quads(NormArgs a) {
  __shared__ float part[16];
  const int i = blockIdx.x, quads = a.width / 4;
  float4 weight[kQuads], v[kQuads];
#pragma unroll
  for (int n = 0; n < kQuads; ++n) {
    const int c = threadIdx.x + 512 * n;
    if (c < quads) weight[n] = reinterpret_cast<const float4*>(a.weight)[c];
  }
  dependency_wait();
  allow_dependents();
  const int row = a.select ? min(max(a.select[i], 0), a.limit - 1) : i;
  float4* x = reinterpret_cast<float4*>(a.x + size_t(row) * a.width);
  float sq = 0.f;
#pragma unroll
  for (int n = 0; n < kQuads; ++n) {
    const int c = threadIdx.x + 512 * n;
    v[n] = c < quads ? x[c] : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  if (a.again) {
    const T* again = static_cast<const T*>(a.again) + size_t(min(max(a.tokens[row], 0), a.vocab - 1)) * a.width;
#pragma unroll
    for (int n = 0; n < kQuads; ++n) {
      const int c = threadIdx.x + 512 * n;
      if (c >= quads) continue;
      v[n].x += to_f(again[4 * c]);
      v[n].y += to_f(again[4 * c + 1]);
      v[n].z += to_f(again[4 * c + 2]);
      v[n].w += to_f(again[4 * c + 3]);
      x[c] = v[n];
    }
  }
#pragma unroll
  for (int n = 0; n < kQuads; ++n) sq += v[n].x * v[n].x + v[n].y * v[n].y + v[n].z * v[n].z + v[n].w * v[n].w;
  sq = warp_sum(sq);
  if ((threadIdx.x & 31) == 0) part[threadIdx.x >> 5] = sq;
  __syncthreads();
  sq = 0.f;
#pragma unroll
  for (int w = 0; w < 16; ++w) sq += part[w];
  const float inv = 1.f / sqrtf(sq / float(a.width) + a.eps);
  T* out = static_cast<T*>(a.out) + size_t(i) * a.out_stride;
#pragma unroll
  for (int n = 0; n < kQuads; ++n) {
    const int c = threadIdx.x + 512 * n;
    if (c >= quads) continue;
    alignas(16) T y[4] = {from_f<T>(v[n].x * inv * weight[n].x), from_f<T>(v[n].y * inv * weight[n].y), from_f<T>(v[n].z * inv * weight[n].z),
                          from_f<T>(v[n].w * inv * weight[n].w)};
    if (sizeof(T) == 2) reinterpret_cast<uint2*>(out)[c] = *reinterpret_cast<const uint2*>(y);
    else reinterpret_cast<uint4*>(out)[c] = *reinterpret_cast<const uint4*>(y);
  }
}

// A sublayer's output normed and added to the stream, see AddNormArgs. QUADS: widths that are multiples of 4 up to 8192
// (the row in registers); otherwise a thread forms the output's columns twice.
template <typename T>
__device__ __forceinline__ float branch_value(const AddNormArgs& a, int row, int c) {
  if (a.parts == 0) return a.branch[size_t(row) * a.width + c];
  const T* at = static_cast<const T*>(a.parts_of) + size_t(row) * a.parts * a.width + c;
  float v = 0.f;
  for (int k = 0; k < a.parts; ++k) v += to_f(at[size_t(k) * a.width]);
  return v;
}
template <typename T> __device__ __forceinline__ float4 four(const T* at);
template <> __device__ __forceinline__ float4 four<float>(const float* at) { return *reinterpret_cast<const float4*>(at); }
template <> __device__ __forceinline__ float4 four<__nv_bfloat16>(const __nv_bfloat16* at) {
  const uint2 w = *reinterpret_cast<const uint2*>(at);
  return make_float4(bf_lo(w.x), bf_hi(w.x), bf_lo(w.y), bf_hi(w.y));
}

template <typename T, bool QUADS>
__global__ void __launch_bounds__(512) add_norm(AddNormArgs a) {
  __shared__ float part[16];
  const int row = blockIdx.x, quads = a.width / 4;
  float4 weight[kQuads], y[kQuads], x[kQuads];
  if (QUADS) {
#pragma unroll
    for (int n = 0; n < kQuads; ++n) {
      const int c = threadIdx.x + 512 * n;
      if (c >= quads) continue;
      weight[n] = reinterpret_cast<const float4*>(a.weight)[c];
    }
  }
  dependency_wait();
  allow_dependents();
  float* line = a.x + size_t(row) * a.width;
  float sq = 0.f;
  if (QUADS) {
#pragma unroll
    for (int n = 0; n < kQuads; ++n) {
      const int c = threadIdx.x + 512 * n;
      y[n] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (c >= quads) continue;
      x[n] = reinterpret_cast<const float4*>(line)[c];
      if (a.parts == 0) {
        y[n] = reinterpret_cast<const float4*>(a.branch + size_t(row) * a.width)[c];
      } else {
        const T* at = static_cast<const T*>(a.parts_of) + size_t(row) * a.parts * a.width + 4 * c;
#pragma unroll 8
        for (int k = 0; k < a.parts; ++k) {
          const float4 v = four<T>(at + size_t(k) * a.width);
          y[n].x += v.x;
          y[n].y += v.y;
          y[n].z += v.z;
          y[n].w += v.w;
        }
      }
    }
#pragma unroll
    for (int n = 0; n < kQuads; ++n) sq += y[n].x * y[n].x + y[n].y * y[n].y + y[n].z * y[n].z + y[n].w * y[n].w;
  } else {
    for (int c = threadIdx.x; c < a.width; c += 512) {
      const float v = branch_value<T>(a, row, c);
      sq = fmaf(v, v, sq);
    }
  }
  sq = warp_sum(sq);
  if ((threadIdx.x & 31) == 0) part[threadIdx.x >> 5] = sq;
  __syncthreads();
  sq = 0.f;
#pragma unroll
  for (int w = 0; w < 16; ++w) sq += part[w];
  const float inv = 1.f / sqrtf(sq / float(a.width) + a.eps);
  T* out = static_cast<T*>(a.out) + size_t(row) * a.out_stride;
  if (QUADS) {
#pragma unroll
    for (int n = 0; n < kQuads; ++n) {
      const int c = threadIdx.x + 512 * n;
      if (c >= quads) continue;
      x[n].x += y[n].x * inv * weight[n].x;
      x[n].y += y[n].y * inv * weight[n].y;
      x[n].z += y[n].z * inv * weight[n].z;
      x[n].w += y[n].w * inv * weight[n].w;
      reinterpret_cast<float4*>(line)[c] = x[n];
      alignas(16) T e[4] = {from_f<T>(x[n].x), from_f<T>(x[n].y), from_f<T>(x[n].z), from_f<T>(x[n].w)};
      if (sizeof(T) == 2) reinterpret_cast<uint2*>(out)[c] = *reinterpret_cast<const uint2*>(e);
      else reinterpret_cast<uint4*>(out)[c] = *reinterpret_cast<const uint4*>(e);
    }
  } else {
    for (int c = threadIdx.x; c < a.width; c += 512) {
      const float v = line[c] + branch_value<T>(a, row, c) * inv * a.weight[c];
      line[c] = v;
      out[c] = from_f<T>(v);
    }
  }
}

// Streams updated by a sublayer's output and collected for the next one, see StreamArgs. S: streams held (at least those there
// are). QUADS: widths that are multiples of 4 up to 8192 (what was collected stays in registers); otherwise a thread collects
// its columns twice.
template <typename T, int S, bool QUADS>
__global__ void __launch_bounds__(512) stream_step(StreamArgs a) {
  using V = std::conditional_t<QUADS, float4, float>;
  constexpr int N = QUADS ? kQuads : 1, E = QUADS ? 4 : 1;   // E: columns of a V
  __shared__ float part[16], mix[S * S], out[S], in[S];
  const int i = blockIdx.x, units = a.width / E;
  V weight[N], u[N];
  if (threadIdx.x < S * S) {
    const int from = threadIdx.x / S, to = threadIdx.x % S;
    mix[threadIdx.x] = from >= a.streams || to >= a.streams ? 0.f : a.mix ? a.mix[from * a.streams + to] : from == to ? 1.f : 0.f;
  }
  if (threadIdx.x < S) {
    const bool live = int(threadIdx.x) < a.streams;
    out[threadIdx.x] = !live ? 0.f : a.out ? a.out[threadIdx.x] : 1.f;
    in[threadIdx.x] = !live ? 0.f : a.in ? a.in[threadIdx.x] : 1.f;
  }
  if (QUADS && a.weight) {
#pragma unroll
    for (int n = 0; n < N; ++n)
      if (int c = threadIdx.x + 512 * n; c < units) weight[n] = reinterpret_cast<const V*>(a.weight)[c];
  }
  dependency_wait();
  allow_dependents();
  __syncthreads();
  const int row = a.select ? min(max(a.select[i], 0), a.limit - 1) : i;
  float* x = a.x + size_t(row) * a.streams * a.width;
  const float opened = a.branch_gate ? 1.f / (1.f + expf(-a.branch_gate[size_t(i) * a.gate_stride])) : 1.f;
  const T* parts_of = static_cast<const T*>(a.parts_of) + size_t(i) * a.parts * a.width;
  const float* scales = a.part_scale + size_t(i) * a.parts;
  auto load = [&](const void* at, int c, float (&v)[E]) {         // fp32
    if constexpr (QUADS) {
      const float4 q = static_cast<const float4*>(at)[c];
      v[0] = q.x, v[1] = q.y, v[2] = q.z, v[3] = q.w;
    } else {
      v[0] = static_cast<const float*>(at)[c];
    }
  };
  auto store = [&](float* at, int c, const float (&v)[E]) {
    if constexpr (QUADS) reinterpret_cast<float4*>(at)[c] = make_float4(v[0], v[1], v[2], v[3]);
    else at[c] = v[0];
  };
  // column unit c of what the next sublayer reads; `write`: the update comes first
  auto visit = [&](int c, bool write, float (&got)[E]) {
    float old[S][E];
#pragma unroll
    for (int s = 0; s < S; ++s) {
#pragma unroll
      for (int e = 0; e < E; ++e) old[s][e] = 0.f;
      if (s < a.streams) load(x + size_t(s) * a.width, c, old[s]);
    }
    if (write) {
      float y[E] = {};
      if (a.branch) {
        load(a.branch + size_t(i) * a.width, c, y);
#pragma unroll
        for (int e = 0; e < E; ++e) y[e] *= opened;
      }
#pragma unroll 8
      for (int k = 0; k < a.parts; ++k) {
        const float f = scales[k];
        if constexpr (QUADS) {
          const float4 v = four<T>(parts_of + size_t(k) * a.width + 4 * c);
          y[0] = fmaf(f, v.x, y[0]), y[1] = fmaf(f, v.y, y[1]), y[2] = fmaf(f, v.z, y[2]), y[3] = fmaf(f, v.w, y[3]);
        } else {
          y[0] = fmaf(f, to_f(parts_of[size_t(k) * a.width + c]), y[0]);
        }
      }
      float sum[E] = {};
#pragma unroll
      for (int e = 0; e < E; ++e) y[e] *= a.gain;
#pragma unroll
      for (int e = 0; e < E; ++e) {
        float now[S];
#pragma unroll
        for (int t = 0; t < S; ++t) {
          now[t] = out[t] * y[e];
#pragma unroll
          for (int s = 0; s < S; ++s) now[t] = fmaf(mix[s * S + t], old[s][e], now[t]);
          sum[e] += now[t];
        }
#pragma unroll
        for (int t = 0; t < S; ++t) old[t][e] = now[t];
      }
#pragma unroll
      for (int t = 0; t < S; ++t)
        if (t < a.streams) store(x + size_t(t) * a.width, c, old[t]);
      if (a.sum_of) store(a.sum_of + size_t(i) * a.width, c, sum);
    }
#pragma unroll
    for (int e = 0; e < E; ++e) {
      got[e] = 0.f;
#pragma unroll
      for (int t = 0; t < S; ++t) got[e] = fmaf(in[t], old[t][e], got[e]);
    }
  };
  float sq = 0.f;
  if constexpr (QUADS) {
#pragma unroll
    for (int n = 0; n < N; ++n) {
      const int c = threadIdx.x + 512 * n;
      float v[E] = {};
      if (c < units) visit(c, a.update, v);
      u[n] = make_float4(v[0], v[1], v[2], v[3]);
      sq += v[0] * v[0] + v[1] * v[1] + v[2] * v[2] + v[3] * v[3];
    }
  } else {
    for (int c = threadIdx.x; c < units; c += 512) {
      float v[E];
      visit(c, a.update, v);
      sq = fmaf(v[0], v[0], sq);
    }
  }
  T* normed = static_cast<T*>(a.normed) + size_t(i) * a.normed_stride;
  if (!a.weight) {
    if (!a.normed) return;
    if constexpr (QUADS) {
#pragma unroll
      for (int n = 0; n < N; ++n) {
        const int c = threadIdx.x + 512 * n;
        if (c >= units) continue;
        alignas(16) T e[4] = {from_f<T>(u[n].x), from_f<T>(u[n].y), from_f<T>(u[n].z), from_f<T>(u[n].w)};
        if (sizeof(T) == 2) reinterpret_cast<uint2*>(normed)[c] = *reinterpret_cast<const uint2*>(e);
        else reinterpret_cast<uint4*>(normed)[c] = *reinterpret_cast<const uint4*>(e);
      }
    } else {
      for (int c = threadIdx.x; c < units; c += 512) {
        float v[E];
        visit(c, false, v);
        normed[c] = from_f<T>(v[0]);
      }
    }
    return;
  }
  sq = warp_sum(sq);
  if ((threadIdx.x & 31) == 0) part[threadIdx.x >> 5] = sq;
  __syncthreads();
  sq = 0.f;
#pragma unroll
  for (int w = 0; w < 16; ++w) sq += part[w];
  const float inv = 1.f / sqrtf(sq / float(a.width) + a.eps);
  if constexpr (QUADS) {
#pragma unroll
    for (int n = 0; n < N; ++n) {
      const int c = threadIdx.x + 512 * n;
      if (c >= units) continue;
      alignas(16) T e[4] = {from_f<T>(u[n].x * inv * weight[n].x), from_f<T>(u[n].y * inv * weight[n].y), from_f<T>(u[n].z * inv * weight[n].z),
                            from_f<T>(u[n].w * inv * weight[n].w)};
      if (sizeof(T) == 2) reinterpret_cast<uint2*>(normed)[c] = *reinterpret_cast<const uint2*>(e);
      else reinterpret_cast<uint4*>(normed)[c] = *reinterpret_cast<const uint4*>(e);
    }
  } else {
    for (int c = threadIdx.x; c < units; c += 512) {   // (each thread re-reads its own columns)
      float v[E];
      visit(c, false, v);
      normed[c] = from_f<T>(v[0] * inv * a.weight[c]);
    }
  }
}

template <typename T, int S> int StreamStepAs(const Queue& q, const StreamArgs& a) {
  const bool quads = a.width % 4 == 0 && a.width <= 512 * 4 * kQuads;
  auto kernel = quads ? stream_step<T, S, true> : stream_step<T, S, false>;
  return int(Launch(kernel, dim3(unsigned(a.rows)), dim3(512), 0, q.stream, q.chained, a));
}
template <typename T> int StreamStepWith(const Queue& q, const StreamArgs& a) {
  return a.streams == 1 ? StreamStepAs<T, 1>(q, a) : a.streams == 2 ? StreamStepAs<T, 2>(q, a) : a.streams <= 4 ? StreamStepAs<T, 4>(q, a)
         : a.streams <= 8 ? StreamStepAs<T, 8>(q, a) : StreamStepAs<T, 16>(q, a);
}

__global__ void __launch_bounds__(1024) arg_max(const float* logits, int vocab, int* next) {
  __shared__ float best_v[32];
  __shared__ int best_i[32];
  dependency_wait();
  allow_dependents();
  const float* line = logits + size_t(blockIdx.x) * vocab;
  float v = -INFINITY;
  int at = 0x7fffffff;
  int rest = 0;
  if (vocab % 4 == 0) {
    rest = vocab;
    const float4* quads = reinterpret_cast<const float4*>(line);
#pragma unroll 8
    for (int i = threadIdx.x; i < vocab / 4; i += 1024) {
      const float4 four = quads[i];
      const float x[4] = {four.x, four.y, four.z, four.w};
#pragma unroll
      for (int j = 0; j < 4; ++j)
        if (x[j] > v || at == 0x7fffffff) {
          v = x[j];
          at = 4 * i + j;
        }
    }
  }
  for (int i = rest + threadIdx.x; i < vocab; i += 1024)
    if (line[i] > v || at == 0x7fffffff) {
      v = line[i];
      at = i;
    }
  auto better = [](float a, int ia, float b, int ib) { return a > b || (a == b && ia < ib); };
  for (int o = 16; o; o >>= 1) {
    const float ov = __shfl_xor_sync(0xffffffffu, v, o);
    const int oi = __shfl_xor_sync(0xffffffffu, at, o);
    if (better(ov, oi, v, at)) {
      v = ov;
      at = oi;
    }
  }
  if ((threadIdx.x & 31) == 0) {
    best_v[threadIdx.x >> 5] = v;
    best_i[threadIdx.x >> 5] = at;
  }
  __syncthreads();
  if (threadIdx.x == 0) {
    for (int w = 1; w < 32; ++w)
      if (better(best_v[w], best_i[w], v, at)) {
        v = best_v[w];
        at = best_i[w];
      }
    next[blockIdx.x] = min(at, vocab - 1);
  }
}

__global__ void feed(Entry* entries, int count, const int* next, int* tokens, int capacity) {
  dependency_wait();
  const int i = blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= count) return;
  tokens[i] = next[i];
  entries[i].first_position = min(entries[i].first_position + 1, capacity - 1);
}

}  // namespace

int StartStep(const Queue& q, const StepRows& r, const int* tokens, const void* embed, float* x, int streams, void* copy, int copy_stride, int width,
              int vocab, float scale) {
  const dim3 grid(unsigned(r.rows));
  if (q.f32)
    return int(Launch(start_step<float>, grid, dim3(256), 0, q.stream, false, r, tokens, static_cast<const float*>(embed), x, streams, static_cast<float*>(copy),
                      copy_stride, width, vocab, scale));
  return int(Launch(start_step<__nv_bfloat16>, grid, dim3(256), 0, q.stream, false, r, tokens, static_cast<const __nv_bfloat16*>(embed), x, streams,
                    static_cast<__nv_bfloat16*>(copy), copy_stride, width, vocab, scale));
}

int RmsNorm(const Queue& q, const NormArgs& a) {
  if (a.rows <= 0) return 0;
  if (a.width % 4 == 0 && a.width <= 512 * 4 * kQuads) {
    auto quads = q.f32 ? rms_norm_quads<float> : rms_norm_quads<__nv_bfloat16>;
    return int(Launch(quads, dim3(unsigned(a.rows)), dim3(512), 0, q.stream, q.chained, a));
  }
  auto kernel = q.f32 ? rms_norm<float> : rms_norm<__nv_bfloat16>;
  return int(Launch(kernel, dim3(unsigned(a.rows)), dim3(256), 0, q.stream, q.chained, a));
}

int AddNorm(const Queue& q, const AddNormArgs& a) {
  if (a.rows <= 0) return 0;
  const bool quads = a.width % 4 == 0 && a.width <= 512 * 4 * kQuads;
  auto kernel = q.f32 ? (quads ? add_norm<float, true> : add_norm<float, false>)
                      : (quads ? add_norm<__nv_bfloat16, true> : add_norm<__nv_bfloat16, false>);
  return int(Launch(kernel, dim3(unsigned(a.rows)), dim3(512), 0, q.stream, q.chained, a));
}

int StreamStep(const Queue& q, const StreamArgs& a) {
  if (a.rows <= 0) return 0;
  if (a.streams < 1 || a.streams > kMaxStreams || (a.update && a.select)) return int(cudaErrorInvalidValue);
  return q.f32 ? StreamStepWith<float>(q, a) : StreamStepWith<__nv_bfloat16>(q, a);
}

int ArgMax(const Queue& q, const float* logits, int rows, int vocab, int* next) {
  if (rows <= 0) return 0;
  return int(Launch(arg_max, dim3(unsigned(rows)), dim3(1024), 0, q.stream, q.chained, logits, vocab, next));
}

int Feed(const Queue& q, Entry* entries, int count, const int* next, int* tokens, int capacity) {
  return int(Launch(feed, dim3(unsigned((count + 127) / 128)), dim3(128), 0, q.stream, q.chained, entries, count, next, tokens, capacity));
}

}  // namespace tmb
