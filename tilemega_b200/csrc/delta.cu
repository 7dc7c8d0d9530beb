// The generalised delta rule of ragged steps, see DeltaArgs, by its recurrence in fp32 (both element types). With the old
// state S, p = u^T S and q = (w r)^T S of a column come out of one pass over it, and with them
//   S' = diag(w) S - (a u) p + k v,      o = S'^T r = q - (r . a u) p + (r . k) v,
// so a token costs one reduction over the key channels. Columns of a state do not meet: a warp owns four, a lane every eighth
// four of a column's key channels, and states lie with a column's key channels contiguous.
#include <cuda_bf16.h>

#include <algorithm>

#include "element.cuh"
#include "mixers.cuh"
#include "ops.h"
#include "ptx.cuh"
#include "tensor_map.h"

namespace tmb {
namespace {

struct DeltaParams {
  const void* proj;
  const float* z;
  float *state, *raw;
  void* out;
  const float* norm;
  int proj_stride, out_stride, heads, dim, padded;
  float decay_scale, unit_eps, eps;
  bool wide;                             // four neighbours of a head can be loaded at a time
};

enum { kUnit, kTurnedDecay, kDecay, kRemoval, kKey, kVectors };   // u, r w, w, a u, k
constexpr int kScalars = 4;              // r . a u, r . k

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

// What one token brings, by one warp: the vectors of its head, DP floats each (zeros behind the head), then the scalars.
template <typename T, int DP> __device__ __forceinline__ void stage_token(const DeltaParams& p, int row, int head, int lane, float* to) {
  constexpr int M = (DP / 4 + 31) / 32;
  const T* r = static_cast<const T*>(p.proj) + size_t(row) * p.proj_stride + size_t(head) * p.dim;
  const size_t all = size_t(p.heads) * p.dim;
  const float* z = p.z + size_t(row) * all + size_t(head) * p.dim;
  float rv[M][4], kv[M][4], av[M][4], zv[M][4], square = 0.f;
#pragma unroll
  for (int m = 0; m < M; ++m) {
    const int d = 4 * (lane + 32 * m), count = min(4, p.dim - d);
    load_four(r + d, count, p.wide, rv[m]);
    load_four(r + all + d, count, p.wide, kv[m]);
    load_four(r + 3 * all + d, count, p.wide, av[m]);
    load_four(z + d, count, p.wide, zv[m]);
#pragma unroll
    for (int i = 0; i < 4; ++i) square = fmaf(kv[m][i], kv[m][i], square);
  }
  const float inv = 1.f / sqrtf(warp_sum(square) + p.unit_eps);
  float ra = 0.f, rk = 0.f;
#pragma unroll
  for (int m = 0; m < M; ++m) {
    const int d = 4 * (lane + 32 * m);
    float vec[kVectors][4];
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const bool live = d + i < p.dim;
      const float u = kv[m][i] * inv, w = live ? expf(-p.decay_scale * sigmoid(zv[m][i])) : 0.f;
      vec[kUnit][i] = u;
      vec[kTurnedDecay][i] = rv[m][i] * w;
      vec[kDecay][i] = w;
      vec[kRemoval][i] = u * sigmoid(av[m][i]);
      vec[kKey][i] = kv[m][i];
      ra = fmaf(rv[m][i], vec[kRemoval][i], ra);
      rk = fmaf(rv[m][i], kv[m][i], rk);
    }
    if (d < DP)
#pragma unroll
      for (int n = 0; n < kVectors; ++n) *reinterpret_cast<float4*>(to + n * DP + d) = make_float4(vec[n][0], vec[n][1], vec[n][2], vec[n][3]);
  }
  ra = warp_sum(ra);
  rk = warp_sum(rk);
  if (lane == 0) {
    to[kVectors * DP] = ra;
    to[kVectors * DP + 1] = rk;
  }
}

// One token on a lane's share of a column: returns o, the same in all lanes of the column.
template <int NQ> __device__ __forceinline__ float advance(float4 (&s)[NQ], const float* token, int group, float v) {
  constexpr int DP = NQ * 32;
  float p0 = 0.f, p1 = 0.f, q0 = 0.f, q1 = 0.f;
  const float4* vec = reinterpret_cast<const float4*>(token) + group;
#pragma unroll
  for (int i = 0; i < NQ; ++i) {
    const float4 u = vec[kUnit * DP / 4 + 8 * i], rw = vec[kTurnedDecay * DP / 4 + 8 * i];
    p0 = fmaf(u.x, s[i].x, p0);
    q0 = fmaf(rw.x, s[i].x, q0);
    p1 = fmaf(u.y, s[i].y, p1);
    q1 = fmaf(rw.y, s[i].y, q1);
    p0 = fmaf(u.z, s[i].z, p0);
    q0 = fmaf(rw.z, s[i].z, q0);
    p1 = fmaf(u.w, s[i].w, p1);
    q1 = fmaf(rw.w, s[i].w, q1);
  }
  float p = p0 + p1, q = q0 + q1;
#pragma unroll
  for (int o = 4; o < 32; o <<= 1) {
    p += __shfl_xor_sync(0xffffffffu, p, o);
    q += __shfl_xor_sync(0xffffffffu, q, o);
  }
#pragma unroll
  for (int i = 0; i < NQ; ++i) {
    const float4 w = vec[kDecay * DP / 4 + 8 * i], a = vec[kRemoval * DP / 4 + 8 * i], k = vec[kKey * DP / 4 + 8 * i];
    s[i].x = fmaf(w.x, s[i].x, fmaf(-a.x, p, k.x * v));
    s[i].y = fmaf(w.y, s[i].y, fmaf(-a.y, p, k.y * v));
    s[i].z = fmaf(w.z, s[i].z, fmaf(-a.z, p, k.z * v));
    s[i].w = fmaf(w.w, s[i].w, fmaf(-a.w, p, k.w * v));
  }
  return fmaf(token[kVectors * DP + 1], v, fmaf(-token[kVectors * DP], p, q));
}

// An entry's rows one after the other, 32 columns of a head a CTA: warps 0 .. 7 own the columns, warps 8 .. 15 stage the next
// batch of tokens meanwhile, one each. blockIdx = (slice, head, entry).
constexpr int kBatch = 8, kSlice = 32, kStepThreads = 512;
template <int NQ> constexpr int kTokenFloats = kVectors * NQ * 32 + kScalars;
template <int NQ> constexpr int kStepMemory = 2 * kBatch * (kTokenFloats<NQ> + kSlice) * 4;

template <typename T, int NQ>
__global__ void __launch_bounds__(kStepThreads, 1) delta_steps(StepRows r, DeltaParams p, bool portions_only) {
  extern __shared__ __align__(16) float tokens[];         // [2][kBatch][vectors, scalars], then [2][kBatch][kSlice] values
  float* values = tokens + 2 * kBatch * kTokenFloats<NQ>;
  dependency_wait();
  allow_dependents();
  const Entry e = r.entry[blockIdx.z];
  if (portions_only && e.rows == 1) return;
  const int head = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, group = lane >> 2;
  const int mine = warp * 4 + (lane & 3), column = blockIdx.x * kSlice + mine;
  const size_t all = size_t(p.heads) * p.dim;
  const bool owner = warp < kBatch, live = owner && column < p.dim;
  float* state = p.state + ((size_t(e.slot) * p.heads + head) * p.dim + min(column, p.dim - 1)) * p.padded;
  float4 s[NQ];
#pragma unroll
  for (int i = 0; i < NQ; ++i) {
    const int d = 4 * (group + 8 * i);
    s[i] = live && e.first_position > 0 && d < p.padded ? *reinterpret_cast<const float4*>(state + d) : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  const int batches = (e.rows + kBatch - 1) / kBatch;
  auto stage = [&](int batch) {                            // (the staging warps)
    const int t = batch * kBatch + warp - kBatch, at = (batch & 1) * kBatch + warp - kBatch;
    if (t >= e.rows) return;
    const int row = e.first_row + t, c = blockIdx.x * kSlice + lane;
    values[at * kSlice + lane] = c < p.dim ? to_f(static_cast<const T*>(p.proj)[size_t(row) * p.proj_stride + 2 * all + size_t(head) * p.dim + c]) : 0.f;
    stage_token<T, NQ * 32>(p, row, head, lane, tokens + at * kTokenFloats<NQ>);
  };
  if (!owner) stage(0);
  for (int batch = 0; batch < batches; ++batch) {
    __syncthreads();
    if (!owner) {
      if (batch + 1 < batches) stage(batch + 1);
      continue;
    }
    const int t0 = batch * kBatch, n = min(kBatch, e.rows - t0);
    for (int t = 0; t < n; ++t) {
      const int at = (batch & 1) * kBatch + t;
      const float o = advance<NQ>(s, tokens + at * kTokenFloats<NQ>, group, values[at * kSlice + mine]);
      if (group == 0 && live) p.raw[size_t(e.first_row + t0 + t) * all + size_t(head) * p.dim + column] = o;
    }
  }
#pragma unroll
  for (int i = 0; i < NQ; ++i) {
    const int d = 4 * (group + 8 * i);
    if (live && d < p.padded) *reinterpret_cast<float4*>(state + d) = s[i];
  }
}

// One decoded token of an entry, whole: recurrence, per-head norm and gate. A CTA holds one head's state, a lane its share of
// PASSES columns; every load of the state is in flight before the first is used. blockIdx = (head, entry).
constexpr int kTokenThreads = 512, kTokenColumns = kTokenThreads / 8;

template <typename T, int NQ, int PASSES>
__global__ void __launch_bounds__(kTokenThreads, NQ * PASSES <= 8 ? 2 : 1) delta_token(StepRows r, DeltaParams p) {
  __shared__ __align__(16) float token[kTokenFloats<NQ>];
  __shared__ float part[kTokenThreads / 32], outputs[PASSES * kTokenColumns];
  const Entry e = r.entry[blockIdx.y];   // (tables and states: written before the kernel this one depends on)
  if (e.rows != 1) {
    dependency_wait();
    allow_dependents();
    return;
  }
  const int head = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, group = lane >> 2;
  float* state = p.state + (size_t(e.slot) * p.heads + head) * p.dim * p.padded;
  float4 s[PASSES][NQ];
#pragma unroll
  for (int n = 0; n < PASSES; ++n) {
    const int column = n * kTokenColumns + warp * 4 + (lane & 3);
#pragma unroll
    for (int i = 0; i < NQ; ++i) {
      const int d = 4 * (group + 8 * i);
      s[n][i] = column < p.dim && d < p.padded && e.first_position > 0 ? __ldcs(reinterpret_cast<const float4*>(state + size_t(column) * p.padded + d))
                                                                      : make_float4(0.f, 0.f, 0.f, 0.f);
    }
  }
  const int c = threadIdx.x;             // (a head has at most kTokenThreads columns)
  const float weight = c < p.dim ? p.norm[size_t(head) * p.dim + c] : 0.f;
  dependency_wait();
  allow_dependents();
  const size_t all = size_t(p.heads) * p.dim;
  const T* line = static_cast<const T*>(p.proj) + size_t(e.first_row) * p.proj_stride + size_t(head) * p.dim;
  const float gate = c < p.dim ? to_f(line[4 * all + c]) : 0.f;
  float v[PASSES];
#pragma unroll
  for (int n = 0; n < PASSES; ++n) {
    const int column = n * kTokenColumns + warp * 4 + (lane & 3);
    v[n] = column < p.dim ? to_f(line[2 * all + column]) : 0.f;
  }
  if (warp == 0) stage_token<T, NQ * 32>(p, e.first_row, head, lane, token);
  __syncthreads();
#pragma unroll
  for (int n = 0; n < PASSES; ++n) {
    const int column = n * kTokenColumns + warp * 4 + (lane & 3);
    const float o = advance<NQ>(s[n], token, group, v[n]);
    if (group == 0) outputs[column] = column < p.dim ? o : 0.f;
    if (column < p.dim)
#pragma unroll
      for (int i = 0; i < NQ; ++i) {
        const int d = 4 * (group + 8 * i);
        if (d < p.padded) __stcs(reinterpret_cast<float4*>(state + size_t(column) * p.padded + d), s[n][i]);
      }
  }
  __syncthreads();
  const float o = c < p.dim ? outputs[c] : 0.f;
  float square = warp_sum(o * o);
  if (lane == 0) part[warp] = square;
  __syncthreads();
  square = 0.f;
#pragma unroll
  for (int w = 0; w < kTokenThreads / 32; ++w) square += part[w];
  if (c < p.dim)
    static_cast<T*>(p.out)[size_t(e.first_row) * p.out_stride + size_t(head) * p.dim + c] =
        from_f<T>(o * (1.f / sqrtf(square / float(p.dim) + p.eps)) * weight * sigmoid(gate));
}

constexpr int kWholeHead = 192;          // widest head whose state one CTA holds

template <typename T, int NQ> int StepsWith(const Queue& q, const StepRows& r, const DeltaParams& p, bool portions_only) {
  return int(Launch(delta_steps<T, NQ>, dim3(unsigned((p.dim + kSlice - 1) / kSlice), unsigned(p.heads), unsigned(r.entries)), dim3(kStepThreads),
                    kStepMemory<NQ>, q.stream, q.chained, r, p, portions_only));
}

template <typename T> int DeltaAs(const Queue& q, const StepRows& r, const DeltaArgs& a) {
  const T* proj = static_cast<const T*>(a.proj);
  const bool wide = a.dim % 4 == 0 && a.proj_stride % 4 == 0 && reinterpret_cast<uintptr_t>(proj) % (4 * sizeof(T)) == 0;
  const DeltaParams p{a.proj, a.z, a.state, a.raw, a.out, a.norm, a.proj_stride, a.out_stride, a.heads, a.dim, a.padded, a.decay_scale, a.unit_eps, a.eps, wide};
  const int quads = (a.dim + 31) / 32;
  const bool whole = a.dim <= kWholeHead;
  int status = 0;
  if (r.singles < r.entries || !whole) {
    status = quads <= 1 ? StepsWith<T, 1>(q, r, p, whole) : quads <= 2 ? StepsWith<T, 2>(q, r, p, whole) : quads <= 3 ? StepsWith<T, 3>(q, r, p, whole)
             : quads <= 4 ? StepsWith<T, 4>(q, r, p, whole) : quads <= 6 ? StepsWith<T, 6>(q, r, p, whole) : StepsWith<T, 8>(q, r, p, whole);
    if (status == 0)
      status = HeadGate(q, {a.raw, a.proj, a.proj_stride, 4 * a.heads * a.dim, a.out, a.out_stride, r.rows, a.heads, a.dim, a.norm, false, a.eps});
  }
  if (status != 0 || r.singles == 0 || !whole) return status;
  // (behind the gate of all rows, whose result for the single tokens it replaces)
  auto kernel = quads <= 1 ? delta_token<T, 1, 1> : quads <= 2 ? delta_token<T, 2, 1> : quads <= 3 ? delta_token<T, 3, 2> : quads <= 4 ? delta_token<T, 4, 2>
                                                                                                                        : delta_token<T, 6, 3>;
  return int(Launch(kernel, dim3(unsigned(a.heads), unsigned(r.entries)), dim3(kTokenThreads), 0, q.stream, q.chained, r, p));
}

template <typename T, int NQ> cudaError_t Raise() {
  return cudaFuncSetAttribute(delta_steps<T, NQ>, cudaFuncAttributeMaxDynamicSharedMemorySize, kStepMemory<NQ>);
}
template <typename T> cudaError_t RaiseAll() {
  for (cudaError_t err : {Raise<T, 1>(), Raise<T, 2>(), Raise<T, 3>(), Raise<T, 4>(), Raise<T, 6>(), Raise<T, 8>()})
    if (err != cudaSuccess) return err;
  return cudaSuccess;
}

}  // namespace

int Delta(const Queue& q, const StepRows& r, const DeltaArgs& a) {
  if (a.dim > kMaxHeadDim || a.padded % 4 || a.padded < a.dim) return int(cudaErrorInvalidValue);
  return q.f32 ? DeltaAs<float>(q, r, a) : DeltaAs<__nv_bfloat16>(q, r, a);
}

int PrepareDelta() {
  const cudaError_t err = RaiseAll<float>();
  return int(err == cudaSuccess ? RaiseAll<__nv_bfloat16>() : err);
}

}  // namespace tmb
