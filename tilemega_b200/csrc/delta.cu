// The generalised delta rule of ragged steps, see DeltaArgs, by its recurrence in fp32: decoded tokens, and the portions of fp32 plans
// (those of bf16 plans: delta_mma.cu). With the old
// state S, p = u^T S and q = (w r)^T S of a column come out of one pass over it, and with them
//   S' = diag(w) S - (a u) p + k v,      o = S'^T r = q - (r . a u) p + (r . k) v,
// so a token costs one reduction over the key channels (and so do two, see below). Columns of a state do not meet: warps own some
// each, lanes some of their key channels, and states lie with a column's key channels contiguous.
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

// One token on a lane's share of a column (every eighth four of its key channels): returns o, the same in all lanes of the column.
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

// ---- portions (fp32 plans): two tokens a turn ------------------------------------------------------------------------------------------
// With the tokens 0 and 1 of a pair, both reductions are taken against the state S before them:
//   p0 = u0^T S,  p1 = (w0 u1)^T S - (u1 . a0) p0 + (u1 . k0) v0,      a = removal rate times unit key
//   o0 = (w0 r0)^T S - (r0 . a0) p0 + (r0 . k0) v0
//   o1 = (w0 w1 r1)^T S - (w1 r1 . a0) p0 + (w1 r1 . k0) v0 - (r1 . a1) p1 + (r1 . k1) v1
//   S' = diag(w0 w1) S - (w1 a0) p0 + (w1 k0) v0 - a1 p1 + k1 v1
// A missing second token is one without a key, a query and a decay. A warp owns 32 / G groups of four columns, a lane every G-th
// four of their key channels; sixteen sums (two kinds, two tokens, four columns) meet by halving the list at every step.
enum { kU0, kR0, kU1, kR1, kW01, kA0, kK0, kA1, kK1, kPairVectors };
enum { kU1A0, kU1K0, kR0A0, kR0K0, kR1A0, kR1K0, kR1A1, kR1K1, kPairScalars };
constexpr int kPairs = 8, kOwners = 4, kPairThreads = 32 * (kOwners + kPairs);   // pairs a batch; warps that own columns
template <int G, int NQ> struct PairShape {
  static constexpr int DP = 4 * G * NQ;                    // key channels, padded
  static constexpr int kColumns = 4 * 32 / G, kSlice = kOwners * kColumns;   // of a warp, of a CTA
  static constexpr int kFloats = kPairVectors * DP + kPairScalars + 2 * kSlice;
  static constexpr int kMemory = 2 * kPairs * kFloats * 4;
};

// Sums over the warp of eight values each, the lane >> 2-th of them in every lane.
__device__ __forceinline__ float sum_eight(float (&v)[8], int lane) {
#pragma unroll
  for (int half = 4; half; half >>= 1) {
    const bool upper = lane & (4 * half);
#pragma unroll
    for (int j = 0; j < half; ++j) {
      const float keep = upper ? v[j + half] : v[j], send = upper ? v[j] : v[j + half];
      v[j] = keep + __shfl_xor_sync(0xffffffffu, send, 4 * half);
    }
  }
  v[0] += __shfl_xor_sync(0xffffffffu, v[0], 2);
  v[0] += __shfl_xor_sync(0xffffffffu, v[0], 1);
  return v[0];
}

// What a pair of tokens brings, by one warp: the vectors, the scalars, then the values of the CTA's columns.
template <int G, int NQ>
__device__ __forceinline__ void stage_pair(const DeltaParams& p, int row, bool second, int head, int column0, int lane, float* to) {
  using Shape = PairShape<G, NQ>;
  constexpr int DP = Shape::DP, M = (DP / 4 + 31) / 32;
  const size_t all = size_t(p.heads) * p.dim;
  const float* line = static_cast<const float*>(p.proj) + size_t(row) * p.proj_stride + size_t(head) * p.dim;
  const float* z = p.z + size_t(row) * all + size_t(head) * p.dim;
  float rv[2][M][4], kv[2][M][4], av[2][M][4], wv[2][M][4], square[2] = {};
#pragma unroll
  for (int t = 0; t < 2; ++t)
#pragma unroll
    for (int m = 0; m < M; ++m) {
      const int d = 4 * (lane + 32 * m), count = t == 0 || second ? min(4, p.dim - d) : 0;
      const float* r = line + size_t(t) * p.proj_stride + d;
      load_four(r, count, p.wide, rv[t][m]);
      load_four(r + all, count, p.wide, kv[t][m]);
      load_four(r + 3 * all, count, p.wide, av[t][m]);
      load_four(z + size_t(t) * all + d, count, p.wide, wv[t][m]);
    }
  float value[2 * Shape::kSlice / 32];
#pragma unroll
  for (int i = 0; i < 2 * Shape::kSlice / 32; ++i) {
    const int at = lane + 32 * i, t = at / Shape::kSlice, c = column0 + at % Shape::kSlice;
    value[i] = c < p.dim && (t == 0 || second) ? line[size_t(t) * p.proj_stride + 2 * all + c] : 0.f;
  }
#pragma unroll
  for (int t = 0; t < 2; ++t) {
#pragma unroll
    for (int m = 0; m < M; ++m)
#pragma unroll
      for (int i = 0; i < 4; ++i) square[t] = fmaf(kv[t][m][i], kv[t][m][i], square[t]);
    square[t] = 1.f / sqrtf(warp_sum(square[t]) + p.unit_eps);
  }
  float scalar[8] = {};
#pragma unroll
  for (int m = 0; m < M; ++m) {
    const int d = 4 * (lane + 32 * m);
    float vec[kPairVectors][4];
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const bool live = d + i < p.dim;
      float u[2], a[2], w[2];
#pragma unroll
      for (int t = 0; t < 2; ++t) {
        u[t] = kv[t][m][i] * square[t];
        a[t] = u[t] * sigmoid(av[t][m][i]);
        w[t] = !live ? 0.f : t == 0 || second ? expf(-p.decay_scale * sigmoid(wv[t][m][i])) : 1.f;
      }
      const float r0 = rv[0][m][i], r1 = rv[1][m][i], k0 = kv[0][m][i], k1 = kv[1][m][i], r1w = r1 * w[1];
      vec[kU0][i] = u[0];
      vec[kR0][i] = r0 * w[0];
      vec[kU1][i] = u[1] * w[0];
      vec[kR1][i] = r1w * w[0];
      vec[kW01][i] = w[0] * w[1];
      vec[kA0][i] = a[0] * w[1];
      vec[kK0][i] = k0 * w[1];
      vec[kA1][i] = a[1];
      vec[kK1][i] = k1;
      scalar[kU1A0] = fmaf(u[1], a[0], scalar[kU1A0]);
      scalar[kU1K0] = fmaf(u[1], k0, scalar[kU1K0]);
      scalar[kR0A0] = fmaf(r0, a[0], scalar[kR0A0]);
      scalar[kR0K0] = fmaf(r0, k0, scalar[kR0K0]);
      scalar[kR1A0] = fmaf(r1w, a[0], scalar[kR1A0]);
      scalar[kR1K0] = fmaf(r1w, k0, scalar[kR1K0]);
      scalar[kR1A1] = fmaf(r1, a[1], scalar[kR1A1]);
      scalar[kR1K1] = fmaf(r1, k1, scalar[kR1K1]);
    }
    if (d < DP)
#pragma unroll
      for (int n = 0; n < kPairVectors; ++n) *reinterpret_cast<float4*>(to + n * DP + d) = make_float4(vec[n][0], vec[n][1], vec[n][2], vec[n][3]);
  }
  const float sum = sum_eight(scalar, lane);
  if ((lane & 3) == 0) to[kPairVectors * DP + lane / 4] = sum;
#pragma unroll
  for (int i = 0; i < 2 * Shape::kSlice / 32; ++i) to[kPairVectors * DP + kPairScalars + lane + 32 * i] = value[i];
}

// An entry's rows in pairs, a slice of a head's columns a CTA: the first warps own the columns, the others stage the next batch of
// pairs meanwhile, one each. blockIdx = (slice, head, entry).
template <int G, int NQ>
__global__ void __launch_bounds__(kPairThreads, 1) delta_pairs(StepRows r, DeltaParams p, bool portions_only) {
  using Shape = PairShape<G, NQ>;
  constexpr int DP = Shape::DP;
  extern __shared__ __align__(16) float pairs[];           // [2][kPairs]
  dependency_wait();
  allow_dependents();
  const Entry e = r.entry[blockIdx.z];
  if (portions_only && e.rows == 1) return;
  const int head = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, part = lane & (G - 1);
  const int column0 = blockIdx.x * Shape::kSlice, mine = warp * Shape::kColumns + lane / G * 4;   // the lane's four columns, in the slice
  const size_t all = size_t(p.heads) * p.dim;
  const bool owner = warp < kOwners;
  float* state = p.state + (size_t(e.slot) * p.heads + head) * p.dim * p.padded;
  float4 s[NQ][4];
  auto each_state = [&](auto&& visit) {
#pragma unroll
    for (int i = 0; i < NQ; ++i)
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        const int column = column0 + mine + c, d = 4 * (part + G * i);
        if (owner && column < p.dim && d < p.padded) visit(*reinterpret_cast<float4*>(state + size_t(column) * p.padded + d), s[i][c]);
      }
  };
#pragma unroll
  for (int i = 0; i < NQ; ++i)
#pragma unroll
    for (int c = 0; c < 4; ++c) s[i][c] = make_float4(0.f, 0.f, 0.f, 0.f);
  if (e.first_position > 0) each_state([](const float4& from, float4& to) { to = from; });
  const int count = (e.rows + 1) / 2, batches = (count + kPairs - 1) / kPairs;
  auto stage = [&](int batch) {                            // (the staging warps)
    const int n = batch * kPairs + warp - kOwners;
    if (n < count)
      stage_pair<G, NQ>(p, e.first_row + 2 * n, 2 * n + 1 < e.rows, head, column0, lane,
                           pairs + size_t((batch & 1) * kPairs + warp - kOwners) * Shape::kFloats);
  };
  if (!owner) stage(0);
  // (which sum a lane ends up with)
  const int held = G == 32 ? lane >> 1 : lane & 15, held_column = held & 3, home = G == 32 ? 0 : lane & 16;
  const bool query = held & 8, later = held & 4, writes = query && (G != 32 || (lane & 1) == 0) && column0 + mine + held_column < p.dim;
  auto pick = [&](const float (&v)[4]) { return held_column & 2 ? (held_column & 1 ? v[3] : v[2]) : (held_column & 1 ? v[1] : v[0]); };
  for (int batch = 0; batch < batches; ++batch) {
    __syncthreads();
    if (!owner) {
      if (batch + 1 < batches) stage(batch + 1);
      continue;
    }
    const int n0 = batch * kPairs, here = min(kPairs, count - n0);
    for (int n = 0; n < here; ++n) {
      const float* pair = pairs + size_t((batch & 1) * kPairs + n) * Shape::kFloats;
      const float4* vec = reinterpret_cast<const float4*>(pair) + part;
      auto get = [&](int which, int i) { return vec[which * (DP / 4) + G * i]; };
      float x[16] = {};                                    // [kind][token][column]
#pragma unroll
      for (int i = 0; i < NQ; ++i) {
        const float4 by[4] = {get(kU0, i), get(kU1, i), get(kR0, i), get(kR1, i)};
#pragma unroll
        for (int b = 0; b < 4; ++b)
#pragma unroll
          for (int c = 0; c < 4; ++c) {
            float v = x[4 * b + c];
            v = fmaf(by[b].x, s[i][c].x, v);
            v = fmaf(by[b].y, s[i][c].y, v);
            v = fmaf(by[b].z, s[i][c].z, v);
            x[4 * b + c] = fmaf(by[b].w, s[i][c].w, v);
          }
      }
#pragma unroll
      for (int half = 8; half; half >>= 1) {
        const int mask = G == 32 ? 2 * half : half;
        const bool upper = lane & mask;
#pragma unroll
        for (int j = 0; j < half; ++j) {
          const float keep = upper ? x[j + half] : x[j], send = upper ? x[j] : x[j + half];
          x[j] = keep + __shfl_xor_sync(0xffffffffu, send, mask);
        }
      }
      float sum = x[0];
      if (G == 32) sum += __shfl_xor_sync(0xffffffffu, sum, 1);
      const float4 c01 = *reinterpret_cast<const float4*>(pair + kPairVectors * DP), c23 = *reinterpret_cast<const float4*>(pair + kPairVectors * DP + 4);
      const float4 v0q = *reinterpret_cast<const float4*>(pair + kPairVectors * DP + kPairScalars + mine);
      const float4 v1q = *reinterpret_cast<const float4*>(pair + kPairVectors * DP + kPairScalars + Shape::kSlice + mine);
      const float v0[4] = {v0q.x, v0q.y, v0q.z, v0q.w}, v1[4] = {v1q.x, v1q.y, v1q.z, v1q.w};
      float p0[4], p1[4];
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        p0[c] = __shfl_sync(0xffffffffu, sum, G == 32 ? 2 * c : home + c);
        p1[c] = __shfl_sync(0xffffffffu, sum, G == 32 ? 8 + 2 * c : home + 4 + c);
        p1[c] = fmaf(c01.y, v0[c], fmaf(-c01.x, p0[c], p1[c]));
      }
#pragma unroll
      for (int i = 0; i < NQ; ++i) {
        const float4 w = get(kW01, i), a0 = get(kA0, i), k0 = get(kK0, i), a1 = get(kA1, i), k1 = get(kK1, i);
#pragma unroll
        for (int c = 0; c < 4; ++c) {
          s[i][c].x = fmaf(w.x, s[i][c].x, fmaf(-a0.x, p0[c], fmaf(k0.x, v0[c], fmaf(-a1.x, p1[c], k1.x * v1[c]))));
          s[i][c].y = fmaf(w.y, s[i][c].y, fmaf(-a0.y, p0[c], fmaf(k0.y, v0[c], fmaf(-a1.y, p1[c], k1.y * v1[c]))));
          s[i][c].z = fmaf(w.z, s[i][c].z, fmaf(-a0.z, p0[c], fmaf(k0.z, v0[c], fmaf(-a1.z, p1[c], k1.z * v1[c]))));
          s[i][c].w = fmaf(w.w, s[i][c].w, fmaf(-a0.w, p0[c], fmaf(k0.w, v0[c], fmaf(-a1.w, p1[c], k1.w * v1[c]))));
        }
      }
      const int t = 2 * (n0 + n) + (later ? 1 : 0);
      if (writes && t < e.rows) {
        float o = fmaf(later ? c23.y : c01.w, pick(v0), fmaf(later ? -c23.x : -c01.z, pick(p0), sum));
        if (later) o = fmaf(c23.w, pick(v1), fmaf(-c23.z, pick(p1), o));
        p.raw[size_t(e.first_row + t) * all + size_t(head) * p.dim + column0 + mine + held_column] = o;
      }
    }
  }
  each_state([](float4& to, const float4& from) { to = from; });
}

// ---- one decoded token ------------------------------------------------------------------------------------------------------
// One decoded token of an entry, whole: recurrence, per-head norm and gate. A CTA holds one head's state, a lane its share of
// PASSES columns; every load of the state is in flight before the first is used. blockIdx = (head, entry).
template <int NQ> constexpr int kTokenFloats = kVectors * NQ * 32 + kScalars;
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

template <int G, int NQ> int PairsWith(const Queue& q, const StepRows& r, const DeltaParams& p, bool portions_only) {
  using Shape = PairShape<G, NQ>;
  return int(Launch(delta_pairs<G, NQ>, dim3(unsigned((p.dim + Shape::kSlice - 1) / Shape::kSlice), unsigned(p.heads), unsigned(r.entries)),
                    dim3(kPairThreads), Shape::kMemory, q.stream, q.chained, r, p, portions_only));
}

template <typename T> int DeltaAs(const Queue& q, const StepRows& r, const DeltaArgs& a) {
  const T* proj = static_cast<const T*>(a.proj);
  const bool wide = a.dim % 4 == 0 && a.proj_stride % 4 == 0 && reinterpret_cast<uintptr_t>(proj) % (4 * sizeof(T)) == 0;
  const DeltaParams p{a.proj, a.z, a.state, a.raw, a.out, a.norm, a.proj_stride, a.out_stride, a.heads, a.dim, a.padded, a.decay_scale, a.unit_eps, a.eps, wide};
  const int quads = (a.dim + 31) / 32;
  const bool whole = a.dim <= kWholeHead;
  int status = 0;
  if (r.singles < r.entries || !whole) {
    if (!q.f32) status = DeltaChunks(q, r, a, whole);
    else status = p.dim <= 64 ? PairsWith<16, 1>(q, r, p, whole) : p.dim <= 128 ? PairsWith<32, 1>(q, r, p, whole) : PairsWith<32, 2>(q, r, p, whole);
    if (status == 0)
      status = HeadGate(q, {a.raw, a.proj, a.proj_stride, 4 * a.heads * a.dim, a.out, a.out_stride, r.rows, a.heads, a.dim, a.norm, false, a.eps});
  }
  if (status != 0 || r.singles == 0 || !whole) return status;
  // (behind the gate of all rows, whose result for the single tokens it replaces)
  auto kernel = quads <= 1 ? delta_token<T, 1, 1> : quads <= 2 ? delta_token<T, 2, 1> : quads <= 3 ? delta_token<T, 3, 2> : quads <= 4 ? delta_token<T, 4, 2>
                                                                                                                        : delta_token<T, 6, 3>;
  return int(Launch(kernel, dim3(unsigned(a.heads), unsigned(r.entries)), dim3(kTokenThreads), 0, q.stream, q.chained, r, p));
}

template <int G, int NQ> cudaError_t Raise() {
  return cudaFuncSetAttribute(delta_pairs<G, NQ>, cudaFuncAttributeMaxDynamicSharedMemorySize, PairShape<G, NQ>::kMemory);
}
}  // namespace

int Delta(const Queue& q, const StepRows& r, const DeltaArgs& a) {
  if (a.dim > kMaxHeadDim || a.padded % 4 || a.padded < a.dim) return int(cudaErrorInvalidValue);
  return q.f32 ? DeltaAs<float>(q, r, a) : DeltaAs<__nv_bfloat16>(q, r, a);
}

int PrepareDelta() {
  for (cudaError_t err : {Raise<16, 1>(), Raise<32, 1>(), Raise<32, 2>()})
    if (err != cudaSuccess) return int(err);
  return PrepareDeltaChunks();
}

}  // namespace tmb
