// Token mixers of a ragged step, in the form that works for every size and both element types: rotary append into the
// paged pools, attention with a sliding window and kept first positions (over latent rows too), retention by its recurrence.
// Attention of bf16 steps and retention inside bf16 prompt portions run in mixers_mma.cu, latent attention of bf16 steps in
// latent.cu.
#include <cuda_bf16.h>

#include <algorithm>
#include <cmath>
#include <type_traits>

#include "element.cuh"
#include "mixers.cuh"
#include "ops.h"
#include "ptx.cuh"
#include "tensor_map.h"

namespace tmb {
namespace {

// ---- rotary + append ------------------------------------------------------------------------------------------------
struct AppendParams {
  int stride, heads, kv_heads, dim, vdim, pool_dim, v_pool_dim;
  bool value_is_key;
  const float *q_norm, *k_norm;
  float eps;
  Rotary rot;
  Blend blend;
};

template <typename T>
__global__ void __launch_bounds__(128) rotate_append(StepRows r, T* proj, T* k_pool, T* v_pool, AppendParams p, bool portions_only) {
  __shared__ float2 part[4];
  dependency_wait();
  allow_dependents();
  const int row = blockIdx.x;
  if (portions_only && r.entry[r.row_entry[row]].rows == 1) return;
  const int half = p.rot.dims / 2, units = p.dim - half;   // a unit: one rotated pair, or one entry behind the rotated ones
  const float2* angle = p.rot.table + size_t(min(r.row_position[row], p.rot.capacity - 1)) * half;
  const int kv = r.row_kv[row];
  T* line = proj + size_t(row) * p.stride;
  const T* keys = line + size_t(p.heads) * p.dim;
  float2 inv = make_float2(1.f, 1.f);
  if (p.q_norm) {
    const int q_count = p.heads * p.dim, k_count = p.kv_heads * p.dim;
    inv = inverse_rms<128>(make_float2(square_sum(line, q_count, 128), square_sum(keys, k_count, 128)), q_count, k_count, p.eps, part);
  }
  const T* values = p.value_is_key ? keys : keys + size_t(p.kv_heads) * p.dim;
  for (int i = threadIdx.x; i < p.kv_heads * p.vdim; i += 128)
    v_pool[pool_offset(kv, i / p.vdim, p.kv_heads, p.v_pool_dim) + i % p.vdim] = blended(p.blend, values, row, i);
  for (int i = threadIdx.x; i < (p.heads + p.kv_heads) * units; i += 128) {
    const int head = i / units, u = i % units, group = head - p.heads;
    if (u >= half && group < 0 && !p.q_norm) continue;      // (an entry of q that stays as it is)
    T* at = line + size_t(head) * p.dim;
    T* to = group < 0 ? at : k_pool + pool_offset(kv, group, p.kv_heads, p.pool_dim);
    const float scale = group < 0 ? inv.x : inv.y;
    const float* weight = group < 0 ? p.q_norm : p.k_norm;
    auto value = [&](int d) { return weight ? to_f(at[d]) * scale * weight[(group < 0 ? head : group) * p.dim + d] : to_f(at[d]); };
    if (u < half) {
      const float a = value(u), b = value(u + half);
      const float2 cs = angle[u];
      to[u] = from_f<T>(a * cs.x - b * cs.y);
      to[u + half] = from_f<T>(b * cs.x + a * cs.y);
    } else {
      to[u + half] = from_f<T>(value(u + half));
    }
  }
}

// The same for bf16 rows whose head sizes and half rotations are multiples of 8: eight pairs, or eight entries behind the
// rotated ones, a turn. Portions only.
__global__ void __launch_bounds__(256) rotate_append_wide(StepRows r, __nv_bfloat16* proj, __nv_bfloat16* k_pool, __nv_bfloat16* v_pool, AppendParams p) {
  __shared__ float2 part[8];
  dependency_wait();
  allow_dependents();
  const int row = blockIdx.x;
  if (r.entry[r.row_entry[row]].rows == 1) return;
  const int half = p.rot.dims / 2, turned = half / 8, units = p.dim / 8 - turned;
  const float2* angle = p.rot.table + size_t(min(r.row_position[row], p.rot.capacity - 1)) * half;
  const int kv = r.row_kv[row];
  __nv_bfloat16* line = proj + size_t(row) * p.stride;
  const __nv_bfloat16* keys = line + size_t(p.heads) * p.dim;
  const __nv_bfloat16* values = p.value_is_key ? keys : keys + size_t(p.kv_heads) * p.dim;
  const int v_units = p.vdim / 8;
  for (int i = threadIdx.x; i < p.kv_heads * v_units; i += 256) {
    uint4 word = reinterpret_cast<const uint4*>(values)[i];
    if (p.blend.by) {
      alignas(16) __nv_bfloat16 mixed[8];
#pragma unroll
      for (int j = 0; j < 8; ++j) mixed[j] = blended(p.blend, values, row, 8 * i + j);
      word = *reinterpret_cast<const uint4*>(mixed);
    }
    *reinterpret_cast<uint4*>(v_pool + pool_offset(kv, i / v_units, p.kv_heads, p.v_pool_dim) + i % v_units * 8) = word;
  }
  float2 inv = make_float2(1.f, 1.f);
  if (p.q_norm) {
    const int q_count = p.heads * p.dim, k_count = p.kv_heads * p.dim;
    inv = inverse_rms<256>(make_float2(square_sum(line, q_count, 256), square_sum(keys, k_count, 256)), q_count, k_count, p.eps, part);
  }
  for (int i = threadIdx.x; i < (p.heads + p.kv_heads) * units; i += 256) {
    const int head = i / units, u = i % units, group = head - p.heads;
    if (u >= turned && group < 0 && !p.q_norm) continue;
    const int d = u < turned ? 8 * u : 8 * u + half;
    __nv_bfloat16* at = line + size_t(head) * p.dim + d;
    __nv_bfloat16* to = group < 0 ? at : k_pool + pool_offset(kv, group, p.kv_heads, p.pool_dim) + d;
    const float* weight = group < 0 ? p.q_norm : p.k_norm;
    const float scale = group < 0 ? inv.x : inv.y;
    auto load = [&](int offset, float (&v)[8]) {
      unpack8(*reinterpret_cast<const uint4*>(at + offset), v);
      if (!weight) return;
      const float4* w = reinterpret_cast<const float4*>(weight + (group < 0 ? head : group) * p.dim + d + offset);
      const float4 lo = w[0], hi = w[1];
      const float by[8] = {lo.x, lo.y, lo.z, lo.w, hi.x, hi.y, hi.z, hi.w};
#pragma unroll
      for (int j = 0; j < 8; ++j) v[j] *= scale * by[j];
    };
    auto store = [&](int offset, const float (&v)[8]) {
      *reinterpret_cast<uint4*>(to + offset) =
          make_uint4(pack_bf16x2(v[0], v[1]), pack_bf16x2(v[2], v[3]), pack_bf16x2(v[4], v[5]), pack_bf16x2(v[6], v[7]));
    };
    float a[8];
    load(0, a);
    if (u < turned) {
      float b[8];
      load(half, b);
      const float4* turn = reinterpret_cast<const float4*>(angle + d);
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const float4 cs = turn[j];
        const float x0 = a[2 * j], y0 = b[2 * j], x1 = a[2 * j + 1], y1 = b[2 * j + 1];
        a[2 * j] = x0 * cs.x - y0 * cs.y;
        b[2 * j] = y0 * cs.x + x0 * cs.y;
        a[2 * j + 1] = x1 * cs.z - y1 * cs.w;
        b[2 * j + 1] = y1 * cs.z + x1 * cs.w;
      }
      store(half, b);
    }
    store(0, a);
  }
}

// ---- attention, one warp per (row, query head) -------------------------------------------------------------------------
// Queries are rows of q_stride, heads q_head apart; outputs likewise. MAXD: most columns of a head's query or value.
constexpr int kPlainWarps = 4;

struct PlainAttend {
  int q_stride, q_head, out_stride, out_head, heads, kv_heads, dim, vdim, pool_dim, v_pool_dim, window, keep;
  float scale, sink;
  const float* sinks;
  int gate_at;
};

template <typename T, int MAXD>
__global__ void __launch_bounds__(32 * kPlainWarps) attend_rows(StepRows r, const T* q, const T* k_pool, const T* v_pool, T* out, PlainAttend p) {
  __shared__ float qs[kPlainWarps][MAXD];
  dependency_wait();
  allow_dependents();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int head = blockIdx.x * kPlainWarps + warp, row = blockIdx.y;
  if (head >= p.heads) return;
  const int group = head / (p.heads / p.kv_heads);
  const int position = r.row_position[row];
  const int slot = r.entry[r.row_entry[row]].slot;
  const int* table = r.block_table + size_t(slot) * r.max_blocks;
  const T* line = q + size_t(row) * p.q_stride;
  for (int d = lane; d < p.dim; d += 32) qs[warp][d] = to_f(line[size_t(head) * p.q_head + d]);
  __syncwarp();
  constexpr int N = MAXD / 32;
  const float sink = p.sinks ? p.sinks[head] : p.sink;
  float acc[N] = {}, top = sink, sum = sink == -INFINITY ? 0.f : 1.f;   // (the null key, if there is one)
  auto walk = [&](int from, int to) {
    for (int base = from; base < to; base += 32) {
      const int j = base + lane;
      long long v_at = 0;
      float score = -INFINITY;
      if (j < to) {
        const int key = key_row(table, j, r);
        const size_t at = pool_offset(key, group, p.kv_heads, p.pool_dim);
        v_at = (long long)(pool_offset(key, group, p.kv_heads, p.v_pool_dim));
        float dot = 0.f;
        for (int d = 0; d < p.dim; ++d) dot = fmaf(qs[warp][d], to_f(k_pool[at + d]), dot);
        score = dot * p.scale;
      }
      const float high = fmaxf(top, warp_max(score));
      const float fade = expf(top - high), w = j < to ? expf(score - high) : 0.f;
      sum = sum * fade + warp_sum(w);
      top = high;
#pragma unroll
      for (int i = 0; i < N; ++i) acc[i] *= fade;
      const int count = min(32, to - base);
      for (int jj = 0; jj < count; ++jj) {
        const float weight = __shfl_sync(0xffffffffu, w, jj);
        const T* v = v_pool + __shfl_sync(0xffffffffu, v_at, jj);
#pragma unroll
        for (int i = 0; i < N; ++i)
          if (lane + 32 * i < p.vdim) acc[i] = fmaf(weight, to_f(v[lane + 32 * i]), acc[i]);
      }
    }
  };
  const int low = max(0, position - p.window + 1);
  walk(0, min(p.keep, low));
  walk(low, position + 1);
#pragma unroll
  for (int i = 0; i < N; ++i) {
    const int c = lane + 32 * i;
    if (c >= p.vdim) continue;
    const float gate = p.gate_at < 0 ? 1.f : sigmoid(to_f(line[p.gate_at + size_t(head) * p.vdim + c]));
    out[size_t(row) * p.out_stride + size_t(head) * p.out_head + c] = from_f<T>(acc[i] / sum * gate);
  }
}

// ---- latent rows: normed (and their last columns rotated) into the pool; rows that queries are images of, normed -------------
struct AppendLatentParams {
  int raw_stride, pool_dim, rank;
  const float* norm;
  Rotary rotary;
  const void* query_raw;
  const float* query_norm;
  void* query;
  int query_rank, query_stride;
  float eps;
};

template <typename T>
__global__ void __launch_bounds__(128) append_latent(StepRows r, const T* raw, T* pool, AppendLatentParams p, bool portions_only) {
  __shared__ float2 part[4];
  dependency_wait();
  allow_dependents();
  const int row = blockIdx.x;
  if (portions_only && r.entry[r.row_entry[row]].rows == 1) return;
  if (blockIdx.y == 1) {
    const T* line = static_cast<const T*>(p.query_raw) + size_t(row) * p.raw_stride;
    T* to = static_cast<T*>(p.query) + size_t(row) * p.query_stride;
    const float inv = inverse_rms<128>(make_float2(square_sum(line, p.query_rank, 128), 0.f), p.query_rank, 1, p.eps, part).x;
    for (int d = threadIdx.x; d < p.query_rank; d += 128) to[d] = from_f<T>(to_f(line[d]) * inv * p.query_norm[d]);
    return;
  }
  const int half = p.rotary.dims / 2, normed = p.rank - p.rotary.dims;
  const T* line = raw + size_t(row) * p.raw_stride;
  T* to = pool + pool_offset(r.row_kv[row], 0, 1, p.pool_dim);
  const float inv = inverse_rms<128>(make_float2(square_sum(line, normed, 128), 0.f), normed, 1, p.eps, part).x;
  for (int d = threadIdx.x; d < normed; d += 128) to[d] = from_f<T>(to_f(line[d]) * inv * p.norm[d]);
  const float2* angle = p.rotary.table + size_t(min(r.row_position[row], p.rotary.capacity - 1)) * half;
  for (int i = threadIdx.x; i < half; i += 128) {
    const int d = normed + 2 * i;
    const float u = to_f(line[d]), v = to_f(line[d + 1]);
    const float2 cs = angle[i];
    to[d] = from_f<T>(u * cs.x - v * cs.y);
    to[d + 1] = from_f<T>(v * cs.x + u * cs.y);
  }
}

// ---- retention by its recurrence ----------------------------------------------------------------------------------------
// A CTA holds a [dim][32] slice of one (entry, head) state in registers (thread: one column, every eighth row) and
// walks the entry's rows, kBatch at a time.
constexpr int kBatch = 8;

template <typename T, int NR>
__global__ void __launch_bounds__(256) retain_steps(StepRows r, const T* proj, int stride, float* states, float* raw, int heads, int dim, int vdim,
                                                    const float* decays, float key_scale, Rotary rot, bool singles_only) {
  __shared__ float qs[kBatch][8 * NR], ks[kBatch][8 * NR], red[kBatch][8][32];
  dependency_wait();
  allow_dependents();
  const Entry e = r.entry[blockIdx.z];
  if (singles_only && e.rows != 1) return;
  const int head = blockIdx.y, lane = threadIdx.x & 31, group = threadIdx.x >> 5;
  const int column = blockIdx.x * 32 + lane;
  const bool live = column < vdim;
  float* state = states + (size_t(e.slot) * heads + head) * dim * vdim + column;
  const float decay = decays[head];
  float s[NR];
#pragma unroll
  for (int i = 0; i < NR; ++i) s[i] = live && e.first_position > 0 && group + 8 * i < dim ? state[size_t(group + 8 * i) * vdim] : 0.f;
  const int half = rot.dims / 2;
  for (int t0 = 0; t0 < e.rows; t0 += kBatch) {
    const int count = min(kBatch, e.rows - t0);
    for (int i = threadIdx.x; i < count * 8 * NR; i += 256) {
      const int t = i / (8 * NR), d = i % (8 * NR);
      float qv = 0.f, kv = 0.f;
      if (d < dim) {
        const T* q = proj + size_t(e.first_row + t0 + t) * stride + size_t(head) * dim;
        const T* k = q + size_t(heads) * dim;
        const int position = min(e.first_position + t0 + t, rot.capacity - 1);
        qv = rotated(q, d, half, rot.table + size_t(position) * half);
        kv = rotated(k, d, half, rot.table + size_t(position) * half) * key_scale;
      }
      qs[t][d] = qv;
      ks[t][d] = kv;
    }
    __syncthreads();
    for (int t = 0; t < count; ++t) {
      const float v = live ? to_f(proj[size_t(e.first_row + t0 + t) * stride + size_t(2 * heads) * dim + size_t(head) * vdim + column]) : 0.f;
      float acc = 0.f;
#pragma unroll
      for (int i = 0; i < NR; ++i) {
        s[i] = fmaf(ks[t][group + 8 * i], v, decay * s[i]);
        acc = fmaf(qs[t][group + 8 * i], s[i], acc);
      }
      red[t][group][lane] = acc;
    }
    __syncthreads();
    if (group < count && live) {
      float sum = 0.f;
#pragma unroll
      for (int i = 0; i < 8; ++i) sum += red[group][i][lane];
      raw[size_t(e.first_row + t0 + group) * heads * vdim + size_t(head) * vdim + column] = sum;
    }
    // (the next batch writes qs/ks, read before the barrier above, and red only behind the next barrier)
  }
#pragma unroll
  for (int i = 0; i < NR; ++i)
    if (live && group + 8 * i < dim) state[size_t(group + 8 * i) * vdim] = s[i];
}

// One decoded token of an entry, whole: recurrence, per-head norm and gate. A CTA holds one head's state, a thread four
// columns of every (512 / columns)-th row; every load of the state is in flight before the first is used.
constexpr int kTokenThreads = 512;

template <typename T, int NR>
__global__ void __launch_bounds__(kTokenThreads, NR <= 8 ? 2 : 1) retain_token(StepRows r, const T* proj, int stride, float* states, T* out, int out_stride, int heads, int dim,
                                                    int vdim, const float* decays, float key_scale, float eps, Rotary rot) {
  __shared__ float qs[kMaxHeadDim], ks[kMaxHeadDim], part[kTokenThreads / 32];
  __shared__ float4 red[kTokenThreads];
  const Entry e = r.entry[blockIdx.y];   // (tables and states: written before the kernel this one depends on)
  if (e.rows != 1) {
    dependency_wait();
    allow_dependents();
    return;
  }
  const int head = blockIdx.x, quads = vdim / 4, groups = kTokenThreads / quads;
  const int quad = threadIdx.x % quads, group = threadIdx.x / quads;
  const bool live = group < groups;
  float4* state = reinterpret_cast<float4*>(states + (size_t(e.slot) * heads + head) * dim * vdim) + quad;
  const float decay = decays[head];
  const T* line = proj + size_t(e.first_row) * stride;
  float4 s[NR];
#pragma unroll
  for (int i = 0; i < NR; ++i) {
    const int row = group + groups * i;
    s[i] = live && e.first_position > 0 && row < dim ? __ldcs(state + size_t(row) * quads) : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  dependency_wait();
  allow_dependents();
  const T* q = line + size_t(head) * dim;
  const T* k = q + size_t(heads) * dim;
  const T* v = line + size_t(2 * heads) * dim + size_t(head) * vdim;
  const T* g = v + size_t(heads) * vdim;
  const int half = rot.dims / 2;
  const float2* angle = rot.table + size_t(min(e.first_position, rot.capacity - 1)) * half;
  for (int d = threadIdx.x; d < dim; d += kTokenThreads) {
    qs[d] = rotated(q, d, half, angle);
    ks[d] = rotated(k, d, half, angle) * key_scale;
  }
  float4 value = make_float4(0.f, 0.f, 0.f, 0.f), acc = value;
  if (live) value = make_float4(to_f(v[4 * quad]), to_f(v[4 * quad + 1]), to_f(v[4 * quad + 2]), to_f(v[4 * quad + 3]));
  __syncthreads();
#pragma unroll
  for (int i = 0; i < NR; ++i) {
    const int row = group + groups * i;
    if (!live || row >= dim) continue;
    const float kd = ks[row], qd = qs[row];
    s[i].x = fmaf(kd, value.x, decay * s[i].x);
    s[i].y = fmaf(kd, value.y, decay * s[i].y);
    s[i].z = fmaf(kd, value.z, decay * s[i].z);
    s[i].w = fmaf(kd, value.w, decay * s[i].w);
    acc.x = fmaf(qd, s[i].x, acc.x);
    acc.y = fmaf(qd, s[i].y, acc.y);
    acc.z = fmaf(qd, s[i].z, acc.z);
    acc.w = fmaf(qd, s[i].w, acc.w);
    __stcs(state + size_t(row) * quads, s[i]);
  }
  red[threadIdx.x] = acc;
  __syncthreads();
  const float* lanes = reinterpret_cast<const float*>(red);
  float sq = 0.f, o[2];
#pragma unroll
  for (int n = 0; n < 2; ++n) {       // vdim <= 1024
    const int c = threadIdx.x + kTokenThreads * n;
    o[n] = 0.f;
    if (c < vdim)
      for (int w = 0; w < groups; ++w) o[n] += lanes[(w * quads + c / 4) * 4 + c % 4];
    sq = fmaf(o[n], o[n], sq);
  }
  sq = warp_sum(sq);
  if ((threadIdx.x & 31) == 0) part[threadIdx.x >> 5] = sq;
  __syncthreads();
  sq = 0.f;
#pragma unroll
  for (int w = 0; w < kTokenThreads / 32; ++w) sq += part[w];
  const float inv = 1.f / sqrtf(sq / float(vdim) + eps);
#pragma unroll
  for (int n = 0; n < 2; ++n) {
    const int c = threadIdx.x + kTokenThreads * n;
    if (c >= vdim) continue;
    const float gate = to_f(g[c]);
    out[size_t(e.first_row) * out_stride + size_t(head) * vdim + c] = from_f<T>(o[n] * inv * (gate / (1.f + expf(-gate))));
  }
}

// A warp per (row, head), see HeadGateArgs.
template <typename T>
__global__ void __launch_bounds__(128) head_gate(HeadGateArgs p) {
  dependency_wait();
  allow_dependents();
  const int unit = blockIdx.x * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31, vdim = p.vdim;
  if (unit >= p.rows * p.heads) return;
  const int row = unit / p.heads, head = unit % p.heads;
  const float* o = p.raw + size_t(row) * p.heads * vdim + size_t(head) * vdim;
  const T* gate = static_cast<const T*>(p.proj) + size_t(row) * p.proj_stride + p.gate_at + size_t(head) * vdim;
  const float* weight = p.weight ? p.weight + size_t(head) * vdim : nullptr;
  T* out = static_cast<T*>(p.out) + size_t(row) * p.out_stride + size_t(head) * vdim;
  auto opened = [&](float x) { return p.silu ? x / (1.f + expf(-x)) : sigmoid(x); };
  float sq = 0.f;
  if (vdim % 4 == 0 && vdim <= 256 && p.proj_stride % 4 == 0 && p.gate_at % 4 == 0 && p.out_stride % 4 == 0) {
    float4 v[2];
    alignas(16) T g[2][4], y[4];
    using Word = std::conditional_t<sizeof(T) == 2, uint2, uint4>;
#pragma unroll
    for (int n = 0; n < 2; ++n) {
      const int d = 4 * (lane + 32 * n);
      if (d >= vdim) continue;
      v[n] = *reinterpret_cast<const float4*>(o + d);
      *reinterpret_cast<Word*>(g[n]) = *reinterpret_cast<const Word*>(gate + d);
      sq += v[n].x * v[n].x + v[n].y * v[n].y + v[n].z * v[n].z + v[n].w * v[n].w;
    }
    const float inv = 1.f / sqrtf(warp_sum(sq) / float(vdim) + p.eps);
#pragma unroll
    for (int n = 0; n < 2; ++n) {
      const int d = 4 * (lane + 32 * n);
      if (d >= vdim) continue;
      const float4 w = weight ? *reinterpret_cast<const float4*>(weight + d) : make_float4(1.f, 1.f, 1.f, 1.f);
      const float value[4] = {v[n].x * w.x, v[n].y * w.y, v[n].z * w.z, v[n].w * w.w};
#pragma unroll
      for (int j = 0; j < 4; ++j) y[j] = from_f<T>(value[j] * inv * opened(to_f(g[n][j])));
      *reinterpret_cast<Word*>(out + d) = *reinterpret_cast<const Word*>(y);
    }
    return;
  }
  for (int d = lane; d < vdim; d += 32) sq = fmaf(o[d], o[d], sq);
  const float inv = 1.f / sqrtf(warp_sum(sq) / float(vdim) + p.eps);
  for (int d = lane; d < vdim; d += 32) out[d] = from_f<T>(o[d] * (weight ? weight[d] : 1.f) * inv * opened(to_f(gate[d])));
}

template <typename T> int RotateAppendAs(const Queue& q, const StepRows& r, const AttentionArgs& a) {
  const AppendParams p{a.proj_stride, a.heads, a.kv_heads, a.dim, a.vdim, a.pool_dim, a.v_pool_dim, a.value_is_key, a.q_norm, a.k_norm, a.eps, a.rotary,
                       {a.blend, a.blend_from, a.blend_stride}};
  if constexpr (sizeof(T) == 2) {
    if (a.dim % 8 == 0 && a.vdim % 8 == 0 && a.rotary.dims % 16 == 0 && a.proj_stride % 8 == 0)
      return int(Launch(rotate_append_wide, dim3(unsigned(r.rows)), dim3(256), 0, q.stream, q.chained, r, static_cast<T*>(a.proj),
                        static_cast<T*>(a.k_pool), static_cast<T*>(a.v_pool), p));
  }
  return int(Launch(rotate_append<T>, dim3(unsigned(r.rows)), dim3(128), 0, q.stream, q.chained, r, static_cast<T*>(a.proj),
                    static_cast<T*>(a.k_pool), static_cast<T*>(a.v_pool), p, !q.f32));
}

dim3 PlainGrid(int heads, int rows) { return dim3(unsigned((heads + kPlainWarps - 1) / kPlainWarps), unsigned(rows)); }

template <typename T> int AttendAs(const Queue& q, const StepRows& r, const AttentionArgs& a) {
  const PlainAttend p{a.proj_stride, a.dim, a.out_stride, a.vdim, a.heads, a.kv_heads, a.dim, a.vdim, a.pool_dim, a.v_pool_dim, a.window, a.keep,
                      a.scale, a.sink, a.sinks, a.gate_at};
  return int(Launch(attend_rows<T, kMaxHeadDim>, PlainGrid(a.heads, r.rows), dim3(32 * kPlainWarps), 0, q.stream, q.chained, r,
                    static_cast<const T*>(a.proj), static_cast<const T*>(a.k_pool), static_cast<const T*>(a.v_pool), static_cast<T*>(a.out), p));
}

template <typename T> int AttendLatentAs(const Queue& q, const StepRows& r, const LatentArgs& a) {
  const int stride = a.heads * a.rank_stride;
  const PlainAttend p{stride, a.rank_stride, stride, a.rank_stride, a.heads, 1, a.rank, a.rank, a.pool_dim, a.pool_dim, a.window, 0,
                      a.scale, a.sink, a.sinks, -1};
  auto kernel = a.rank <= kMaxHeadDim ? attend_rows<T, kMaxHeadDim> : attend_rows<T, kMaxLatent>;
  return int(Launch(kernel, PlainGrid(a.heads, r.rows), dim3(32 * kPlainWarps), 0, q.stream, q.chained, r, static_cast<const T*>(a.q),
                    static_cast<const T*>(a.pool), static_cast<const T*>(a.pool), static_cast<T*>(a.out), p));
}

template <typename T> int AppendLatentAs(const Queue& q, const StepRows& r, const LatentArgs& a, bool portions_only) {
  const AppendLatentParams p{a.raw_stride, a.pool_dim, a.rank, a.norm, a.rotary, a.query_raw, a.query_norm, a.query, a.query_rank, a.query_stride, a.eps};
  return int(Launch(append_latent<T>, dim3(unsigned(r.rows), a.query_raw ? 2u : 1u), dim3(128), 0, q.stream, q.chained, r, static_cast<const T*>(a.raw),
                    static_cast<T*>(a.pool), p, portions_only));
}

template <typename T> int RetainAs(const Queue& q, const StepRows& r, const RetentionArgs& a, bool singles_only) {
  auto kernel = a.dim <= 64 ? retain_steps<T, 8> : a.dim <= 128 ? retain_steps<T, 16> : retain_steps<T, 32>;
  const dim3 grid(unsigned((a.vdim + 31) / 32), unsigned(a.heads), unsigned(r.entries));
  return int(Launch(kernel, grid, dim3(256), 0, q.stream, q.chained, r, static_cast<const T*>(a.proj), a.proj_stride, a.state, a.raw, a.heads,
                    a.dim, a.vdim, a.decay, a.key_scale, a.rotary, singles_only));
}

// Rows of a head's state one thread of retain_token holds: 0 when the sizes do not suit it.
int TokenRows(const RetentionArgs& a) {
  if (a.vdim % 4 || a.vdim > 1024) return 0;
  const int groups = kTokenThreads / (a.vdim / 4), rows = (a.dim + groups - 1) / groups;
  return rows <= 4 ? 4 : rows <= 8 ? 8 : rows <= 16 ? 16 : 0;
}

template <typename T> int RetainTokenAs(const Queue& q, const StepRows& r, const RetentionArgs& a) {
  const int rows = TokenRows(a);
  auto kernel = rows == 4 ? retain_token<T, 4> : rows == 8 ? retain_token<T, 8> : retain_token<T, 16>;
  return int(Launch(kernel, dim3(unsigned(a.heads), unsigned(r.entries)), dim3(kTokenThreads), 0, q.stream, q.chained, r, static_cast<const T*>(a.proj),
                    a.proj_stride, a.state, static_cast<T*>(a.out), a.out_stride, a.heads, a.dim, a.vdim, a.decay, a.key_scale, a.eps, a.rotary));
}

int Gate(const Queue& q, const StepRows& r, const RetentionArgs& a) {
  return HeadGate(q, {a.raw, a.proj, a.proj_stride, a.heads * (2 * a.dim + a.vdim), a.out, a.out_stride, r.rows, a.heads, a.vdim, nullptr, true, a.eps});
}

}  // namespace

int RotateAppend(const Queue& q, const StepRows& r, const AttentionArgs& a) {
  if (!q.f32 && r.singles == r.entries) return 0;
  return q.f32 ? RotateAppendAs<float>(q, r, a) : RotateAppendAs<__nv_bfloat16>(q, r, a);
}

int Attend(const Queue& q, const StepRows& r, const AttentionArgs& a) {
  return q.f32 ? AttendAs<float>(q, r, a) : AttendTiles(q, r, a);
}

int AppendLatent(const Queue& q, const StepRows& r, const LatentArgs& a) {
  if (q.f32 || a.query_raw || !LatentTiled(a)) return q.f32 ? AppendLatentAs<float>(q, r, a, false) : AppendLatentAs<__nv_bfloat16>(q, r, a, false);
  return r.singles == r.entries ? 0 : AppendLatentAs<__nv_bfloat16>(q, r, a, true);
}

int AttendLatent(const Queue& q, const StepRows& r, const LatentArgs& a) {
  if (q.f32) return AttendLatentAs<float>(q, r, a);
  return LatentTiled(a) ? AttendLatentTiles(q, r, a) : AttendLatentAs<__nv_bfloat16>(q, r, a);
}

int HeadGate(const Queue& q, const HeadGateArgs& a) {
  const unsigned blocks = unsigned((size_t(a.rows) * a.heads + 3) / 4);
  return int(Launch(q.f32 ? head_gate<float> : head_gate<__nv_bfloat16>, dim3(blocks), dim3(128), 0, q.stream, q.chained, a));
}

int Retain(const Queue& q, const StepRows& r, const RetentionArgs& a) {
  if (q.f32) {
    // a step of decoded tokens only takes the whole-token form; anything else the recurrence row by row
    if (r.singles == r.entries && TokenRows(a)) return RetainTokenAs<float>(q, r, a);
    const int status = RetainAs<float>(q, r, a, false);
    return status != 0 ? status : Gate(q, r, a);
  }
  // bf16: single tokens advance their states by the recurrence, portions by chunks
  const bool whole = TokenRows(a) != 0;
  int status = 0;
  if (r.singles < r.entries) status = RetainChunks(q, r, a);
  if (status == 0 && r.singles > 0 && !whole) status = RetainAs<__nv_bfloat16>(q, r, a, true);
  if (status == 0 && (r.singles < r.entries || !whole)) status = Gate(q, r, a);
  // (behind the gate of all rows, whose result for the single tokens it replaces)
  if (status == 0 && r.singles > 0 && whole) status = RetainTokenAs<__nv_bfloat16>(q, r, a);
  return status;
}

}  // namespace tmb
