// Token mixers of bf16 ragged steps on the tensor pipe (mma.sync; the tiles are too small and too irregular for
// tcgen05): attention over the paged pools, for prompt portions and for decoded tokens (a long window cut over several
// CTAs), and retention inside prompt portions, a chunk of positions at a time.
#include <cuda_bf16.h>

#include <algorithm>
#include <cmath>

#include "element.cuh"
#include "mixers.cuh"
#include "mma.cuh"
#include "ops.h"
#include "ptx.cuh"
#include "tensor_map.h"

namespace tmb {
namespace {

// ---- attention ---------------------------------------------------------------------------------------------------------
constexpr int kKeys = 64;   // keys per block

struct AttendParams {
  const bf16* proj;
  bf16* k_pool;
  bf16* v_pool;
  bf16* out;
  float* part;
  unsigned* count;
  const float *q_norm, *k_norm;
  int proj_stride, out_stride, heads, kv_heads, dim, vdim, pool_dim, v_pool_dim, window, keep, splits, gate_at;
  int subs, sub_heads;      // query heads of one key head are served in `subs` units of up to `sub_heads`
  int q_head;               // elements from one query head to the next
  const int* context;       // portions whose keys and values are rows [.. + position] of k_pool and v_pool (see AttendContext), or null
  int context_stride;
  float scale_log2, sink_log2, eps;
  bool value_is_key, even;
  Rotary rotary;
  Blend blend;
  const float* sinks;
  __device__ float sink_of(int head) const { return sinks ? sinks[head] * 1.4426950408889634f : sink_log2; }
};

template <int DT, int WM> struct AttendShape {
  static constexpr int kThreads = WM == 1 ? 128 : 32 * WM;
  static constexpr int kPitch = DT * 16 + 8;
  static constexpr int kRows = 16 * WM;
  static constexpr int kTile = kKeys * kPitch;                        // elements of one K or V block
  static constexpr int kSmem = (kRows * kPitch + 4 * kTile) * 2;      // q, two stages of K and V
};

// Rows of a tile are (token, query head of the unit) pairs, token-major. WM = 8: a prompt portion, 128 rows, each warp 16
// of them against all keys of a block; q is rotated and the portion's keys are in the pools already (RotateAppend).
// WM = 1: one decoded token, 16 rows, each of the four warps a quarter of a block's keys; the CTA rotates q itself, and
// the one that holds the newest position rotates and appends its key and value (both norm them first, if the model does,
// which takes the squares of the whole projected row). DT: 16-column tiles of the wider of keys and values; FULL: both
// fill them. blockIdx = (token tile | split, unit, entry).
template <int DT, int WM, bool FULL>
__global__ void __launch_bounds__(AttendShape<DT, WM>::kThreads, DT > 8 ? 1 : WM > 1 ? 2 : 3) attend_tiles(StepRows r, AttendParams p) {
  using Shape = AttendShape<DT, WM>;
  constexpr int WN = WM == 1 ? 4 : 1, KN = kKeys / WN, P = Shape::kPitch, NT = Shape::kThreads;
  extern __shared__ __align__(16) unsigned char smem_raw[];
  bf16* qs = reinterpret_cast<bf16*>(smem_raw);
  bf16* ks = qs + Shape::kRows * P;
  bf16* vs = ks + 2 * Shape::kTile;
  __shared__ unsigned last;
  __shared__ float2 square_part[NT / 32];
  __shared__ long long key_at[2][kKeys], value_at[2][kKeys];   // element offsets of a block's keys (-1: none) and values
  // Every kernel of a step lets the next one start only behind its own dependency wait, so what kernels before the last
  // one wrote is there already: the step's tables, and the keys of earlier steps. A decoded token's first block of keys
  // is therefore requested before the wait (its own key, if the block holds it, is put over the copy later).
  if (WM > 1) dependency_wait();
  const Entry e = r.entry[blockIdx.z];
  if ((e.rows == 1) != (WM == 1)) {
    if (WM == 1) dependency_wait();
    allow_dependents();
    return;
  }
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int group = blockIdx.y / p.subs, first_head = (blockIdx.y % p.subs) * p.sub_heads;
  const int gq = min(p.sub_heads, p.heads / p.kv_heads - first_head);
  const int head0 = group * (p.heads / p.kv_heads) + first_head;
  const int per_tile = Shape::kRows / gq;
  const int t0 = WM == 1 ? 0 : blockIdx.x * per_tile, split = WM == 1 ? blockIdx.x : 0;
  if (t0 >= e.rows) return;   // (prompt portions only)
  const int tokens = min(per_tile, e.rows - t0);
  const int p0 = e.first_position + t0, p1 = p0 + tokens - 1;
  const int* table = r.block_table + size_t(e.slot) * r.max_blocks;

  // the keys any row of the tile sees: [0, kept) and [low, p1], in blocks of kKeys
  const int low = max(0, p0 - p.window + 1), kept = min(p.keep, low);
  const int kept_blocks = (kept + kKeys - 1) / kKeys, blocks = kept_blocks + (p1 + 1 - low + kKeys - 1) / kKeys;
  const int share = (blocks + p.splits - 1) / p.splits;
  const int from = WM == 1 ? min(blocks, split * share) : 0, to = WM == 1 ? min(blocks, from + share) : blocks;
  auto block_base = [&](int b) { return b < kept_blocks ? b * kKeys : low + (b - kept_blocks) * kKeys; };
  auto block_limit = [&](int b) { return b < kept_blocks ? kept : p1 + 1; };
  const int context = WM > 1 && p.context ? p.context[blockIdx.z] - max(0, e.first_position - p.window + 1) : 0;
  auto locate = [&](int b) {   // one block ahead of its fetch: the block-table loads are then off the copies' path
    if (threadIdx.x < kKeys && b < to) {
      const int j = block_base(b) + int(threadIdx.x), stage = (b - from) & 1;
      long long key = -1, value = -1;
      if (j < block_limit(b)) {
        if (WM > 1 && p.context) {
          key = (long long)(context + j) * p.context_stride;
          value = key + group * p.v_pool_dim;
          key += group * p.pool_dim;
        } else {
          const int row = key_row(table, j, r);
          key = (long long)(pool_offset(row, group, p.kv_heads, p.pool_dim));
          value = (long long)(pool_offset(row, group, p.kv_heads, p.v_pool_dim));
        }
      }
      key_at[stage][threadIdx.x] = key;
      value_at[stage][threadIdx.x] = value;
    }
  };
  auto fetch = [&](int b) {
    const int stage = (b - from) & 1;
    constexpr int C = DT * 2;   // 16-byte pieces of a row
#pragma unroll 4
    for (int i = threadIdx.x; i < kKeys * C; i += NT) {
      const int key = i / C, c = (i % C) * 8;
      const long long at = key_at[stage][key];
      const bool live = at >= 0;
      if (FULL || c < p.pool_dim) copy16(ks + stage * Shape::kTile + key * P + c, p.k_pool + (live ? at + c : 0), live);
      if (FULL || c < p.v_pool_dim) copy16(vs + stage * Shape::kTile + key * P + c, p.v_pool + (live ? value_at[stage][key] + c : 0), live);
    }
    copy_commit();
  };
  locate(from);
  locate(from + 1);
  __syncthreads();
  if (from < to) fetch(from);
  if (WM == 1) dependency_wait();
  allow_dependents();

  const int half = p.rotary.dims / 2;
  const float2* angle = p.rotary.table + size_t(min(p1, p.rotary.capacity - 1)) * half;   // WM == 1: the token's
  float2 inv = make_float2(1.f, 1.f);
  if constexpr (WM == 1) {
    const bf16* line = p.proj + size_t(e.first_row) * p.proj_stride;
    for (int i = threadIdx.x; i < Shape::kRows * (P / 8); i += NT) *reinterpret_cast<uint4*>(qs + 8 * i) = make_uint4(0, 0, 0, 0);
    if (p.q_norm) {
      const int q_count = p.heads * p.dim, k_count = p.kv_heads * p.dim;
      inv = inverse_rms<NT>(make_float2(square_sum(line, q_count, NT), square_sum(line + q_count, k_count, NT)), q_count, k_count, p.eps, square_part);
    } else {
      __syncthreads();
    }
    const int units = p.dim - half;                      // a unit: one rotated pair, or one entry behind the rotated ones
#pragma unroll 4
    for (int i = threadIdx.x; i < gq * units; i += NT) {
      const int m = i / units, u = i % units, d = u < half ? u : u + half, head = head0 + m;
      const bf16* q = line + size_t(head) * p.dim;
      const float* weight = p.q_norm ? p.q_norm + size_t(head) * p.dim : nullptr;
      float a = __bfloat162float(q[d]);
      if (weight) a *= inv.x * weight[d];
      if (u < half) {
        float b = __bfloat162float(q[d + half]);
        if (weight) b *= inv.x * weight[d + half];
        const float2 cs = angle[u];
        qs[m * P + d + half] = __float2bfloat16_rn(b * cs.x + a * cs.y);
        a = a * cs.x - b * cs.y;
      }
      qs[m * P + d] = __float2bfloat16_rn(a);
    }
  } else {
    const bool wide = (p.dim & 7) == 0 && (p.q_head & 7) == 0;
    for (int i = threadIdx.x; i < Shape::kRows * (P / 8); i += NT) {
      const int m = i / (P / 8), c = (i % (P / 8)) * 8, t = m / gq;
      const bf16* head = p.proj + size_t(e.first_row + t0 + t) * p.proj_stride + size_t(head0 + m % gq) * p.q_head;
      uint4 word = make_uint4(0, 0, 0, 0);
      if (t < tokens && c < p.dim) {
        if (wide) {
          word = *reinterpret_cast<const uint4*>(head + c);
        } else {
          bf16 e8[8];
#pragma unroll
          for (int j = 0; j < 8; ++j) e8[j] = c + j >= p.dim ? __float2bfloat16_rn(0.f) : head[c + j];
          word = *reinterpret_cast<uint4*>(e8);
        }
      }
      *reinterpret_cast<uint4*>(qs + m * P + c) = word;
    }
  }

  const int row0 = WM == 1 ? 0 : warp * 16, key0 = WM == 1 ? warp * KN : 0;
  const int ra = row0 + (lane >> 2), rb = ra + 8;                     // this thread's rows of the score tile
  const int pa = p0 + min(ra / gq, tokens - 1), pb = p0 + min(rb / gq, tokens - 1);
  float o[2 * DT][4];
#pragma unroll
  for (int i = 0; i < 2 * DT; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
  float top_a = -INFINITY, top_b = -INFINITY, sum_a = 0.f, sum_b = 0.f;

  for (int b = from; b < to; ++b) {
    const int stage = (b - from) & 1;
    if (b + 1 < to) {
      fetch(b + 1);
      copy_wait<1>();
    } else {
      copy_wait<0>();
    }
    __syncthreads();
    locate(b + 2);
    if (WM == 1 && b + 1 == blocks) {   // the newest position: over whatever the copy found in its pool row
      const bf16* k = p.proj + size_t(e.first_row) * p.proj_stride + size_t(p.heads + group) * p.dim;
      const bf16* v = p.value_is_key ? k : k + size_t(p.kv_heads) * p.dim;
      v += size_t(group) * (p.vdim - p.dim);
      const float* weight = p.k_norm ? p.k_norm + group * p.dim : nullptr;
      const int row = key_row(table, p1, r), key = p1 - block_base(b);
      bf16* k_to = p.k_pool + pool_offset(row, group, p.kv_heads, p.pool_dim);
      bf16* v_to = p.v_pool + pool_offset(row, group, p.kv_heads, p.v_pool_dim);
      for (int d = threadIdx.x; d < p.dim; d += NT) {
        const bf16 kd = __float2bfloat16_rn(normed_rotated(k, weight, inv.y, d, half, angle));
        ks[stage * Shape::kTile + key * P + d] = kd;
        if (first_head == 0) k_to[d] = kd;
      }
      for (int d = threadIdx.x; d < p.vdim; d += NT) {
        const bf16 vd = blended(p.blend, v - size_t(group) * p.vdim, e.first_row, group * p.vdim + d);
        vs[stage * Shape::kTile + key * P + d] = vd;
        if (first_head == 0) v_to[d] = vd;
      }
      __syncthreads();
    }
    const bf16* kt = ks + stage * Shape::kTile + key0 * P;
    const bf16* vt = vs + stage * Shape::kTile + key0 * P;
    float s[KN / 8][4];
#pragma unroll
    for (int t = 0; t < KN / 8; ++t) s[t][0] = s[t][1] = s[t][2] = s[t][3] = 0.f;
#pragma unroll
    for (int kk = 0; kk < DT; ++kk) {
      if (!FULL && kk * 16 >= p.pool_dim) break;
      uint32_t a[4];
      load_a(a, qs, P, row0, kk * 16, lane);
#pragma unroll
      for (int t = 0; t < KN / 16; ++t) {
        uint32_t bb[4];
        load_b(bb, kt, P, t * 16, kk * 16, lane);
        mma16816(s[2 * t], a, bb[0], bb[1]);
        mma16816(s[2 * t + 1], a, bb[2], bb[3]);
      }
    }
    const int limit = block_limit(b), first = block_base(b) + key0 + 2 * (lane & 3);
    float high_a = top_a, high_b = top_b;
#pragma unroll
    for (int t = 0; t < KN / 8; ++t)
#pragma unroll
      for (int c = 0; c < 2; ++c) {
        const int j = first + 8 * t + c;
        const bool in_a = j < limit && j <= pa && (pa - j < p.window || j < p.keep);
        const bool in_b = j < limit && j <= pb && (pb - j < p.window || j < p.keep);
        s[t][c] = in_a ? s[t][c] * p.scale_log2 : -INFINITY;
        s[t][2 + c] = in_b ? s[t][2 + c] * p.scale_log2 : -INFINITY;
        high_a = fmaxf(high_a, s[t][c]);
        high_b = fmaxf(high_b, s[t][2 + c]);
      }
#pragma unroll
    for (int x = 1; x <= 2; x <<= 1) {
      high_a = fmaxf(high_a, __shfl_xor_sync(0xffffffffu, high_a, x));
      high_b = fmaxf(high_b, __shfl_xor_sync(0xffffffffu, high_b, x));
    }
    const float ref_a = high_a == -INFINITY ? 0.f : high_a, ref_b = high_b == -INFINITY ? 0.f : high_b;
    const float fade_a = ex2(top_a - ref_a), fade_b = ex2(top_b - ref_b);
    top_a = high_a;
    top_b = high_b;
    float add_a = 0.f, add_b = 0.f;
#pragma unroll
    for (int t = 0; t < KN / 8; ++t)
#pragma unroll
      for (int c = 0; c < 2; ++c) {
        s[t][c] = ex2(s[t][c] - ref_a);
        s[t][2 + c] = ex2(s[t][2 + c] - ref_b);
        add_a += s[t][c];
        add_b += s[t][2 + c];
      }
    sum_a = sum_a * fade_a + add_a;
    sum_b = sum_b * fade_b + add_b;
#pragma unroll
    for (int i = 0; i < 2 * DT; ++i) {
      o[i][0] *= fade_a;
      o[i][1] *= fade_a;
      o[i][2] *= fade_b;
      o[i][3] *= fade_b;
    }
    // the weights enter the product as a bf16 head and a bf16 remainder, about 16 bits of each
#pragma unroll
    for (int kk = 0; kk < KN / 16; ++kk) {
      uint32_t hi[4], lo[4];
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        const float(&w)[4] = s[2 * kk + h];
        hi[2 * h] = pack(w[0], w[1]);
        hi[2 * h + 1] = pack(w[2], w[3]);
        lo[2 * h] = pack(rest(w[0]), rest(w[1]));
        lo[2 * h + 1] = pack(rest(w[2]), rest(w[3]));
      }
#pragma unroll
      for (int d = 0; d < DT; ++d) {
        if (!FULL && d * 16 >= p.v_pool_dim) break;
        uint32_t bb[4];
        load_b_transposed(bb, vt, P, kk * 16, d * 16, lane);
        mma16816(o[2 * d], hi, bb[0], bb[1]);
        mma16816(o[2 * d + 1], hi, bb[2], bb[3]);
        mma16816(o[2 * d], lo, bb[0], bb[1]);
        mma16816(o[2 * d + 1], lo, bb[2], bb[3]);
      }
    }
    __syncthreads();
  }
#pragma unroll
  for (int x = 1; x <= 2; x <<= 1) {
    sum_a += __shfl_xor_sync(0xffffffffu, sum_a, x);
    sum_b += __shfl_xor_sync(0xffffffffu, sum_b, x);
  }
  if constexpr (WM > 1) {
    // (a null key that stands above every key takes the maximum's place: the values then count by the distance)
    auto share = [&](int m, float top, float sum) {
      const float sink = p.sink_of(head0 + m % gq);
      if (sink == -INFINITY) return 1.f / sum;
      const float high = fmaxf(top, sink), f = ex2(top - high);
      return f / fmaf(sum, f, ex2(sink - high));
    };
    const float inv_a = share(ra, top_a, sum_a), inv_b = share(rb, top_b, sum_b);
    auto write = [&](int m, float inv, int i, int at) {
      const int t = m / gq, c = i * 8 + 2 * (lane & 3);
      if (t >= tokens || c >= p.vdim) return;
      const size_t row = size_t(e.first_row + t0 + t), column = size_t(head0 + m % gq) * p.vdim + c;
      bf16* dst = p.out + row * p.out_stride + column;
      float y0 = o[i][at] * inv, y1 = o[i][at + 1] * inv;
      const bool pair = c + 1 < p.vdim;
      if (p.even) {                                      // both columns, and words of two at the addresses
        if (p.gate_at >= 0) {
          const uint32_t gate = *reinterpret_cast<const uint32_t*>(p.proj + row * p.proj_stride + p.gate_at + column);
          y0 = __fdividef(y0, 1.f + ex2(-1.4426950408889634f * bf_lo(gate)));
          y1 = __fdividef(y1, 1.f + ex2(-1.4426950408889634f * bf_hi(gate)));
        }
        *reinterpret_cast<uint32_t*>(dst) = pack(y0, y1);
        return;
      }
      if (p.gate_at >= 0) {
        const bf16* gate = p.proj + row * p.proj_stride + p.gate_at + column;
        y0 *= sigmoid(__bfloat162float(gate[0]));
        if (pair) y1 *= sigmoid(__bfloat162float(gate[1]));
      }
      dst[0] = __float2bfloat16_rn(y0);
      if (pair) dst[1] = __float2bfloat16_rn(y1);
    };
#pragma unroll
    for (int i = 0; i < 2 * DT; ++i) {
      write(ra, inv_a, i, 0);
      write(rb, inv_b, i, 2);
    }
  } else {
    // the four warps' states meet in shared memory: [4][16] maxima, [4][16] sums, [4][16][16 DT] values
    float* ms = reinterpret_cast<float*>(smem_raw);
    float* ls = ms + 64;
    float* os = ls + 64;
    constexpr int D = DT * 16;
    __syncthreads();   // (a split without keys comes here straight from the query tile)
    if ((lane & 3) == 0) {
      ms[warp * 16 + ra] = top_a;
      ms[warp * 16 + rb] = top_b;
      ls[warp * 16 + ra] = sum_a;
      ls[warp * 16 + rb] = sum_b;
    }
#pragma unroll
    for (int i = 0; i < 2 * DT; ++i) {
      const int c = i * 8 + 2 * (lane & 3);
      *reinterpret_cast<float2*>(os + (warp * 16 + ra) * D + c) = make_float2(o[i][0], o[i][1]);
      *reinterpret_cast<float2*>(os + (warp * 16 + rb) * D + c) = make_float2(o[i][2], o[i][3]);
    }
    __syncthreads();
    const bf16* gates = p.proj + size_t(e.first_row) * p.proj_stride + p.gate_at + size_t(head0) * p.vdim;   // [head of the unit][column]
    bf16* dst = p.out + size_t(e.first_row) * p.out_stride + size_t(head0) * p.vdim;
    auto gated = [&](float v, int i) { return __float2bfloat16_rn(p.gate_at < 0 ? v : v * sigmoid(__bfloat162float(gates[i]))); };
    const int record = p.vdim + 2;
    float* parts = p.part + (size_t(blockIdx.z) * p.heads + head0) * p.splits * record;   // [head of the unit][split][record]
    for (int i = threadIdx.x; i < gq * p.vdim; i += NT) {
      const int h = i / p.vdim, c = i % p.vdim;
      const float sink = p.sink_of(head0 + h);
      float high = p.splits == 1 ? sink : -INFINITY, sum = 0.f, value = 0.f;
#pragma unroll
      for (int w = 0; w < 4; ++w) high = fmaxf(high, ms[w * 16 + h]);
      const float ref = high == -INFINITY ? 0.f : high;
#pragma unroll
      for (int w = 0; w < 4; ++w) {
        const float f = ex2(ms[w * 16 + h] - ref);
        sum = fmaf(ls[w * 16 + h], f, sum);
        value = fmaf(os[(w * 16 + h) * D + c], f, value);
      }
      if (p.splits == 1) {
        dst[i] = gated(value / (sum + ex2(sink - ref)), i);
      } else {
        float* mine = parts + (size_t(h) * p.splits + split) * record;
        mine[2 + c] = value;
        if (c == 0) {
          mine[0] = high;
          mine[1] = sum;
        }
      }
    }
    if (p.splits > 1) {
      unsigned* counter = p.count + size_t(blockIdx.z) * (p.kv_heads * p.subs) + blockIdx.y;
      __syncthreads();
      if (threadIdx.x == 0) last = atom_acq_rel_add(counter, 1u) == unsigned(p.splits) - 1 ? 1u : 0u;
      __syncthreads();
      if (!last) return;
      if (threadIdx.x == 0) *counter = 0;   // for the next launch
      // every split's share of the whole, once per head; then the values, several splits' loads in flight at a time
      float* factor = os;                            // [gq][splits]
      for (int i = threadIdx.x; i < gq * p.splits; i += NT) {
        factor[i] = __ldcg(parts + size_t(i) * record);
        factor[gq * p.splits + i] = __ldcg(parts + size_t(i) * record + 1);
      }
      __syncthreads();
      if (int(threadIdx.x) < gq) {
        float* f = factor + threadIdx.x * p.splits;
        const float* l = f + gq * p.splits;
        const float sink = p.sink_of(head0 + int(threadIdx.x));
        float high = sink;
        for (int s = 0; s < p.splits; ++s) high = fmaxf(high, f[s]);
        float sum = ex2(sink - high);
        for (int s = 0; s < p.splits; ++s) {         // in split order
          f[s] = ex2(f[s] - high);
          sum = fmaf(l[s], f[s], sum);
        }
        for (int s = 0; s < p.splits; ++s) f[s] /= sum;
      }
      __syncthreads();
      const int outputs = gq * p.vdim;
      for (int i0 = threadIdx.x; i0 < outputs; i0 += 4 * NT) {
        float value[4] = {};
        const float* at[4];
        const float* f[4];
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const int i = min(i0 + j * NT, outputs - 1), h = i / p.vdim;
          at[j] = parts + size_t(h) * p.splits * record + 2 + i % p.vdim;
          f[j] = factor + h * p.splits;
        }
#pragma unroll 8
        for (int s = 0; s < p.splits; ++s)
#pragma unroll
          for (int j = 0; j < 4; ++j) value[j] = fmaf(__ldcg(at[j] + size_t(s) * record), f[j][s], value[j]);
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const int i = i0 + j * NT;
          if (i < outputs) dst[i] = gated(value[j], i);
        }
      }
    }
  }
}

// ---- retention inside a prompt portion -----------------------------------------------------------------------------------
// With C positions a chunk, local index a, decay d and the state S before the chunk:
//   o_a = d^(a+1) q_a S + sum_{b <= a} d^(a-b) (q_a . k_b) v_b,    S' = d^n S + sum_b d^(n-1-b) k_b v_b^T.
// A CTA walks one (entry, head) over a slice of 32 value columns; the state stays in fp32 accumulators. q, k, the state,
// the score weights and the decayed values enter the products as bf16 heads plus bf16 remainders (v is bf16 as it is),
// leaving out remainder x remainder: about 16 bits of every operand. Rotated q and k arrive split already
// (retention_split), so that a chunk is plain 16-byte copies, the next one under the products of this one.
constexpr int kSlice = 32, kSlicePitch = kSlice + 8;

template <int DT> struct RetainShape {
  static constexpr int kStages = DT <= 8 ? 2 : 1;
  static constexpr int kPitch = DT * 16 + 8;
  static constexpr int kTile = kRetentionChunk * kPitch;
  static constexpr int kStage = 4 * kTile + kRetentionChunk * kSlicePitch;    // q, k heads and remainders, v
  static constexpr int kSmem = (kStages * kStage + 2 * kRetentionChunk * kSlicePitch + 2 * DT * 16 * kSlicePitch) * 2 + (kRetentionChunk + 1) * 4;
};

// Rotated q and scaled rotated k of portions' rows as [row][head][q head | q remainder | k head | k remainder][padded],
// zeros behind `dim`.
__global__ void __launch_bounds__(256) retention_split(StepRows r, const bf16* proj, int stride, bf16* split, int heads, int dim, int padded,
                                                       float key_scale, Rotary rot) {
  dependency_wait();
  allow_dependents();
  const int row = blockIdx.x;
  if (r.entry[r.row_entry[row]].rows == 1) return;
  const int half = rot.dims / 2, units = padded - half;
  const float2* angle = rot.table + size_t(min(r.row_position[row], rot.capacity - 1)) * half;
  const bf16* line = proj + size_t(row) * stride;
#pragma unroll 4
  for (int i = threadIdx.x; i < heads * units; i += 256) {
    const int head = i / units, u = i % units;
    const bf16* q = line + size_t(head) * dim;
    const bf16* k = q + size_t(heads) * dim;
    bf16* out = split + (size_t(row) * heads + head) * 4 * padded;
    auto put = [&](bf16* at, int d, float v) {
      at[d] = __float2bfloat16_rn(v);
      at[padded + d] = __float2bfloat16_rn(rest(v));
    };
    if (u < half) {
      const float2 cs = angle[u];
      const float q1 = __bfloat162float(q[u]), q2 = __bfloat162float(q[u + half]);
      const float k1 = __bfloat162float(k[u]), k2 = __bfloat162float(k[u + half]);
      put(out, u, q1 * cs.x - q2 * cs.y);
      put(out, u + half, q2 * cs.x + q1 * cs.y);
      put(out + 2 * padded, u, (k1 * cs.x - k2 * cs.y) * key_scale);
      put(out + 2 * padded, u + half, (k2 * cs.x + k1 * cs.y) * key_scale);
    } else {
      const int d = u + half;
      put(out, d, d < dim ? __bfloat162float(q[d]) : 0.f);
      put(out + 2 * padded, d, d < dim ? __bfloat162float(k[d]) * key_scale : 0.f);
    }
  }
}

template <int DT>
__global__ void __launch_bounds__(128) retain_chunks(StepRows r, const bf16* proj, int stride, const bf16* split, int padded, float* states, float* raw,
                                                     int heads, int dim, int vdim, const float* decays) {
  using Shape = RetainShape<DT>;
  constexpr int C = kRetentionChunk, P = Shape::kPitch, MT = (DT + 3) / 4, S = Shape::kStages;   // MT: state row tiles per warp
  extern __shared__ __align__(16) unsigned char smem_raw[];
  bf16* stages = reinterpret_cast<bf16*>(smem_raw);
  bf16* wh = stages + S * Shape::kStage;           // decayed values
  bf16* wl = wh + C * kSlicePitch;
  bf16* sh = wl + C * kSlicePitch;                 // [16 DT][slice]
  bf16* sl = sh + DT * 16 * kSlicePitch;
  float* power = reinterpret_cast<float*>(sl + DT * 16 * kSlicePitch);   // d^0 .. d^C
  dependency_wait();
  allow_dependents();
  const Entry e = r.entry[blockIdx.z];
  if (e.rows == 1) return;
  const int head = blockIdx.y, c0 = blockIdx.x * kSlice;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const float decay = decays[head];
  const int chunks = (e.rows + C - 1) / C;
  const int v_at = 2 * heads * dim + head * vdim + c0;
  const bool wide = (v_at & 7) == 0 && (vdim & 7) == 0;
  auto fetch = [&](int chunk) {
    if (chunk < chunks) {
      bf16* tile = stages + (chunk % S) * Shape::kStage;
      bf16* vt = tile + 4 * Shape::kTile;
      const int t0 = chunk * C, n = min(C, e.rows - t0), pieces = padded / 8;
#pragma unroll 8
      for (int i = threadIdx.x; i < C * 4 * pieces; i += 128) {
        const int t = i / (4 * pieces), piece = i % (4 * pieces), part = piece / pieces, c = (piece % pieces) * 8;
        const size_t row = size_t(e.first_row + t0 + (t < n ? t : 0));
        copy16(tile + part * Shape::kTile + t * P + c, split + ((row * heads + head) * 4 + part) * padded + c, t < n);
      }
      if (wide) {
        for (int i = threadIdx.x; i < C * (kSlice / 8); i += 128) {
          const int t = i / (kSlice / 8), c = (i % (kSlice / 8)) * 8;
          const bool live = t < n && c0 + c < vdim;
          copy16(vt + t * kSlicePitch + c, proj + size_t(e.first_row + t0 + (live ? t : 0)) * stride + v_at + (live ? c : 0), live);
        }
      } else {
        for (int i = threadIdx.x; i < C * kSlice; i += 128) {
          const int t = i / kSlice, c = i % kSlice;
          vt[t * kSlicePitch + c] = t < n && c0 + c < vdim ? proj[size_t(e.first_row + t0 + t) * stride + v_at + c] : __float2bfloat16_rn(0.f);
        }
      }
    }
    copy_commit();
  };
  // columns between the padded head size and the tile stay zero
  for (int i = threadIdx.x; i < S * 4 * C * (DT * 16 - padded); i += 128) {
    const int width = DT * 16 - padded, d = padded + i % width, t = i / width % C, part = i / width / C;
    stages[(part / 4) * Shape::kStage + (part % 4) * Shape::kTile + t * P + d] = __float2bfloat16_rn(0.f);
  }
  for (int s = 0; s < S; ++s) fetch(s);
  for (int i = threadIdx.x; i <= C; i += 128) power[i] = powf(decay, float(i));
  float* state = states + (size_t(e.slot) * heads + head) * dim * vdim;

  float st[MT][kSlice / 8][4];
  auto each_state = [&](auto&& visit) {
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int n = 0; n < kSlice / 8; ++n)
#pragma unroll
        for (int x = 0; x < 4; ++x) {
          const int row = (warp + 4 * m) * 16 + (lane >> 2) + (x >> 1) * 8, col = n * 8 + 2 * (lane & 3) + (x & 1);
          visit(row, col, st[m][n][x]);
        }
  };
  each_state([&](int row, int col, float& v) {
    v = e.first_position > 0 && row < dim && c0 + col < vdim ? state[size_t(row) * vdim + c0 + col] : 0.f;
  });
  auto publish = [&]() {   // the state as an operand
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int i = 0; i < kSlice / 8; ++i)
#pragma unroll
        for (int h = 0; h < 2; ++h) {
          const int row = (warp + 4 * m) * 16 + (lane >> 2) + 8 * h, col = i * 8 + 2 * (lane & 3);
          const float a = st[m][i][2 * h], b = st[m][i][2 * h + 1];
          if (row < DT * 16) {
            *reinterpret_cast<uint32_t*>(sh + row * kSlicePitch + col) = pack(a, b);
            *reinterpret_cast<uint32_t*>(sl + row * kSlicePitch + col) = pack(rest(a), rest(b));
          }
        }
  };
  publish();

  for (int chunk = 0; chunk < chunks; ++chunk) {
    const int t0 = chunk * C, n = min(C, e.rows - t0);
    const bf16* qh = stages + (chunk % S) * Shape::kStage;
    const bf16* ql = qh + Shape::kTile;
    const bf16* kh = ql + Shape::kTile;
    const bf16* kl = kh + Shape::kTile;
    const bf16* vt = kl + Shape::kTile;
    copy_wait<S - 1>();
    __syncthreads();   // the chunk is there, and the state before it
    for (int i = threadIdx.x; i < C * kSlice / 2; i += 128) {
      const int t = i / (kSlice / 2), c = (i % (kSlice / 2)) * 2;
      const float f = t < n ? power[n - 1 - t] : 0.f;
      const float a = __bfloat162float(vt[t * kSlicePitch + c]) * f, b = __bfloat162float(vt[t * kSlicePitch + c + 1]) * f;
      *reinterpret_cast<uint32_t*>(wh + t * kSlicePitch + c) = pack(a, b);
      *reinterpret_cast<uint32_t*>(wl + t * kSlicePitch + c) = pack(rest(a), rest(b));
    }
    __syncthreads();
    const int row0 = warp * 16, ra = row0 + (lane >> 2), rb = ra + 8;
    if (row0 < n) {
      float o[kSlice / 8][4], s[C / 8][4];
#pragma unroll
      for (int i = 0; i < kSlice / 8; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
#pragma unroll
      for (int i = 0; i < C / 8; ++i) s[i][0] = s[i][1] = s[i][2] = s[i][3] = 0.f;
#pragma unroll 2
      for (int kk = 0; kk < DT; ++kk) {
        uint32_t ah[4], al[4];
        load_a(ah, qh, P, row0, kk * 16, lane);
        load_a(al, ql, P, row0, kk * 16, lane);
#pragma unroll
        for (int t = 0; t < kSlice / 16; ++t) {
          uint32_t bh[4], bl[4];
          load_b_transposed(bh, sh, kSlicePitch, kk * 16, t * 16, lane);
          load_b_transposed(bl, sl, kSlicePitch, kk * 16, t * 16, lane);
#pragma unroll
          for (int h = 0; h < 2; ++h) {
            mma16816(o[2 * t + h], ah, bh[2 * h], bh[2 * h + 1]);
            mma16816(o[2 * t + h], al, bh[2 * h], bh[2 * h + 1]);
            mma16816(o[2 * t + h], ah, bl[2 * h], bl[2 * h + 1]);
          }
        }
#pragma unroll
        for (int t = 0; t < C / 16; ++t) {
          if (t > warp) continue;                      // keys behind every row of the tile
          uint32_t bh[4], bl[4];
          load_b(bh, kh, P, t * 16, kk * 16, lane);
          load_b(bl, kl, P, t * 16, kk * 16, lane);
#pragma unroll
          for (int h = 0; h < 2; ++h) {
            mma16816(s[2 * t + h], ah, bh[2 * h], bh[2 * h + 1]);
            mma16816(s[2 * t + h], al, bh[2 * h], bh[2 * h + 1]);
            mma16816(s[2 * t + h], ah, bl[2 * h], bl[2 * h + 1]);
          }
        }
      }
      const float da = power[ra + 1], db = power[rb + 1];
#pragma unroll
      for (int i = 0; i < kSlice / 8; ++i) {
        o[i][0] *= da;
        o[i][1] *= da;
        o[i][2] *= db;
        o[i][3] *= db;
      }
#pragma unroll
      for (int kk = 0; kk < C / 16; ++kk) {
        if (kk > warp) continue;
        uint32_t hi[4], lo[4];
#pragma unroll
        for (int h = 0; h < 2; ++h) {
          float w[4];
#pragma unroll
          for (int x = 0; x < 4; ++x) {
            const int a = x < 2 ? ra : rb, b = (2 * kk + h) * 8 + 2 * (lane & 3) + (x & 1);
            w[x] = b <= a ? s[2 * kk + h][x] * power[max(a - b, 0)] : 0.f;
          }
          hi[2 * h] = pack(w[0], w[1]);
          hi[2 * h + 1] = pack(w[2], w[3]);
          lo[2 * h] = pack(rest(w[0]), rest(w[1]));
          lo[2 * h + 1] = pack(rest(w[2]), rest(w[3]));
        }
#pragma unroll
        for (int t = 0; t < kSlice / 16; ++t) {
          uint32_t bb[4];
          load_b_transposed(bb, vt, kSlicePitch, kk * 16, t * 16, lane);
#pragma unroll
          for (int h = 0; h < 2; ++h) {
            mma16816(o[2 * t + h], hi, bb[2 * h], bb[2 * h + 1]);
            mma16816(o[2 * t + h], lo, bb[2 * h], bb[2 * h + 1]);
          }
        }
      }
#pragma unroll
      for (int i = 0; i < kSlice / 8; ++i)
#pragma unroll
        for (int x = 0; x < 4; ++x) {
          const int a = x < 2 ? ra : rb, c = c0 + i * 8 + 2 * (lane & 3) + (x & 1);
          if (a < n && c < vdim) raw[size_t(e.first_row + t0 + a) * heads * vdim + size_t(head) * vdim + c] = o[i][x];
        }
    }
    const float whole = power[n];
#pragma unroll
    for (int m = 0; m < MT; ++m) {
      const int row = (warp + 4 * m) * 16;
      if (row >= DT * 16) continue;
#pragma unroll
      for (int i = 0; i < kSlice / 8; ++i)
#pragma unroll
        for (int x = 0; x < 4; ++x) st[m][i][x] *= whole;
#pragma unroll
      for (int kk = 0; kk < C / 16; ++kk) {
        uint32_t ah[4], al[4];
        load_a_transposed(ah, kh, P, kk * 16, row, lane);
        load_a_transposed(al, kl, P, kk * 16, row, lane);
#pragma unroll
        for (int t = 0; t < kSlice / 16; ++t) {
          uint32_t bh[4], bl[4];
          load_b_transposed(bh, wh, kSlicePitch, kk * 16, t * 16, lane);
          load_b_transposed(bl, wl, kSlicePitch, kk * 16, t * 16, lane);
#pragma unroll
          for (int h = 0; h < 2; ++h) {
            mma16816(st[m][2 * t + h], ah, bh[2 * h], bh[2 * h + 1]);
            mma16816(st[m][2 * t + h], al, bh[2 * h], bh[2 * h + 1]);
            mma16816(st[m][2 * t + h], ah, bl[2 * h], bl[2 * h + 1]);
          }
        }
      }
    }
    __syncthreads();   // every warp has read the chunk and the state before it
    fetch(chunk + S);
    if (chunk + 1 < chunks) publish();
  }
  each_state([&](int row, int col, float& v) {
    if (row < dim && c0 + col < vdim) state[size_t(row) * vdim + c0 + col] = v;
  });
}

template <int DT, int WM> int LaunchAttend(const Queue& q, const StepRows& r, const AttendParams& p, int x) {
  const int units = p.kv_heads * p.subs;
  auto kernel = p.pool_dim == 16 * DT && p.v_pool_dim == 16 * DT ? attend_tiles<DT, WM, true> : attend_tiles<DT, WM, false>;
  return int(Launch(kernel, dim3(unsigned(x), unsigned(units), unsigned(r.entries)), dim3(AttendShape<DT, WM>::kThreads), AttendShape<DT, WM>::kSmem, q.stream,
                    q.chained, r, p));
}

template <int DT> int AttendWith(const Queue& q, const StepRows& r, const AttentionArgs& a, AttendParams p) {
  if (r.singles > 0) {
    // A decoded token's keys are cut over several CTAs. Three CTAs fit an SM; a CTA costs its blocks plus about four
    // blocks' time to start and merge (more with more parts to merge): the cut that ends soonest by that measure.
    const int reach = std::min(a.window, r.capacity) + std::min(a.keep, r.capacity), blocks = reach / kKeys + 1;
    const int units = p.kv_heads * p.subs, resident = 3 * q.sm_count;
    AttendParams one = p;
    float least = 0.f;
    for (int s = 1; s <= std::min(blocks, 64); ++s) {
      if (s > 1 && size_t(r.singles) * units * s > size_t(8 * q.sm_count)) break;
      const int waves = (r.singles * units * s + resident - 1) / resident;
      const float cost = float(waves) * (float((blocks + s - 1) / s) + 4.f + float(s) / 8.f);
      if (s == 1 || cost < least) {
        least = cost;
        one.splits = s;
      }
    }
    if (size_t(r.entries) * a.heads * one.splits * (a.vdim + 2) > a.part_floats || r.entries * units > a.count_words) one.splits = 1;
    const int status = LaunchAttend<DT, 1>(q, r, one, one.splits);
    if (status != 0) return status;
  }
  if (r.singles < r.entries) {
    p.splits = 1;
    const int per_tile = 128 / p.sub_heads;
    return LaunchAttend<DT, 8>(q, r, p, (r.longest + per_tile - 1) / per_tile);
  }
  return 0;
}

template <int DT> int RetainWith(const Queue& q, const StepRows& r, const RetentionArgs& a) {
  const int padded = (a.dim + 15) / 16 * 16;
  const int status = int(Launch(retention_split, dim3(unsigned(r.rows)), dim3(256), 0, q.stream, q.chained, r, static_cast<const bf16*>(a.proj),
                                a.proj_stride, static_cast<bf16*>(a.split), a.heads, a.dim, padded, a.key_scale, a.rotary));
  if (status != 0) return status;
  const dim3 grid(unsigned((a.vdim + kSlice - 1) / kSlice), unsigned(a.heads), unsigned(r.entries));
  return int(Launch(retain_chunks<DT>, grid, dim3(128), RetainShape<DT>::kSmem, q.stream, q.chained, r, static_cast<const bf16*>(a.proj),
                    a.proj_stride, static_cast<const bf16*>(a.split), padded, a.state, a.raw, a.heads, a.dim, a.vdim, a.decay));
}

template <int DT> cudaError_t Raise() {
  cudaError_t err = cudaFuncSetAttribute(retain_chunks<DT>, cudaFuncAttributeMaxDynamicSharedMemorySize, RetainShape<DT>::kSmem);
  for (auto kernel : {attend_tiles<DT, 1, false>, attend_tiles<DT, 1, true>})
    if (err == cudaSuccess) err = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, AttendShape<DT, 1>::kSmem);
  for (auto kernel : {attend_tiles<DT, 8, false>, attend_tiles<DT, 8, true>})
    if (err == cudaSuccess) err = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, AttendShape<DT, 8>::kSmem);
  return err;
}

}  // namespace

namespace {

AttendParams ParamsOf(const AttentionArgs& a) {
  AttendParams p{};
  p.proj = static_cast<const bf16*>(a.proj);
  p.k_pool = static_cast<bf16*>(a.k_pool);
  p.v_pool = static_cast<bf16*>(a.v_pool);
  p.value_is_key = a.value_is_key;
  p.rotary = a.rotary;
  p.out = static_cast<bf16*>(a.out);
  p.part = a.part;
  p.count = a.count;
  p.proj_stride = a.proj_stride;
  p.out_stride = a.out_stride;
  p.heads = a.heads;
  p.kv_heads = a.kv_heads;
  p.dim = a.dim;
  p.vdim = a.vdim;
  p.pool_dim = a.pool_dim;
  p.v_pool_dim = a.v_pool_dim;
  p.q_norm = a.q_norm;
  p.k_norm = a.k_norm;
  p.eps = a.eps;
  p.gate_at = a.gate_at;
  p.even = a.vdim % 2 == 0 && a.out_stride % 2 == 0 && a.proj_stride % 2 == 0 && (a.gate_at < 0 || a.gate_at % 2 == 0);
  p.window = a.window;
  p.keep = a.keep;
  const int gq = a.heads / a.kv_heads;
  p.subs = (gq + 15) / 16;
  p.sub_heads = (gq + p.subs - 1) / p.subs;
  p.subs = (gq + p.sub_heads - 1) / p.sub_heads;
  p.scale_log2 = a.scale * 1.4426950408889634f;
  p.sink_log2 = a.sink * 1.4426950408889634f;
  p.sinks = a.sinks;
  p.blend = {a.blend, a.blend_from, a.blend_stride};
  p.q_head = a.dim;
  return p;
}

}  // namespace

int AttendTiles(const Queue& q, const StepRows& r, const AttentionArgs& a) {
  const AttendParams p = ParamsOf(a);
  const int tiles = (std::max(a.dim, a.vdim) + 15) / 16;
  return tiles <= 2 ? AttendWith<2>(q, r, a, p) : tiles <= 4 ? AttendWith<4>(q, r, a, p) : tiles <= 6 ? AttendWith<6>(q, r, a, p)
         : tiles <= 8 ? AttendWith<8>(q, r, a, p) : tiles <= 12 ? AttendWith<12>(q, r, a, p) : AttendWith<16>(q, r, a, p);
}

int AttendContext(const Queue& q, const StepRows& r, const AttentionArgs& a, int q_head, const int* context, int context_stride) {
  AttendParams p = ParamsOf(a);
  p.q_head = q_head;
  p.context = context;
  p.context_stride = context_stride;
  p.splits = 1;
  const int tiles = (std::max(a.dim, a.vdim) + 15) / 16, per_tile = 128 / p.sub_heads, x = (r.longest + per_tile - 1) / per_tile;
  return tiles <= 2 ? LaunchAttend<2, 8>(q, r, p, x) : tiles <= 4 ? LaunchAttend<4, 8>(q, r, p, x) : tiles <= 6 ? LaunchAttend<6, 8>(q, r, p, x)
         : tiles <= 8 ? LaunchAttend<8, 8>(q, r, p, x) : tiles <= 12 ? LaunchAttend<12, 8>(q, r, p, x) : LaunchAttend<16, 8>(q, r, p, x);
}

int RetainChunks(const Queue& q, const StepRows& r, const RetentionArgs& a) {
  const int tiles = (a.dim + 15) / 16;
  return tiles <= 2 ? RetainWith<2>(q, r, a) : tiles <= 4 ? RetainWith<4>(q, r, a) : tiles <= 6 ? RetainWith<6>(q, r, a)
         : tiles <= 8 ? RetainWith<8>(q, r, a) : tiles <= 12 ? RetainWith<12>(q, r, a) : RetainWith<16>(q, r, a);
}

int PrepareMixers() {
  cudaError_t err = Raise<2>();
  if (err == cudaSuccess) err = Raise<4>();
  if (err == cudaSuccess) err = Raise<6>();
  if (err == cudaSuccess) err = Raise<8>();
  if (err == cudaSuccess) err = Raise<12>();
  if (err == cudaSuccess) err = Raise<16>();
  return int(err);
}

}  // namespace tmb
