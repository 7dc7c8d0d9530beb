// Latent attention of bf16 ragged steps on the tensor pipe (mma.sync): every head of a token reads the same cached rows, as
// keys and as values, so a tile holds (token, head) rows against blocks of latent rows that are copied once for both.
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

constexpr int kKeys = 64;          // latent rows per block
constexpr int kWeightPitch = kKeys + 8;

struct LatentParams {
  const bf16* q;
  const bf16* raw;
  bf16* pool;
  bf16* out;
  float* part;                     // split sums: [entry][head][split][rank_stride] latent columns, then [entry][head][split] maxima and sums
  const float *norm, *sinks;
  int raw_stride, heads, rank, rank_stride, pool_dim, window, splits;
  int subs, sub_heads;             // the heads are served in `subs` units of up to `sub_heads`
  float scale_log2, sink_log2, eps;
  __device__ float2* stats(int entries) const { return reinterpret_cast<float2*>(part + size_t(entries) * heads * splits * rank_stride); }
  __device__ float sink_of(int head) const { return sinks ? sinks[head] * 1.4426950408889634f : sink_log2; }
};

template <int RT, int WM> struct LatentShape {
  static constexpr int kWarps = WM == 1 ? 8 : 16;
  static constexpr int kThreads = 32 * kWarps;
  static constexpr int kPitch = RT * 16 + 8;
  static constexpr int kRows = 16 * WM;
  static constexpr int kTile = kKeys * kPitch;                                    // elements of one block
  static constexpr int kSmem = (kRows * kPitch + 2 * kTile + 2 * kRows * kWeightPitch) * 2;   // q, two blocks, weights as heads and remainders
};

// Rows of a tile are (token, head of the unit) pairs, token-major; the warps are WM row tiles times WN parts: of a
// block's keys for the scores, of the latent columns for the sums. ONE: one decoded token, the keys cut over gridDim.x CTAs
// (merge_latent follows if there are several); the CTA with the newest position norms and appends the token's own row. Otherwise a portion, whose rows are in the pool
// already. RT: 16-column tiles of a latent row; FULL: it fills them. blockIdx = (token tile | split, unit, entry).
template <int RT, int WM, bool ONE, bool FULL>
__global__ void __launch_bounds__(LatentShape<RT, WM>::kThreads, 1) attend_latent(StepRows r, LatentParams p) {
  using Shape = LatentShape<RT, WM>;
  constexpr int kWarps = Shape::kWarps, kThreads = Shape::kThreads;
  constexpr int WN = kWarps / WM, KN = kKeys / WN, P = Shape::kPitch, CT = RT / WN;   // CT: column tiles of a warp
  static_assert(CT >= 1, "a warp sums at least one column tile");
  extern __shared__ __align__(16) unsigned char smem_raw[];
  bf16* qs = reinterpret_cast<bf16*>(smem_raw);
  bf16* cs = qs + Shape::kRows * P;
  bf16* wh = cs + 2 * Shape::kTile;
  bf16* wl = wh + Shape::kRows * kWeightPitch;
  __shared__ float high_part[WN][Shape::kRows], sum_part[WN][Shape::kRows];
  __shared__ float2 square_part[kWarps];
  __shared__ int key_at[2][kKeys];   // pool rows of a block's keys (-1: none)
  if (!ONE) dependency_wait();
  const Entry e = r.entry[blockIdx.z];
  if ((e.rows == 1) != ONE) {
    if (ONE) dependency_wait();
    allow_dependents();
    return;
  }
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int head0 = blockIdx.y * p.sub_heads, gq = min(p.sub_heads, p.heads - head0);
  const int per_tile = Shape::kRows / p.sub_heads;
  const int t0 = ONE ? 0 : blockIdx.x * per_tile, split = ONE ? blockIdx.x : 0;
  if (t0 >= e.rows) return;          // (portions only)
  const int tokens = min(per_tile, e.rows - t0);
  const int p0 = e.first_position + t0, p1 = p0 + tokens - 1;
  const int* table = r.block_table + size_t(e.slot) * r.max_blocks;

  const int low = max(0, p0 - p.window + 1), blocks = (p1 + 1 - low + kKeys - 1) / kKeys;   // any row of the tile sees [low, p1]
  const int share = (blocks + p.splits - 1) / p.splits;
  const int from = ONE ? min(blocks, split * share) : 0, to = ONE ? min(blocks, from + share) : blocks;
  auto locate = [&](int b) {         // one block ahead of its fetch
    if (threadIdx.x < kKeys && b < to) {
      const int j = low + b * kKeys + int(threadIdx.x);
      key_at[(b - from) & 1][threadIdx.x] = j <= p1 ? key_row(table, j, r) : -1;
    }
  };
  auto fetch = [&](int b) {
    const int stage = (b - from) & 1;
    constexpr int C = RT * 2;        // 16-byte pieces of a row
#pragma unroll 4
    for (int i = threadIdx.x; i < kKeys * C; i += kThreads) {
      const int key = i / C, c = (i % C) * 8, row = key_at[stage][key];
      const bool live = row >= 0;
      if (FULL || c < p.pool_dim) copy16(cs + stage * Shape::kTile + key * P + c, p.pool + size_t(live ? row : 0) * p.pool_dim + c, live);
    }
    copy_commit();
  };
  locate(from);
  locate(from + 1);
  __syncthreads();
  if (from < to) fetch(from);        // (earlier steps' rows, and this portion's, are there; a token's own row comes later)
  float inv = 1.f;
  const bf16* raw = p.raw + size_t(e.first_row) * p.raw_stride;
  const bool newest = ONE && to == blocks && from < to;
  if (newest)                        // (the projection ran two kernels ago: there before the dependency wait)
    inv = inverse_rms<kThreads>(make_float2(square_sum(raw, p.rank, kThreads), 0.f), p.rank, 1, p.eps, square_part).x;
  if (ONE) dependency_wait();
  allow_dependents();

  for (int i = threadIdx.x; i < Shape::kRows * (P / 8); i += kThreads) {
    const int m = i / (P / 8), c = (i % (P / 8)) * 8, t = m / gq;
    uint4 word = make_uint4(0, 0, 0, 0);
    if (t < tokens && c < p.rank) {
      word = *reinterpret_cast<const uint4*>(p.q + (size_t(e.first_row + t0 + t) * p.heads + head0 + m % gq) * p.rank_stride + c);
      if (c + 8 > p.rank) {          // columns behind the rank hold nothing
        alignas(16) bf16 e8[8];
        *reinterpret_cast<uint4*>(e8) = word;
#pragma unroll
        for (int j = 0; j < 8; ++j)
          if (c + j >= p.rank) e8[j] = __float2bfloat16_rn(0.f);
        word = *reinterpret_cast<const uint4*>(e8);
      }
    }
    *reinterpret_cast<uint4*>(qs + m * P + c) = word;
  }

  const int wm = warp % WM, wn = warp / WM, row0 = wm * 16, key0 = wn * KN;
  const int ra = row0 + (lane >> 2), rb = ra + 8;                     // this thread's rows
  const int pa = p0 + min(ra / gq, tokens - 1), pb = p0 + min(rb / gq, tokens - 1);
  float o[2 * CT][4];
#pragma unroll
  for (int i = 0; i < 2 * CT; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
  float top_a = -INFINITY, top_b = -INFINITY, sum_a = 0.f, sum_b = 0.f;   // maxima of all keys, sums of this warp's

  for (int b = from; b < to; ++b) {
    const int stage = (b - from) & 1;
    bf16* tile = cs + stage * Shape::kTile;
    if (b + 1 < to) {
      fetch(b + 1);
      copy_wait<1>();
    } else {
      copy_wait<0>();
    }
    __syncthreads();
    locate(b + 2);
    if (newest && b + 1 == blocks) {   // the token's own row: over whatever the copy found in its place
      bf16* to_pool = p.pool + size_t(key_row(table, p1, r)) * p.pool_dim;
      bf16* to_tile = tile + (p1 - low - b * kKeys) * P;
      for (int d = threadIdx.x; d < p.rank; d += kThreads) {
        const bf16 c = __float2bfloat16_rn(__bfloat162float(raw[d]) * inv * p.norm[d]);
        to_tile[d] = c;
        if (blockIdx.y == 0) to_pool[d] = c;
      }
      __syncthreads();
    }
    float s[KN / 8][4];
#pragma unroll
    for (int t = 0; t < KN / 8; ++t) s[t][0] = s[t][1] = s[t][2] = s[t][3] = 0.f;
    if constexpr (KN >= 16) {
#pragma unroll 8
      for (int kk = 0; kk < RT; ++kk) {
        if (!FULL && kk * 16 >= p.pool_dim) break;
        uint32_t a[4];
        load_a(a, qs, P, row0, kk * 16, lane);
#pragma unroll
        for (int t = 0; t < KN / 16; ++t) {
          uint32_t bb[4];
          load_b(bb, tile + key0 * P, P, t * 16, kk * 16, lane);
          mma16816(s[2 * t], a, bb[0], bb[1]);
          mma16816(s[2 * t + 1], a, bb[2], bb[3]);
        }
      }
    } else {
      float other[4] = {};             // two chains: the odd k steps apart
#pragma unroll 8
      for (int kk = 0; kk < RT; kk += 2) {
        if (!FULL && kk * 16 >= p.pool_dim) break;
        uint32_t a[4], bb[4];
        load_b_narrow(bb, tile + key0 * P, P, 0, kk * 16, lane);
        load_a(a, qs, P, row0, kk * 16, lane);
        mma16816(s[0], a, bb[0], bb[1]);
        if (!FULL && kk * 16 + 16 >= p.pool_dim) break;
        load_a(a, qs, P, row0, kk * 16 + 16, lane);
        mma16816(other, a, bb[2], bb[3]);
      }
#pragma unroll
      for (int x = 0; x < 4; ++x) s[0][x] += other[x];
    }
    const int first = low + b * kKeys + key0 + 2 * (lane & 3);
    float high_a = -INFINITY, high_b = -INFINITY;
#pragma unroll
    for (int t = 0; t < KN / 8; ++t)
#pragma unroll
      for (int c = 0; c < 2; ++c) {
        const int j = first + 8 * t + c;
        s[t][c] = j <= pa && pa - j < p.window ? s[t][c] * p.scale_log2 : -INFINITY;
        s[t][2 + c] = j <= pb && pb - j < p.window ? s[t][2 + c] * p.scale_log2 : -INFINITY;
        high_a = fmaxf(high_a, s[t][c]);
        high_b = fmaxf(high_b, s[t][2 + c]);
      }
#pragma unroll
    for (int x = 1; x <= 2; x <<= 1) {
      high_a = fmaxf(high_a, __shfl_xor_sync(0xffffffffu, high_a, x));
      high_b = fmaxf(high_b, __shfl_xor_sync(0xffffffffu, high_b, x));
    }
    if ((lane & 3) == 0) {
      high_part[wn][ra] = high_a;
      high_part[wn][rb] = high_b;
    }
    __syncthreads();
    high_a = top_a;
    high_b = top_b;
#pragma unroll
    for (int w = 0; w < WN; ++w) {
      high_a = fmaxf(high_a, high_part[w][ra]);
      high_b = fmaxf(high_b, high_part[w][rb]);
    }
    const float ref_a = high_a == -INFINITY ? 0.f : high_a, ref_b = high_b == -INFINITY ? 0.f : high_b;
    const float fade_a = ex2(top_a - ref_a), fade_b = ex2(top_b - ref_b);
    top_a = high_a;
    top_b = high_b;
    float add_a = 0.f, add_b = 0.f;
#pragma unroll
    for (int t = 0; t < KN / 8; ++t) {
#pragma unroll
      for (int c = 0; c < 2; ++c) {
        s[t][c] = ex2(s[t][c] - ref_a);
        s[t][2 + c] = ex2(s[t][2 + c] - ref_b);
        add_a += s[t][c];
        add_b += s[t][2 + c];
      }
      // the weights enter the sums as a bf16 head and a bf16 remainder, about 16 bits of each
      const int col = key0 + 8 * t + 2 * (lane & 3);
      *reinterpret_cast<uint32_t*>(wh + ra * kWeightPitch + col) = pack(s[t][0], s[t][1]);
      *reinterpret_cast<uint32_t*>(wl + ra * kWeightPitch + col) = pack(rest(s[t][0]), rest(s[t][1]));
      *reinterpret_cast<uint32_t*>(wh + rb * kWeightPitch + col) = pack(s[t][2], s[t][3]);
      *reinterpret_cast<uint32_t*>(wl + rb * kWeightPitch + col) = pack(rest(s[t][2]), rest(s[t][3]));
    }
    sum_a = sum_a * fade_a + add_a;
    sum_b = sum_b * fade_b + add_b;
#pragma unroll
    for (int i = 0; i < 2 * CT; ++i) {
      o[i][0] *= fade_a;
      o[i][1] *= fade_a;
      o[i][2] *= fade_b;
      o[i][3] *= fade_b;
    }
    __syncthreads();
#pragma unroll
    for (int kk = 0; kk < kKeys / 16; ++kk) {
      uint32_t hi[4], lo[4];
      load_a(hi, wh, kWeightPitch, row0, kk * 16, lane);
      load_a(lo, wl, kWeightPitch, row0, kk * 16, lane);
#pragma unroll
      for (int d = 0; d < CT; ++d) {
        const int column = (wn * CT + d) * 16;
        if (!FULL && column >= p.pool_dim) break;
        uint32_t bb[4];
        load_b_transposed(bb, tile, P, kk * 16, column, lane);
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
  if ((lane & 3) == 0) {
    sum_part[wn][ra] = sum_a;
    sum_part[wn][rb] = sum_b;
  }
  __syncthreads();
  sum_a = sum_b = 0.f;
#pragma unroll
  for (int w = 0; w < WN; ++w) {
    sum_a += sum_part[w][ra];
    sum_b += sum_part[w][rb];
  }
  const bool whole = !ONE || p.splits == 1;
  auto finish = [&](int m, float top, float sum, int at) {
    const int t = m / gq, h = m % gq;
    if (t >= tokens) return;
    float f = 1.f;
    if (whole) {
      const float sink = p.sink_of(head0 + h), high = fmaxf(top, sink), fade = ex2(top - high);
      f = fade / fmaf(sum, fade, ex2(sink - high));
    }
    bf16* dst = p.out + (size_t(e.first_row + t0 + t) * p.heads + head0 + h) * p.rank_stride;
    const size_t record = (size_t(blockIdx.z) * p.heads + head0 + h) * p.splits + split;
    float* mine = p.part + record * p.rank_stride;
#pragma unroll
    for (int i = 0; i < 2 * CT; ++i) {
      const int c = wn * CT * 16 + i * 8 + 2 * (lane & 3);
      if (c >= p.rank) continue;
      const float y0 = o[i][at] * f, y1 = o[i][at + 1] * f;
      if (whole) {                   // (a row has an even number of columns; the one behind an odd rank meets zero weights)
        *reinterpret_cast<uint32_t*>(dst + c) = pack(y0, c + 1 < p.rank ? y1 : 0.f);
      } else {
        *reinterpret_cast<float2*>(mine + c) = make_float2(y0, y1);
      }
    }
    if (!whole && wn == 0 && (lane & 3) == 0) p.stats(r.entries)[record] = make_float2(top, sum);
  };
  finish(ra, top_a, sum_a, 0);
  finish(rb, top_b, sum_b, 2);
}

// A decoded token's splits put together, a CTA per head. blockIdx = (head, entry).
constexpr int kMostSplits = 64;
__global__ void __launch_bounds__(128) merge_latent(StepRows r, LatentParams p) {
  __shared__ float factor[kMostSplits];
  dependency_wait();
  allow_dependents();
  const Entry e = r.entry[blockIdx.y];
  if (e.rows != 1) return;
  const int head = blockIdx.x, lane = threadIdx.x & 31;
  const size_t record = (size_t(blockIdx.y) * p.heads + head) * p.splits;
  if (threadIdx.x < 32) {
    const float2 none = make_float2(-INFINITY, 0.f);
    const float2 a = lane < p.splits ? p.stats(r.entries)[record + lane] : none, b = lane + 32 < p.splits ? p.stats(r.entries)[record + lane + 32] : none;
    const float sink = p.sink_of(head), high = fmaxf(warp_max(fmaxf(a.x, b.x)), sink), fa = ex2(a.x - high), fb = ex2(b.x - high);
    const float sum = warp_sum(a.y * fa + b.y * fb) + ex2(sink - high);
    factor[lane] = fa / sum;
    factor[lane + 32] = fb / sum;
  }
  __syncthreads();
  const float4* parts = reinterpret_cast<const float4*>(p.part + record * p.rank_stride);
  bf16* dst = p.out + (size_t(e.first_row) * p.heads + head) * p.rank_stride;
  for (int c = threadIdx.x; c < p.rank_stride / 4; c += 128) {
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 8
    for (int s = 0; s < p.splits; ++s) {
      const float4 w = parts[size_t(s) * (p.rank_stride / 4) + c];
      v.x = fmaf(w.x, factor[s], v.x);
      v.y = fmaf(w.y, factor[s], v.y);
      v.z = fmaf(w.z, factor[s], v.z);
      v.w = fmaf(w.w, factor[s], v.w);
    }
    // (columns behind the rank were never written: they meet zero weights, as zeros)
    const float y[4] = {v.x, v.y, v.z, v.w};
    float z[4];
#pragma unroll
    for (int j = 0; j < 4; ++j) z[j] = 4 * c + j < p.rank ? y[j] : 0.f;
    *reinterpret_cast<uint2*>(dst + 4 * c) = make_uint2(pack(z[0], z[1]), pack(z[2], z[3]));
  }
}

// First expanded row of every entry: the portions' reaches one after the other, decoded tokens' empty.
__global__ void __launch_bounds__(256) latent_context(StepRows r, int window, int* context, int* context_rows) {
  __shared__ int part[8];
  dependency_wait();
  allow_dependents();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  int before = 0;
  for (int base = 0; base < r.entries; base += 256) {
    const int n = base + int(threadIdx.x);
    int reach = 0;
    if (n < r.entries) {
      const Entry e = r.entry[n];
      if (e.rows > 1) reach = e.first_position + e.rows - max(0, e.first_position - window + 1);
    }
    int sum = reach;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const int s = __shfl_up_sync(0xffffffffu, sum, o);
      if (lane >= o) sum += s;
    }
    if (lane == 31) part[warp] = sum;
    __syncthreads();
    int all = 0;
#pragma unroll
    for (int w = 0; w < 8; ++w) {
      if (w < warp) sum += part[w];
      all += part[w];
    }
    if (n < r.entries) context[n] = before + sum - reach;
    before += all;
    __syncthreads();
  }
  if (threadIdx.x == 0) *context_rows = before;
}

// One expanded row's latent row out of the pool, a warp each. The entry is the last one that starts at or before it.
__global__ void __launch_bounds__(256) gather_latent(StepRows r, int window, const uint4* pool, int pool_pieces, const int* context, const int* context_rows,
                                                     int most, uint4* out, int pieces) {
  dependency_wait();
  allow_dependents();
  const int i = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (i >= min(*context_rows, most)) return;
  int lo = 0, hi = r.entries - 1;
  while (lo < hi) {
    const int mid = (lo + hi + 1) / 2;
    if (context[mid] <= i) lo = mid;
    else hi = mid - 1;
  }
  const Entry e = r.entry[lo];
  const int position = min(max(0, e.first_position - window + 1) + i - context[lo], r.capacity - 1);
  const int row = key_row(r.block_table + size_t(e.slot) * r.max_blocks, position, r);
  for (int c = lane; c < pieces; c += 32) out[size_t(i) * pieces + c] = pool[size_t(row) * pool_pieces + c];
}

template <int RT, int WM, bool ONE> int LaunchLatent(const Queue& q, const StepRows& r, const LatentParams& p, int x) {
  auto kernel = p.pool_dim == 16 * RT ? attend_latent<RT, WM, ONE, true> : attend_latent<RT, WM, ONE, false>;
  return int(Launch(kernel, dim3(unsigned(x), unsigned(p.subs), unsigned(r.entries)), dim3(LatentShape<RT, WM>::kThreads), LatentShape<RT, WM>::kSmem, q.stream, q.chained, r, p));
}

template <int RT> int LatentWith(const Queue& q, const StepRows& r, const LatentArgs& a, LatentParams p) {
  auto divide = [&](int most) {      // the heads in as few units of at most this many as there can be
    p.subs = (a.heads + most - 1) / most;
    p.sub_heads = (a.heads + p.subs - 1) / p.subs;
    p.subs = (a.heads + p.sub_heads - 1) / p.sub_heads;
  };
  if (r.singles > 0) {
    // Units of 16 heads while these do not fill the GPU, else as few as there can be; then the cut of a decoded token's keys
    // that ends soonest: a CTA costs its blocks plus a few blocks' time to start, a merge behind it two.
    const int blocks = std::min(a.window, r.capacity) / kKeys + 1;
    divide(size_t(r.singles) * ((a.heads + 15) / 16) * blocks <= size_t(q.sm_count) ? 16 : 64);
    LatentParams one = p;
    one.splits = 1;
    float least = 0.f;
    for (int s = 1; s <= std::min(blocks, kMostSplits); ++s) {
      if (size_t(r.entries) * a.heads * s * (a.rank_stride + 2) > a.part_floats) break;
      const int waves = (r.singles * p.subs * s + q.sm_count - 1) / q.sm_count;
      const float cost = float(waves) * (float((blocks + s - 1) / s) + 2.f) + (s > 1 ? 2.f + float(s) / 16.f : 0.f);
      if (s == 1 || cost < least) {
        least = cost;
        one.splits = s;
      }
    }
    int status = p.sub_heads <= 16 ? LaunchLatent<RT, 1, true>(q, r, one, one.splits) : p.sub_heads <= 32 ? LaunchLatent<RT, 2, true>(q, r, one, one.splits)
                 : LaunchLatent<RT, 4, true>(q, r, one, one.splits);
    if (status == 0 && one.splits > 1)
      status = int(Launch(merge_latent, dim3(unsigned(a.heads), unsigned(r.entries)), dim3(128), 0, q.stream, q.chained, r, one));
    if (status != 0) return status;
  }
  divide(64);
  if (r.singles < r.entries && !a.singles_only) {
    const int per_tile = 64 / p.sub_heads;
    p.splits = 1;
    return LaunchLatent<RT, 4, false>(q, r, p, (r.longest + per_tile - 1) / per_tile);
  }
  return 0;
}

template <int RT, int WM, bool ONE> cudaError_t RaiseOne() {
  for (auto kernel : {attend_latent<RT, WM, ONE, false>, attend_latent<RT, WM, ONE, true>}) {
    const cudaError_t err = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, LatentShape<RT, WM>::kSmem);
    if (err != cudaSuccess) return err;
  }
  return cudaSuccess;
}
template <int RT> cudaError_t Raise() {
  cudaError_t err = RaiseOne<RT, 1, true>();
  if (err == cudaSuccess) err = RaiseOne<RT, 2, true>();
  if (err == cudaSuccess) err = RaiseOne<RT, 4, true>();
  if (err == cudaSuccess) err = RaiseOne<RT, 4, false>();
  return err;
}

}  // namespace

int AttendLatentTiles(const Queue& q, const StepRows& r, const LatentArgs& a) {
  LatentParams p{};
  p.q = static_cast<const bf16*>(a.q);
  p.raw = static_cast<const bf16*>(a.raw);
  p.pool = static_cast<bf16*>(a.pool);
  p.out = static_cast<bf16*>(a.out);
  p.part = a.part;
  p.norm = a.norm;
  p.sinks = a.sinks;
  p.raw_stride = a.raw_stride;
  p.heads = a.heads;
  p.rank = a.rank;
  p.rank_stride = a.rank_stride;
  p.pool_dim = a.pool_dim;
  p.window = a.window;
  p.scale_log2 = a.scale * 1.4426950408889634f;
  p.sink_log2 = a.sink * 1.4426950408889634f;
  p.eps = a.eps;
  return a.rank <= 128 ? LatentWith<8>(q, r, a, p) : a.rank <= 256 ? LatentWith<16>(q, r, a, p) : LatentWith<32>(q, r, a, p);
}

int LatentContext(const Queue& q, const StepRows& r, int window, int* context, int* context_rows) {
  return int(Launch(latent_context, dim3(1), dim3(256), 0, q.stream, q.chained, r, window, context, context_rows));
}

int GatherLatent(const Queue& q, const StepRows& r, const LatentArgs& a, const int* context, const int* context_rows, int most, void* out) {
  if (q.f32) return int(cudaErrorInvalidValue);
  return int(Launch(gather_latent, dim3(unsigned((most + 7) / 8)), dim3(256), 0, q.stream, q.chained, r, a.window, static_cast<const uint4*>(a.pool),
                    a.pool_dim / 8, context, context_rows, most, static_cast<uint4*>(out), a.rank_stride / 8));
}

int PrepareLatent() {
  cudaError_t err = Raise<8>();
  if (err == cudaSuccess) err = Raise<16>();
  if (err == cudaSuccess) err = Raise<32>();
  return int(err);
}

}  // namespace tmb
