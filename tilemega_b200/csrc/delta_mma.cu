// The generalised delta rule over portions in bf16 plans, see DeltaArgs: sixteen tokens at a time on the tensor pipe (mma.sync),
// the state in fp32 accumulators. Within a chunk, with c_t the sum of the log decays up to token t (per key channel), u the unit key,
// b = removal rate times u, and S the state before the chunk, what token t reads of the old state (p_t) and its output (o_t) are
//   p_t = (u_t e^c_(t-1))^T S - sum_(j<t) L_tj p_j + sum_(j<t) M_tj v_j,    L_tj = u_t^T e^(c_(t-1) - c_j) b_j,   M: k_j in place of b_j
//   o_t = (r_t e^c_t)^T S - sum_(j<=t) Lr_tj p_j + sum_(j<=t) Mr_tj v_j,     Lr, Mr: r_t and c_t in place of u_t and c_(t-1)
// which is linear in S and in the values. Solved for p (I + L is unit lower triangular) a chunk is
//   P = U S + G V,   O = R S + H V,   S' = diag(e^c) S + B^T P + K^T V,      B_j = -b_j e^(c - c_j),   K_j = k_j e^(c - c_j)
// with U = (I + L)^-1 (u e^c), G = (I + L)^-1 M, R = (r e^c) - Lr U, H = Mr - Lr G: small, and without the state, so delta_split forms
// them for all chunks at once, in fp32. Columns of a state do not meet: in delta_chunks a CTA owns sixteen and walks the chunks. Operands
// enter the products as bf16 heads and remainders (the values are bf16 as they are).
#include <algorithm>
#include <initializer_list>

#include "mixers.cuh"
#include "mma.cuh"
#include "ops.h"
#include "tensor_map.h"

namespace tmb {
namespace {

constexpr int kChunk = 16;

// A chunk of a head as delta_split leaves it: operands in the order in which lanes hold them (head and remainder of both pairs: 16
// bytes a lane), then the whole chunk's decays.
template <int KS> struct Record {        // KS: sixteens of key channels
  static constexpr int kPadded = 16 * KS;
  static constexpr int kRows = 0;                          // [KS][4: U, U, R, R by eight rows][32 lanes]
  static constexpr int kColumns = KS * 4 * 512;            // [2 KS eights of channels][2: B, K][32 lanes]
  static constexpr int kWithin = 2 * kColumns;             // [4: G, G, H, H by eight rows][32 lanes]
  static constexpr int kDecay = kWithin + 4 * 512;
  static constexpr int kBytes = kDecay + kPadded * 4;
};

struct SplitParams {
  const bf16* proj;
  const float* z;
  unsigned char* chunks;
  int proj_stride, heads, dim;
  float decay_scale, unit_eps;
  bool wide, portions_only;
};

__device__ __forceinline__ int first_chunk(const Entry& e, int entry) { return e.first_row / kChunk + entry; }

__device__ __forceinline__ uint4 heads_and_rests(float a, float b, float c, float d) {
  return make_uint4(pack(a, b), pack(c, d), pack(rest(a), rest(b)), pack(rest(c), rest(d)));
}

// blockIdx = (chunk, head, entry)
constexpr int kSplitThreads = 288, kSplitWarps = kSplitThreads / 32;
template <int KS> constexpr int kSplitMemory = (4 * kChunk * (16 * KS + 4) + 4 * kChunk * kChunk + 16 * KS + kChunk) * 4;
template <int KS> __global__ void __launch_bounds__(kSplitThreads) delta_split(StepRows r, SplitParams p) {
  using Layout = Record<KS>;
  constexpr int DP = Layout::kPadded, kPitch = DP + 4, M = (DP / 4 + 31) / 32;
  extern __shared__ __align__(16) float memory[];
  float *us = memory, *rs = us + kChunk * kPitch, *bs = rs + kChunk * kPitch, *ks = bs + kChunk * kPitch;   // [token][channel]
  float *ub = ks + kChunk * kPitch, *uk = ub + kChunk * kChunk, *rb = uk + kChunk * kChunk, *rk = rb + kChunk * kChunk;   // L, M, Lr, Mr
  float *decay = rk + kChunk * kChunk, *inverse = decay + DP;
  dependency_wait();
  allow_dependents();
  const Entry e = r.entry[blockIdx.z];
  const int from = blockIdx.x * kChunk, count = min(kChunk, e.rows - from), head = blockIdx.y;
  if (count <= 0 || (p.portions_only && e.rows == 1)) return;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const size_t all = size_t(p.heads) * p.dim;
  for (int t = warp; t < kChunk; t += kSplitWarps) {       // r, k, removal rate times k, log decay (us)
    const size_t row = size_t(e.first_row) + from + t;
    const bf16* line = p.proj + row * p.proj_stride + size_t(head) * p.dim;
    const float* z = p.z + row * all + size_t(head) * p.dim;
    float square = 0.f;
#pragma unroll
    for (int m = 0; m < M; ++m) {
      const int d = 4 * (lane + 32 * m), here = t < count ? min(4, p.dim - d) : 0;
      float rv[4], kv[4], av[4], zv[4];
      load_four(line + d, here, p.wide, rv);
      load_four(line + all + d, here, p.wide, kv);
      load_four(line + 3 * all + d, here, p.wide, av);
      load_four(z + d, here, p.wide, zv);
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        square = fmaf(kv[i], kv[i], square);
        av[i] = kv[i] * sigmoid(av[i]);
        zv[i] = i < here ? -p.decay_scale * sigmoid(zv[i]) : 0.f;
      }
      if (d < DP) {
        const int at = t * kPitch + d;
        *reinterpret_cast<float4*>(us + at) = make_float4(zv[0], zv[1], zv[2], zv[3]);
        *reinterpret_cast<float4*>(rs + at) = make_float4(rv[0], rv[1], rv[2], rv[3]);
        *reinterpret_cast<float4*>(bs + at) = make_float4(av[0], av[1], av[2], av[3]);
        *reinterpret_cast<float4*>(ks + at) = make_float4(kv[0], kv[1], kv[2], kv[3]);
      }
    }
    square = warp_sum(square);
    if (lane == 0) inverse[t] = 1.f / sqrtf(square + p.unit_eps);
  }
  __syncthreads();
  if (const int d = threadIdx.x; d < DP) {                 // decays
    float sum = 0.f, before = 1.f;
    for (int t = 0; t < kChunk; ++t) {
      const int at = t * kPitch + d;
      sum += us[at];
      const float after = expf(sum), grown = expf(-sum), k = ks[at], inv = inverse[t];
      us[at] = k * inv * before;
      rs[at] *= after;
      bs[at] *= inv * grown;
      ks[at] = k * grown;
      before = after;
    }
    decay[d] = before;
  }
  __syncthreads();
  for (int i = threadIdx.x; i < kChunk * kChunk; i += kSplitThreads) {
    const int t = i / kChunk, j = i % kChunk;
    float sum[4] = {};
    if (j <= t) {
      const float4 *u = reinterpret_cast<const float4*>(us + t * kPitch), *v = reinterpret_cast<const float4*>(rs + t * kPitch);
      const float4 *b = reinterpret_cast<const float4*>(bs + j * kPitch), *k = reinterpret_cast<const float4*>(ks + j * kPitch);
#pragma unroll 4
      for (int d = 0; d < DP / 4; ++d) {
        const float4 uq = u[d], rq = v[d], bq = b[d], kq = k[d];
        auto dot = [](float s, const float4& x, const float4& y) { return fmaf(x.w, y.w, fmaf(x.z, y.z, fmaf(x.y, y.y, fmaf(x.x, y.x, s)))); };
        sum[0] = dot(sum[0], uq, bq);
        sum[1] = dot(sum[1], uq, kq);
        sum[2] = dot(sum[2], rq, bq);
        sum[3] = dot(sum[3], rq, kq);
      }
    }
    ub[i] = j < t ? sum[0] : 0.f;
    uk[i] = j < t ? sum[1] : 0.f;
    rb[i] = sum[2];
    rk[i] = sum[3];
  }
  __syncthreads();
  // forward substitution, a channel of U and R or (the last warp) a column of G and H each
  const bool within = threadIdx.x >= kSplitThreads - 32;
  const int column = within ? threadIdx.x - (kSplitThreads - 32) : threadIdx.x;
  if (column < (within ? kChunk : DP)) {
    float *first = (within ? uk : us) + column, *second = (within ? rk : rs) + column, x[kChunk];
    const int pitch = within ? kChunk : kPitch;
#pragma unroll
    for (int t = 0; t < kChunk; ++t) {
      float a = first[t * pitch], b = second[t * pitch];
      const float4 *l = reinterpret_cast<const float4*>(ub + t * kChunk), *lr = reinterpret_cast<const float4*>(rb + t * kChunk);
      float row[kChunk];
#pragma unroll
      for (int j = 0; j < t; j += 4) {
        const float4 q = l[j / 4];
        row[j] = q.x, row[j + 1] = q.y, row[j + 2] = q.z, row[j + 3] = q.w;
      }
#pragma unroll
      for (int j = 0; j < t; ++j) a = fmaf(-row[j], x[j], a);
      x[t] = a;
#pragma unroll
      for (int j = 0; j <= t; j += 4) {
        const float4 q = lr[j / 4];
        row[j] = q.x, row[j + 1] = q.y, row[j + 2] = q.z, row[j + 3] = q.w;
      }
#pragma unroll
      for (int j = 0; j <= t; ++j) b = fmaf(-row[j], x[j], b);
      first[t * pitch] = a;
      second[t * pitch] = b;
    }
  }
  __syncthreads();
  unsigned char* out = p.chunks + (size_t(first_chunk(e, blockIdx.z) + blockIdx.x) * p.heads + head) * Layout::kBytes;
  for (int i = threadIdx.x; i < KS * 4 * 32; i += kSplitThreads) {
    const int owner = i & 31, n = (i >> 5 & 1) * 8 + (owner >> 2), d = (i >> 7) * 16 + 2 * (owner & 3);
    const float* row = (i & 64 ? rs : us) + n * kPitch + d;
    const float2 a = *reinterpret_cast<const float2*>(row), b = *reinterpret_cast<const float2*>(row + 8);
    reinterpret_cast<uint4*>(out + Layout::kRows)[i] = heads_and_rests(a.x, a.y, b.x, b.y);
  }
  for (int i = threadIdx.x; i < KS * 4 * 32; i += kSplitThreads) {
    const int owner = i & 31, d = (i >> 6) * 8 + (owner >> 2), t = 2 * (owner & 3);
    const float* x = (i & 32 ? ks : bs) + d;
    const float w = i & 32 ? decay[d] : -decay[d];
    reinterpret_cast<uint4*>(out + Layout::kColumns)[i] =
        heads_and_rests(w * x[t * kPitch], w * x[(t + 1) * kPitch], w * x[(t + 8) * kPitch], w * x[(t + 9) * kPitch]);
  }
  for (int i = threadIdx.x; i < 4 * 32; i += kSplitThreads) {
    const int owner = i & 31;
    const float* x = (i & 64 ? rk : uk) + ((i >> 5 & 1) * 8 + (owner >> 2)) * kChunk + 2 * (owner & 3);
    reinterpret_cast<uint4*>(out + Layout::kWithin)[i] = heads_and_rests(x[0], x[1], x[8], x[9]);
  }
  for (int d = threadIdx.x; d < DP; d += kSplitThreads) reinterpret_cast<float*>(out + Layout::kDecay)[d] = decay[d];
}

struct ChunkParams {
  const bf16* values;                    // of the first row and head
  const unsigned char* chunks;
  float *state, *raw;
  unsigned* status;
  int proj_stride, heads, dim, padded;
  bool portions_only;
};

// An entry's chunks in order, sixteen columns of a head's state a CTA, each of its warps a quarter of the key channels: their shares of
// P and O meet in shared memory. blockIdx = (columns, head, entry).
constexpr int kWalkers = 4, kWalkThreads = 32 * kWalkers, kSlots = 3;
constexpr int kShares = 2 * kWalkers * 4 * 32 * 16;        // [chunk & 1][warp][4][32 lanes] four floats
template <int KS> constexpr int kWalkMemory = kSlots * Record<KS>::kBytes + kShares + kSlots * 8;
template <int KS> __global__ void __launch_bounds__(kWalkThreads) delta_chunks(StepRows r, ChunkParams p) {
  using Layout = Record<KS>;
  constexpr int KW = KS / kWalkers;      // sixteens of channels of a warp
  extern __shared__ __align__(128) unsigned char slots[];
  float4* shares = reinterpret_cast<float4*>(slots + kSlots * Layout::kBytes);
  uint64_t* full = reinterpret_cast<uint64_t*>(slots + kSlots * Layout::kBytes + kShares);
  const Entry e = r.entry[blockIdx.z];   // (tables and states: written before the kernel this one depends on)
  if (p.portions_only && e.rows == 1) {
    dependency_wait();
    allow_dependents();
    return;
  }
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, head = blockIdx.y, pair = 2 * (lane & 3);
  const int column = blockIdx.x * 16 + (lane >> 2);        // and the eighth behind it
  const size_t all = size_t(p.heads) * p.dim;
  float* state = p.state + (size_t(e.slot) * p.heads + head) * p.dim * p.padded;
  float s[2 * KW][4];                    // columns x channels
  auto each_state = [&](auto&& visit) {
#pragma unroll
    for (int n = 0; n < 2 * KW; ++n)
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int c = column + 8 * half, d = 8 * (2 * KW * warp + n) + pair;
        if (c < p.dim && d < p.padded) visit(*reinterpret_cast<float2*>(state + size_t(c) * p.padded + d), s[n][2 * half], s[n][2 * half + 1]);
      }
  };
#pragma unroll
  for (int n = 0; n < 2 * KW; ++n)
#pragma unroll
    for (int i = 0; i < 4; ++i) s[n][i] = 0.f;
  if (e.first_position > 0)
    each_state([](const float2& at, float& a, float& b) {
      const float2 v = __ldcs(&at);
      a = v.x, b = v.y;
    });
  const int chunks = (e.rows + kChunk - 1) / kChunk;
  const unsigned char* record = p.chunks + (size_t(first_chunk(e, blockIdx.z)) * p.heads + head) * Layout::kBytes;
  int issued = 0;
  auto fetch = [&]() {                   // (one thread)
    uint64_t* bar = &full[issued % kSlots];
    mbar_expect_tx(bar, Layout::kBytes);
    bulk_g2s(slots + size_t(issued % kSlots) * Layout::kBytes, record + size_t(issued) * p.heads * Layout::kBytes, Layout::kBytes, bar);
    ++issued;
  };
  if (threadIdx.x == 0) {
    for (int i = 0; i < kSlots; ++i) mbar_init(&full[i], 1);
    mbar_fence_init();
  }
  dependency_wait();
  allow_dependents();
  __syncthreads();
  if (threadIdx.x == 0)
    while (issued < min(kSlots, chunks)) fetch();
  uint32_t values[4], next[4];           // columns x tokens
  auto load_values = [&](int chunk) {
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int c = column + 8 * (i & 1), t = chunk * kChunk + pair + 8 * (i >> 1);
      const unsigned short* at = reinterpret_cast<const unsigned short*>(p.values) + size_t(e.first_row + t) * p.proj_stride + size_t(head) * p.dim + c;
      const uint32_t low = c < p.dim && t < e.rows ? at[0] : 0, high = c < p.dim && t + 1 < e.rows ? at[p.proj_stride] : 0;
      next[i] = low | high << 16;
    }
  };
  load_values(0);
  bool ok = true;
  for (int chunk = 0; chunk < chunks; ++chunk) {
    const unsigned char* slot = slots + size_t(chunk % kSlots) * Layout::kBytes;
#pragma unroll
    for (int i = 0; i < 4; ++i) values[i] = next[i];
    if (chunk + 1 < chunks) load_values(chunk + 1);
    ok = __all_sync(0xffffffffu, wait_bounded(&full[chunk % kSlots], uint32_t(chunk / kSlots) & 1u, p.status, 16)) && ok;
    const uint4* rows = reinterpret_cast<const uint4*>(slot + Layout::kRows) + KW * warp * 128 + lane;
    const uint4* columns = reinterpret_cast<const uint4*>(slot + Layout::kColumns) + KW * warp * 128 + lane;
    const float* decay = reinterpret_cast<const float*>(slot + Layout::kDecay) + KW * warp * 16 + pair;
    float x[4][4] = {}, y[4][4] = {};    // P, P, O, O by eight tokens: products of heads, and those with a remainder
#pragma unroll
    for (int k = 0; k < KW; ++k) {
      const float (&f)[4] = s[2 * k], (&g)[4] = s[2 * k + 1];
      const uint32_t high[4] = {pack(f[0], f[1]), pack(f[2], f[3]), pack(g[0], g[1]), pack(g[2], g[3])};
      const uint32_t low[4] = {pack(rest(f[0]), rest(f[1])), pack(rest(f[2]), rest(f[3])), pack(rest(g[0]), rest(g[1])), pack(rest(g[2]), rest(g[3]))};
      uint4 b[4];
#pragma unroll
      for (int n = 0; n < 4; ++n) b[n] = rows[(k * 4 + n) * 32];
#pragma unroll
      for (int n = 0; n < 4; ++n) mma16816(x[n], high, b[n].x, b[n].y);
#pragma unroll
      for (int n = 0; n < 4; ++n) mma16816(y[n], low, b[n].x, b[n].y);
#pragma unroll
      for (int n = 0; n < 4; ++n) mma16816(y[n], high, b[n].z, b[n].w);
    }
    const uint4 within = reinterpret_cast<const uint4*>(slot + Layout::kWithin)[warp * 32 + lane];
    float4* share = shares + (chunk & 1) * kWalkers * 4 * 32 + lane;
#pragma unroll
    for (int n = 0; n < 4; ++n) {        // (what comes of the values: by one warp per eight tokens)
      if (n == warp) {
        mma16816(x[n], values, within.x, within.y);
        mma16816(y[n], values, within.z, within.w);
      }
      share[(warp * 4 + n) * 32] = make_float4(x[n][0] + y[n][0], x[n][1] + y[n][1], x[n][2] + y[n][2], x[n][3] + y[n][3]);
    }
    __syncthreads();                     // (and nobody reads the slot of the chunk before any more)
    if (threadIdx.x == 0 && ok && chunk > 0 && issued < chunks) fetch();
    auto sum = [&](int n) {
      float4 v = share[n * 32];
#pragma unroll
      for (int w = 1; w < kWalkers; ++w) {
        const float4 more = share[(w * 4 + n) * 32];
        v.x += more.x, v.y += more.y, v.z += more.z, v.w += more.w;
      }
      return v;
    };
    const float4 p0 = sum(0), p1 = sum(1);
    const uint32_t high[4] = {pack(p0.x, p0.y), pack(p0.z, p0.w), pack(p1.x, p1.y), pack(p1.z, p1.w)};
    const uint32_t low[4] = {pack(rest(p0.x), rest(p0.y)), pack(rest(p0.z), rest(p0.w)), pack(rest(p1.x), rest(p1.y)), pack(rest(p1.z), rest(p1.w))};
#pragma unroll
    for (int group = 0; group < 2 * KW; group += 2) {
      uint4 b[2], k[2];
#pragma unroll
      for (int n = 0; n < 2; ++n) {
        float (&f)[4] = s[group + n];
        const float2 w = *reinterpret_cast<const float2*>(decay + 8 * (group + n));
        f[0] *= w.x, f[1] *= w.y, f[2] *= w.x, f[3] *= w.y;
        b[n] = columns[(group + n) * 64];
        k[n] = columns[(group + n) * 64 + 32];
      }
#pragma unroll
      for (int n = 0; n < 2; ++n) mma16816(s[group + n], values, k[n].x, k[n].y);
#pragma unroll
      for (int n = 0; n < 2; ++n) mma16816(s[group + n], values, k[n].z, k[n].w);
#pragma unroll
      for (int n = 0; n < 2; ++n) mma16816(s[group + n], high, b[n].x, b[n].y);
#pragma unroll
      for (int n = 0; n < 2; ++n) mma16816(s[group + n], low, b[n].x, b[n].y);
#pragma unroll
      for (int n = 0; n < 2; ++n) mma16816(s[group + n], high, b[n].z, b[n].w);
    }
    if (warp < 2) {
      const float4 o = sum(2 + warp);
      const float v[4] = {o.x, o.y, o.z, o.w};
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int t = chunk * kChunk + warp * 8 + pair + (i & 1), c = column + 8 * (i >> 1);
        if (c < p.dim && t < e.rows) p.raw[size_t(e.first_row + t) * all + size_t(head) * p.dim + c] = v[i];
      }
    }
  }
  if (!ok && threadIdx.x == 0)           // copies still under way
    for (int i = max(0, issued - kSlots); i < issued; ++i) wait_bounded(&full[i % kSlots], uint32_t(i / kSlots) & 1u, p.status, 17);
  if (ok)
    each_state([](float2& at, const float& a, const float& b) { at = make_float2(a, b); });
}

template <int KS> int ChunksWith(const Queue& q, const StepRows& r, const SplitParams& split, const ChunkParams& p) {
  const int status = int(Launch(delta_split<KS>, dim3(unsigned((r.longest + kChunk - 1) / kChunk), unsigned(p.heads), unsigned(r.entries)), dim3(kSplitThreads),
                                kSplitMemory<KS>, q.stream, q.chained, r, split));
  if (status != 0) return status;
  return int(Launch(delta_chunks<KS>, dim3(unsigned((p.dim + 15) / 16), unsigned(p.heads), unsigned(r.entries)), dim3(kWalkThreads),
                    kWalkMemory<KS>, q.stream, q.chained, r, p));
}

int Sixteens(int dim) {
  return std::min(16, (dim + 63) / 64 * 4);   // (the warps of a walk share the channels)
}
template <typename F> auto WithSixteens(int dim, F&& f) {
  switch (Sixteens(dim)) {
    case 4: return f(std::integral_constant<int, 4>());
    case 8: return f(std::integral_constant<int, 8>());
    case 12: return f(std::integral_constant<int, 12>());
    default: return f(std::integral_constant<int, 16>());
  }
}

}  // namespace

size_t DeltaChunkBytes(int rows, int slots, int heads, int dim) {
  const size_t bytes = WithSixteens(dim, [](auto k) { return size_t(Record<k.value>::kBytes); });
  return bytes * size_t(heads) * size_t(rows / kChunk + slots + 1);
}

int DeltaChunks(const Queue& q, const StepRows& r, const DeltaArgs& a, bool portions_only) {
  if (!a.chunks || a.decay_scale > kMostDecay) return int(cudaErrorInvalidValue);   // (keys are multiplied by e^(16 decay_scale) at most)
  const bf16* proj = static_cast<const bf16*>(a.proj);
  const bool wide = a.dim % 4 == 0 && a.proj_stride % 4 == 0 && reinterpret_cast<uintptr_t>(proj) % 8 == 0;
  unsigned char* chunks = static_cast<unsigned char*>(a.chunks);
  const SplitParams split{proj, a.z, chunks, a.proj_stride, a.heads, a.dim, a.decay_scale, a.unit_eps, wide, portions_only};
  const ChunkParams p{proj + 2 * size_t(a.heads) * a.dim, chunks, a.state, a.raw, q.status, a.proj_stride, a.heads, a.dim, a.padded, portions_only};
  return WithSixteens(a.dim, [&](auto k) { return ChunksWith<k.value>(q, r, split, p); });
}

int PrepareDeltaChunks() {
  for (int dim : {64, 128, 192, 256}) {
    const cudaError_t err = WithSixteens(dim, [](auto k) {
      const cudaError_t split = cudaFuncSetAttribute(delta_split<k.value>, cudaFuncAttributeMaxDynamicSharedMemorySize, kSplitMemory<k.value>);
      return split != cudaSuccess ? split : cudaFuncSetAttribute(delta_chunks<k.value>, cudaFuncAttributeMaxDynamicSharedMemorySize, kWalkMemory<k.value>);
    });
    if (err != cudaSuccess) return int(err);
  }
  return 0;
}

}  // namespace tmb
