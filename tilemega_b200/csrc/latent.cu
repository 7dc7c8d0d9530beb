// Latent attention of bf16 ragged steps on the tensor pipe: every head of a token reads the same cached rows, as keys and as
// values, so blocks of latent rows are copied once for both. Decoded tokens (decode_latent): tcgen05, latent rows by TMA.
// Short portions (attend_latent): mma.sync tiles of (token, head) rows; long ones expand the rows they see first.
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

struct LatentParams {
  const bf16* q;
  const bf16* raw;                 // null: every row of the step lies in the pool already
  bf16* pool;
  bf16* out;
  float* part;                     // split sums: [entry][head][split][rank_stride] latent columns, then [entry][head][split] references and sums
  unsigned* status;
  const float *norm, *sinks;
  int raw_stride, heads, rank, rank_stride, pool_dim, window, splits;
  int subs, sub_heads;             // the heads are served in `subs` units of up to `sub_heads`
  float scale_log2, sink_log2, eps;
  __device__ float2* stats(int entries) const { return reinterpret_cast<float2*>(part + size_t(entries) * heads * splits * rank_stride); }
  __device__ float sink_of(int head) const { return sinks ? sinks[head] * 1.4426950408889634f : sink_log2; }
};

// ---- one decoded token ---------------------------------------------------------------------------------------------------
// With C [64 keys][latent columns] a block of rows as TMA leaves it (128-byte swizzled chunks of 64 columns, two to a slot):
//   S [head][key] = Q C^T       A = Q, B = C; of the 128 rows of the tile only a unit's (up to 32) mean anything
//   O^T [column][head] += C^T P^T   A = C read transposed, 128 columns a slot; B = the weights P, each as a bf16 head (rows
//                                   0 .. 31) and a bf16 remainder (rows 32 .. 63), summed at the end
// so both products stream the rows through the tensor core from the one copy. Warp 0 requests rows, warp 1 issues products,
// warps 4 to 7 share the softmax (a lane per head, 16 keys a warp), own the columns of O (rescaled only when a maximum outgrows
// its reference by 2^8) and put the token's own row, normed, and zeros for rows out of sight into the edge blocks.
// A ring of slots holds blocks ahead: up to 256 columns four of them, two CTAs then share an SM and hide each other's waits.
constexpr int kUnitHeads = 32, kLatentThreads = 256, kMostSlots = 10, kSharedSlots = 4, kSharedChunks = 4;
constexpr int kChunkBytes = kKeys * 128, kSlotBytes = 2 * kChunkBytes, kQueryChunk = kUnitHeads * 128, kMostChunks = kTiledLatent / 64;
constexpr int kWeightBytes = 2 * kUnitHeads * 128;
constexpr int kScorePitch = kKeys + 4;
__host__ __device__ constexpr int DecodeSmem(int chunks, int ring) {
  return chunks * kQueryChunk + ring * kSlotBytes + 2 * kWeightBytes + kUnitHeads * kScorePitch * 4 + 1024;
}
static_assert(kMostSlots * kSlotBytes >= 128 * 128, "a score product reads 128 query rows, past the last chunk's own");
static_assert(kSharedSlots * kSlotBytes >= 128 * 128, "a score product reads 128 query rows, past the last chunk's own");
constexpr int kScoreColumns = kKeys, kSumColumns = 2 * kUnitHeads;   // tensor memory: two blocks' scores, then a slot's sums each
constexpr float kGrowth = 8.f;

__device__ __forceinline__ void column_sync() { asm volatile("bar.sync 1, 128;" ::: "memory"); }

template <bool SHARED>
__global__ void __launch_bounds__(kLatentThreads, SHARED ? 2 : 1) decode_latent(const __grid_constant__ CUtensorMap pool_map, const __grid_constant__ CUtensorMap q_map,
                                                                   StepRows r, LatentParams p) {
  constexpr int kSlots = SHARED ? kSharedSlots : kMostSlots, kQueryBytes = (SHARED ? kSharedChunks : kMostChunks) * kQueryChunk;
  constexpr int kTensorColumns = SHARED ? 256 : 512;
  extern __shared__ unsigned char smem_raw[];
  unsigned char* queries = reinterpret_cast<unsigned char*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  unsigned char* slots = queries + kQueryBytes;        // (the score product reads rows behind a unit's out of whatever follows)
  unsigned char* weights = slots + kSlots * kSlotBytes;
  float* scores = reinterpret_cast<float*>(weights + 2 * kWeightBytes);
  __shared__ uint64_t full[kSlots], empty[kSlots], query_full, score_full[2], weight_full[2], sum_done[2], patched;
  __shared__ uint32_t tmem_slot;
  __shared__ float exchange[4][kUnitHeads], factor[kUnitHeads], square_part[4];
  const Entry e = r.entry[blockIdx.z];   // (tables, the rows of earlier steps, this step's projection: there before the dependency wait)
  if (e.rows != 1) {
    dependency_wait();
    allow_dependents();
    return;
  }
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int head0 = blockIdx.y * p.sub_heads, heads = min(p.sub_heads, p.heads - head0), split = blockIdx.x;
  const int p1 = e.first_position, low = max(0, p1 - p.window + 1), start = low / kRaggedBlock * kRaggedBlock;
  const int* table = r.block_table + size_t(e.slot) * r.max_blocks;
  const int blocks = (p1 - start) / kKeys + 1, share = (blocks + p.splits - 1) / p.splits;
  const int from = min(blocks, split * share), count = min(blocks, from + share) - from;
  const int chunks = (p.pool_dim + 63) / 64, pairs = (chunks + 1) / 2;
  auto edge = [&](int i) { return start + (from + i) * kKeys < low || from + i == blocks - 1; };   // a block with rows to put in

  if (threadIdx.x == 0) {
    prefetch_map(&pool_map);
    prefetch_map(&q_map);
    for (int s = 0; s < kSlots; ++s) {
      mbar_init(&full[s], 1);
      mbar_init(&empty[s], 1);
    }
    mbar_init(&query_full, 1);
    for (int s = 0; s < 2; ++s) {
      mbar_init(&score_full[s], 1);
      mbar_init(&weight_full[s], 4);
      mbar_init(&sum_done[s], 1);
    }
    mbar_init(&patched, 128);
    mbar_fence_init();
  }
  if (warp == 1) tmem_alloc(&tmem_slot, kTensorColumns);
  tcgen05_fence_before();
  __syncthreads();
  tcgen05_fence_after();
  const uint32_t tmem = tmem_slot;

  if (warp == 0) {
    // lane = (chunk of the slot, page of the block): one box of 16 rows x 64 columns each
    const int total = count * pairs, page = lane & 3, chunk = (lane >> 2) & 1;
    int issued = 0;
    bool ok = true;
    auto request = [&](int it) {
      const int s = it % kSlots, block = it / pairs, pair = it % pairs, live = min(2, chunks - 2 * pair);
      if (it >= kSlots) ok = __all_sync(0xffffffffu, wait_bounded(&empty[s], uint32_t(it / kSlots - 1) & 1u, p.status, 5));
      if (!ok) return;
      if (lane == 0) mbar_expect_tx(&full[s], uint32_t(live * kChunkBytes));
      __syncwarp();
      if (lane < 4 * live) {
        const int position = min(start + (from + block) * kKeys + page * kRaggedBlock, r.capacity - 1);
        tma_load_2d(slots + s * kSlotBytes + chunk * kChunkBytes + page * kRaggedBlock * 128, &pool_map, (2 * pair + chunk) * 64,
                    key_row(table, position / kRaggedBlock * kRaggedBlock, r), &full[s]);
      }
      issued = it + 1;
    };
    const int early = min(total, kSlots);
    for (int it = 0; it < early; ++it) request(it);
    dependency_wait();
    if (lane == 0 && count > 0) {
      mbar_expect_tx(&query_full, uint32_t(chunks * kQueryChunk));
      for (int c = 0; c < chunks; ++c) tma_load_2d(queries + c * kQueryChunk, &q_map, 64 * c, e.first_row * p.heads + head0, &query_full);
    }
    for (int it = early; it < total && ok; ++it) request(it);
    if (!ok) {   // leaving early: let the copies already issued land first
      for (int it = max(0, issued - kSlots); it < issued; ++it) wait_bounded(&full[it % kSlots], uint32_t(it / kSlots) & 1u, p.status, 6);
      wait_bounded(&query_full, 0, p.status, 6);
    }
  } else {
    dependency_wait();
  }
  allow_dependents();

  if (warp == 1 && lane == 0) {
    const uint32_t score_idesc = umma_idesc_bf16(128, kKeys), sum_idesc = umma_idesc_bf16(128, kSumColumns) | kUmmaATransposed;
    bool ok = count > 0 && wait_bounded(&query_full, 0, p.status, 7);
    unsigned patches = 0;
    auto score = [&](int i) {
      if (edge(i)) ok = ok && wait_bounded(&patched, patches++ & 1u, p.status, 8);
      for (int j = 0; j < pairs && ok; ++j) {
        const int it = i * pairs + j, s = it % kSlots;
        ok = wait_bounded(&full[s], uint32_t(it / kSlots) & 1u, p.status, 9);
        if (!ok) break;
        tcgen05_fence_after();
        for (int c = 2 * j; c < min(2 * j + 2, chunks); ++c) {
          const uint32_t q = smem_u32(queries + c * kQueryChunk), k = smem_u32(slots + s * kSlotBytes + (c & 1) * kChunkBytes);
#pragma unroll
          for (int step = 0; step < 4; ++step)
            umma_bf16(tmem + (i & 1) * kScoreColumns, umma_desc_k_sw128(q + 32 * step, 1024), umma_desc_k_sw128(k + 32 * step, 1024), score_idesc,
                      uint32_t((c | step) != 0));
        }
      }
      if (ok) umma_commit(&score_full[i & 1]);
    };
    if (ok) score(0);
    for (int i = 0; i < count && ok; ++i) {
      if (i + 1 < count) score(i + 1);
      ok = ok && wait_bounded(&weight_full[i & 1], uint32_t(i >> 1) & 1u, p.status, 10);
      if (!ok) break;
      tcgen05_fence_after();
      const uint32_t w = smem_u32(weights + (i & 1) * kWeightBytes);
      for (int j = 0; j < pairs; ++j) {
        const int s = (i * pairs + j) % kSlots;
        const uint32_t c = smem_u32(slots + s * kSlotBytes);
#pragma unroll
        for (int step = 0; step < kKeys / 16; ++step)
          umma_bf16(tmem + 2 * kScoreColumns + j * kSumColumns, umma_desc_mn_sw128(c + 2048 * step, kChunkBytes, 1024),
                    umma_desc_k_sw128(w + 32 * step, 1024), sum_idesc, uint32_t((i | step) != 0));
        umma_commit(&empty[s]);
      }
      umma_commit(&sum_done[i & 1]);
    }
  } else if (warp >= 4) {
    // a wait that gave up does not leave the loop: its four warps meet at named barriers
    const int quarter = warp - 4, t = threadIdx.x - 128, column = 32 * quarter + lane;
    const uint32_t lanes = uint32_t(32 * quarter) << 16;
    bool ok = true;
    float inv = 1.f;
    const bf16* raw = p.raw + size_t(e.first_row) * p.raw_stride;
    const bool newest = p.raw && count > 0 && from + count == blocks;
    if (newest) {
      float sq = 0.f;
      for (int d = t; d < p.rank; d += 128) sq = fmaf(__bfloat162float(raw[d]), __bfloat162float(raw[d]), sq);
      sq = warp_sum(sq);
      if (lane == 0) square_part[quarter] = sq;
      column_sync();
      inv = 1.f / sqrtf((square_part[0] + square_part[1] + square_part[2] + square_part[3]) / float(p.rank) + p.eps);
    }
    float reference = -INFINITY, sum = 0.f;              // of the head `lane`: what its weights are relative to, this warp's sum
    for (int i = 0; i < count; ++i) {
      const int base = start + (from + i) * kKeys;
      if (edge(i)) {
        for (int j = 0; j < pairs; ++j) {
          const int it = i * pairs + j;
          ok = wait_bounded(&full[it % kSlots], uint32_t(it / kSlots) & 1u, p.status, 11) && ok;
        }
        auto place = [&](int key, int unit) {            // 16 bytes: columns 8 unit ... of the block's row `key`
          const int it = i * pairs + unit / 16;
          return reinterpret_cast<uint4*>(slots + (it % kSlots) * kSlotBytes + (unit / 8 % 2) * kChunkBytes + key * 128 + ((unit % 8) ^ (key & 7)) * 16);
        };
        const int units = chunks * 8, first = max(0, low - base), behind = min(kKeys, p1 + 1 - base);   // rows in sight: [first, behind)
        for (int n = t; n < (first + kKeys - behind) * units; n += 128) {
          const int row = n / units;
          *place(row < first ? row : behind + row - first, n % units) = make_uint4(0, 0, 0, 0);
        }
        if (p.raw && from + i == blocks - 1) {
          bf16* to_pool = p.pool + size_t(key_row(table, p1, r)) * p.pool_dim;
          for (int unit = t; unit < p.pool_dim / 8; unit += 128) {
            float c[8];
#pragma unroll
            for (int x = 0; x < 8; ++x) {
              const int d = 8 * unit + x;
              c[x] = d < p.rank ? __bfloat162float(raw[d]) * inv * p.norm[d] : 0.f;
            }
            const uint4 word = make_uint4(pack(c[0], c[1]), pack(c[2], c[3]), pack(c[4], c[5]), pack(c[6], c[7]));
            *place(p1 - base, unit) = word;
            if (blockIdx.y == 0) *reinterpret_cast<uint4*>(to_pool + 8 * unit) = word;
          }
        }
        fence_proxy_async();
        mbar_arrive(&patched);
      }
      // the scores lie in the first 32 lanes of tensor memory, which warp 4 alone reads: through shared memory every warp
      // gets 16 keys of every head (a lane's)
      if (quarter == 0) {
        ok = wait_bounded(&score_full[i & 1], uint32_t(i >> 1) & 1u, p.status, 12) && ok;
        __syncwarp();
        tcgen05_fence_after();
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          float v[32];
          tmem_load_32(tmem + uint32_t((i & 1) * kScoreColumns + 32 * half), v);
#pragma unroll
          for (int k = 0; k < 32; k += 4) *reinterpret_cast<float4*>(scores + lane * kScorePitch + 32 * half + k) = make_float4(v[k], v[k + 1], v[k + 2], v[k + 3]);
        }
      }
      column_sync();
      float s[16], high = -INFINITY;
#pragma unroll
      for (int k = 0; k < 16; k += 4) {
        const float4 v = *reinterpret_cast<const float4*>(scores + lane * kScorePitch + 16 * quarter + k);
        s[k] = v.x * p.scale_log2;
        s[k + 1] = v.y * p.scale_log2;
        s[k + 2] = v.z * p.scale_log2;
        s[k + 3] = v.w * p.scale_log2;
      }
      if (edge(i)) {
#pragma unroll
        for (int k = 0; k < 16; ++k) {
          const int j = base + 16 * quarter + k;
          if (j < low || j > p1) s[k] = -INFINITY;
        }
      }
#pragma unroll
      for (int k = 0; k < 16; ++k) high = fmaxf(high, s[k]);
      exchange[quarter][lane] = high;
      column_sync();
      high = fmaxf(fmaxf(exchange[0][lane], exchange[1][lane]), fmaxf(exchange[2][lane], exchange[3][lane]));
      const bool live = lane < heads, grows = live && high > reference + kGrowth;   // (the first block: from -infinity)
      const float next = grows ? high : reference, fade = grows && i > 0 ? ex2(reference - next) : 1.f;
      reference = next;
      sum *= fade;
      if (__any_sync(0xffffffffu, grows) && i > 0) {
        ok = wait_bounded(&sum_done[(i - 1) & 1], uint32_t((i - 1) >> 1) & 1u, p.status, 13) && ok;
        __syncwarp();
        tcgen05_fence_after();
        for (int c = 0; c < pairs * kSumColumns; c += 32) {
          float v[32];
          tmem_load_32(tmem + lanes + uint32_t(2 * kScoreColumns + c), v);
#pragma unroll
          for (int k = 0; k < 32; ++k) v[k] *= __shfl_sync(0xffffffffu, fade, k);
          tmem_store_32(tmem + lanes + uint32_t(2 * kScoreColumns + c), v);
        }
      }
      // the weights' place is free once the sums two blocks before are done
      if (i >= 2) ok = wait_bounded(&sum_done[i & 1], uint32_t((i - 2) >> 1) & 1u, p.status, 14) && ok;
      unsigned char* rows = weights + (i & 1) * kWeightBytes + lane * 128;
#pragma unroll
      for (int unit = 0; unit < 2; ++unit) {
        float w[8], left[8];
        uint32_t word[4];
#pragma unroll
        for (int x = 0; x < 8; ++x) {
          w[x] = live ? ex2(s[8 * unit + x] - reference) : 0.f;
          sum += w[x];
        }
#pragma unroll
        for (int x = 0; x < 4; ++x) {
          word[x] = pack(w[2 * x], w[2 * x + 1]);
          left[2 * x] = w[2 * x] - bf_lo(word[x]);
          left[2 * x + 1] = w[2 * x + 1] - bf_hi(word[x]);
        }
        const int at = ((2 * quarter + unit) ^ (lane & 7)) * 16;
        *reinterpret_cast<uint4*>(rows + at) = make_uint4(word[0], word[1], word[2], word[3]);
        *reinterpret_cast<uint4*>(rows + kUnitHeads * 128 + at) =
            make_uint4(pack(left[0], left[1]), pack(left[2], left[3]), pack(left[4], left[5]), pack(left[6], left[7]));
      }
      fence_proxy_async();
      tcgen05_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&weight_full[i & 1]);
    }
    column_sync();                                       // (the last maxima have been read)
    exchange[quarter][lane] = sum;
    column_sync();
    sum = exchange[0][lane] + exchange[1][lane] + exchange[2][lane] + exchange[3][lane];
    const bool whole = p.splits == 1;
    const size_t record = (size_t(blockIdx.z) * p.heads + head0) * p.splits + split;   // of the unit's head 0; heads are `splits` apart
    if (quarter == 0 && lane < heads) {
      if (whole) {
        const float sink = p.sink_of(head0 + lane), high = fmaxf(reference, sink), f = ex2(reference - high);
        factor[lane] = f / fmaf(sum, f, ex2(sink - high));
      } else {
        factor[lane] = 1.f;
        p.stats(r.entries)[record + size_t(lane) * p.splits] = make_float2(reference, sum);
      }
    }
    column_sync();
    if (count > 0) {
      ok = wait_bounded(&sum_done[(count - 1) & 1], uint32_t((count - 1) >> 1) & 1u, p.status, 15) && ok;
      __syncwarp();
      tcgen05_fence_after();
    }
    bf16* dst = p.out + (size_t(e.first_row) * p.heads + head0) * p.rank_stride;
    for (int j = 0; j < pairs; ++j) {
      float hi[32], lo[32];
      const uint32_t at = tmem + lanes + uint32_t(2 * kScoreColumns + j * kSumColumns);
      if (count > 0) {
        tmem_load_32(at, hi);
        tmem_load_32(at + kUnitHeads, lo);
      }
      const int c = 128 * j + column;
      if (c < p.rank_stride) {
#pragma unroll
        for (int h = 0; h < kUnitHeads; ++h) {
          if (h >= heads) break;
          const float v = count > 0 && c < p.rank ? (hi[h] + lo[h]) * factor[h] : 0.f;
          if (whole) dst[size_t(h) * p.rank_stride + c] = __float2bfloat16_rn(v);
          else p.part[(record + size_t(h) * p.splits) * p.rank_stride + c] = v;
        }
      }
      __syncwarp();
    }
  }
  tcgen05_fence_before();
  __syncthreads();
  if (warp == 1) {
    tcgen05_fence_after();
    tmem_dealloc(tmem, kTensorColumns);
  }
}

// A decoded token's splits put together, a CTA per head. blockIdx = (head, entry).
constexpr int kMostSplits = 64;
constexpr int kMergeThreads = kTiledLatent / 4;   // a thread per four columns
__global__ void __launch_bounds__(kMergeThreads) merge_latent(StepRows r, LatentParams p) {
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
  for (int c = threadIdx.x; c < p.rank_stride / 4; c += kMergeThreads) {
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 8
    for (int s = 0; s < p.splits; ++s) {
      const float4 w = parts[size_t(s) * (p.rank_stride / 4) + c];
      v.x = fmaf(w.x, factor[s], v.x);
      v.y = fmaf(w.y, factor[s], v.y);
      v.z = fmaf(w.z, factor[s], v.z);
      v.w = fmaf(w.w, factor[s], v.w);
    }
    *reinterpret_cast<uint2*>(dst + 4 * c) = make_uint2(pack(v.x, v.y), pack(v.z, v.w));
  }
}

// ---- a portion ------------------------------------------------------------------------------------------------------------
constexpr int kWeightPitch = kKeys + 8;

template <int RT> struct LatentShape {
  static constexpr int WM = 4, kWarps = 16, kThreads = 32 * kWarps;
  static constexpr int kPitch = RT * 16 + 8;
  static constexpr int kRows = 16 * WM;
  static constexpr int kTile = kKeys * kPitch;                                    // elements of one block
  static constexpr int kStages = RT <= 32 ? 2 : 1;
  static constexpr int kSmem = (kRows * kPitch + kStages * kTile + 2 * kRows * kWeightPitch) * 2;   // q, blocks, weights as heads and remainders
};

// Rows of a tile are (token, head of the unit) pairs, token-major; the warps are four row tiles times WN parts: of a block's
// keys for the scores, of the latent columns for the sums. The portion's own rows are in the pool already. RT: 16-column
// tiles of a latent row; FULL: it fills them. blockIdx = (token tile, unit, entry).
template <int RT, bool FULL>
__global__ void __launch_bounds__(LatentShape<RT>::kThreads, 1) attend_latent(StepRows r, LatentParams p) {
  using Shape = LatentShape<RT>;
  constexpr int WM = Shape::WM, kWarps = Shape::kWarps, kThreads = Shape::kThreads;
  constexpr int WN = kWarps / WM, KN = kKeys / WN, P = Shape::kPitch, CT = RT / WN, S = Shape::kStages;   // CT: column tiles of a warp
  static_assert(CT >= 1, "a warp sums at least one column tile");
  extern __shared__ __align__(16) unsigned char smem_raw[];
  bf16* qs = reinterpret_cast<bf16*>(smem_raw);
  bf16* cs = qs + Shape::kRows * P;
  bf16* wh = cs + S * Shape::kTile;
  bf16* wl = wh + Shape::kRows * kWeightPitch;
  __shared__ float high_part[WN][Shape::kRows], sum_part[WN][Shape::kRows];
  __shared__ int key_at[2][kKeys];   // pool rows of a block's keys (-1: none)
  dependency_wait();
  allow_dependents();
  const Entry e = r.entry[blockIdx.z];
  if (e.rows == 1) return;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int head0 = blockIdx.y * p.sub_heads, gq = min(p.sub_heads, p.heads - head0);
  const int per_tile = Shape::kRows / p.sub_heads;
  const int t0 = blockIdx.x * per_tile;
  if (t0 >= e.rows) return;
  const int tokens = min(per_tile, e.rows - t0);
  const int p0 = e.first_position + t0, p1 = p0 + tokens - 1;
  const int* table = r.block_table + size_t(e.slot) * r.max_blocks;

  const int low = max(0, p0 - p.window + 1), blocks = (p1 + 1 - low + kKeys - 1) / kKeys;   // any row of the tile sees [low, p1]
  auto locate = [&](int b) {         // one block ahead of its fetch
    if (threadIdx.x < kKeys && b < blocks) {
      const int j = low + b * kKeys + int(threadIdx.x);
      key_at[b & 1][threadIdx.x] = j <= p1 ? key_row(table, j, r) : -1;
    }
  };
  auto fetch = [&](int b) {
    constexpr int C = RT * 2;        // 16-byte pieces of a row
#pragma unroll 4
    for (int i = threadIdx.x; i < kKeys * C; i += kThreads) {
      const int key = i / C, c = (i % C) * 8, row = key_at[b & 1][key];
      const bool live = row >= 0;
      if (FULL || c < p.pool_dim) copy16(cs + (b % S) * Shape::kTile + key * P + c, p.pool + size_t(live ? row : 0) * p.pool_dim + c, live);
    }
    copy_commit();
  };
  locate(0);
  locate(1);
  __syncthreads();
  fetch(0);

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

  for (int b = 0; b < blocks; ++b) {
    bf16* tile = cs + (b % S) * Shape::kTile;
    if (S == 1 && b > 0) fetch(b);
    if (S > 1 && b + 1 < blocks) {
      fetch(b + 1);
      copy_wait<1>();
    } else {
      copy_wait<0>();
    }
    __syncthreads();
    locate(b + 2);
    float s[KN / 8][4];
#pragma unroll
    for (int t = 0; t < KN / 8; ++t) s[t][0] = s[t][1] = s[t][2] = s[t][3] = 0.f;
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
  auto finish = [&](int m, float top, float sum, int at) {
    const int t = m / gq, h = m % gq;
    if (t >= tokens) return;
    const float sink = p.sink_of(head0 + h), high = fmaxf(top, sink), fade = ex2(top - high);
    const float f = fade / fmaf(sum, fade, ex2(sink - high));
    bf16* dst = p.out + (size_t(e.first_row + t0 + t) * p.heads + head0 + h) * p.rank_stride;
#pragma unroll
    for (int i = 0; i < 2 * CT; ++i) {
      const int c = wn * CT * 16 + i * 8 + 2 * (lane & 3);
      if (c >= p.rank) continue;     // (a row has an even number of columns; the one behind an odd rank meets zero weights)
      *reinterpret_cast<uint32_t*>(dst + c) = pack(o[i][at] * f, c + 1 < p.rank ? o[i][at + 1] * f : 0.f);
    }
  };
  finish(ra, top_a, sum_a, 0);
  finish(rb, top_b, sum_b, 2);
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

// The heads in as few units of at most `most` as there can be.
void Divide(LatentParams* p, int most) {
  p->subs = (p->heads + most - 1) / most;
  p->sub_heads = (p->heads + p->subs - 1) / p->subs;
  p->subs = (p->heads + p->sub_heads - 1) / p->sub_heads;
}

int DecodeLatent(const Queue& q, const StepRows& r, const LatentArgs& a, LatentParams p) {
  // the cut of a token's keys that ends soonest: a CTA costs its blocks plus a few blocks' time to start, a merge behind it three
  const int blocks = (std::min(a.window, r.capacity) + kRaggedBlock - 2) / kKeys + 1;
  const bool shared = a.pool_dim <= 64 * kSharedChunks;
  const int resident = (shared ? 2 : 1) * q.sm_count;
  Divide(&p, kUnitHeads);
  p.splits = 1;
  float least = 0.f;
  for (int s = 1; s <= std::min(blocks, kMostSplits); ++s) {
    if (size_t(r.entries) * a.heads * s * (a.rank_stride + 2) > a.part_floats) break;
    const int waves = (r.singles * p.subs * s + resident - 1) / resident;
    const float cost = float(waves) * (float((blocks + s - 1) / s) + 3.f) + (s > 1 ? 3.f + float(s) / 16.f : 0.f);
    if (s == 1 || cost < least) {
      least = cost;
      p.splits = s;
    }
  }
  auto kernel = shared ? decode_latent<true> : decode_latent<false>;
  const int smem = shared ? DecodeSmem(kSharedChunks, kSharedSlots) : DecodeSmem(kMostChunks, kMostSlots);
  const int status = int(Launch(kernel, dim3(unsigned(p.splits), unsigned(p.subs), unsigned(r.entries)), dim3(kLatentThreads), smem, q.stream,
                                q.chained, *a.pool_map, *a.q_map, r, p));
  if (status != 0 || p.splits == 1) return status;
  return int(Launch(merge_latent, dim3(unsigned(a.heads), unsigned(r.entries)), dim3(kMergeThreads), 0, q.stream, q.chained, r, p));
}

template <int RT> int AttendWith(const Queue& q, const StepRows& r, LatentParams p) {
  Divide(&p, 64);
  auto kernel = p.pool_dim == 16 * RT ? attend_latent<RT, true> : attend_latent<RT, false>;
  const int per_tile = 64 / p.sub_heads;
  return int(Launch(kernel, dim3(unsigned((r.longest + per_tile - 1) / per_tile), unsigned(p.subs), unsigned(r.entries)), dim3(LatentShape<RT>::kThreads),
                    LatentShape<RT>::kSmem, q.stream, q.chained, r, p));
}

template <int RT> cudaError_t Raise() {
  for (auto kernel : {attend_latent<RT, false>, attend_latent<RT, true>}) {
    const cudaError_t err = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, LatentShape<RT>::kSmem);
    if (err != cudaSuccess) return err;
  }
  return cudaSuccess;
}

}  // namespace

int AttendLatentTiles(const Queue& q, const StepRows& r, const LatentArgs& a) {
  LatentParams p{};
  p.q = static_cast<const bf16*>(a.q);
  p.raw = a.query_raw ? nullptr : static_cast<const bf16*>(a.raw);
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
  p.status = q.status;
  if (r.singles > 0) {
    const int status = DecodeLatent(q, r, a, p);
    if (status != 0) return status;
  }
  if (r.singles == r.entries || a.singles_only) return 0;
  return a.rank <= 128 ? AttendWith<8>(q, r, p) : a.rank <= 256 ? AttendWith<16>(q, r, p) : a.rank <= 512 ? AttendWith<32>(q, r, p) : AttendWith<40>(q, r, p);
}

bool EncodeLatent(CUtensorMap* pool_map, const void* pool, uint64_t rows, uint64_t pool_dim) {
  return EncodeMatrix(pool_map, false, pool, rows, pool_dim, kRaggedBlock);
}
bool EncodeLookup(CUtensorMap* q_map, const void* q, uint64_t rows, uint64_t rank_stride) {
  return EncodeMatrix(q_map, false, q, rows, rank_stride, kUnitHeads);
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
  cudaError_t err = cudaFuncSetAttribute(decode_latent<false>, cudaFuncAttributeMaxDynamicSharedMemorySize, DecodeSmem(kMostChunks, kMostSlots));
  if (err == cudaSuccess)
    err = cudaFuncSetAttribute(decode_latent<true>, cudaFuncAttributeMaxDynamicSharedMemorySize, DecodeSmem(kSharedChunks, kSharedSlots));
  if (err == cudaSuccess) err = Raise<8>();
  if (err == cudaSuccess) err = Raise<16>();
  if (err == cudaSuccess) err = Raise<32>();
  if (err == cudaSuccess) err = Raise<40>();
  return int(err);
}

}  // namespace tmb
