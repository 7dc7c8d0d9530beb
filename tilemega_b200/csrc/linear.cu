// Matrix products of a ragged step: D[t][n] = sum_k activations[t][k] weight[n][k] for any t, n and k.
//
// bf16: weights fill the M side of a tcgen05 tile (128 weight rows), the step's tokens the N side (16 .. 256), so one
// kernel serves a single decoded token (a weight stream: many small stages in flight, K split over the CTAs of a
// cluster, whose partial tiles meet in distributed shared memory) and a prompt of thousands (128 x 256 tiles). Both
// operands arrive by TMA in 128-byte-swizzled stages; weight tiles of the first stages are requested before the
// dependency wait. A thread of the epilogue owns one weight row (output feature), so a warp's stores are runs of 32
// consecutive features of one token. fp32: a tiled kernel of plain fused multiply-adds.
#include <cuda_bf16.h>

#include <algorithm>

#include "element.cuh"
#include "ops.h"
#include "ptx.cuh"
#include "tensor_map.h"

namespace tmb {
namespace {

constexpr int kRowsM = 128;                 // weight rows per tile
constexpr int kStepK = 64;                  // 16-bit elements per 128-byte swizzle row
constexpr int kWeightBytes = kRowsM * kStepK * 2;
constexpr int kLinearThreads = 320;         // producer warp, issuing warp, eight epilogue warps
constexpr int kMaxCluster = 8;

struct LinearParams {
  const float* bias;
  void* out;
  int t, n, out_stride, outputs;
  int head_in, head_out;
  const int* rows_there;
  int chunks, chunks_per_split;
  Glu glu;
  int tanh_below;
  float gain;
  RotateHeads rotate;
  SideGate side;
  ExpertSlots slots;
  unsigned* status;
};

// Which products read gathered rows, and which run per expert.
__host__ __device__ constexpr bool Gathers(int epilogue, int tokens) {
  return (epilogue == kLinearExpertUp || epilogue == kLinearExpertGlu) && tokens <= kGatherRows;
}
__host__ __device__ constexpr bool PerExpert(int epilogue) {
  return epilogue == kLinearExpertUp || epilogue == kLinearExpertDown || epilogue == kLinearExpertGlu || epilogue == kLinearExpertStore;
}
// Gated units: products of interleaved gate and up rows.
__host__ __device__ constexpr bool IsGlu(int epilogue) { return epilogue == kLinearGlu || epilogue == kLinearExpertGlu; }

template <int BN> struct LinearShape {
  static constexpr int kStages = BN == 256 ? 4 : BN == 128 ? 3 : BN == 64 ? 4 : 5;   // about 100 KB (two CTAs per SM), 192 KB for the widest
  static constexpr int kTokenBytes = BN * kStepK * 2;
  static constexpr int kStageBytes = kWeightBytes + kTokenBytes;
  static constexpr int kSmem = kStages * kStageBytes + 1024 + 256;
  static constexpr int kTmemCols = BN < 32 ? 32 : BN;
  static constexpr bool kStaged = BN <= 128;   // the epilogue goes through shared memory (needed to sum K splits)
  static_assert(!kStaged || kStages * kStageBytes >= kRowsM * BN * 4, "the fp32 tile must fit the stages");
};

// gelu(g) = g (1 + tanh(z)) / 2 = g / (1 + exp(-2 z)), z = sqrt(2 / pi) (g + 0.044715 g^3)
__device__ __forceinline__ float glu_value(float g, float u, const Glu& p) {
  if (p.gelu) return g / (1.f + __expf(-1.5957691216057308f * (g + 0.044715f * g * g * g))) * u;
  g = fminf(g, p.limit);
  u = fminf(fmaxf(u, -p.limit), p.limit);
  return g / (1.f + __expf(-p.alpha * g)) * (u + p.shift);
}

// Output column n of a product with rotated heads: whether it turns, by which angles, and with which sign its neighbour enters.
struct Turn {
  bool on;
  const float2* angles;      // of position 0
  int half;
  float sign;
};
__device__ __forceinline__ Turn turn_of(const RotateHeads& p, int n) {
  const int d = n % p.head - p.lead;
  return {d >= 0 && d < p.rotary.dims, p.rotary.table + d / 2, p.rotary.dims / 2, d & 1 ? 1.f : -1.f};
}
__device__ __forceinline__ float2 angle_at(const RotateHeads& p, const Turn& turn, int t) {
  return turn.on ? __ldg(turn.angles + size_t(min(__ldg(p.positions + t), p.rotary.capacity - 1)) * turn.half) : make_float2(1.f, 0.f);
}
__device__ __forceinline__ float turned(const Turn& turn, float2 angle, float v, float other) { return v * angle.x + turn.sign * other * angle.y; }

// gelu(z) times column n of the row's token's part
template <typename T> __device__ __forceinline__ float side_value(const SideGate& p, int t, int n, float z) {
  const T* part = static_cast<const T*>(p.part) + size_t(min(max(p.tokens[t], 0), p.vocab - 1)) * p.stride;
  const float y = 0.7978845608028654f * (z + 0.044715f * z * z * z);
  return (sizeof(T) == 4 ? 0.5f * z * (1.f + tanhf(y)) : z / (1.f + __expf(-2.f * y))) * to_f(part[n]);
}

// tanh to the precision of a 16-bit element
__device__ __forceinline__ float tanh16(float v) {
  float y;
  asm("tanh.approx.f32 %0, %1;" : "=f"(y) : "f"(v));
  return y;
}

__device__ __forceinline__ uint32_t cluster_rank() {
  uint32_t r;
  asm volatile("mov.u32 %0, %%cluster_ctarank;" : "=r"(r));
  return r;
}
__device__ __forceinline__ void cluster_sync() {
  asm volatile("barrier.cluster.arrive.release;\nbarrier.cluster.wait.acquire;" ::: "memory");
}
__device__ __forceinline__ float ld_peer(uint32_t local, uint32_t rank) {
  uint32_t remote;
  float v;
  asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(remote) : "r"(local), "r"(rank));
  asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(v) : "r"(remote) : "memory");
  return v;
}

template <int EPI> __device__ __forceinline__ void emit(const LinearParams& g, int t, int n, float v) {
  if (EPI == kLinearSide) v = side_value<__nv_bfloat16>(g.side, t, n, v);
  if (EPI == kLinearStore || EPI == kLinearHeads || EPI == kLinearRotate || EPI == kLinearSide)
    static_cast<__nv_bfloat16*>(g.out)[size_t(t) * g.out_stride + n] = __float2bfloat16_rn(v);
  if (EPI == kLinearAdd) static_cast<float*>(g.out)[size_t(t) * g.out_stride + n] += v;
  if (EPI == kLinearFloat) static_cast<float*>(g.out)[size_t(t) * g.out_stride + n] = v * g.gain;
  if (EPI == kLinearExpertUp) {
    const float r = fmaxf(v * g.slots.score[t], 0.f);
    static_cast<__nv_bfloat16*>(g.out)[size_t(t) * g.out_stride + n] = __float2bfloat16_rn(r * r);
  }
  if (EPI == kLinearExpertDown) static_cast<__nv_bfloat16*>(g.out)[size_t(g.slots.list[t]) * g.out_stride + n] = __float2bfloat16_rn(v);
}

// blockIdx = (token tile, weight tile, K split): CTAs that run together share weight tiles, so a prompt's weights are read
// once while its activations stay in L2. The CTAs of one (weight, token) tile form a cluster along z. Per expert the
// first two axes change places (an expert's weights are read by few tiles, its tokens by all of its weight tiles), token
// tiles are those of the slot table (the grid holds as many as there could be), tokens are slots, and weight tiles start at
// the expert's rows; what a tile computes beyond its slots or its expert's rows is dropped. Products by heads count the weight
// tiles of one head after the other; columns behind a head's in its chunks of activations meet zeros, the map's fill
// behind a weight row.
template <int BN, int EPI>
__global__ void __launch_bounds__(kLinearThreads) linear_tiles(const __grid_constant__ CUtensorMap wmap, const __grid_constant__ CUtensorMap tmap,
                                                               const LinearParams g) {
  using Shape = LinearShape<BN>;
  constexpr int S = Shape::kStages;
  extern __shared__ unsigned char smem_raw[];
  unsigned char* tiles = reinterpret_cast<unsigned char*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint64_t* full = reinterpret_cast<uint64_t*>(tiles + S * Shape::kStageBytes);
  uint64_t* empty = full + S;
  uint64_t* accum = empty + S;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(accum + 1);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  int n0 = (PerExpert(EPI) ? blockIdx.x : blockIdx.y) * kRowsM;
  const int token_tile = PerExpert(EPI) ? blockIdx.y : blockIdx.x;
  int t0 = token_tile * BN, t_end = g.t, weight_row = n0, k_at = 0, out_at = 0;
  if constexpr (EPI == kLinearHeads) {
    const int tiles = (g.n + kRowsM - 1) / kRowsM, head = blockIdx.y / tiles;
    n0 = (blockIdx.y % tiles) * kRowsM;
    weight_row = head * g.n + n0;
    k_at = head * g.head_in;
    out_at = head * g.head_out;
  }
  if constexpr (EPI == kLinearStore) {
    if (g.rows_there) {
      t_end = min(t_end, *g.rows_there);
      if (t0 >= t_end) {
        dependency_wait();
        return;
      }
    }
  }
  // per expert only the tokens there are cost anything: wide tiles load them 32 rows at a time
  constexpr bool kGather = Gathers(EPI, BN);
  constexpr int kBoxes = PerExpert(EPI) && BN > 32 ? BN / 32 : 1;
  int columns = BN, boxes = kBoxes;
  if constexpr (PerExpert(EPI)) {
    // a product that gathers follows the kernel that writes the table; for the others it is there before the wait
    if (kGather) dependency_wait();
    const ExpertTile tile = g.slots.tiles[token_tile];
    if (token_tile >= *g.slots.tile_count) {
      if (!kGather) dependency_wait();
      return;
    }
    t0 = tile.first;
    t_end = tile.first + min(tile.count, BN);
    weight_row = tile.expert * g.n + n0;
    columns = (t_end - t0 + 15) / 16 * 16;
    if (kBoxes > 1) boxes = (t_end - t0 + 31) / 32;
  }
  const uint32_t stage_bytes = uint32_t(kWeightBytes + boxes * (Shape::kTokenBytes / kBoxes));
  const int splits = gridDim.z;
  const int c0 = blockIdx.z * g.chunks_per_split;
  const int chunks = max(0, min(g.chunks_per_split, g.chunks - c0));

  if (threadIdx.x == 0) {
    prefetch_map(&wmap);
    prefetch_map(&tmap);
    for (int s = 0; s < S; ++s) {
      mbar_init(&full[s], 1);
      mbar_init(&empty[s], 1);
    }
    mbar_init(accum, 1);
    mbar_fence_init();
  }
  if (warp == 1) tmem_alloc(tmem_slot, Shape::kTmemCols);
  tcgen05_fence_before();
  __syncthreads();
  tcgen05_fence_after();
  const uint32_t tmem = *tmem_slot;
  const int early = chunks < S ? chunks : S;
  if (threadIdx.x == 0)
    for (int c = 0; c < early; ++c) {   // weights do not depend on the kernel before this one
      mbar_expect_tx(&full[c], stage_bytes);
      tma_load_2d(tiles + c * Shape::kStageBytes, &wmap, (c0 + c) * kStepK, weight_row, &full[c]);
    }
  if (!kGather) dependency_wait();

  if (kGather && warp == 0) {
    int rows[4];                                        // every lane of the first BN / 4 fetches four rows of the tile
#pragma unroll
    for (int i = 0; i < 4; ++i) rows[i] = g.slots.list[min(t0 + lane * 4 + i, t_end - 1)] / g.slots.top;
    int issued = 0;
    bool ok = true;
    for (int c = 0; c < chunks; ++c) {
      const int s = c % S;
      if (c >= S) ok = __all_sync(0xffffffffu, wait_bounded(&empty[s], uint32_t((c / S) - 1) & 1u, g.status, 1));
      if (!ok) break;
      unsigned char* w = tiles + s * Shape::kStageBytes;
      if (lane == 0 && c >= early) {
        mbar_expect_tx(&full[s], stage_bytes);
        tma_load_2d(w, &wmap, (c0 + c) * kStepK, weight_row, &full[s]);
      }
      __syncwarp();
      if (lane < BN / 4) tma_gather_rows(w + kWeightBytes + lane * 4 * kStepK * 2, &tmap, (c0 + c) * kStepK, rows, &full[s]);
      issued = c + 1;
    }
    if (!ok)
      for (int c = issued > S ? issued - S : 0; c < issued; ++c) wait_bounded(&full[c % S], uint32_t(c / S) & 1u, g.status, 2);
  } else if (warp == 0) {
    if (lane == 0) {
      int issued = 0;
      bool ok = true;
      for (int c = 0; c < chunks; ++c) {
        const int s = c % S;
        if (c >= S) ok = wait_bounded(&empty[s], uint32_t((c / S) - 1) & 1u, g.status, 1);
        if (!ok) break;
        unsigned char* w = tiles + s * Shape::kStageBytes;
        if (c >= early) {
          mbar_expect_tx(&full[s], stage_bytes);
          tma_load_2d(w, &wmap, (c0 + c) * kStepK, weight_row, &full[s]);
        }
        if constexpr (kBoxes == 1) tma_load_2d(w + kWeightBytes, &tmap, k_at + (c0 + c) * kStepK, t0, &full[s]);
        else
          for (int i = 0; i < boxes; ++i) tma_load_2d(w + kWeightBytes + i * 32 * kStepK * 2, &tmap, (c0 + c) * kStepK, t0 + 32 * i, &full[s]);
        issued = c + 1;
      }
      if (!ok)   // leaving early: let the copies already issued land first
        for (int c = issued > S ? issued - S : 0; c < issued; ++c) wait_bounded(&full[c % S], uint32_t(c / S) & 1u, g.status, 2);
    }
  } else if (warp == 1) {
    if (lane == 0) {
      const uint32_t idesc = umma_idesc_bf16(kRowsM, columns);
      for (int c = 0; c < chunks; ++c) {
        const int s = c % S;
        if (!wait_bounded(&full[s], uint32_t(c / S) & 1u, g.status, 3)) break;
        tcgen05_fence_after();
        const uint32_t w = smem_u32(tiles + s * Shape::kStageBytes), t = w + kWeightBytes;
#pragma unroll
        for (int j = 0; j < kStepK / 16; ++j)
          umma_bf16(tmem, umma_desc_k_sw128(w + 32 * j, 1024), umma_desc_k_sw128(t + 32 * j, 1024), idesc, uint32_t((c | j) != 0));
        umma_commit(&empty[s]);
      }
      umma_commit(accum);   // arrives once everything issued above is done
    }
  }
  const int worker = int(threadIdx.x) - 64;           // epilogue thread
  const int quarter = warp & 3, column_half = (warp - 2) >> 2;
  bool ok = true;
  if (worker >= 0) {
    ok = wait_bounded(accum, 0, g.status, 4);
    tcgen05_fence_after();
    allow_dependents();
  }
  if constexpr (Shape::kStaged) {
    float* tile = reinterpret_cast<float*>(tiles);    // [BN][128]: every stage has been consumed
    if (worker >= 0) {
      constexpr int W = BN >= 64 ? 32 : BN == 32 ? 16 : 8;
      constexpr int L = W == 8 ? 16 : W;              // columns per tensor-memory load
#pragma unroll
      for (int c = column_half * (BN / 2); c < (column_half + 1) * (BN / 2); c += W) {
        if (PerExpert(EPI) && c >= columns) break;
        float v[L];
        const uint32_t at = tmem + (uint32_t(32 * quarter) << 16) + uint32_t(W == 8 ? 0 : c);
        if constexpr (L == 32) tmem_load_32(at, v);
        else tmem_load_16(at, v);
#pragma unroll
        for (int i = 0; i < W; ++i)
          tile[(c + i) * kRowsM + 32 * quarter + lane] = chunks ? (W == 8 ? (column_half ? v[(i + 8) % L] : v[i]) : v[i]) : 0.f;
      }
    }
    if (splits > 1) cluster_sync();
    else __syncthreads();
    if (worker >= 0 && ok) {
      const uint32_t rank = splits > 1 ? cluster_rank() : 0;
      const int per = (BN + splits - 1) / splits, first = int(rank) * per;
      const int cols = min(min(per, BN - first), t_end - t0 - first);   // this CTA's tokens of the tile
      const uint32_t base = smem_u32(tile);
      auto total = [&](int c, int row) {
        if (splits == 1) return tile[c * kRowsM + row];
        float sum = 0.f, part[kMaxCluster];
#pragma unroll
        for (int p = 0; p < kMaxCluster; ++p)
          if (p < splits) part[p] = ld_peer(base + uint32_t(c * kRowsM + row) * 4, uint32_t(p));
#pragma unroll
        for (int p = 0; p < kMaxCluster; ++p)
          if (p < splits) sum += part[p];               // in split order
        return sum;
      };
      if constexpr (IsGlu(EPI)) {
        for (int i = worker; i < cols * (kRowsM / 2); i += 256) {
          const int c = first + i / (kRowsM / 2), pair = i % (kRowsM / 2);
          const int row = (pair / kGluUnit) * 2 * kGluUnit + pair % kGluUnit, out = n0 / 2 + pair;
          if (out >= g.outputs) continue;
          const float v = glu_value(total(c, row), total(c, row + kGluUnit), g.glu);
          static_cast<__nv_bfloat16*>(g.out)[size_t(t0 + c) * g.out_stride + out] = __float2bfloat16_rn(v);
        }
      } else {
        const int row = worker & (kRowsM - 1), n = n0 + row;
        if (n < g.n) {
          const float bias = g.bias ? g.bias[n] : 0.f;
          if constexpr (EPI == kLinearRotate) {           // (neighbours lie in one tile)
            const Turn turn = turn_of(g.rotate, n);
            constexpr int U = 8;
            for (int c0 = first + (worker >> 7); c0 < first + cols; c0 += 2 * U) {
              float2 angle[U];
#pragma unroll
              for (int i = 0; i < U; ++i) angle[i] = angle_at(g.rotate, turn, t0 + min(c0 + 2 * i, first + cols - 1));
#pragma unroll
              for (int i = 0; i < U; ++i)
                if (const int c = c0 + 2 * i; c < first + cols) {
                  const float v = total(c, row);
                  emit<EPI>(g, t0 + c, n, turn.on ? turned(turn, angle[i], v, total(c, row ^ 1)) : v);
                }
            }
          } else {
            const bool bent = EPI == kLinearStore && n < g.tanh_below;
            for (int c = first + (worker >> 7); c < first + cols; c += 2) {
              const float v = total(c, row) + bias;
              emit<EPI>(g, t0 + c, out_at + n, bent ? tanh16(v) : v);
            }
          }
        }
      }
    }
    if (splits > 1) cluster_sync();   // the peers have read this CTA's tile
  } else if (worker >= 0 && ok) {
    const int n = n0 + 32 * quarter + lane;
    const float bias = g.bias && n < g.n ? g.bias[n] : 0.f;
    for (int c = column_half * (BN / 2); c < (column_half + 1) * (BN / 2); c += 32) {
      if (t0 + c >= t_end) break;
      float v[32];
      tmem_load_32(tmem + (uint32_t(32 * quarter) << 16) + uint32_t(c), v);
      const int cols = min(32, t_end - t0 - c);
      if constexpr (IsGlu(EPI)) {
        const bool upper = lane >= kGluUnit;          // lanes 0..15 hold gate rows, 16..31 the matching up rows
        const int out = (n0 + 32 * quarter) / 2 + (lane & (kGluUnit - 1));
#pragma unroll
        for (int i = 0; i < 32; i += 2) {             // lower lanes finish column i, upper lanes column i + 1
          const float other = __shfl_xor_sync(0xffffffffu, upper ? v[i] : v[i + 1], kGluUnit);
          const float y = glu_value(upper ? other : v[i], upper ? v[i + 1] : other, g.glu);
          const int col = i + (upper ? 1 : 0);
          if (out < g.outputs && col < cols)
            static_cast<__nv_bfloat16*>(g.out)[size_t(t0 + c + col) * g.out_stride + out] = __float2bfloat16_rn(y);
        }
      } else if constexpr (EPI == kLinearRotate) {
        const Turn turn = turn_of(g.rotate, n);
        if (__any_sync(0xffffffffu, turn.on)) {
#pragma unroll
          for (int i0 = 0; i0 < 32; i0 += 8) {
            float2 angle[8];
#pragma unroll
            for (int i = 0; i < 8; ++i) angle[i] = angle_at(g.rotate, turn, t0 + c + min(i0 + i, cols - 1));
#pragma unroll
            for (int i = 0; i < 8; ++i) v[i0 + i] = turned(turn, angle[i], v[i0 + i], __shfl_xor_sync(0xffffffffu, v[i0 + i], 1));
          }
        }
        if (n < g.n) {
#pragma unroll
          for (int i = 0; i < 32; ++i)
            if (i < cols) emit<EPI>(g, t0 + c + i, n, v[i]);
        }
      } else if (n < g.n) {
        if constexpr (EPI == kLinearAdd) {
          float* x = static_cast<float*>(g.out) + size_t(t0 + c) * g.out_stride + n;
          float old[32];
#pragma unroll
          for (int i = 0; i < 32; ++i)
            if (i < cols) old[i] = x[size_t(i) * g.out_stride];
#pragma unroll
          for (int i = 0; i < 32; ++i)
            if (i < cols) x[size_t(i) * g.out_stride] = old[i] + (v[i] + bias);
        } else {
          if (EPI == kLinearStore && n0 < g.tanh_below) {
#pragma unroll
            for (int i = 0; i < 32; ++i)
              if (n < g.tanh_below) v[i] = tanh16(v[i] + bias) - bias;
          }
#pragma unroll
          for (int i = 0; i < 32; ++i)
            if (i < cols) emit<EPI>(g, t0 + c + i, out_at + n, v[i] + bias);
        }
      }
    }
  }
  tcgen05_fence_before();
  __syncthreads();
  if (warp == 1) {
    tcgen05_fence_after();
    tmem_dealloc(tmem, Shape::kTmemCols);
  }
}

// ---- fp32 --------------------------------------------------------------------------------------------------------
constexpr int kTile32 = 64, kStep32 = 16;

template <int EPI>
__global__ void __launch_bounds__(256) linear_f32(const float* activations, const float* weight, const LinearParams g, int k_stride, int in_stride) {
  __shared__ float as[kStep32][kTile32 + 4], ws[kStep32][kTile32 + 4];
  const int n0 = blockIdx.x * kTile32;
  int t0 = blockIdx.y * kTile32, t_end = g.t;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  dependency_wait();
  allow_dependents();
  if constexpr (PerExpert(EPI)) {
    if (int(blockIdx.y) >= *g.slots.tile_count) return;
    const ExpertTile tile = g.slots.tiles[blockIdx.y];
    t0 = tile.first;
    t_end = tile.first + min(tile.count, kTile32);
    weight += size_t(tile.expert) * g.n * k_stride;
  }
  const int head = blockIdx.z;                          // (products by heads only)
  activations += size_t(head) * g.head_in;
  weight += size_t(head) * g.n * k_stride;
  auto row_of = [&](int t) { return EPI == kLinearExpertUp || EPI == kLinearExpertStore ? g.slots.list[t] / g.slots.top : t; };
  float acc[4][4] = {};
  for (int k0 = 0; k0 < k_stride; k0 += kStep32) {
#pragma unroll
    for (int i = threadIdx.x; i < kTile32 * kStep32; i += 256) {
      const int r = i / kStep32, k = i % kStep32;
      as[k][r] = t0 + r < t_end && k0 + k < k_stride ? activations[size_t(row_of(t0 + r)) * in_stride + k0 + k] : 0.f;
      ws[k][r] = n0 + r < g.n && k0 + k < k_stride ? weight[size_t(n0 + r) * k_stride + k0 + k] : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < kStep32; ++k)
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(as[k][ty * 4 + i], ws[k][tx * 4 + j], acc[i][j]);
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int t = t0 + ty * 4 + i, n = n0 + tx * 4 + j;
      if (t >= t_end || n >= g.n) continue;
      float v = acc[i][j] + (g.bias ? g.bias[n] : 0.f);
      if (EPI == kLinearStore && n < g.tanh_below) v = tanhf(v);
      if (EPI == kLinearSide) v = side_value<float>(g.side, t, n, v);
      if (EPI == kLinearFloat) v *= g.gain;
      if constexpr (EPI == kLinearRotate) {
        const Turn turn = turn_of(g.rotate, n);
        if (turn.on) v = turned(turn, angle_at(g.rotate, turn, t), v, acc[i][j ^ 1]);
      }
      float* out = static_cast<float*>(g.out) + size_t(EPI == kLinearExpertDown ? g.slots.list[t] : t) * g.out_stride + size_t(head) * g.head_out + n;
      const float positive = fmaxf(EPI == kLinearExpertUp ? v * g.slots.score[t] : 0.f, 0.f);
      *out = EPI == kLinearAdd ? *out + v : EPI == kLinearExpertUp ? positive * positive : v;
    }
}

template <typename T>
__global__ void __launch_bounds__(256) glu_rows(const T* in, T* out, int t, int in_stride, int out_stride, int outputs, Glu glu) {
  dependency_wait();
  allow_dependents();
  const int j = blockIdx.x * 256 + threadIdx.x, row = blockIdx.y;
  if (j >= outputs || row >= t) return;
  const T* pair = in + size_t(row) * in_stride + (j / kGluUnit) * 2 * kGluUnit + j % kGluUnit;
  if (glu.gelu) {
    const float z = to_f(pair[0]);
    out[size_t(row) * out_stride + j] = from_f<T>(z / (1.f + expf(-1.5957691216057308f * (z + 0.044715f * z * z * z))) * to_f(pair[kGluUnit]));
    return;
  }
  const float g = fminf(to_f(pair[0]), glu.limit), u = fminf(fmaxf(to_f(pair[kGluUnit]), -glu.limit), glu.limit);
  out[size_t(row) * out_stride + j] = from_f<T>(g / (1.f + expf(-glu.alpha * g)) * (u + glu.shift));
}

template <int BN> cudaError_t RaiseLimit() {
  const int smem = LinearShape<BN>::kSmem;
  for (auto kernel : {linear_tiles<BN, kLinearStore>, linear_tiles<BN, kLinearAdd>, linear_tiles<BN, kLinearGlu>, linear_tiles<BN, kLinearFloat>,
                      linear_tiles<BN, kLinearExpertUp>, linear_tiles<BN, kLinearExpertDown>, linear_tiles<BN, kLinearHeads>,
                      linear_tiles<BN, kLinearExpertGlu>, linear_tiles<BN, kLinearRotate>, linear_tiles<BN, kLinearSide>}) {
    const cudaError_t err = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (err != cudaSuccess) return err;
  }
  return cudaSuccess;
}

// Most tiles the slots of a step can fall into: full ones, and one more for every expert in use.
int MostTiles(const ExpertSlots& s) { return s.slots / s.tile_rows + std::min(s.experts, s.slots); }

template <int BN>
cudaError_t LaunchTiles(const Queue& q, const LinearArgs& a, const LinearParams& p, int map, int splits) {
  auto kernel = a.epilogue == kLinearAdd ? linear_tiles<BN, kLinearAdd> : a.epilogue == kLinearGlu ? linear_tiles<BN, kLinearGlu>
                : a.epilogue == kLinearFloat ? linear_tiles<BN, kLinearFloat> : a.epilogue == kLinearExpertUp ? linear_tiles<BN, kLinearExpertUp>
                : a.epilogue == kLinearExpertDown ? linear_tiles<BN, kLinearExpertDown> : a.epilogue == kLinearHeads ? linear_tiles<BN, kLinearHeads>
                : a.epilogue == kLinearExpertGlu ? linear_tiles<BN, kLinearExpertGlu> : a.epilogue == kLinearRotate ? linear_tiles<BN, kLinearRotate>
                : a.epilogue == kLinearSide ? linear_tiles<BN, kLinearSide> : linear_tiles<BN, kLinearStore>;
  cudaLaunchConfig_t config{};
  const unsigned weight_tiles = unsigned((a.n + kRowsM - 1) / kRowsM) * unsigned(std::max(a.heads, 1));
  config.gridDim = PerExpert(a.epilogue) ? dim3(weight_tiles, unsigned(MostTiles(a.slots)), unsigned(splits))
                                         : dim3(unsigned((a.t + BN - 1) / BN), weight_tiles, unsigned(splits));
  config.blockDim = dim3(kLinearThreads);
  config.dynamicSmemBytes = LinearShape<BN>::kSmem;
  config.stream = q.stream;
  cudaLaunchAttribute attributes[2];
  int count = 0;
  if (q.chained) {
    attributes[count].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attributes[count++].val.programmaticStreamSerializationAllowed = 1;
  }
  if (splits > 1) {
    attributes[count].id = cudaLaunchAttributeClusterDimension;
    attributes[count].val.clusterDim.x = 1;
    attributes[count].val.clusterDim.y = 1;
    attributes[count++].val.clusterDim.z = unsigned(splits);
  }
  config.attrs = attributes;
  config.numAttrs = unsigned(count);
  return cudaLaunchKernelEx(&config, kernel, a.maps->weight, Gathers(a.epilogue, BN) ? a.maps->row : a.maps->rows[PerExpert(a.epilogue) ? std::min(map, 1) : map], p);
}

// Tile width (index into 16, 32, 64, 128, 256 tokens) and K splits: the widest tile that gives most SMs a CTA, else
// the narrowest that covers the tokens (at most 128), with K split over a cluster until the SMs are covered; further, up
// to two CTAs per SM, where a part keeps a long run of K.
void ChooseLinear(int t, int n, int heads, int chunks, int sms, int* index, int* splits) {
  const int tiles = (n + kRowsM - 1) / kRowsM * heads;
  *splits = 1;
  if (t > 128 && tiles * ((t + 255) / 256) * 10 >= sms * 8) {
    *index = 4;
    return;
  }
  *index = 0;
  while (*index < 3 && (16 << *index) < t) ++*index;
  const int grid = tiles * ((t + (16 << *index) - 1) / (16 << *index));
  while (*splits < kMaxCluster && grid * *splits <= sms && chunks / (*splits * 2) >= (grid * *splits * 10 < sms * 8 ? 4 : 16)) *splits *= 2;
}

// The same per expert: the tile width is that of the slot table; K splits until the tiles to be expected cover the SMs.
void ChooseExpertLinear(const ExpertSlots& s, int n, int chunks, int sms, int* index, int* splits) {
  *index = 0;
  while ((16 << *index) < s.tile_rows) ++*index;
  *splits = 1;
  if (*index == 4) return;
  const int grid = MostTiles(s) * ((n + kRowsM - 1) / kRowsM);
  while (*splits < kMaxCluster && grid * *splits <= sms && chunks / (*splits * 2) >= 4) *splits *= 2;
}

}  // namespace

int ExpertTileRows(const Queue& q, int slots, int experts) {
  if (q.f32) return kTile32;
  const int share = (slots + experts - 1) / experts;   // slots of an expert on average; most have no more than 4/3 of it
  int rows = 16;
  while (rows < 128 && rows * 3 < share * 4) rows *= 2;
  return rows;
}

int PrepareLinear() {
  cudaError_t err = RaiseLimit<16>();
  if (err == cudaSuccess) err = RaiseLimit<32>();
  if (err == cudaSuccess) err = RaiseLimit<64>();
  if (err == cudaSuccess) err = RaiseLimit<128>();
  if (err == cudaSuccess) err = RaiseLimit<256>();
  return int(err);
}

bool EncodeLinear(LinearMaps* maps, const void* weight, uint64_t n, const void* activations, uint64_t rows, uint64_t k_stride) {
  return EncodeHeads(maps, weight, n, k_stride, activations, rows, k_stride);
}

bool EncodeHeads(LinearMaps* maps, const void* weight, uint64_t n, uint64_t k_stride, const void* activations, uint64_t rows, uint64_t in_stride) {
  if (!EncodeMatrix(&maps->weight, false, weight, n, k_stride, kRowsM)) return false;
  for (int i = 0; i < 5; ++i)
    if (!EncodeMatrix(&maps->rows[i], false, activations, rows, in_stride, 16u << i)) return false;
  return true;
}

bool EncodeGathered(LinearMaps* maps, const void* activations, uint64_t rows, uint64_t k_stride) {
  return EncodeMatrix(&maps->row, false, activations, rows, k_stride, 1);
}

int Linear(const Queue& q, const LinearArgs& a) {
  if (a.t <= 0) return 0;
  const bool experts = PerExpert(a.epilogue);
  if (experts && (a.slots.slots <= 0 || a.slots.tile_rows < 16 || !a.slots.tiles)) return int(cudaErrorInvalidValue);
  if (a.epilogue == kLinearHeads ? a.heads < 1 || a.head_in % 8 != 0 || a.bias : a.heads != 0) return int(cudaErrorInvalidValue);
  if (a.rows_there && (q.f32 || a.epilogue != kLinearStore)) return int(cudaErrorInvalidValue);
  if (a.epilogue == kLinearExpertStore && !q.f32) return int(cudaErrorInvalidValue);
  if (a.epilogue == kLinearRotate && (a.rotate.head < 2 || a.rotate.head % 2 || a.rotate.lead % 2 || a.bias)) return int(cudaErrorInvalidValue);
  LinearParams p{};
  p.tanh_below = a.tanh_below;
  p.gain = a.gain;
  p.rotate = a.rotate;
  p.side = a.side;
  p.head_in = a.head_in;
  p.head_out = a.head_out;
  p.rows_there = a.rows_there;
  p.bias = a.bias;
  p.out = a.out;
  p.t = a.t;
  p.n = a.n;
  p.out_stride = a.out_stride;
  p.outputs = a.outputs;
  p.glu = a.glu;
  p.slots = a.slots;
  p.status = q.status;
  if (q.f32) {
    if (IsGlu(a.epilogue)) return int(cudaErrorInvalidValue);   // two operations in fp32: the product, then GluRows
    auto kernel = a.epilogue == kLinearAdd ? linear_f32<kLinearAdd> : a.epilogue == kLinearExpertUp ? linear_f32<kLinearExpertUp>
                  : a.epilogue == kLinearExpertDown ? linear_f32<kLinearExpertDown>
                  : a.epilogue == kLinearExpertStore ? linear_f32<kLinearExpertStore> : a.epilogue == kLinearFloat ? linear_f32<kLinearFloat>
                  : a.epilogue == kLinearRotate ? linear_f32<kLinearRotate> : a.epilogue == kLinearSide ? linear_f32<kLinearSide> : linear_f32<kLinearStore>;
    if (experts && a.slots.tile_rows != kTile32) return int(cudaErrorInvalidValue);
    const dim3 grid(unsigned((a.n + kTile32 - 1) / kTile32), unsigned(experts ? MostTiles(a.slots) : (a.t + kTile32 - 1) / kTile32), unsigned(std::max(a.heads, 1)));
    return int(Launch(kernel, grid, dim3(256), 0, q.stream, q.chained, static_cast<const float*>(a.activations),
                      static_cast<const float*>(a.weight), p, a.k_stride, a.in_stride ? a.in_stride : a.k_stride));
  }
  p.chunks = (a.k_stride + kStepK - 1) / kStepK;
  int index = 0, splits = 1;
  if (experts) ChooseExpertLinear(a.slots, a.n, p.chunks, q.sm_count, &index, &splits);
  else ChooseLinear(a.t, a.n, std::max(a.heads, 1), p.chunks, q.sm_count, &index, &splits);
  p.chunks_per_split = (p.chunks + splits - 1) / splits;
  switch (index) {
    case 0: return int(LaunchTiles<16>(q, a, p, 0, splits));
    case 1: return int(LaunchTiles<32>(q, a, p, 1, splits));
    case 2: return int(LaunchTiles<64>(q, a, p, 2, splits));
    case 3: return int(LaunchTiles<128>(q, a, p, 3, splits));
    default: return int(LaunchTiles<256>(q, a, p, 4, splits));
  }
}

int GluRows(const Queue& q, const void* in, void* out, int t, int in_stride, int out_stride, int outputs, const Glu& glu) {
  if (t <= 0) return 0;
  const dim3 grid(unsigned((outputs + 255) / 256), unsigned(t));
  if (q.f32)
    return int(Launch(glu_rows<float>, grid, dim3(256), 0, q.stream, q.chained, static_cast<const float*>(in), static_cast<float*>(out), t,
                      in_stride, out_stride, outputs, glu));
  return int(Launch(glu_rows<__nv_bfloat16>, grid, dim3(256), 0, q.stream, q.chained, static_cast<const __nv_bfloat16*>(in),
                    static_cast<__nv_bfloat16*>(out), t, in_stride, out_stride, outputs, glu));
}

}  // namespace tmb
