// The operations a ragged-step plan (csrc/ragged.cu) is put together from, each with the constants of a model as
// parameters. A step runs `rows` tokens: every ENTRY of the step is one sequence with one or more consecutive
// positions (a portion of its prompt, or one decoded token). Every launcher queues one kernel on `Queue::stream` and
// returns a cudaError_t as int; element buffers are bf16 (Queue::f32 false) or fp32.
#pragma once
#include <cuda.h>
#include <cuda_runtime.h>
#include <stdint.h>

#include "ragged_limits.h"

namespace tmb {

// One sequence of a step: its rows are [first_row, first_row + rows), their positions first_position, ... , its
// block-table row and its recurrent state are those of `slot`. (Four ints, as the host writes them.)
struct Entry {
  int first_row, rows, first_position, slot;
};

struct Queue {
  cudaStream_t stream = nullptr;
  bool f32 = false;        // element type of activations, weights and pools: fp32 (true) or bf16
  bool chained = true;     // launch as a programmatic dependent of the kernel before it
  int sm_count = 148;
  unsigned* status = nullptr;   // first device wait that gave up (0: none)
};

// What a step's kernels know about its rows. entry/position/kv_row are written by StartStep.
struct StepRows {
  int rows = 0, entries = 0, longest = 0;   // longest: most rows of one entry
  int singles = 0;                          // entries of exactly one row
  const Entry* entry = nullptr;             // [entries]
  const int* block_table = nullptr;         // [slots][max_blocks]
  int max_blocks = 0, num_blocks = 0, capacity = 0, slots = 0;
  int* row_entry = nullptr;                 // [rows]
  int* row_position = nullptr;              // [rows]
  int* row_kv = nullptr;                    // [rows] pool row: block * 16 + position mod 16
};

// Each of the `streams` copies of x[row] = embed[token] * scale (and embed[token] as an element in `copy`, rows of copy_stride, unless null);
// the row tables.
int StartStep(const Queue& q, const StepRows& r, const int* tokens, const void* embed, float* x, int streams, void* copy, int copy_stride, int width,
              int vocab, float scale);

// out[i] = x[r] / sqrt(mean(x[r]^2) + eps) * weight, r = select ? select[i] : i. With `again`, x[r] += embed[token[r]]
// first (and is written back). Rows of `out` are out_stride elements apart.
struct NormArgs {
  float* x;
  const float* weight;
  void* out;
  const int* select;
  const int* tokens;
  const void* again;
  int rows, width, out_stride, vocab, limit;   // limit: rows of x (select is clamped to it)
  float eps;
};
int RmsNorm(const Queue& q, const NormArgs& a);

// A sublayer's output normed and added: x[i] += y / sqrt(mean(y^2) + eps) * weight, and out[i] = x[i] as elements. y is
// branch[i] (fp32 [rows][width]), or with `parts` > 0 the sum of the elements parts_of[i * parts + 0 .. parts - 1].
struct AddNormArgs {
  float* x;
  const float* branch;
  const void* parts_of;
  int parts;
  const float* weight;
  void* out;
  int rows, width, out_stride;
  float eps;
};
int AddNorm(const Queue& q, const AddNormArgs& a);

// One row operation between two sublayers of a model with residual streams x [row][streams][width]:
//   update    x_t <- sum_s mix[s][t] x_s + out[t] y    (mix null: x_t itself, out null: 1), all t from the old streams
//   collect   u = sum_t in[t] x_t (in null: 1), normed[i] = u / sqrt(mean(u^2) + eps) * weight, as elements
// y = the weighted sum of `parts` elements rows, parts_of[i * parts + k] by part_scale[i * parts + k], plus branch[i] (fp32)
// times sigmoid(branch_gate[i * gate_stride]) (null: 1), the sum times `gain`; either may be absent. Without an update a row may be
// chosen: r = select[i]. sum_of (or null): the streams' plain sum after the update. weight null: normed (or null) is u itself.
struct StreamArgs {
  float* x;
  int streams, rows, width, limit;
  bool update;
  const float *mix, *out;
  const void* parts_of;
  const float* part_scale;
  int parts;
  const float *branch, *branch_gate;
  int gate_stride;
  float gain = 1.f;
  float* sum_of;
  const float *in, *weight;
  void* normed;
  int normed_stride;
  const int* select;
  float eps;
};
int StreamStep(const Queue& q, const StreamArgs& a);

// The row operation in front of a layer whose mixer reads its norm through a short convolution over time:
//   x'   = x + gain * side / sqrt(mean(side^2) + eps) * side_weight      (side null: x), written to x_out (or null; not x itself)
//   h    = x' in `groups` runs of columns, each over its own root mean square, times weight; as elements in normed
//   read = h + sum_j taps[j] h at position p - (count - 1) + j, as elements in convolved (count 0: none)
// The h of the last count - 1 positions of a sequence lie in history [slots][count - 1][width], position p in row p mod
// (count - 1); positions before the first count as zeros. With `select` (and no convolution) row i is row select[i] of x.
struct ConvNormArgs {
  const float* x;
  const float* side;
  const float* side_weight;
  float* x_out;
  float gain, eps;
  const float* weight;
  int groups, rows, width, limit;
  void* normed;
  int stride;                // of normed and convolved
  const float* taps;         // [count][width]
  int count;
  float* history;
  void* convolved;
  const int* select;
};
int ConvNorm(const Queue& q, const StepRows& r, const ConvNormArgs& a);
int PrepareConv();

// Rotary table [capacity][dims / 2] of (cos, sin), or dims = 0: none.
struct Rotary {
  const float2* table = nullptr;
  int dims = 0, capacity = 0;
};

// y = min(g, limit) sigmoid(alpha min(g, limit)) (clamp(u, -limit, limit) + shift), or with `gelu` y = gelu(g) u, the
// tanh form
struct Glu {
  float limit = 0.f, alpha = 1.f, shift = 0.f;
  bool gelu = false;
};

enum LinearEpilogue { kLinearStore = 0, kLinearAdd = 1, kLinearGlu = 2, kLinearFloat = 3, kLinearExpertUp = 4, kLinearExpertDown = 5,
                      kLinearHeads = 6, kLinearExpertGlu = 7, kLinearExpertStore = 8, kLinearRotate = 9, kLinearSide = 10 };

// kLinearRotate: output columns are heads of head_out, and in each the columns rotary.dims behind `lead` turn, neighbours 2i and
// 2i + 1 by the row's position's angle i.
struct RotateHeads {
  Rotary rotary;
  const int* positions = nullptr;   // [rows]
  int lead = 0, head = 0;           // a head's columns: head
};
// kLinearSide: y = gelu(D) * part[token of the row], the tanh form; part rows of `stride` elements.
struct SideGate {
  const void* part = nullptr;
  const int* tokens = nullptr;      // [rows]
  int stride = 0, vocab = 0;
};

// The assignments of a step's rows to experts, sorted by expert (written by Route). Assignment a is the a % top-th choice
// of row a / top; slot s, in sorted order, runs assignment list[s] on the expert of its tile.
struct ExpertTile {
  int expert, first, count, unused;   // slots [first, first + count)
};
struct ExpertSlots {
  const ExpertTile* tiles = nullptr;
  const int* tile_count = nullptr;
  const int* list = nullptr;          // [slots]
  const float* score = nullptr;       // [slots]
  int experts = 0, top = 1, slots = 0, tile_rows = 0;
};

// D[t][n] = sum_k activations[t][k] weight[n][k] (+ bias[n]), then by epilogue: store as an element; x[t][n] += D; the
// gated unit of interleaved gate/up rows, stored as an element (column n of the output is pair n); store as fp32.
// Activation and weight rows are k_stride elements long (a multiple of 8, zero weights behind k).
// Per expert (weight rows expert * n ..., slots in place of t): ExpertUp reads activation row list[s] / top for slot s
// (from `activations`; bf16 tiles of more than kGatherRows slots read row s of rows gathered before, see GatherRows) and
// stores relu(score[s] D)^2 in row s; ExpertGlu reads the same and stores the gated unit, ExpertStore (fp32) D itself;
// ExpertDown reads row s and stores D in row list[s]; all as elements.
// Rotate and Side store elements as their structs say. Store: columns below tanh_below as their hyperbolic tangent.
// Heads: `heads` products side by side, head h of weight rows h * n ..., activation columns h * head_in ... and output
// columns h * head_out ... (head_in a multiple of 8; n and k are one head's), stored as elements.
constexpr int kGatherRows = 32;
struct LinearMaps {
  CUtensorMap weight;        // bf16 only: 128-row boxes
  CUtensorMap rows[5];       // boxes of 16, 32, 64, 128, 256 activation rows
  CUtensorMap row;           // boxes of one activation row (gathered rows)
};
struct LinearArgs {
  const void* activations;
  const void* weight;
  const float* bias;         // or null
  void* out;                 // element buffer, or the fp32 residual stream, or fp32
  const LinearMaps* maps;    // bf16 only
  int t, n, k_stride, out_stride;
  const int* rows_there;     // bf16: of the t rows only the first *rows_there are needed (null: all); written two kernels before, or earlier
  int in_stride;             // elements of an activation row, if it is not k_stride (0)
  int heads, head_in, head_out;   // kLinearHeads
  int outputs;               // kLinearGlu: columns stored (pairs beyond it are padding)
  int tanh_below;            // kLinearStore
  float gain = 1.f;          // kLinearFloat: factor of what is stored
  int epilogue;
  RotateHeads rotate;
  SideGate side;
  Glu glu;
  ExpertSlots slots;         // expert epilogues
};
int ExpertTileRows(const Queue& q, int slots, int experts);   // slots per tile that suits this many
int PrepareLinear();         // raises the kernels' shared-memory limits (once per device)
bool EncodeLinear(LinearMaps* maps, const void* weight, uint64_t n, const void* activations, uint64_t rows, uint64_t k_stride);
bool EncodeHeads(LinearMaps* maps, const void* weight, uint64_t n, uint64_t k_stride, const void* activations, uint64_t rows, uint64_t in_stride);
bool EncodeGathered(LinearMaps* maps, const void* activations, uint64_t rows, uint64_t k_stride);   // maps->row only
int Linear(const Queue& q, const LinearArgs& a);

// The gated unit by itself: in [t][2 * padded] interleaved pairs, out [t][outputs].
int GluRows(const Queue& q, const void* in, void* out, int t, int in_stride, int out_stride, int outputs, const Glu& glu);

// Mixture of experts: per row z = router h, scores sigmoid(z) or softmax(z) over the experts, and the `top` largest of score
// + correction (null: 0; the smaller index on a tie) among the keep_groups groups of neighbours whose largest is largest. `chosen`: ranked
// by z, scores are a softmax over the chosen experts' z alone.
// `weights`: the scores handed on are over their sum (+ 1e-20). `extra` more router rows are only multiplied. And the
// assignments sorted by expert in tiles of slots->tile_rows. RouteFused: does Route compute z itself? (If not, the
// caller has put it into `logits`.)
struct RouteArgs {
  const void* h;             // elements, rows of k_stride
  const void* router;        // [experts][k_stride]
  int k_stride, rows, experts, top, tile_rows;
  int extra;
  bool softmax, weights, chosen;
  const float* correction;
  int groups, keep_groups;
  float* ranks;              // [rows][experts], scratch (softmax scores, corrections or groups)
  float* logits;             // [rows][experts + extra]
  int* choice;               // [rows * top]
  float* score;              // [rows * top]
  int* list;                 // [rows * top], sorted
  float* slot_score;         // [rows * top], sorted
  ExpertTile* tiles;
  int* tile_count;
  unsigned* count;           // kRouteCounters arrival counters, zero between launches
};
constexpr int kRouteCounters = 9;
bool RouteFused(int rows);
int Route(const Queue& q, const RouteArgs& a);
// out[slot] = h[list[slot] / top] (bf16 rows of k_stride).
int GatherRows(const Queue& q, const void* h, int k_stride, const ExpertSlots& slots, void* out);

// Attention with grouped heads, a sliding window of `window` positions and the first `keep` positions always seen.
// proj rows hold q | k (| v) (| g): q heads x dim, k kv_heads x dim, v kv_heads x vdim, g heads x vdim; the values are v,
// or k before rotation (value_is_key). q_norm / k_norm: RMS norm over all heads together before the rotation. A null key
// of score `sink` (-infinity: none), or of sinks[head], without a value joins the softmax. Values are blended with
// blend_from, those of another layer for the same rows: (1 - *blend) v + *blend * theirs. gate_at >= 0: outputs times sigmoid(g).
struct AttentionArgs {
  void* proj;
  int proj_stride;
  void* k_pool;              // [num_blocks][kv_heads][16][pool_dim]
  void* v_pool;              // [num_blocks][kv_heads][16][v_pool_dim]
  void* out;                 // [rows][out_stride], heads x vdim
  int out_stride;
  int heads, kv_heads, dim, vdim, pool_dim, v_pool_dim;
  bool value_is_key;
  const float* q_norm;       // [heads * dim], or null
  const float* k_norm;       // [kv_heads * dim]
  float eps, sink;
  const float* sinks;        // [heads], or null
  const float* blend;        // or null
  const void* blend_from;    // element rows of blend_stride, kv_heads x vdim
  int blend_stride;
  int gate_at;               // first gate column of a projected row, or -1
  int window, keep;
  float scale;
  Rotary rotary;
  float* part;               // decode partials, part_floats floats
  size_t part_floats;
  unsigned* count;           // arrival counters, zero between launches
  int count_words;
};
// Norms and rotates q in place and appends such k, and v, to the pools. (bf16: rows of portions only; a decoded token's attention
// does it itself.)
int RotateAppend(const Queue& q, const StepRows& r, const AttentionArgs& a);
int Attend(const Queue& q, const StepRows& r, const AttentionArgs& a);
int AttendTiles(const Queue& q, const StepRows& r, const AttentionArgs& a);   // the bf16 form
// The portions of a step over keys and values that lie in rows of context_stride elements: position j of entry n in row
// context[n] + j - max(0, first_position - window + 1), keys of head g at k_pool + g * pool_dim there, values at
// v_pool + g * v_pool_dim. Query heads are q_head elements apart; nothing is rotated, normed or appended.
int AttendContext(const Queue& q, const StepRows& r, const AttentionArgs& a, int q_head, const int* context, int context_stride);
int PrepareMixers();

// Attention whose keys and values are images, per head, of one cached latent row per token: scores and sums are taken
// against the latent rows themselves, with queries `q` already multiplied by their heads' key matrices; `out` rows are the
// heads' weighted sums of latent rows, for the heads' value matrices to follow. latent rows come from `raw` ([rows] of
// raw_stride, normed by AppendLatent on their way into the pool).
struct LatentArgs {
  const void* q;             // [rows][heads][rank_stride], zeros behind the rank
  void* out;                 // [rows][heads][rank_stride]
  const void* raw;
  int raw_stride;
  const float* norm;         // [rank]
  void* pool;                // [num_blocks][16][pool_dim]
  const CUtensorMap *pool_map, *q_map;   // bf16, tiled form: see EncodeLatent, EncodeLookup
  int heads, rank, rank_stride, pool_dim;   // rank: columns of a row, the rotated ones included
  Rotary rotary;             // the last rotary.dims columns of a row turn, neighbours together, in place of being normed
  const void* query_raw;     // rows of raw_stride beside `raw` that AppendLatent norms into query (null: none; then the heads' queries are images
  const float* query_norm;   // of these, and AppendLatent takes every row)
  void* query;               // [rows][query_stride]
  int query_rank, query_stride;
  float eps, scale, sink;
  const float* sinks;        // [heads], or null
  int window;
  bool singles_only;         // portions are attended to elsewhere
  float* part;               // decode partials, part_floats floats
  size_t part_floats;
};
// (bf16 rows that suit the tiled form: AppendLatent takes portions only, a decoded token's attention appends its own row.)
int AppendLatent(const Queue& q, const StepRows& r, const LatentArgs& a);
int AttendLatent(const Queue& q, const StepRows& r, const LatentArgs& a);
constexpr int kTiledLatent = 640;   // widest latent row of the tiled form
inline bool LatentTiled(const LatentArgs& a) { return a.rank <= kTiledLatent; }
int AttendLatentTiles(const Queue& q, const StepRows& r, const LatentArgs& a);   // the tiled form
int PrepareLatent();
bool EncodeLatent(CUtensorMap* pool_map, const void* pool, uint64_t rows, uint64_t pool_dim);
bool EncodeLookup(CUtensorMap* q_map, const void* q, uint64_t rows, uint64_t rank_stride);   // rows: one per token and head
// Long portions expand the latent rows they see into keys and values first: where each entry's rows start in the expanded
// ones (context [entries], and how many there are in all), and those rows gathered from the pool, `most` at most.
int LatentContext(const Queue& q, const StepRows& r, int window, int* context, int* context_rows);
int GatherLatent(const Queue& q, const StepRows& r, const LatentArgs& a, const int* context, const int* context_rows, int most, void* out);

// Retention: per head S <- decay S + k v^T, o = S^T q, with rotary q and k, k scaled by key_scale. proj rows hold
// q | k | v | g. state [slots][heads][dim][vdim] fp32; an entry that starts at position 0 starts from a zero state.
struct RetentionArgs {
  const void* proj;
  int proj_stride;
  float* state;
  float* raw;                // [rows][heads * vdim]
  void* split;               // bf16: [rows][heads][4][dim padded to 16], q and k of portions as heads and remainders
  void* out;                 // [rows][out_stride]
  int out_stride;
  int heads, dim, vdim;
  const float* decay;        // [heads]
  float key_scale, eps;
  Rotary rotary;
};
// The mixer's output in a.out: o / rms(o) per head, times silu(g).
int Retain(const Queue& q, const StepRows& r, const RetentionArgs& a);
int RetainChunks(const Queue& q, const StepRows& r, const RetentionArgs& a);  // the bf16 form of entries of several rows

// out = o / rms(o) of every head, times weight (null: 1), times the gate's sigmoid, or (silu) the gate times its sigmoid. o fp32
// [rows][heads * vdim], gates at column gate_at of rows of `proj`.
struct HeadGateArgs {
  const float* raw;
  const void* proj;
  int proj_stride, gate_at;
  void* out;
  int out_stride, rows, heads, vdim;
  const float* weight;       // [heads * vdim]
  bool silu;
  float eps;
};
int HeadGate(const Queue& q, const HeadGateArgs& a);

// Generalised delta rule with a decay and a removal rate per head and key channel:
//   u = k / sqrt(k^2 + unit_eps), w = exp(-decay_scale sigmoid(z)), S <- diag(w) S - (sigmoid(a) u) (u^T S) + k v^T, o = S^T r
// proj rows hold r | k | v | a | g, heads x dim each; z fp32 [rows][heads * dim]. state [slots][heads][dim: value columns][padded dim: key
// channels] fp32; an entry that starts at position 0 starts from a zero state. Out: o / rms(o) per head, times norm, times sigmoid(g).
struct DeltaArgs {
  const void* proj;
  int proj_stride;
  const float* z;
  float* state;
  float* raw;                // [rows][heads * dim]
  void* out;
  int out_stride;
  int heads, dim, padded;
  const float* norm;         // [heads * dim]
  float decay_scale, unit_eps, eps;
  void* chunks;              // bf16: DeltaChunkBytes bytes, the portions' chunks
};
int Delta(const Queue& q, const StepRows& r, const DeltaArgs& a);
int PrepareDelta();
size_t DeltaChunkBytes(int rows, int slots, int heads, int dim);
// The bf16 form of portions (portions_only: of these alone), up to the heads' raw outputs.
int DeltaChunks(const Queue& q, const StepRows& r, const DeltaArgs& a, bool portions_only);
int PrepareDeltaChunks();

// next[i] = index of the largest of logits[i][0..vocab), the smallest such index on a tie.
int ArgMax(const Queue& q, const float* logits, int rows, int vocab, int* next);
// After a step of single-row entries whose rows are all wanted: tokens[row] = next[row], first_position += 1.
int Feed(const Queue& q, Entry* entries, int count, const int* next, int* tokens, int capacity);

}  // namespace tmb
