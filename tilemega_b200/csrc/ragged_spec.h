// Description of a ragged-step plan: a decoder given as a list of layers, each with its own kind of token mixer and
// its own sizes, run in a given order (a layer may run several times). Read from the "model" object of the sidecar,
// which registry.py derives from a model's config.json.
#pragma once
#include <stdint.h>

#include <vector>

#include "json.h"

namespace tmb {

struct BufferSpec;

struct RaggedMixer {
  enum Kind { kAttention, kRetention, kLatent };
  Kind kind = kAttention;
  int heads = 0, kv_heads = 0, dim = 0, vdim = 0;
  int rot_dims = 0, rotary = -1;          // rotary: index into RaggedSpec::rotaries (-1: no rotation)
  int rank = 0;                           // latent attention: size of the cached row that every head's key and value are images of
  // attention
  bool value_is_key = false;
  bool qk_norm = false;                   // RMS norm over all query heads together, and over all key heads, before the rotation
  bool gate = false;                      // the heads' outputs are multiplied by sigmoid of a projection of their own
  bool sink = false;                      // a null key of score sink_score without a value joins every softmax
  double sink_score = 0;
  enum ValueMix { kOwn, kSource, kBlend };   // kBlend: values are a blend with those the kSource layer projected for the same token
  ValueMix value_mix = kOwn;
  int window = 0, keep = 0;
  double scale = 1.0;
  // retention
  std::vector<float> decay;

  int proj_rows() const {                 // rows of the stacked input projection: q | k (| v) (| g), or q | k | v | g, or q | latent
    if (kind == kLatent) return heads * head_stride() + rank;
    if (kind == kRetention) return 2 * heads * dim + 2 * heads * vdim;
    return (heads + kv_heads) * dim + (value_is_key ? 0 : kv_heads * vdim) + (gate ? heads * vdim : 0);
  }
  int gate_at() const { return gate ? proj_rows() - heads * vdim : -1; }   // attention: first gate column of a projected row
  int out_columns() const { return heads * vdim; }
  int head_stride() const { return (dim + 7) / 8 * 8; }      // latent attention: columns of one head's query
  int rank_stride() const { return (rank + 7) / 8 * 8; }     // ... and of its query or output against latent rows
  int expanded_key() const { return (dim + 15) / 16 * 16; }  // ... and of its key and value expanded from latent rows
  int expanded_columns() const { return heads * (expanded_key() + v_pool_dim()); }
  int pool_dim() const { return ((kind == kLatent ? rank : dim) + 15) / 16 * 16; }
  int v_pool_dim() const { return (vdim + 15) / 16 * 16; }
};

struct RaggedMlp {
  enum Kind { kNone, kGlu, kExperts };
  Kind kind = kNone;
  int ff = 0;
  // gated unit
  bool gelu = false;                      // tanh form of GELU on the gate, else the clipped SiLU
  double limit = 0, alpha = 1, shift = 0;
  int packed_rows() const { return (ff + 15) / 16 * 32; }
  // mixture of experts
  int experts = 0, top = 0;
  bool output_weighted = false;           // gated units whose outputs are weighted (else relu^2 units whose inputs are)
  bool softmax = false, correction = false;   // scores: softmax over all experts (else sigmoid), ranked with a correction added
  int groups = 1, keep_groups = 1;        // experts are taken from the best groups of neighbours only
  int shared_ff = 0;                      // a gated unit every token runs, times the sigmoid of one more row of the router
  double shared_limit = 0;
  int logits() const { return experts + (shared_ff ? 1 : 0); }   // router rows
  int shared_rows() const { return (shared_ff + 15) / 16 * 32; }
};

// Weights of one sublayer on several residual streams, indices into the plan's buffer table.
struct RaggedStreams {
  int in = -1, out = -1, mix = -1;
};

struct RaggedLayer {
  RaggedMixer mixer;
  RaggedMlp mlp;
  bool norm_output = false;               // the norms act on the sublayers' outputs; the sublayers read the stream itself
  // indices into the plan's buffer table
  int norm1 = -1, in_weight = -1, in_bias = -1, out_weight = -1, out_bias = -1, norm2 = -1, gate_up = -1, down = -1, decay = -1,
      q_norm = -1, k_norm = -1, router = -1, expert_up = -1, expert_down = -1, sinks = -1, blend = -1, latent_norm = -1, key_up = -1, value_up = -1, expand = -1,
      correction = -1, shared_up = -1, shared_down = -1;
  RaggedStreams streams[2];               // of the mixer and of the feed-forward
};

struct RaggedRun {
  int layer = 0;
  bool add_embedding = false;             // the embedding output is added to the residual stream first
  int k_pool = -1, v_pool = -1, state = -1;   // (latent attention: k_pool holds the latent rows)
};

struct RotaryTable {
  double base = 0, factor = 1;
  int dims = 0, buffer = -1;
};

struct RaggedSpec {
  bool f32 = false;
  int width = 0, vocab = 0, slots = 0, capacity = 0, max_blocks = 0, num_blocks = 0, max_rows = 0, max_wanted = 0;
  double eps = 0;
  int streams = 1;                        // residual streams
  bool combined = false;                  // sublayer outputs enter the streams in a kernel of their own, see StreamStep in ops.h
  bool write_residuals = false;
  std::vector<RaggedLayer> layers;
  std::vector<RaggedRun> runs;
  std::vector<RotaryTable> rotaries;
  int tokens = -1, entries = -1, wanted = -1, block_table = -1, logits = -1, next = -1, embed = -1, final_norm = -1, head = -1, hidden = -1,
      residuals = -1;

  // Fills the description and appends the plan's buffer table. Throws std::invalid_argument on anything unsupported.
  static RaggedSpec FromJson(const Json& plan, std::vector<BufferSpec>* buffers);
  uint64_t weight_bytes = 0;              // matrices a step of one token reads (every layer run, and the head)
};

inline int padded_columns(int k) { return (k + 7) / 8 * 8; }   // 16-byte rows for bf16

}  // namespace tmb
