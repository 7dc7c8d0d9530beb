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
  enum Kind { kAttention, kRetention, kLatent, kDelta };
  Kind kind = kAttention;
  int heads = 0, kv_heads = 0, dim = 0, vdim = 0;
  int rot_dims = 0, rotary = -1;          // rotary: index into RaggedSpec::rotaries (-1: no rotation)
  int rank = 0;                           // latent attention: size of the normed row that every head's key and value are images of
  int q_rank = 0;                         // ... and of the normed row that the queries are images of (0: of the layer's input itself)
                                          // ... rot_dims: rotated columns behind both, of every head's query and of one key part that all heads share
  int decay_rank = 0;                     // delta rule: size of the row that the decays are images of
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
  // delta rule: a decay is exp(-decay_scale sigmoid(..)), a unit key k / sqrt(k^2 + unit_eps)
  double decay_scale = 0, unit_eps = 0;

  int proj_rows() const {                 // rows of the stacked input projection: q | k (| v) (| g), or q | k | v | g, or q | latent, or decays | r | k | v | a | g
    if (kind == kLatent) return latent_at() + columns();
    if (kind == kDelta) return delta_at() + 5 * heads * dim;
    if (kind == kRetention) return 2 * heads * dim + 2 * heads * vdim;
    return (heads + kv_heads) * dim + (value_is_key ? 0 : kv_heads * vdim) + (gate ? heads * vdim : 0);
  }
  int gate_at() const { return gate ? proj_rows() - heads * vdim : -1; }   // attention: first gate column of a projected row
  int out_columns() const { return heads * vdim; }
  int columns() const { return rank + rot_dims; }            // latent attention: columns of a cached row
  int head_lead() const { return (dim + 7) / 8 * 8; }        // ... where the rotated part of a head's query starts
  int head_key() const { return rot_dims ? head_lead() + rot_dims : dim; }   // ... columns of its key
  int head_stride() const { return head_lead() + (rot_dims + 7) / 8 * 8; }   // ... and of its query
  int rank_stride() const { return (columns() + 7) / 8 * 8; }     // ... and of its query or output against latent rows
  int latent_at() const { return q_rank ? (q_rank + 7) / 8 * 8 : heads * head_stride(); }   // ... where the latent row starts in a projected one
  int expanded_key() const { return (head_key() + 15) / 16 * 16; }  // ... and of its key and value expanded from latent rows
  int expanded_columns() const { return heads * (expanded_key() + v_pool_dim()); }
  int delta_at() const { return (decay_rank + 7) / 8 * 8; }  // delta rule: where r starts in a projected row
  int state_dim() const { return (dim + 3) / 4 * 4; }        // ... key channels of a state, padded
  int pool_dim() const { return ((kind == kLatent ? columns() : dim) + 15) / 16 * 16; }
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
  bool chosen = false;                    // scores: softmax over the chosen experts' logits, ranked by logit
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

// A second embedding's part for a layer, gated by the stream: y = proj (gelu(gate x) * part), normed and added.
struct RaggedSide {
  int gate = -1, proj = -1, norm = -1;
  int from = 0;                           // first column of the layer's part
};

struct RaggedLayer {
  RaggedMixer mixer;
  RaggedMlp mlp;
  bool norm_output = false;               // the norms act on the sublayers' outputs; the sublayers read the stream itself
  // indices into the plan's buffer table
  int norm1 = -1, in_weight = -1, in_bias = -1, out_weight = -1, out_bias = -1, norm2 = -1, gate_up = -1, down = -1, decay = -1,
      q_norm = -1, k_norm = -1, router = -1, expert_up = -1, expert_down = -1, sinks = -1, blend = -1, latent_norm = -1, key_up = -1, value_up = -1, expand = -1,
      correction = -1, shared_up = -1, shared_down = -1;
  int q_latent_norm = -1, query_up = -1, decay_up = -1, decay_bias = -1, out_norm = -1, conv = -1;
  RaggedStreams streams[2];               // of the mixer and of the feed-forward
  RaggedSide side;
};

struct RaggedRun {
  int layer = 0;
  bool add_embedding = false;             // the embedding output is added to the residual stream first
  int k_pool = -1, v_pool = -1, state = -1;   // (latent attention: k_pool holds the latent rows)
  int history = -1;                       // inputs of the short convolution that are still to be read
};

struct RotaryTable {
  double base = 0, factor = 1;
  int dims = 0, buffer = -1;
  double yarn[4] = {1, 0, 0, 0};          // factor (1: none), original length, fast and slow turns
};

struct RaggedSpec {
  bool f32 = false;
  int width = 0, vocab = 0, slots = 0, capacity = 0, max_blocks = 0, num_blocks = 0, max_rows = 0, max_wanted = 0;
  double eps = 0;
  int streams = 1;                        // residual streams
  bool combined = false;                  // sublayer outputs enter the streams in a kernel of their own, see StreamStep in ops.h
  bool parallel = false;                  // a layer's mixer and feed-forward read one norm and enter the stream together
  int norm_groups = 1, taps = 0;          // (parallel) the norms' groups of columns; taps of the convolution in front of every mixer (0: none)
  int side_dim = 0, side_embed = -1;      // (parallel) columns of a layer's part of the second embedding (0: none)
  int side_columns = 0;
  double residual_mult = 1, embed_scale = 1, logit_scale = 1;
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
