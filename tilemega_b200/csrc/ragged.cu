// Ragged-step plans: the layer list of a decoder lowered to the operations of ops.h. See ragged.h.
#include "ragged.h"

#include <algorithm>
#include <cmath>
#include <cstdlib>
#include <map>
#include <tuple>

#include "ops.h"
#include "plan_spec.h"
#include "tensor_map.h"

namespace tmb {

struct RaggedPlan {
  RaggedSpec spec;
  Queue queue;
  StepRows rows;
  std::vector<void*> buffers;
  std::vector<void*> owned;
  void* normed = nullptr;      // [max_rows][padded width]
  void* picked = nullptr;      // [max_wanted][padded width]: normed rows the head scores
  void* proj = nullptr;        // [max_rows][widest input projection]
  void* mixed = nullptr;       // [max_rows][widest mixer output]
  void* source = nullptr;      // [max_rows][its input projection]: the projected rows of the layer whose values others blend in
  int source_stride = 0, source_at = 0;   // ... and where its values start in a row
  void *lookup = nullptr, *looked = nullptr;   // latent attention: queries against latent rows, weighted sums of latent rows
  void* mlp = nullptr;         // [max_rows][widest feed-forward]
  void* pairs = nullptr;       // fp32 plans: gate/up rows before the gated unit
  float* branch = nullptr;     // fp32 outputs of sublayers that are normed, or summed, before they are added
  // parallel layers: the stream's other place (rows are formed anew next to rows that still read the old ones), the stream and the
  // convolved norm as elements, the side input's hidden rows and output
  float* other = nullptr;
  void *elements = nullptr, *convolved = nullptr, *side_hidden = nullptr;
  float* side_out = nullptr;
  void *query_latent = nullptr, *queries = nullptr;   // latent attention: normed rows that queries are images of, and these
  float* decay_in = nullptr;   // delta rule: what decays are made of, [max_rows][heads * dim]
  void* chunks = nullptr;      // ... bf16 plans: operands of the portions' chunks
  // bf16 plans with latent attention: the latent rows that portions see, gathered, and their keys and values
  void *context = nullptr, *expanded = nullptr;
  int *context_at = nullptr, *context_count = nullptr;
  int context_rows = 0;
  // mixtures of experts: logits, choices and scores per row, the assignments sorted by expert, their hidden rows and outputs
  float* logits = nullptr;
  int *choice = nullptr, *list = nullptr, *tile_count = nullptr;
  float *score = nullptr, *slot_score = nullptr;
  ExpertTile* tiles = nullptr;
  unsigned* route_count = nullptr;
  void* gathered = nullptr;        // bf16 plans: [max_rows * most experts of a token][padded width]
  float* ranks = nullptr;          // [max_rows][most experts]
  void* expert_pairs = nullptr;    // fp32 plans: gate/up rows of experts before the gated unit
  void* expert_hidden = nullptr;   // [max_rows * most experts of a token][widest expert]
  void* expert_out = nullptr;      // [max_rows * most experts of a token][width]
  float* raw = nullptr;        // retention outputs before their norm
  void* split = nullptr;       // bf16 plans: rotated retention queries and keys of portions
  float* part = nullptr;       // attention partials
  size_t part_floats = 0;
  unsigned* count = nullptr;
  int count_words = 0;
  std::vector<float*> decay;   // per layer
  struct Maps {
    LinearMaps in, out, gate_up, down, router;   // (gate_up, down: of the gated unit or of the experts)
    LinearMaps shared_up, shared_down, key_up, value_up, expand, query_up, decay_up, side_gate, side_proj;
    CUtensorMap lookup;
  };
  std::vector<Maps> maps;      // per layer (bf16 plans)
  std::vector<CUtensorMap> latent;   // per run (bf16 plans): pools of latent rows
  LinearMaps head;
  // recorded steps of single-row entries, by (entries, wanted, feed)
  std::map<std::tuple<uint32_t, uint32_t, bool>, cudaGraphExec_t> graphs;
  std::map<std::tuple<uint32_t, uint32_t, bool>, int> seen;
};

namespace {

template <typename T> bool Own(RaggedPlan* plan, T** out, size_t bytes) {
  void* p = nullptr;
  bytes = (bytes + 255) / 256 * 256 + 256;
  if (cudaMalloc(&p, bytes) != cudaSuccess) return false;
  plan->owned.push_back(p);
  *out = static_cast<T*>(p);
  return cudaMemset(p, 0, bytes) == cudaSuccess;
}

// Rows (at most) that a step's portions see of a latent layer, if these are to be expanded into keys and values: for long
// portions that is less work than scores and sums over latent rows, by about three products' cost to one of attention.
int ContextRows(const RaggedPlan* plan, const StepRows& r, const RaggedMixer& m) {
  const int portions = r.entries - r.singles, rows = r.rows - r.singles;
  if (!plan->context_rows || portions == 0) return 0;
  const double reach = std::min(m.window, r.capacity), each = double(rows) / portions, head = m.head_key() + m.vdim;
  const double most = rows + portions * (reach - 1);
  if (most > plan->context_rows) return 0;
  return each * reach * (2.0 * m.columns() - head) > (each + reach) * m.columns() * head / 3.0 ? int(most) : 0;
}

int Enqueue(RaggedPlan* plan, uint32_t entries, uint32_t rows, uint32_t longest, uint32_t singles, uint32_t wanted, bool feed, cudaStream_t stream) {
  const RaggedSpec& s = plan->spec;
  Queue q = plan->queue;
  q.stream = stream;
  StepRows r = plan->rows;
  r.rows = int(rows);
  r.entries = int(entries);
  r.longest = int(longest);
  r.singles = int(singles);
  auto buffer = [&](int index) -> void* { return index >= 0 ? plan->buffers[size_t(index)] : nullptr; };
  auto floats = [&](int index) { return static_cast<float*>(buffer(index)); };
  float* x = floats(s.hidden);
  const int* tokens = static_cast<const int*>(buffer(s.tokens));
  const int W = s.width, W8 = padded_columns(s.width);
#define TMB_TRY(call)                \
  do {                               \
    const int status_ = (call);      \
    if (status_ != 0) return status_; \
  } while (0)
  const bool norm_output = s.layers[0].norm_output;   // sublayers then read the stream itself: `normed` holds it as elements
  TMB_TRY(StartStep(q, r, tokens, buffer(s.embed), x, s.streams, norm_output ? plan->normed : nullptr, W8, W, s.vocab, float(s.embed_scale)));
  auto norm = [&](int weight, bool again) {
    NormArgs a{};
    a.x = x;
    a.weight = floats(weight);
    a.out = plan->normed;
    a.tokens = tokens;
    a.again = again ? buffer(s.embed) : nullptr;
    a.rows = r.rows;
    a.width = W;
    a.out_stride = W8;
    a.vocab = s.vocab;
    a.limit = r.rows;
    a.eps = float(s.eps);
    return RmsNorm(q, a);
  };
  auto linear = [&](const void* in, int weight, int bias, const LinearMaps* maps, int n, int k, void* out, int out_stride, int epilogue) {
    LinearArgs a{};
    a.activations = in;
    a.weight = buffer(weight);
    a.bias = floats(bias);
    a.out = out;
    a.maps = maps;
    a.t = r.rows;
    a.n = n;
    a.k_stride = padded_columns(k);
    a.out_stride = out_stride;
    a.epilogue = epilogue;
    return a;
  };
  // a sublayer's last product (rows of `in` times `weight`): added to the stream, or normed and added
  auto add_output = [&](const void* in, int weight, int bias, const LinearMaps* maps, int k) {
    if (!norm_output && !s.combined && !s.parallel) return Linear(q, linear(in, weight, bias, maps, W, k, x, W, kLinearAdd));
    return Linear(q, linear(in, weight, bias, maps, W, k, plan->branch, W, kLinearFloat));
  };
  auto add_norm = [&](int weight, int parts) {
    AddNormArgs a{};
    a.x = x;
    a.branch = plan->branch;
    a.parts_of = plan->expert_out;
    a.parts = parts;
    a.weight = floats(weight);
    a.out = plan->normed;
    a.rows = r.rows;
    a.width = W;
    a.out_stride = W8;
    a.eps = float(s.eps);
    return AddNorm(q, a);
  };
  // Several streams (combined): one row operation adds a sublayer's output and collects what the next one reads. `done`: the
  // sublayer that ran (null: none yet), `next`: the one to come (null: the model's end).
  StreamArgs step{};
  step.x = x;
  step.streams = s.streams;
  step.rows = step.limit = r.rows;
  step.width = W;
  step.normed = plan->normed;
  step.normed_stride = W8;
  step.eps = float(s.eps);
  auto restream = [&](const RaggedStreams* done, const RaggedMlp* mixture, const RaggedStreams* next, int norm_weight, float* sum_of) {
    StreamArgs a = step;
    if (done) {
      a.update = true;
      a.mix = floats(done->mix);
      a.out = floats(done->out);
      a.branch = plan->branch;
      if (mixture) {
        a.parts_of = plan->expert_out;
        a.part_scale = plan->score;
        a.parts = mixture->top;
        a.branch = mixture->shared_ff ? plan->branch : nullptr;
        a.branch_gate = mixture->shared_ff ? plan->logits + mixture->experts : nullptr;
        a.gate_stride = mixture->logits();
      }
    }
    if (next) {
      a.in = floats(next->in);
      a.weight = floats(norm_weight);
    } else {
      a.normed = nullptr;
    }
    a.sum_of = sum_of;
    return StreamStep(q, a);
  };
  if (s.combined) {
    const RaggedLayer& first = s.layers[size_t(s.runs[0].layer)];
    TMB_TRY(restream(nullptr, nullptr, &first.streams[0], first.norm1, nullptr));
  }
  // Parallel layers. In front of a layer: the side input of the layer before added, the grouped norm, the convolution. Behind it: both
  // sublayers' outputs added at once, and the side input's products.
  bool side_waits = false;
  const RaggedSide* side = nullptr;
  auto conv_norm = [&](int weight, const RaggedLayer* layer, const RaggedRun* run, const int* select, int count, void* normed) {
    ConvNormArgs a{};
    a.x = x;
    if (side_waits) {
      a.side = plan->side_out;
      a.side_weight = floats(side->norm);
      a.gain = float(s.residual_mult);
    }
    if (side_waits && !select) {
      a.x_out = x == floats(s.hidden) ? plan->other : floats(s.hidden);
      x = a.x_out;
      side_waits = false;
    }
    a.eps = float(s.eps);
    a.weight = floats(weight);
    a.groups = s.norm_groups;
    a.rows = count;
    a.limit = r.rows;
    a.width = W;
    a.normed = normed;
    a.stride = W8;
    if (layer) {
      a.taps = floats(layer->conv);
      a.count = s.taps;
      a.history = floats(run->history);
      a.convolved = plan->convolved;
    }
    a.select = select;
    return ConvNorm(q, r, a);
  };
  auto add_sublayers = [&](const RaggedLayer& layer, const RaggedPlan::Maps* maps) {
    StreamArgs a{};
    a.x = x;
    a.streams = 1;
    a.rows = a.limit = r.rows;
    a.width = W;
    a.update = true;
    a.branch = plan->branch;
    a.gain = float(s.residual_mult);
    if (layer.mlp.kind == RaggedMlp::kExperts) {
      a.parts_of = plan->expert_out;
      a.part_scale = plan->score;
      a.parts = layer.mlp.top;
    }
    if (s.side_dim) {
      a.normed = plan->elements;
      a.normed_stride = W8;
    }
    TMB_TRY(StreamStep(q, a));
    if (!s.side_dim) return 0;
    const int stride = padded_columns(s.side_dim);
    LinearArgs gate = linear(plan->elements, layer.side.gate, -1, maps ? &maps->side_gate : nullptr, s.side_dim, W, plan->side_hidden, stride, kLinearSide);
    gate.side.part = static_cast<const char*>(buffer(s.side_embed)) + size_t(layer.side.from) * (s.f32 ? 4 : 2);
    gate.side.tokens = tokens;
    gate.side.stride = s.side_columns;
    gate.side.vocab = s.vocab;
    TMB_TRY(Linear(q, gate));
    TMB_TRY(Linear(q, linear(plan->side_hidden, layer.side.proj, -1, maps ? &maps->side_proj : nullptr, W, s.side_dim, plan->side_out, W, kLinearFloat)));
    side = &layer.side;
    side_waits = true;
    return 0;
  };
  auto keep_stream = [&](size_t run) {       // (plans that write residuals)
    return int(cudaMemcpyAsync(floats(s.residuals) + run * size_t(s.max_rows) * W, x, size_t(rows) * W * sizeof(float), cudaMemcpyDeviceToDevice, stream));
  };
  int context_window = -1;               // the window that the table of expanded rows is for
  for (size_t i = 0; i < s.runs.size(); ++i) {
    const RaggedRun& run = s.runs[i];
    const RaggedLayer* next = i + 1 < s.runs.size() ? &s.layers[size_t(s.runs[i + 1].layer)] : nullptr;
    float* kept = s.write_residuals ? floats(s.residuals) + i * size_t(s.max_rows) * W : nullptr;
    const RaggedLayer& layer = s.layers[size_t(run.layer)];
    const RaggedMixer& m = layer.mixer;
    const RaggedPlan::Maps* maps = s.f32 ? nullptr : &plan->maps[size_t(run.layer)];
    const int stride = (m.proj_rows() + 7) / 8 * 8, mixed_stride = padded_columns(m.out_columns());
    if (s.parallel) {
      TMB_TRY(conv_norm(layer.norm1, s.taps ? &layer : nullptr, &run, nullptr, r.rows, plan->normed));
      if (s.write_residuals && i > 0) TMB_TRY(keep_stream(i - 1));
    } else if (!norm_output && !s.combined) {
      TMB_TRY(norm(layer.norm1, run.add_embedding));
    }
    void* proj = m.value_mix == RaggedMixer::kSource ? plan->source : plan->proj;
    LinearArgs in = linear(s.taps ? plan->convolved : plan->normed, layer.in_weight, layer.in_bias, maps ? &maps->in : nullptr, m.proj_rows(), W, proj, stride, kLinearStore);
    if (m.kind == RaggedMixer::kDelta) in.tanh_below = m.decay_rank;
    TMB_TRY(Linear(q, in));
    Rotary rotary;
    if (m.rotary >= 0) {
      rotary.table = static_cast<const float2*>(buffer(s.rotaries[size_t(m.rotary)].buffer));
      rotary.dims = m.rot_dims;
    }
    rotary.capacity = s.capacity;
    if (m.kind == RaggedMixer::kRetention) {
      RetentionArgs a{};
      a.proj = plan->proj;
      a.proj_stride = stride;
      a.state = floats(run.state);
      a.raw = plan->raw;
      a.split = plan->split;
      a.out = plan->mixed;
      a.out_stride = mixed_stride;
      a.heads = m.heads;
      a.dim = m.dim;
      a.vdim = m.vdim;
      a.decay = plan->decay[size_t(run.layer)];
      a.key_scale = float(1.0 / std::sqrt(double(m.dim)));
      a.eps = float(s.eps);
      a.rotary = rotary;
      TMB_TRY(Retain(q, r, a));
    } else if (m.kind == RaggedMixer::kDelta) {
      const int all = m.heads * m.dim;
      LinearArgs up = linear(proj, layer.decay_up, layer.decay_bias, maps ? &maps->decay_up : nullptr, all, m.decay_rank, plan->decay_in, all, kLinearFloat);
      up.in_stride = stride;
      TMB_TRY(Linear(q, up));
      DeltaArgs a{};
      a.proj = static_cast<const char*>(proj) + size_t(m.delta_at()) * (s.f32 ? 4 : 2);
      a.proj_stride = stride;
      a.z = plan->decay_in;
      a.state = floats(run.state);
      a.raw = plan->raw;
      a.out = plan->mixed;
      a.out_stride = mixed_stride;
      a.heads = m.heads;
      a.dim = m.dim;
      a.padded = m.state_dim();
      a.norm = floats(layer.out_norm);
      a.decay_scale = float(m.decay_scale);
      a.unit_eps = float(m.unit_eps);
      a.eps = float(s.eps);
      a.chunks = plan->chunks;
      TMB_TRY(Delta(q, r, a));
    } else if (m.kind == RaggedMixer::kLatent) {
      LatentArgs a{};
      a.q = plan->lookup;
      a.out = plan->looked;
      a.raw = static_cast<const char*>(proj) + size_t(m.latent_at()) * (s.f32 ? 4 : 2);
      a.raw_stride = stride;
      a.norm = floats(layer.latent_norm);
      a.pool = buffer(run.k_pool);
      a.pool_map = maps ? &plan->latent[i] : nullptr;
      a.q_map = maps ? &maps->lookup : nullptr;
      a.heads = m.heads;
      a.rank = m.columns();
      a.rotary = rotary;
      if (m.q_rank) {
        a.query_raw = proj;
        a.query_norm = floats(layer.q_latent_norm);
        a.query = plan->query_latent;
        a.query_rank = m.q_rank;
        a.query_stride = padded_columns(m.q_rank);
      }
      a.rank_stride = m.rank_stride();
      a.pool_dim = m.pool_dim();
      a.eps = float(s.eps);
      a.scale = float(m.scale);
      a.sink = -INFINITY;
      a.sinks = floats(layer.sinks);
      a.window = m.window;
      a.part = plan->part;
      a.part_floats = plan->part_floats;
      const int wide = m.heads * m.rank_stride();
      TMB_TRY(AppendLatent(q, r, a));
      const void* heads = proj;            // the heads' queries
      int heads_stride = stride;
      if (m.q_rank) {
        heads = plan->queries;
        heads_stride = m.heads * m.head_stride();
        LinearArgs up = linear(plan->query_latent, layer.query_up, -1, maps ? &maps->query_up : nullptr, heads_stride, m.q_rank, plan->queries, heads_stride,
                               m.rot_dims ? kLinearRotate : kLinearStore);
        up.rotate.rotary = rotary;
        up.rotate.positions = r.row_position;
        up.rotate.lead = m.head_lead();
        up.rotate.head = m.head_stride();
        TMB_TRY(Linear(q, up));
      }
      const int context = ContextRows(plan, r, m);
      a.singles_only = context > 0;
      if (!context || r.singles) {
        LinearArgs up = linear(heads, layer.key_up, -1, maps ? &maps->key_up : nullptr, m.rank_stride(), m.head_stride(), plan->lookup, wide, kLinearHeads);
        up.in_stride = heads_stride;
        up.heads = m.heads;
        up.head_in = m.head_stride();
        up.head_out = m.rank_stride();
        TMB_TRY(Linear(q, up));
        TMB_TRY(AttendLatent(q, r, a));
        LinearArgs down = linear(plan->looked, layer.value_up, -1, maps ? &maps->value_up : nullptr, m.vdim, m.rank_stride(), plan->mixed, mixed_stride, kLinearHeads);
        down.in_stride = wide;
        down.heads = m.heads;
        down.head_in = m.rank_stride();
        down.head_out = m.vdim;
        TMB_TRY(Linear(q, down));
      }
      if (context) {                     // (behind the products of all rows, whose result for the portions' rows it replaces)
        if (context_window != m.window) TMB_TRY(LatentContext(q, r, m.window, plan->context_at, plan->context_count));
        context_window = m.window;
        TMB_TRY(GatherLatent(q, r, a, plan->context_at, plan->context_count, context, plan->context));
        const int columns = m.expanded_columns();
        LinearArgs expand = linear(plan->context, layer.expand, -1, &maps->expand, columns, m.rank_stride(), plan->expanded, columns, kLinearStore);
        expand.t = context;
        expand.rows_there = plan->context_count;
        TMB_TRY(Linear(q, expand));
        AttentionArgs seen{};
        seen.proj = const_cast<void*>(heads);
        seen.proj_stride = heads_stride;
        seen.k_pool = plan->expanded;
        seen.v_pool = static_cast<char*>(plan->expanded) + size_t(m.heads) * m.expanded_key() * 2;
        seen.out = plan->mixed;
        seen.out_stride = mixed_stride;
        seen.heads = seen.kv_heads = m.heads;
        seen.dim = m.head_key();
        seen.vdim = m.vdim;
        seen.pool_dim = m.expanded_key();
        seen.v_pool_dim = m.v_pool_dim();
        seen.sink = a.sink;
        seen.sinks = a.sinks;
        seen.gate_at = -1;
        seen.window = m.window;
        seen.scale = a.scale;
        TMB_TRY(AttendContext(q, r, seen, m.head_stride(), plan->context_at, columns));
      }
    } else {
      AttentionArgs a{};
      a.proj = proj;
      a.proj_stride = stride;
      a.k_pool = buffer(run.k_pool);
      a.v_pool = buffer(run.v_pool);
      a.out = plan->mixed;
      a.out_stride = mixed_stride;
      a.heads = m.heads;
      a.kv_heads = m.kv_heads;
      a.dim = m.dim;
      a.vdim = m.vdim;
      a.pool_dim = m.pool_dim();
      a.v_pool_dim = m.v_pool_dim();
      a.q_norm = floats(layer.q_norm);
      a.k_norm = floats(layer.k_norm);
      a.eps = float(s.eps);
      a.sink = m.sink ? float(m.sink_score) : -INFINITY;
      a.sinks = floats(layer.sinks);
      a.blend = floats(layer.blend);
      a.blend_from = static_cast<const char*>(plan->source) + size_t(plan->source_at) * (s.f32 ? 4 : 2);
      a.blend_stride = plan->source_stride;
      a.gate_at = m.gate_at();
      a.value_is_key = m.value_is_key;
      a.window = m.window;
      a.keep = m.keep;
      a.scale = float(m.scale);
      a.rotary = rotary;
      a.part = plan->part;
      a.part_floats = plan->part_floats;
      a.count = plan->count;
      a.count_words = plan->count_words;
      TMB_TRY(RotateAppend(q, r, a));
      TMB_TRY(Attend(q, r, a));
    }
    TMB_TRY(add_output(plan->mixed, layer.out_weight, layer.out_bias, maps ? &maps->out : nullptr, m.out_columns()));
    if (norm_output) TMB_TRY(add_norm(layer.norm1, 0));
    const RaggedMlp& mlp = layer.mlp;
    // what follows the mixer and what follows the layer, on several streams
    const bool last = mlp.kind == RaggedMlp::kNone;
    auto leave = [&](const RaggedStreams* done, const RaggedMlp* mixture) {
      return restream(done, mixture, next ? &next->streams[0] : nullptr, next ? next->norm1 : -1, kept);
    };
    if (s.combined) TMB_TRY(last ? leave(&layer.streams[0], nullptr) : restream(&layer.streams[0], nullptr, &layer.streams[1], layer.norm2, nullptr));
    if (mlp.kind == RaggedMlp::kGlu) {
      const Glu glu{float(mlp.limit), float(mlp.alpha), float(mlp.shift), mlp.gelu};
      const int packed = mlp.packed_rows(), mlp_stride = padded_columns(mlp.ff);
      if (!norm_output && !s.combined && !s.parallel) TMB_TRY(norm(layer.norm2, false));
      if (s.f32) {
        TMB_TRY(Linear(q, linear(plan->normed, layer.gate_up, -1, nullptr, packed, W, plan->pairs, packed, kLinearStore)));
        TMB_TRY(GluRows(q, plan->pairs, plan->mlp, r.rows, packed, mlp_stride, mlp.ff, glu));
      } else {
        LinearArgs a = linear(plan->normed, layer.gate_up, -1, &maps->gate_up, packed, W, plan->mlp, mlp_stride, kLinearGlu);
        a.outputs = mlp.ff;
        a.glu = glu;
        TMB_TRY(Linear(q, a));
      }
      if (s.parallel) TMB_TRY(Linear(q, linear(plan->mlp, layer.down, -1, maps ? &maps->down : nullptr, W, mlp.ff, plan->branch, W, kLinearAdd)));
      else TMB_TRY(add_output(plan->mlp, layer.down, -1, maps ? &maps->down : nullptr, mlp.ff));
      if (norm_output) TMB_TRY(add_norm(layer.norm2, 0));
      if (s.combined) TMB_TRY(leave(&layer.streams[1], nullptr));
    } else if (mlp.kind == RaggedMlp::kExperts) {
      ExpertSlots slots;
      slots.tiles = plan->tiles;
      slots.tile_count = plan->tile_count;
      slots.list = plan->list;
      slots.score = plan->slot_score;
      slots.experts = mlp.experts;
      slots.top = mlp.top;
      slots.slots = r.rows * mlp.top;
      slots.tile_rows = ExpertTileRows(q, slots.slots, slots.experts);
      RouteArgs a{};
      a.h = plan->normed;
      a.router = buffer(layer.router);
      a.k_stride = W8;
      a.rows = r.rows;
      a.experts = mlp.experts;
      a.top = mlp.top;
      a.tile_rows = slots.tile_rows;
      a.extra = mlp.logits() - mlp.experts;
      a.softmax = mlp.softmax;
      a.weights = mlp.output_weighted;
      a.correction = floats(layer.correction);
      a.groups = mlp.groups;
      a.keep_groups = mlp.keep_groups;
      a.chosen = mlp.chosen;
      a.ranks = mlp.output_weighted && !mlp.chosen ? plan->ranks : nullptr;
      a.logits = plan->logits;
      a.choice = plan->choice;
      a.score = plan->score;
      a.list = plan->list;
      a.slot_score = plan->slot_score;
      a.tiles = plan->tiles;
      a.tile_count = plan->tile_count;
      a.count = plan->route_count;
      if (!RouteFused(r.rows))
        TMB_TRY(Linear(q, linear(plan->normed, layer.router, -1, maps ? &maps->router : nullptr, mlp.logits(), W, plan->logits, mlp.logits(), kLinearFloat)));
      TMB_TRY(Route(q, a));
      if (!s.f32 && slots.tile_rows > kGatherRows) TMB_TRY(GatherRows(q, plan->normed, W8, slots, plan->gathered));
      const int stride = padded_columns(mlp.ff);
      const Glu glu{float(mlp.limit), float(mlp.alpha), float(mlp.shift), false};
      LinearArgs up = linear(plan->normed, layer.expert_up, -1, maps ? &maps->gate_up : nullptr, mlp.ff, W, plan->expert_hidden, stride, kLinearExpertUp);
      up.slots = slots;
      if (mlp.output_weighted) {
        up.n = mlp.packed_rows();
        up.epilogue = s.f32 ? kLinearExpertStore : kLinearExpertGlu;
        up.outputs = mlp.ff;
        up.glu = glu;
        if (s.f32) {
          up.out = plan->expert_pairs;
          up.out_stride = up.n;
        }
      }
      TMB_TRY(Linear(q, up));
      if (mlp.output_weighted && s.f32) TMB_TRY(GluRows(q, plan->expert_pairs, plan->expert_hidden, slots.slots, up.n, stride, mlp.ff, glu));
      LinearArgs down = linear(plan->expert_hidden, layer.expert_down, -1, maps ? &maps->down : nullptr, W, mlp.ff, plan->expert_out, W, kLinearExpertDown);
      down.slots = slots;
      TMB_TRY(Linear(q, down));
      if (norm_output) TMB_TRY(add_norm(layer.norm2, mlp.top));
      if (mlp.shared_ff) {
        const Glu unit{float(mlp.shared_limit), float(mlp.alpha), float(mlp.shift), false};
        const int packed = mlp.shared_rows(), unit_stride = padded_columns(mlp.shared_ff);
        LinearArgs first = linear(plan->normed, layer.shared_up, -1, maps ? &maps->shared_up : nullptr, packed, W, s.f32 ? plan->pairs : plan->mlp,
                                  s.f32 ? packed : unit_stride, s.f32 ? kLinearStore : kLinearGlu);
        first.outputs = mlp.shared_ff;
        first.glu = unit;
        TMB_TRY(Linear(q, first));
        if (s.f32) TMB_TRY(GluRows(q, plan->pairs, plan->mlp, r.rows, packed, unit_stride, mlp.shared_ff, unit));
        TMB_TRY(add_output(plan->mlp, layer.shared_down, -1, maps ? &maps->shared_down : nullptr, mlp.shared_ff));
      }
      if (s.combined) TMB_TRY(leave(&layer.streams[1], &mlp));
    }
    if (s.parallel) {
      TMB_TRY(add_sublayers(layer, maps));
    } else if (kept && !s.combined) {
      const cudaError_t err = cudaMemcpyAsync(kept, x, size_t(rows) * W * sizeof(float),
                                              cudaMemcpyDeviceToDevice, stream);
      if (err != cudaSuccess) return int(err);
    }
  }
  if (s.parallel && s.write_residuals) {       // (the norm is not read)
    TMB_TRY(conv_norm(s.final_norm, nullptr, nullptr, nullptr, r.rows, plan->normed));
    TMB_TRY(keep_stream(s.runs.size() - 1));
  }
  if (wanted) {
    const int* select = static_cast<const int*>(buffer(s.wanted));
    if (s.parallel) {
      TMB_TRY(conv_norm(s.final_norm, nullptr, nullptr, select, int(wanted), plan->picked));
    } else if (s.combined) {
      StreamArgs a = step;
      a.rows = int(wanted);
      a.weight = floats(s.final_norm);
      a.normed = plan->picked;
      a.select = select;
      TMB_TRY(StreamStep(q, a));
    } else {
      NormArgs a{};
      a.x = x;
      a.weight = floats(s.final_norm);
      a.out = plan->picked;
      a.select = select;
      a.rows = int(wanted);
      a.width = W;
      a.out_stride = W8;
      a.limit = r.rows;
      a.eps = float(s.eps);
      TMB_TRY(RmsNorm(q, a));
    }
    LinearArgs h = linear(plan->picked, s.head, -1, s.f32 ? nullptr : &plan->head, s.vocab, W, buffer(s.logits), s.vocab, kLinearFloat);
    h.t = int(wanted);
    h.gain = float(s.logit_scale);
    TMB_TRY(Linear(q, h));
    TMB_TRY(ArgMax(q, floats(s.logits), int(wanted), s.vocab, static_cast<int*>(buffer(s.next))));
    if (feed)
      TMB_TRY(Feed(q, static_cast<Entry*>(buffer(s.entries)), int(entries), static_cast<const int*>(buffer(s.next)),
                   static_cast<int*>(buffer(s.tokens)), s.capacity));
  }
#undef TMB_TRY
  return 0;
}

}  // namespace

RaggedPlan* RaggedCreate(const RaggedSpec& spec, const std::vector<void*>& buffers, int sm_count, std::string* error) {
  auto plan = new RaggedPlan;
  plan->spec = spec;
  plan->buffers = buffers;
  auto fail = [&](const char* what) -> RaggedPlan* {
    *error = what;
    RaggedDestroy(plan);
    return nullptr;
  };
  const size_t element = spec.f32 ? 4 : 2;
  size_t proj = 0, mixed = 0, mlp = 0, pairs = 0, raw = 0, split = 0, heads = 1, partial = 0, query_latent = 0, queries = 0, decays = 0, chunks = 0;
  size_t top = 0, experts = 0, expert_columns = 0, expert_pairs = 0, source = 0, latent = 0, ranks = 0, context = 0, expanded = 0;
  int reach = 0;
  for (const RaggedLayer& layer : spec.layers) {
    const RaggedMixer& m = layer.mixer;
    proj = std::max(proj, size_t(m.proj_rows() + 7) / 8 * 8);
    mixed = std::max(mixed, size_t(padded_columns(m.out_columns())));
    if (m.value_mix == RaggedMixer::kSource) {
      source = size_t(m.proj_rows() + 7) / 8 * 8;
      plan->source_stride = int(source);
      plan->source_at = (m.heads + m.kv_heads) * m.dim;
    }
    if (layer.mlp.kind == RaggedMlp::kGlu) {
      mlp = std::max(mlp, size_t(padded_columns(layer.mlp.ff)));
      pairs = std::max(pairs, size_t(layer.mlp.packed_rows()));
    } else if (layer.mlp.kind == RaggedMlp::kExperts) {
      top = std::max(top, size_t(layer.mlp.top));
      experts = std::max(experts, size_t(layer.mlp.logits()));
      expert_columns = std::max(expert_columns, size_t(padded_columns(layer.mlp.ff)));
      if (layer.mlp.output_weighted) {
        ranks = std::max(ranks, size_t(layer.mlp.experts));
        expert_pairs = std::max(expert_pairs, size_t(layer.mlp.packed_rows()));
      }
      if (layer.mlp.shared_ff) {
        mlp = std::max(mlp, size_t(padded_columns(layer.mlp.shared_ff)));
        pairs = std::max(pairs, size_t(layer.mlp.shared_rows()));
      }
    }
    if (m.kind == RaggedMixer::kRetention) {
      raw = std::max(raw, size_t(m.out_columns()));
      split = std::max(split, size_t(m.heads) * 4 * m.pool_dim());
    } else if (m.kind == RaggedMixer::kDelta) {
      raw = std::max(raw, size_t(m.out_columns()));
      decays = std::max(decays, size_t(m.out_columns()));
      chunks = std::max(chunks, DeltaChunkBytes(spec.max_rows, spec.slots, m.heads, m.dim));
    } else {
      const size_t columns = m.kind == RaggedMixer::kLatent ? size_t(m.rank_stride()) : size_t(m.vdim);
      heads = std::max(heads, size_t(m.heads));
      // (latent attention fills an SM with one or two CTAs: a fourth of the parts)
      partial = std::max(partial, size_t(m.heads) * (columns + 2) / (m.kind == RaggedMixer::kLatent ? 4 : 1));
      if (m.kind == RaggedMixer::kLatent) {
        latent = std::max(latent, size_t(m.heads) * m.rank_stride());
        if (m.q_rank) {
          query_latent = std::max(query_latent, size_t(padded_columns(m.q_rank)));
          queries = std::max(queries, size_t(m.heads) * m.head_stride());
        }
        context = std::max(context, size_t(m.rank_stride()));
        expanded = std::max(expanded, size_t(m.expanded_columns()));
        reach = std::max(reach, std::min(m.window, spec.capacity));
      }
    }
  }
  const size_t rows = size_t(spec.max_rows), W8 = size_t(padded_columns(spec.width)), slots = rows * top;
  if (context && !spec.f32) plan->context_rows = int(std::min(size_t(spec.max_rows) + 2 * size_t(reach), size_t(spec.slots) * spec.capacity + spec.max_rows));
  const size_t context_rows = size_t(plan->context_rows);
  plan->count_words = int(heads) * spec.slots;
  // a decode step cuts a long window into parts: at most eight CTAs per SM's worth of parts in all, one per head at least
  plan->part_floats = partial * (size_t(spec.slots) + 8 * size_t(sm_count));
  if (!Own(plan, &plan->normed, rows * W8 * element) || !Own(plan, &plan->picked, size_t(spec.max_wanted) * W8 * element) ||
      !Own(plan, &plan->proj, rows * proj * element) || !Own(plan, &plan->mixed, rows * mixed * element) ||
      !Own(plan, &plan->mlp, rows * mlp * element) || !Own(plan, &plan->pairs, spec.f32 ? rows * pairs * element : 0) ||
      !Own(plan, &plan->branch, spec.layers[0].norm_output || spec.combined || spec.parallel ? rows * size_t(spec.width) * sizeof(float) : 0) ||
      !Own(plan, &plan->other, spec.side_dim ? rows * size_t(spec.width) * sizeof(float) : 0) || !Own(plan, &plan->elements, spec.side_dim ? rows * W8 * element : 0) ||
      !Own(plan, &plan->convolved, spec.taps ? rows * W8 * element : 0) ||
      !Own(plan, &plan->side_hidden, spec.side_dim ? rows * size_t(padded_columns(spec.side_dim)) * element : 0) ||
      !Own(plan, &plan->side_out, spec.side_dim ? rows * size_t(spec.width) * sizeof(float) : 0) ||
      !Own(plan, &plan->query_latent, rows * query_latent * element) || !Own(plan, &plan->queries, rows * queries * element) ||
      !Own(plan, &plan->decay_in, rows * decays * sizeof(float)) || !Own(plan, &plan->chunks, spec.f32 ? 0 : chunks) ||
      !Own(plan, &plan->context, context_rows * context * element) || !Own(plan, &plan->expanded, context_rows * expanded * element) ||
      !Own(plan, &plan->context_at, size_t(spec.slots) * sizeof(int)) || !Own(plan, &plan->context_count, sizeof(int)) ||
      !Own(plan, &plan->source, rows * source * element) || !Own(plan, &plan->lookup, rows * latent * element) ||
      !Own(plan, &plan->looked, rows * latent * element) || !Own(plan, &plan->ranks, rows * ranks * sizeof(float)) ||
      !Own(plan, &plan->expert_pairs, spec.f32 ? slots * expert_pairs * element : 0) ||
      !Own(plan, &plan->logits, rows * experts * sizeof(float)) || !Own(plan, &plan->choice, slots * sizeof(int)) ||
      !Own(plan, &plan->list, slots * sizeof(int)) || !Own(plan, &plan->tile_count, sizeof(int)) ||
      !Own(plan, &plan->score, slots * sizeof(float)) || !Own(plan, &plan->slot_score, slots * sizeof(float)) ||
      !Own(plan, &plan->tiles, (slots / 16 + experts) * sizeof(ExpertTile)) || !Own(plan, &plan->route_count, kRouteCounters * sizeof(unsigned)) ||
      !Own(plan, &plan->gathered, spec.f32 ? 0 : slots * W8 * element) ||
      !Own(plan, &plan->expert_hidden, slots * expert_columns * element) || !Own(plan, &plan->expert_out, slots * size_t(spec.width) * element) ||
      !Own(plan, &plan->raw, rows * raw * sizeof(float)) || !Own(plan, &plan->split, spec.f32 ? 0 : rows * split * 2) ||
      !Own(plan, &plan->part, plan->part_floats * sizeof(float)) ||
      !Own(plan, &plan->count, size_t(plan->count_words) * sizeof(unsigned)) || !Own(plan, &plan->queue.status, 64) ||
      !Own(plan, &plan->rows.row_entry, rows * sizeof(int)) || !Own(plan, &plan->rows.row_position, rows * sizeof(int)) ||
      !Own(plan, &plan->rows.row_kv, rows * sizeof(int)))
    return fail("no device memory for the step's activations");
  plan->decay.assign(spec.layers.size(), nullptr);
  for (size_t i = 0; i < spec.layers.size(); ++i) {
    const std::vector<float>& decay = spec.layers[i].mixer.decay;
    if (decay.empty()) continue;
    if (!Own(plan, &plan->decay[i], decay.size() * sizeof(float)) ||
        cudaMemcpy(plan->decay[i], decay.data(), decay.size() * sizeof(float), cudaMemcpyHostToDevice) != cudaSuccess)
      return fail("no device memory for the decays");
  }
  plan->queue.f32 = spec.f32;
  plan->queue.sm_count = sm_count;
  // TILEMEGA_RAGGED_CHAIN=0: plain launches (each kernel starts when the one before it has ended)
  const char* chain = std::getenv("TILEMEGA_RAGGED_CHAIN");
  plan->queue.chained = !(chain && chain[0] == '0');
  StepRows& r = plan->rows;
  r.entry = static_cast<const Entry*>(buffers[size_t(spec.entries)]);
  r.block_table = static_cast<const int*>(buffers[size_t(spec.block_table)]);
  r.max_blocks = spec.max_blocks;
  r.num_blocks = spec.num_blocks;
  r.capacity = spec.capacity;
  r.slots = spec.slots;
  if (!spec.f32) {
    if (!TensorMapEncoder()) return fail("the driver does not offer cuTensorMapEncodeTiled");
    plan->maps.resize(spec.layers.size());
    auto at = [&](int index) { return buffers[size_t(index)]; };
    for (size_t i = 0; i < spec.layers.size(); ++i) {
      const RaggedLayer& layer = spec.layers[i];
      const RaggedMixer& m = layer.mixer;
      RaggedPlan::Maps& maps = plan->maps[i];
      bool ok = EncodeLinear(&maps.in, at(layer.in_weight), uint64_t(m.proj_rows()), spec.taps ? plan->convolved : plan->normed, rows, W8) &&
                EncodeLinear(&maps.out, at(layer.out_weight), uint64_t(spec.width), plan->mixed, rows, uint64_t(padded_columns(m.out_columns())));
      const RaggedMlp& mlp = layer.mlp;
      if (m.kind == RaggedMixer::kLatent)
        ok = ok && EncodeLookup(&maps.lookup, plan->lookup, rows * m.heads, uint64_t(m.rank_stride())) &&
             EncodeHeads(&maps.key_up, at(layer.key_up), uint64_t(m.heads) * m.rank_stride(), uint64_t(m.head_stride()),
                         m.q_rank ? plan->queries : plan->proj, rows, m.q_rank ? uint64_t(m.heads) * m.head_stride() : uint64_t(m.proj_rows() + 7) / 8 * 8) &&
             EncodeHeads(&maps.value_up, at(layer.value_up), uint64_t(m.heads) * m.vdim, uint64_t(m.rank_stride()), plan->looked, rows,
                         uint64_t(m.heads) * m.rank_stride()) &&
             EncodeLinear(&maps.expand, at(layer.expand), uint64_t(m.expanded_columns()), plan->context, context_rows, uint64_t(m.rank_stride()));
      if (m.q_rank)
        ok = ok && EncodeLinear(&maps.query_up, at(layer.query_up), uint64_t(m.heads) * m.head_stride(), plan->query_latent, rows, uint64_t(padded_columns(m.q_rank)));
      if (m.kind == RaggedMixer::kDelta)
        ok = ok && EncodeHeads(&maps.decay_up, at(layer.decay_up), uint64_t(m.out_columns()), uint64_t(padded_columns(m.decay_rank)), plan->proj, rows,
                               uint64_t(m.proj_rows() + 7) / 8 * 8);
      if (spec.side_dim)
        ok = ok && EncodeLinear(&maps.side_gate, at(layer.side.gate), uint64_t(spec.side_dim), plan->elements, rows, W8) &&
             EncodeLinear(&maps.side_proj, at(layer.side.proj), uint64_t(spec.width), plan->side_hidden, rows, uint64_t(padded_columns(spec.side_dim)));
      if (mlp.kind == RaggedMlp::kExperts)
        ok = ok && EncodeLinear(&maps.router, at(layer.router), uint64_t(mlp.logits()), plan->normed, rows, W8) &&
             EncodeLinear(&maps.gate_up, at(layer.expert_up), uint64_t(mlp.experts) * (mlp.output_weighted ? mlp.packed_rows() : mlp.ff), plan->gathered,
                          slots, W8) &&
             EncodeGathered(&maps.gate_up, plan->normed, rows, W8) &&
             EncodeLinear(&maps.down, at(layer.expert_down), uint64_t(mlp.experts) * spec.width, plan->expert_hidden, slots,
                          uint64_t(padded_columns(mlp.ff)));
      if (mlp.shared_ff)
        ok = ok && EncodeLinear(&maps.shared_up, at(layer.shared_up), uint64_t(mlp.shared_rows()), plan->normed, rows, W8) &&
             EncodeLinear(&maps.shared_down, at(layer.shared_down), uint64_t(spec.width), plan->mlp, rows, uint64_t(padded_columns(mlp.shared_ff)));
      if (mlp.kind == RaggedMlp::kGlu)
        ok = ok && EncodeLinear(&maps.gate_up, at(layer.gate_up), uint64_t(mlp.packed_rows()), plan->normed, rows, W8) &&
             EncodeLinear(&maps.down, at(layer.down), uint64_t(spec.width), plan->mlp, rows, uint64_t(padded_columns(mlp.ff)));
      if (!ok) return fail("cuTensorMapEncodeTiled rejected a layer's buffers");
    }
    plan->latent.resize(spec.runs.size());
    for (size_t i = 0; i < spec.runs.size(); ++i) {
      const RaggedMixer& m = spec.layers[size_t(spec.runs[i].layer)].mixer;
      if (m.kind == RaggedMixer::kLatent &&
          !EncodeLatent(&plan->latent[i], at(spec.runs[i].k_pool), uint64_t(spec.num_blocks) * kRaggedBlock, uint64_t(m.pool_dim())))
        return fail("cuTensorMapEncodeTiled rejected a pool of latent rows");
    }
    if (!EncodeLinear(&plan->head, at(spec.head), uint64_t(spec.vocab), plan->picked, uint64_t(spec.max_wanted), W8))
      return fail("cuTensorMapEncodeTiled rejected the head");
  }
  if (PrepareLinear() != 0 || PrepareMixers() != 0 || PrepareLatent() != 0 || PrepareConv() != 0 || PrepareDelta() != 0) return fail("cannot raise the kernels' shared-memory limit");
  return plan;
}

int RaggedLaunch(RaggedPlan* plan, uint32_t entries, uint32_t rows, uint32_t longest, uint32_t singles, uint32_t wanted, bool feed,
                 cudaStream_t stream) {
  const bool decode = singles == entries && !plan->spec.write_residuals;
  if (!decode) return Enqueue(plan, entries, rows, longest, singles, wanted, feed, stream);
  // A decode step's launches depend on its counts only: the second step of a kind is recorded and replayed from then on.
  const auto key = std::make_tuple(entries, wanted, feed);
  auto found = plan->graphs.find(key);
  if (found == plan->graphs.end()) {
    if (plan->seen[key]++ == 0) return Enqueue(plan, entries, rows, longest, singles, wanted, feed, stream);
    cudaStream_t recorder = nullptr;
    cudaGraph_t graph = nullptr;
    cudaGraphExec_t exec = nullptr;
    cudaError_t err = cudaStreamCreateWithFlags(&recorder, cudaStreamNonBlocking);
    if (err != cudaSuccess) return int(err);
    err = cudaStreamBeginCapture(recorder, cudaStreamCaptureModeThreadLocal);
    if (err == cudaSuccess) {
      const int status = Enqueue(plan, entries, rows, longest, singles, wanted, feed, recorder);
      err = cudaStreamEndCapture(recorder, &graph);
      if (status != 0) err = cudaError_t(status);
    }
    if (err == cudaSuccess) err = cudaGraphInstantiate(&exec, graph, 0);
    if (graph) cudaGraphDestroy(graph);
    cudaStreamDestroy(recorder);
    if (err != cudaSuccess) return int(err);
    found = plan->graphs.emplace(key, exec).first;
  }
  return int(cudaGraphLaunch(found->second, stream));
}

int RaggedStatus(RaggedPlan* plan, uint64_t* record12) {
  unsigned words[4] = {0, 0, 0, 0};
  if (cudaMemcpy(words, plan->queue.status, sizeof(words), cudaMemcpyDeviceToHost) != cudaSuccess) return -1;
  if (record12) {
    for (int i = 0; i < 12; ++i) record12[i] = 0;
    record12[0] = words[0];
  }
  return words[0] ? 1 : 0;
}

void RaggedClear(RaggedPlan* plan) { cudaMemset(plan->queue.status, 0, 64); }

void RaggedDestroy(RaggedPlan* plan) {
  if (!plan) return;
  for (auto& item : plan->graphs) cudaGraphExecDestroy(item.second);
  for (void* p : plan->owned) cudaFree(p);
  delete plan;
}

}  // namespace tmb
