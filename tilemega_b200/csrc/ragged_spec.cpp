#include "ragged_spec.h"

#include <algorithm>
#include <stdexcept>
#include <string>

#include "plan_spec.h"
#include "ragged_limits.h"

namespace tmb {
namespace {

void Require(bool condition, const std::string& message) {
  if (!condition) throw std::invalid_argument(message);
}

std::string Quoted(const Json& names, std::initializer_list<const char*> keys) {
  std::string out = "[";
  bool first = true;
  for (const char* key : keys) {
    Require(names.has(key) && names.at(key).kind == Json::kString, std::string("a layer names no tensor for '") + key + "'");
    out += (first ? "" : ",") + Json::Quote(names.at(key).text);
    first = false;
  }
  return out + "]";
}

std::string Name(const Json& object, const char* key) {
  const std::string name = object.str(key, "");
  Require(!name.empty(), std::string("the model names no tensor for '") + key + "'");
  return name;
}

std::string AliasRecipe(const std::string& name) { return "{\"kind\":\"alias\",\"source\":" + Json::Quote(name) + "}"; }

std::string OffsetRecipe(const std::string& name, double offset) {
  return offset == 0 ? AliasRecipe(name) : "{\"kind\":\"offset\",\"value\":" + std::to_string(offset) + ",\"source\":" + Json::Quote(name) + "}";
}

// Recipes one under the other, each a JSON object or a quoted tensor name.
std::string Stack(const std::vector<std::string>& recipes) {
  std::string out = "{\"kind\":\"stack\",\"sources\":[";
  for (size_t i = 0; i < recipes.size(); ++i) out += (i ? "," : "") + recipes[i];
  return out + "]}";
}
std::string PadColumns(const std::string& recipe, int columns) {
  return "{\"kind\":\"pad_columns\",\"columns\":" + std::to_string(columns) + ",\"source\":" + recipe + "}";
}
std::string PerHead(const char* kind, const std::string& recipe, int heads, const char* key, int value) {
  return "{\"kind\":\"" + std::string(kind) + "\",\"heads\":" + std::to_string(heads) + ",\"" + key + "\":" + std::to_string(value) +
         ",\"source\":" + recipe + "}";
}
std::string GluRecipe(const std::string& gate, const std::string& up) {
  return "{\"kind\":\"gate_up_interleave\",\"pad\":true,\"u\":" + std::to_string(kGluUnit) + ",\"sources\":[" + gate + "," + up + "]}";
}

// Every head's matrix with an identity of `size` behind its rows and columns.
std::string WithIdentity(const std::string& recipe, int heads, int size) { return size ? PerHead("append_identity", recipe, heads, "size", size) : recipe; }
// Heads whose last `dims` rows are rotated: these as neighbours behind `lead` rows for the others, zero rows up to `rows`.
std::string RotaryTail(const std::string& recipe, int heads, int dims, bool neighbours, int lead, int rows) {
  return "{\"kind\":\"rotary_tail\",\"heads\":" + std::to_string(heads) + ",\"dims\":" + std::to_string(dims) + ",\"layout\":\"" +
         (neighbours ? "pairs" : "halves") + "\",\"lead\":" + std::to_string(lead) + ",\"rows\":" + std::to_string(rows) + ",\"source\":" + recipe + "}";
}
// A vector between zeros.
std::string Between(const std::string& name, int before, int behind) {
  return "{\"kind\":\"pad_vector\",\"before\":" + std::to_string(before) + ",\"behind\":" + std::to_string(behind) + ",\"source\":" + Json::Quote(name) + "}";
}

std::string QuotedList(const Json& names, const char* key, int count) {
  Require(names.has(key) && names.at(key).kind == Json::kArray && int(names.at(key).items.size()) == count,
          std::string("a layer needs one tensor per expert for '") + key + "'");
  std::string out = "[";
  for (const Json& name : names.at(key).items) out += (out.size() > 1 ? "," : "") + Json::Quote(name.text);
  return out + "]";
}

// Matrices stacked by rows, each row zero-padded to `columns`.
std::string StackRecipe(const std::string& sources, int columns) {
  return "{\"kind\":\"pad_columns\",\"columns\":" + std::to_string(columns) + ",\"source\":{\"kind\":\"stack_rows\",\"sources\":" + sources + "}}";
}

}  // namespace

RaggedSpec RaggedSpec::FromJson(const Json& plan, std::vector<BufferSpec>* buffers) {
  RaggedSpec s;
  const Json& model = plan.at("model");
  const std::string dtype = plan.str("dtype", "bf16");
  Require(dtype == "bf16" || dtype == "f32", "a ragged plan computes in bf16 or f32 (dtype)");
  s.f32 = dtype == "f32";
  s.width = int(model.integer("width", 0));
  s.vocab = int(model.integer("vocab", 0));
  s.eps = model.num("eps", -1);
  s.streams = int(model.integer("streams", 1));
  const double offset = model.num("norm_offset", 0);   // added to the stored weights of the residual norms
  s.slots = int(plan.integer("batch_hi", 0));
  s.capacity = int(plan.integer("capacity", 0));
  s.max_rows = int(plan.integer("max_rows", 0));
  s.max_wanted = int(plan.integer("max_wanted", 0));
  s.write_residuals = plan.flag("write_residuals", false);
  s.num_blocks = int(plan.at("kv").integer("num_blocks", 0));
  s.max_blocks = (s.capacity + kRaggedBlock - 1) / kRaggedBlock;
  Require(s.width > 0 && s.vocab > 0 && s.eps >= 0, "width, vocab and eps must be given");
  Require(s.slots >= 1 && s.slots <= 4096, "a ragged plan has 1..4096 sequence slots (batch_hi)");
  Require(s.capacity >= kRaggedBlock && s.capacity % kRaggedBlock == 0, "capacity must be a positive multiple of 16");
  Require(s.max_rows >= 1 && s.max_rows <= 65535, "max_rows must lie in [1, 65535]");
  Require(s.max_wanted >= 1 && s.max_wanted <= 65535, "max_wanted must lie in [1, 65535]");
  Require(s.num_blocks >= 1, "kv.num_blocks must be positive");
  Require(s.streams >= 1 && s.streams <= kMaxStreams, "a model has 1..16 residual streams");
  s.combined = s.streams > 1;
  s.parallel = model.str("form", "sequential") == "parallel";
  s.norm_groups = int(model.integer("norm_groups", 1));
  s.taps = int(model.integer("taps", 0));
  s.residual_mult = model.num("residual_mult", 1);
  s.embed_scale = model.num("embed_scale", 1);
  s.logit_scale = model.num("logit_scale", 1);
  Require(s.norm_groups >= 1 && s.width % s.norm_groups == 0, "the norms' groups are equal runs of columns");
  Require(s.taps >= 0 && s.taps <= kMaxTaps, "a short convolution has 1..16 taps");
  Require(s.parallel || (s.norm_groups == 1 && s.taps == 0 && s.residual_mult == 1 && s.embed_scale == 1 && !model.has("side")),
          "grouped norms, short convolutions, factors of the residual and side inputs are built for parallel layers");
  Require(!s.parallel || (s.streams == 1 && s.width <= kMaxConvWidth && std::max(0, s.taps - 1) * s.width <= 40 * 1024 && offset == 0),
          "parallel layers have one stream of at most 8192 columns, and at most 40960 values of a convolution's history");
  if (!s.parallel) for (const Json& in : model.at("layers").items) {
    if (in.has("streams")) s.combined = true;
    if (in.has("mlp") && in.at("mlp").str("weighted", "") == "output") s.combined = true;
  }

  const uint32_t element = s.f32 ? 1u : 0u;
  const uint64_t element_bytes = s.f32 ? 4 : 2;
  auto add = [&](const std::string& name, uint32_t role, uint32_t type, uint64_t constant, uint64_t per_batch, const std::string& recipe) {
    BufferSpec b;
    b.name = name;
    b.role = role;
    b.dtype = type;
    b.elements_constant = constant;
    b.elements_per_batch = per_batch;
    b.pack_json = recipe;
    buffers->push_back(b);
    return int(buffers->size()) - 1;
  };
  auto matrix = [&](const std::string& name, const std::string& recipe, int rows, int columns) {
    return add(name, 1, element, uint64_t(rows) * padded_columns(columns), 0, recipe);
  };
  const uint64_t W = uint64_t(s.width);
  s.tokens = add("step.tokens", 1, 2, uint64_t(s.max_rows), 0, "");
  s.entries = add("step.entries", 1, 2, 0, 4, "");
  s.wanted = add("step.wanted", 1, 2, uint64_t(s.max_wanted), 0, "");
  s.block_table = add("serving.block_table", 1, 2, 0, uint64_t(s.max_blocks), "");
  s.logits = add("step.logits", 1, 1, uint64_t(s.max_wanted) * s.vocab, 0, "");
  s.next = add("step.next", 1, 2, uint64_t(s.max_wanted), 0, "");
  s.hidden = add("step.hidden", 0, 1, uint64_t(s.max_rows) * s.streams * W, 0, "");
  s.embed = add("embed", 1, element, uint64_t(s.vocab) * W, 0, AliasRecipe(Name(model, "embed")));
  if (model.has("side") && model.at("side").kind == Json::kObject) {
    s.side_dim = int(model.at("side").integer("dim", 0));
    s.side_columns = s.side_dim * int(model.at("layers").items.size());
    Require(s.side_dim >= 1, "a layer's part of the second embedding has at least one column");
    s.side_embed = add("side.embed", 1, element, uint64_t(s.vocab) * s.side_columns, 0, AliasRecipe(Name(model.at("side"), "embed")));
  }

  Require(model.at("layers").kind == Json::kArray && !model.at("layers").items.empty(), "the model has no layers");
  for (size_t i = 0; i < model.at("layers").items.size(); ++i) {
    const Json& in = model.at("layers").items[i];
    const std::string p = "l" + std::to_string(i) + ".";
    RaggedLayer layer;
    RaggedMixer& m = layer.mixer;
    const Json& mixer = in.at("mixer");
    const Json& names = mixer.at("tensors");
    const std::string kind = mixer.str("kind", "");
    Require(kind == "attention" || kind == "retention" || kind == "latent" || kind == "delta", "unknown kind of mixer '" + kind + "'");
    m.kind = kind == "retention" ? RaggedMixer::kRetention : kind == "latent" ? RaggedMixer::kLatent : kind == "delta" ? RaggedMixer::kDelta : RaggedMixer::kAttention;
    m.heads = int(mixer.integer("heads", 0));
    m.kv_heads = int(mixer.integer("kv_heads", m.heads));
    m.dim = int(mixer.integer("dim", 0));
    m.vdim = int(mixer.integer("vdim", m.dim));
    Require(m.heads > 0 && m.kv_heads > 0 && m.heads % m.kv_heads == 0, "heads must be a positive multiple of kv_heads");
    Require(m.dim >= 1 && m.dim <= kMaxHeadDim && m.vdim >= 1, "head sizes must lie in [1, 256]");
    if (mixer.has("rotary") && mixer.at("rotary").kind == Json::kObject) {
      const Json& rot = mixer.at("rotary");
      const double base = rot.num("base", 0);
      const double factor = rot.num("factor", 1);
      m.rot_dims = int(rot.integer("dims", 0));
      Require(factor > 0, "the rotary scaling factor must be positive");
      Require(base > 0 && m.rot_dims >= 0 && m.rot_dims % 2 == 0 && (m.rot_dims <= m.dim || m.kind == RaggedMixer::kLatent),
              "rotary dims must be even and at most the head size");
      if (m.rot_dims) {
        RotaryTable table;
        if (rot.has("yarn") && rot.at("yarn").kind == Json::kObject) {
          const char* keys[4] = {"factor", "original", "fast", "slow"};
          for (int i = 0; i < 4; ++i) {
            table.yarn[i] = rot.at("yarn").num(keys[i], 0);
            Require(table.yarn[i] > 0, "a rotation's length scaling has a positive factor, original length and turns");
          }
        }
        for (size_t r = 0; r < s.rotaries.size(); ++r)
          if (s.rotaries[r].base == base && s.rotaries[r].dims == m.rot_dims && s.rotaries[r].factor == factor &&
              std::equal(table.yarn, table.yarn + 4, s.rotaries[r].yarn))
            m.rotary = int(r);
        if (m.rotary < 0) {
          table.base = base;
          table.factor = factor;
          table.dims = m.rot_dims;
          m.rotary = int(s.rotaries.size());
          table.buffer = add("rotary." + std::to_string(m.rotary), 1, 1, uint64_t(s.capacity) * m.rot_dims, 0, "");
          s.rotaries.push_back(table);
        }
      }
    }
    std::string stacked;                 // recipe of the input projection
    const bool bias = mixer.flag("bias", false);
    const bool neighbours = m.rot_dims && mixer.at("rotary").str("layout", "halves") == "pairs";
    const bool pairs = m.kind != RaggedMixer::kLatent && neighbours;   // (latent attention turns neighbours where they are)
    // entries 2i and 2i + 1 of a head turn together: stored as i and i + dims/2, in queries and keys alike
    auto arranged = [&](const std::string& name, int heads) {
      return pairs ? PerHead("pairs_to_halves", name, heads, "dims", m.rot_dims) : name;
    };
    auto masked = [&]() {
      const Json none;
      const Json& mask = mixer.has("mask") && mixer.at("mask").kind == Json::kObject ? mixer.at("mask") : none;
      m.window = int(std::min<long long>(mask.integer("size", s.capacity), s.capacity));   // no window: everything before
      m.keep = int(std::min<long long>(mask.integer("keep_first", 0), s.capacity));
      m.scale = mixer.num("scale", 0);
      Require(m.window >= 1 && m.keep >= 0, "a window holds at least one position");
    };
    if (names.has("sink")) layer.sinks = add(p + "sinks", 1, 1, uint64_t(m.heads), 0, AliasRecipe(Name(names, "sink")));
    if (m.kind == RaggedMixer::kRetention) {
      Require(m.kv_heads == m.heads, "retention has one key and value head per query head");
      Require(m.vdim <= 4096 && !bias, "retention value heads are at most 4096 wide and its projections have no biases");
      Require(mixer.at("decay").kind == Json::kArray && int(mixer.at("decay").items.size()) == m.heads, "retention needs one decay per head");
      for (const Json& d : mixer.at("decay").items) m.decay.push_back(float(d.number));
      Require(!pairs, "retention turns the halves of a head");
      stacked = "{\"kind\":\"stack_rows\",\"sources\":" + Quoted(names, {"q", "k", "v", "g"}) + "}";
    } else if (m.kind == RaggedMixer::kLatent) {
      m.rank = int(mixer.integer("rank", 0));
      m.q_rank = int(mixer.integer("q_rank", 0));
      Require(m.kv_heads == m.heads && !bias, "latent attention has a key and a value per head and no biases");
      Require(m.rotary < 0 || m.q_rank > 0, "latent attention turns queries that are images of a row of their own (q_rank)");
      Require(m.vdim <= kMaxHeadDim && m.head_key() <= kMaxHeadDim, "head sizes must lie in [1, 256]");
      Require(m.rank >= 1 && m.columns() <= kMaxLatent, "a latent row has 1..1024 columns (rank, rotated ones)");
      masked();
      Require(m.keep == 0, "latent attention keeps no first positions");
      const std::string row = RotaryTail(Json::Quote(Name(names, "dkv")), 1, m.rot_dims, neighbours, m.rank, m.columns());
      if (m.q_rank)
        stacked = Stack({PerHead("pad_heads", Json::Quote(Name(names, "dq")), 1, "rows", m.latent_at()), row});
      else
        stacked = Stack({PerHead("pad_heads", Json::Quote(Name(names, "q")), m.heads, "rows", m.head_stride()), Json::Quote(Name(names, "dkv"))});
    } else if (m.kind == RaggedMixer::kDelta) {
      m.decay_rank = int(mixer.integer("decay_rank", 0));
      m.decay_scale = mixer.num("decay_scale", 0);
      m.unit_eps = mixer.num("unit_eps", 0);
      Require(m.kv_heads == m.heads && m.vdim == m.dim && m.rotary < 0, "a delta rule has a key and a value of one size per head and no rotation");
      Require(s.f32 || m.decay_scale <= kMostDecay, "a bf16 plan's delta rule forgets at most a factor of e^4 per token (decay_scale)");
      Require(m.decay_rank >= 1 && m.decay_scale > 0 && m.unit_eps > 0, "a delta rule needs the size of its decays' row (decay_rank), decay_scale and unit_eps");
      std::vector<std::string> parts = {PerHead("pad_heads", Json::Quote(Name(names, "w1")), 1, "rows", m.delta_at())};
      for (const char* part : {"r", "k", "v", "a", "g"}) parts.push_back(Json::Quote(Name(names, part)));
      stacked = Stack(parts);
    } else {
      m.value_is_key = mixer.str("values", "projected") == "keys";
      Require(m.vdim <= kMaxHeadDim, "head sizes must lie in [1, 256]");
      Require(!m.value_is_key || m.vdim == m.dim, "values that are keys are as wide as keys");
      m.qk_norm = mixer.flag("qk_norm", false);
      m.gate = mixer.flag("gate", false);
      m.sink = mixer.has("sink") && mixer.at("sink").kind == Json::kNumber;
      m.sink_score = mixer.num("sink", 0);
      masked();
      Require(!pairs || !m.value_is_key, "values that are keys take heads whose halves turn");
      std::vector<std::string> parts = {arranged(Json::Quote(Name(names, "q")), m.heads), arranged(Json::Quote(Name(names, "k")), m.kv_heads)};
      if (!m.value_is_key) parts.push_back(Json::Quote(Name(names, "v")));
      if (m.gate) parts.push_back(Json::Quote(Name(names, "g")));
      stacked = Stack(parts);
      const std::string mixing = mixer.str("value_mix", "");
      Require(mixing.empty() || mixing == "source" || mixing == "blend", "unknown way of mixing values");
      m.value_mix = mixing.empty() ? RaggedMixer::kOwn : mixing == "source" ? RaggedMixer::kSource : RaggedMixer::kBlend;
      if (m.value_mix != RaggedMixer::kOwn) {
        Require(!m.value_is_key, "values that are keys are not mixed");
        int sources = 0;
        for (const RaggedLayer& before : s.layers)
          if (before.mixer.value_mix == RaggedMixer::kSource) {
            ++sources;
            Require(before.mixer.kv_heads * before.mixer.vdim == m.kv_heads * m.vdim, "layers that mix values have as many of them");
          }
        Require(sources == (m.value_mix == RaggedMixer::kBlend ? 1 : 0), "values are mixed with those of one layer before");
      }
      if (m.value_mix == RaggedMixer::kBlend) layer.blend = add(p + "blend", 1, 1, 1, 0, AliasRecipe(Name(names, "vmix")));
      Require(!bias || !m.gate, "gated attention has no projection biases");
    }
    const std::string place = in.str("norm_at", "input");
    Require(place == "input" || place == "output", "a layer's norms act on its sublayers' input or output (norm_at)");
    layer.norm_output = place == "output";
    Require(i == 0 || layer.norm_output == s.layers[0].norm_output, "every layer of a model has its norms in the same place");
    Require(!s.parallel || !layer.norm_output, "parallel layers read one norm");
    Require(!s.combined || !layer.norm_output, "layers with norms on their outputs have one stream, and experts with weights on their inputs");
    auto streams = [&](int which) {
      if (!in.has("streams")) {
        Require(s.streams == 1, "every layer of a model with several streams says how its sublayers use them");
        return;
      }
      Require(int(in.at("streams").items.size()) > which, "a layer has stream weights for each of its sublayers");
      const Json& parts = in.at("streams").items[size_t(which)];
      const std::string at = p + "streams" + std::to_string(which + 1) + ".";
      RaggedStreams& out = layer.streams[which];
      out.in = add(at + "in", 1, 1, uint64_t(s.streams), 0, AliasRecipe(Name(parts, "in")));
      out.out = add(at + "out", 1, 1, uint64_t(s.streams), 0, AliasRecipe(Name(parts, "out")));
      out.mix = add(at + "mix", 1, 1, uint64_t(s.streams) * s.streams, 0, AliasRecipe(Name(parts, "mix")));
    };
    streams(0);
    layer.norm1 = add(p + "norm1", 1, 1, W, 0, OffsetRecipe(Name(in, "norm1"), offset));
    layer.in_weight = matrix(p + "in.weight", PadColumns(stacked, padded_columns(s.width)), m.proj_rows(), s.width);
    if (m.kind == RaggedMixer::kLatent) {
      const int rank = m.rank_stride();
      const std::string uk = Json::Quote(Name(names, "uk"));
      layer.latent_norm = add(p + "latent.norm", 1, 1, uint64_t(m.rank), 0, AliasRecipe(Name(names, "dkv.norm")));
      if (m.q_rank) {
        layer.q_latent_norm = add(p + "query.norm", 1, 1, uint64_t(m.q_rank), 0, AliasRecipe(Name(names, "dq.norm")));
        layer.query_up = matrix(p + "query_up.weight",
                                PadColumns(RotaryTail(Json::Quote(Name(names, "uq")), m.heads, m.rot_dims, neighbours, m.head_lead(), m.head_stride()),
                                           padded_columns(m.q_rank)),
                                m.heads * m.head_stride(), m.q_rank);
      }
      // a query against latent rows is its head's key matrix, transposed, times the query, and its rotated part as it is
      std::string key_up = PerHead("transpose_heads", uk, m.heads, "rows", m.dim);
      std::string key = uk;              // a key is the head's key matrix times the normed columns of a latent row, and the rotated ones as they are
      if (m.rot_dims) {
        key_up = WithIdentity(PadColumns(key_up, m.head_lead()), m.heads, m.rot_dims);
        key = WithIdentity(PerHead("pad_heads", uk, m.heads, "rows", m.head_lead()), m.heads, m.rot_dims);
      }
      layer.key_up = add(p + "key_up.weight", 1, element, uint64_t(m.heads) * rank * m.head_stride(), 0,
                         PadColumns(PerHead("pad_heads", key_up, m.heads, "rows", rank), m.head_stride()));
      if (!s.f32)
        layer.expand = add(p + "expand.weight", 1, element, uint64_t(m.expanded_columns()) * rank, 0,
                           PadColumns(Stack({PadColumns(PerHead("pad_heads", key, m.heads, "rows", m.expanded_key()), rank),
                                             PadColumns(PerHead("pad_heads", Json::Quote(Name(names, "uv")), m.heads, "rows", m.v_pool_dim()), rank)}), rank));
      layer.value_up = add(p + "value_up.weight", 1, element, uint64_t(m.heads) * m.vdim * rank, 0,
                           PadColumns(Stack({Json::Quote(Name(names, "uv"))}), rank));
    }
    if (m.kind == RaggedMixer::kDelta) {
      const int all = m.heads * m.dim;
      layer.in_bias = add(p + "in.bias", 1, 1, uint64_t(m.proj_rows()), 0, Between(Name(names, "a.b"), m.delta_at() + 3 * all, all));
      layer.decay_up = matrix(p + "decay_up.weight", PadColumns(Stack({Json::Quote(Name(names, "w2"))}), padded_columns(m.decay_rank)), all, m.decay_rank);
      layer.decay_bias = add(p + "decay.bias", 1, 1, uint64_t(all), 0, AliasRecipe(Name(names, "w0")));
      layer.out_norm = add(p + "out.norm", 1, 1, uint64_t(all), 0, AliasRecipe(Name(names, "norm")));
    }
    if (s.taps) {                        // one row per tap
      layer.conv = add(p + "conv", 1, 1, uint64_t(s.taps) * W, 0, PerHead("transpose_heads", Json::Quote(Name(in, "conv")), 1, "rows", s.width));
    }
    if (s.side_dim) {
      const Json& side = in.at("side");
      layer.side.gate = matrix(p + "side.gate", StackRecipe(Quoted(side, {"gate"}), padded_columns(s.width)), s.side_dim, s.width);
      layer.side.proj = matrix(p + "side.proj", StackRecipe(Quoted(side, {"proj"}), padded_columns(s.side_dim)), s.width, s.side_dim);
      layer.side.norm = add(p + "side.norm", 1, 1, W, 0, AliasRecipe(Name(side, "norm")));
      layer.side.from = int(side.integer("from", -1));
      Require(layer.side.from >= 0 && layer.side.from + s.side_dim <= s.side_columns, "a layer's part lies inside the second embedding");
    }
    layer.out_weight = matrix(p + "out.weight", StackRecipe(Quoted(names, {"o"}), padded_columns(m.out_columns())), s.width, m.out_columns());
    if (m.qk_norm) {
      layer.q_norm = add(p + "q.norm", 1, 1, uint64_t(m.heads) * m.dim, 0, Stack({arranged(Json::Quote(Name(names, "q.norm")), m.heads)}));
      layer.k_norm = add(p + "k.norm", 1, 1, uint64_t(m.kv_heads) * m.dim, 0, Stack({arranged(Json::Quote(Name(names, "k.norm")), m.kv_heads)}));
    }
    if (bias && m.kind == RaggedMixer::kAttention) {
      std::vector<std::string> biases = {arranged(Json::Quote(Name(names, "q.b")), m.heads), arranged(Json::Quote(Name(names, "k.b")), m.kv_heads)};
      if (!m.value_is_key) biases.push_back(Json::Quote(Name(names, "v.b")));
      layer.in_bias = add(p + "in.bias", 1, 1, uint64_t(m.proj_rows()), 0, Stack(biases));
      if (names.has("o.b")) layer.out_bias = add(p + "out.bias", 1, 1, W, 0, AliasRecipe(Name(names, "o.b")));
    }
    if (in.has("mlp") && in.at("mlp").kind == Json::kObject) {
      const Json& mlp = in.at("mlp");
      const Json& parts = mlp.at("tensors");
      const std::string unit = mlp.str("kind", "");
      Require(unit == "glu" || unit == "experts", "unknown kind of feed-forward");
      layer.mlp.kind = unit == "glu" ? RaggedMlp::kGlu : RaggedMlp::kExperts;
      layer.mlp.ff = int(mlp.integer("ff", 0));
      Require(layer.mlp.ff > 0, "the feed-forward width must be positive");
      if (!s.parallel) {
        layer.norm2 = add(p + "norm2", 1, 1, W, 0, OffsetRecipe(Name(in, "norm2"), offset));
        streams(1);
      }
      const std::string activation = mlp.str("activation", "silu");
      if (layer.mlp.kind == RaggedMlp::kGlu) {
        Require(activation == "silu" || activation == "gelu_tanh", "unknown activation of a gated unit");
        layer.mlp.gelu = activation == "gelu_tanh";
        layer.mlp.limit = mlp.num("limit", 3.0e38);
        layer.mlp.alpha = mlp.num("alpha", 1.0);
        layer.mlp.shift = mlp.num("shift", 0.0);
        layer.gate_up = matrix(p + "gate_up.weight",
                               "{\"kind\":\"pad_columns\",\"columns\":" + std::to_string(padded_columns(s.width)) +
                                   ",\"source\":{\"kind\":\"gate_up_interleave\",\"pad\":true,\"u\":" + std::to_string(kGluUnit) +
                                   ",\"sources\":" + Quoted(parts, {"gate", "up"}) + "}}",
                               layer.mlp.packed_rows(), s.width);
        layer.down = matrix(p + "down.weight", StackRecipe(Quoted(parts, {"down"}), padded_columns(layer.mlp.ff)), s.width, layer.mlp.ff);
      } else {
        RaggedMlp& e = layer.mlp;
        e.experts = int(mlp.integer("experts", 0));
        e.top = int(mlp.integer("top", 0));
        Require(e.experts >= 1 && e.experts <= kMaxExperts, "a layer has 1..1024 experts");
        Require(e.top >= 1 && e.top <= e.experts && e.top <= kMaxTop, "a token uses 1..32 of a layer's experts (top)");
        Require(uint64_t(s.max_rows) * e.top <= (1u << 20), "max_rows times the experts of a token is at most 2^20");
        const std::string scores = mlp.str("scores", "");
        e.output_weighted = mlp.str("weighted", "") == "output";
        e.softmax = scores == "softmax";
        e.chosen = scores == "softmax_chosen";
        e.correction = parts.has("correction");
        if (mlp.has("groups") && mlp.at("groups").kind == Json::kObject) {
          e.groups = int(mlp.at("groups").integer("count", 1));
          e.keep_groups = int(mlp.at("groups").integer("keep", e.groups));
        }
        Require(e.groups >= 1 && e.experts % e.groups == 0 && e.keep_groups >= 1 && e.keep_groups <= e.groups, "experts form equal groups, at least one of them kept");
        Require(e.top <= e.keep_groups * (e.experts / e.groups), "the kept groups hold the experts of a token");
        std::string router = Quoted(parts, {"router"});
        if (e.output_weighted) {
          Require(activation == "silu" && (e.softmax || e.chosen || scores == "sigmoid"),
                  "experts with weighted outputs are gated units with softmax or sigmoid scores");
          Require(!e.chosen || (e.groups == 1 && !e.correction), "experts weighted among the chosen ones are ranked by their logits alone");
          Require(!s.parallel || !mlp.has("shared") || mlp.at("shared").kind != Json::kObject, "parallel layers have no shared expert");
          e.limit = mlp.num("limit", 3.0e38);
          e.alpha = mlp.num("alpha", 1.0);
          e.shift = mlp.num("shift", 0.0);
          std::vector<std::string> units;
          Require(parts.has("gate") && parts.has("up") && int(parts.at("gate").items.size()) == e.experts && int(parts.at("up").items.size()) == e.experts,
                  "a layer needs one tensor per expert for 'gate' and 'up'");
          for (int i = 0; i < e.experts; ++i)
            units.push_back(GluRecipe(Json::Quote(parts.at("gate").items[size_t(i)].text), Json::Quote(parts.at("up").items[size_t(i)].text)));
          layer.expert_up = matrix(p + "experts.gate_up", PadColumns(Stack(units), padded_columns(s.width)), e.experts * e.packed_rows(), s.width);
          if (mlp.has("shared") && mlp.at("shared").kind == Json::kObject) {
            e.shared_ff = int(mlp.at("shared").integer("ff", 0));
            e.shared_limit = mlp.at("shared").num("limit", 3.0e38);
            Require(e.shared_ff > 0, "the feed-forward width must be positive");
            layer.shared_up = matrix(p + "shared.gate_up", PadColumns(GluRecipe(Json::Quote(Name(parts, "shared.gate")), Json::Quote(Name(parts, "shared.up"))),
                                                                     padded_columns(s.width)), e.shared_rows(), s.width);
            layer.shared_down = matrix(p + "shared.down", StackRecipe(Quoted(parts, {"shared.down"}), padded_columns(e.shared_ff)), s.width, e.shared_ff);
            router = Quoted(parts, {"router", "shared.sg"});
          }
          if (e.correction) layer.correction = add(p + "correction", 1, 1, uint64_t(e.experts), 0, AliasRecipe(Name(parts, "correction")));
        } else {
          Require(activation == "relu2" && scores == "sigmoid" && mlp.str("weighted", "") == "input",
                  "experts use the square of relu, sigmoid scores and weights on their inputs");
          Require(layer.norm_output, "expert layers need their norms on the sublayers' outputs");
          Require(e.groups == 1 && !e.correction && !mlp.has("shared"), "experts with weighted inputs are ranked by their scores alone, without a shared one");
          layer.expert_up = matrix(p + "experts.up", StackRecipe(QuotedList(parts, "up", e.experts), padded_columns(s.width)), e.experts * e.ff, s.width);
        }
        layer.router = matrix(p + "router.weight", StackRecipe(router, padded_columns(s.width)), e.logits(), s.width);
        layer.expert_down = matrix(p + "experts.down", StackRecipe(QuotedList(parts, "down", e.experts), padded_columns(e.ff)), e.experts * s.width, e.ff);
      }
    }
    s.layers.push_back(layer);
  }
  for (const Json& in : model.at("runs").items) {
    RaggedRun run;
    run.layer = int(in.integer("layer", -1));
    run.add_embedding = in.flag("add_embedding", false);
    Require(run.layer >= 0 && run.layer < int(s.layers.size()), "a run names a layer the model does not have");
    const RaggedMixer& m = s.layers[size_t(run.layer)].mixer;
    const std::string at = std::to_string(s.runs.size());
    if (s.taps > 1) run.history = add("history." + at, 1, 1, 0, uint64_t(s.taps - 1) * W, "");
    if (m.kind == RaggedMixer::kRetention) {
      run.state = add("retention." + at, 1, 1, 0, uint64_t(m.heads) * m.dim * m.vdim, "");
    } else if (m.kind == RaggedMixer::kDelta) {
      run.state = add("delta." + at, 1, 1, 0, uint64_t(m.heads) * m.dim * m.state_dim(), "");
    } else if (m.kind == RaggedMixer::kLatent) {
      run.k_pool = add("kv_pool.latent." + at, 1, element, uint64_t(s.num_blocks) * kRaggedBlock * m.pool_dim(), 0, "");
    } else {
      const uint64_t rows = uint64_t(s.num_blocks) * m.kv_heads * kRaggedBlock;
      run.k_pool = add("kv_pool.k." + at, 1, element, rows * m.pool_dim(), 0, "");
      run.v_pool = add("kv_pool.v." + at, 1, element, rows * m.v_pool_dim(), 0, "");
    }
    const RaggedMlp& mlp = s.layers[size_t(run.layer)].mlp;
    Require(!run.add_embedding || !s.layers[size_t(run.layer)].norm_output, "layers with norms on their outputs are not looped");
    Require(!run.add_embedding || (!s.combined && !s.parallel), "layers of several streams, and parallel ones, are not looped with the embedding added");
    const int unit = mlp.output_weighted ? 3 : 2;              // matrices of an expert
    const int mlp_rows = mlp.kind == RaggedMlp::kGlu ? 3 * mlp.ff : mlp.kind == RaggedMlp::kExperts ? unit * mlp.top * mlp.ff + 3 * mlp.shared_ff + mlp.logits() : 0;
    s.weight_bytes += element_bytes * W * uint64_t(m.proj_rows() + m.out_columns() + mlp_rows);
    if (m.kind == RaggedMixer::kLatent)
      s.weight_bytes += element_bytes * uint64_t(m.heads) * (uint64_t(m.rank) * (m.dim + m.vdim) + uint64_t(m.q_rank) * (m.dim + m.rot_dims));
    if (m.kind == RaggedMixer::kDelta) s.weight_bytes += element_bytes * uint64_t(m.heads) * m.dim * m.decay_rank;
    s.weight_bytes += element_bytes * 2 * W * uint64_t(s.side_dim);
    s.runs.push_back(run);
  }
  Require(!s.runs.empty(), "the model runs no layer");
  s.weight_bytes += element_bytes * W * uint64_t(s.vocab);
  if (s.write_residuals) s.residuals = add("step.residuals", 0, 1, uint64_t(s.runs.size()) * s.max_rows * W, 0, "");
  s.final_norm = add("final.norm", 1, 1, W, 0, OffsetRecipe(Name(model, "final_norm"), offset));
  s.head = matrix("head.weight", StackRecipe("[" + Json::Quote(Name(model, "head")) + "]", padded_columns(s.width)), s.vocab, s.width);
  return s;
}

}  // namespace tmb
