// The decoder block graph of Context: an F32 residual stream, one mixer and an optional feed-forward per
// block, each with its own sizes (DecoderBlock).  It uses the context's arena, caches, per-operator timing,
// captured decode step and pipeline hand-off like the StripedHyena2 graph; what differs is here.
//
// Per block: norm -> fused input projection -> mixer -> output projection added to the residual;
// norm -> up projection -> polynomial activation -> down projection added to the residual.  Designs with norms
// on the sublayers' outputs (ModelConfig::output_norms): the sublayers read the stream itself, their F32 results
// go through a layer norm whose kernel also adds them to the residual and leaves the next sublayer's input.
// In the F32 profile the activations, caches and products are F32 (linear_f32); otherwise they are BF16 with
// F32 accumulation and the residual takes F32 values directly.
#include <algorithm>

#include "stage.hpp"

namespace evob {

// One projection of a decoder block: output (activation type) or output_f32 [+]= alpha input weight^T + bias, soft
// cap last (both F32 results only).
struct DecoderProduct {
  const void *input = nullptr, *weight = nullptr;
  std::size_t rows = 0, in_features = 0, out_features = 0;
  void *output = nullptr;
  float *output_f32 = nullptr;
  bool accumulate = false;
  const float *bias = nullptr;
  float alpha = 1.0F, softcap = 0.0F;
};

namespace {

Activation activation_type(const ExecutionProfile profile) {
  return profile == ExecutionProfile::kFloat32 ? Activation::kF32 : Activation::kBf16;
}

// Row of F32 or BF16 values at `row` of a [*, stride] buffer.
const void *element(const void *base, const std::size_t index, const Activation type) {
  return static_cast<const unsigned char *>(base) + index * activation_bytes(type);
}

int emit_activation(cudaStream_t stream, const DumpPlan &plan, const std::size_t layer, const DumpPoint point,
                    const void *device, const std::size_t rows, const std::size_t columns, const Activation type) {
  if (type == Activation::kBf16) return emit_bf16(stream, plan, layer, point, device, rows, columns);
  return emit_f32(stream, plan, layer, point, static_cast<const float *>(device), rows, columns, columns);
}

// The taps that a decoder block has a buffer for.
bool decoder_tap(const ModelConfig &c, const DumpPoint point) {
  switch (point) {
    case DumpPoint::kBlockOutput: case DumpPoint::kMixerInputProjection: case DumpPoint::kMixerOutput:
    case DumpPoint::kMixerResidual:
      return true;
    case DumpPoint::kPreNorm: case DumpPoint::kPostNorm: case DumpPoint::kMlpL1: case DumpPoint::kMlpActivation:
      return !c.output_norms;
    case DumpPoint::kMixerProjection: return c.output_norms;
    default: return false;
  }
}

// Rows up to which a mixture of experts runs pair by pair instead of grouped by expert.
constexpr std::size_t kPairwiseRows = 8;
// Rows per expert from which its tiles are 256 rows high (CTA pairs).
constexpr std::size_t kPairTileRows = 512;
constexpr std::size_t kWidestTile = 256;

std::size_t grouped_capacity(const DecoderBlock &b, const std::size_t rows) {
  return std::max(grouped_tiles(rows, b.top, b.experts, kWidestTile) * kWidestTile,
                  grouped_tiles(rows, b.top, b.experts, 128) * 128);
}

// Whether the projection kernels apply a gate to these weights themselves (else the products go through memory).
bool gate_fusable(const ExecutionProfile profile, const std::size_t width) {
  return profile != ExecutionProfile::kFloat32 && width % 8 == 0 && width >= 64;
}
// Whether grouped down projections run on the tensor cores.
bool grouped_down(const ExecutionProfile profile, const std::size_t width) {
  return profile != ExecutionProfile::kFloat32 && width >= 32;
}

}  // namespace

int Context::allocate_decoder_stage(Stage &stage) {
  const ModelConfig &c = weights_->config;
  const Activation type = activation_type(profile_);
  const std::size_t T = arena_rows_, bytes = activation_bytes(type);
  std::size_t projection = 0, query = 0, output = 0, inner = 0, workspace = 0;
  std::size_t query_latent = 0, absorbed = 0, keys = 0, values = 0;            // latent attention
  std::size_t gated = 0, pairs = 0, tiles = 0, slots = 0, experts = 0, logits = 0;  // gated feed-forwards, experts
  const bool unfused = !gate_fusable(profile_, c.width);
  for (const DecoderBlock &b : c.blocks) {
    projection = std::max(projection, b.projection_width());
    output = std::max(output, b.output_width());
    if (b.feed_forward == FeedForward::kPolyNorm) inner = std::max(inner, b.inner_width);
    if (b.feed_forward == FeedForward::kReluGated) gated = std::max(gated, T * b.inner_columns());
    if (b.feed_forward == FeedForward::kExperts) {
      const std::size_t capacity = grouped_capacity(b, T);
      gated = std::max(gated, capacity * b.inner_columns());
      pairs = std::max(pairs, T * b.top);
      tiles = std::max(tiles, grouped_tiles(T, b.top, b.experts, 128));
      slots = std::max(slots, capacity);
      experts = std::max(experts, b.experts);
      logits = std::max(logits, b.router_rows());
    }
    if (b.mixer == MixerType::kWindowAttention) query = std::max(query, b.query_width());
    else if (b.mixer == MixerType::kLatentAttention) {
      query = std::max(query, b.query_width());
      query_latent = std::max(query_latent, b.query_rank);
      absorbed = std::max(absorbed, kLatentRows * b.heads * b.latent_rank);
      const std::size_t span = std::min(context_size_, T + b.window - 1);  // tokens that a pass of T rows sees
      keys = std::max(keys, span * b.heads * b.dim);
      values = std::max(values, span * b.heads * b.value_dim);
    } else
      workspace = std::max(workspace, recurrent_workspace_bytes(b.mixer == MixerType::kGatedDelta, T, b.heads,
                                                                b.kv_heads, b.dim, b.value_dim, type));
  }
  std::size_t *const arena = &stage.arena_bytes, *const cache = &stage.cache_bytes;
  EVOB_TRY(stage.allocate(&stage.hidden, T * c.width * sizeof(float), arena));
  EVOB_TRY(stage.allocate(&stage.normalized, T * c.width * bytes, arena));
  EVOB_TRY(stage.allocate(&stage.projection, T * projection * bytes, arena));
  EVOB_TRY(stage.allocate(&stage.query, T * query * bytes, arena));
  EVOB_TRY(stage.allocate(&stage.mixer_out, T * output * bytes, arena));
  EVOB_TRY(stage.allocate(&stage.mlp_first, T * inner * bytes, arena));
  EVOB_TRY(stage.allocate(&stage.gated, std::max(T * inner, gated) * bytes, arena));
  EVOB_TRY(stage.allocate(&stage.recurrent_workspace, workspace, arena));
  void *p = nullptr;
  if (c.output_norms) EVOB_TRY(stage.allocate(&stage.sublayer, T * c.width * sizeof(float), arena));
  if (query_latent != 0) {
    EVOB_TRY(stage.allocate(&stage.query_latent, T * query_latent * bytes, arena));
    EVOB_TRY(stage.allocate(&stage.absorbed, absorbed * bytes, arena));
    EVOB_TRY(stage.allocate(&stage.latent_mix, absorbed * bytes, arena));
    EVOB_TRY(stage.allocate(&stage.expanded_keys, keys * bytes, arena));
    EVOB_TRY(stage.allocate(&stage.expanded_values, values * bytes, arena));
  }
  if (gated != 0 && unfused) EVOB_TRY(stage.allocate(&stage.gate_products, 2 * gated * sizeof(float), arena));
  if (pairs != 0) {
    EVOB_TRY(stage.allocate(&stage.grouped_rows, slots * c.width * bytes, arena));
    EVOB_TRY(stage.allocate(&stage.expert_out, slots * c.width * sizeof(float), arena));
    EVOB_TRY(stage.allocate(&p, T * logits * sizeof(float), arena));
    stage.router_logits = static_cast<float *>(p);
    EVOB_TRY(stage.allocate(&p, (pairs + slots) * sizeof(float), arena));
    stage.pair_score = static_cast<float *>(p);
    stage.slot_score = stage.pair_score + pairs;
    EVOB_TRY(stage.allocate(&p, (3 * pairs + experts + tiles + 1) * sizeof(int), arena));
    stage.pair_expert = static_cast<int *>(p);
    stage.pair_rank = stage.pair_expert + pairs;
    stage.pair_slot = stage.pair_rank + pairs;
    stage.expert_counts = stage.pair_slot + pairs;
    stage.tile_group = stage.expert_counts + experts;
    stage.tile_count = stage.tile_group + tiles;
  }
  EVOB_TRY(stage.allocate(&p, T * sizeof(std::uint32_t), arena));
  stage.tokens = static_cast<std::uint32_t *>(p);
  EVOB_TRY(stage.allocate(&stage.logits, T * c.vocab * sizeof(float), arena));
  EVOB_TRY(stage.allocate(&stage.split_workspace, kSplitWorkspaceBytes, arena));
  stage.layers.resize(stage.weights->layers.size());
  for (std::size_t i = 0; i < stage.layers.size(); ++i) {
    const DecoderBlock &b = c.blocks[stage.weights->layer_begin + i];
    LayerState &state = stage.layers[i];
    if (b.mixer == MixerType::kWindowAttention) {
      EVOB_TRY(stage.allocate(&state.key_cache, context_size_ * b.key_width() * bytes, cache));
      EVOB_TRY(stage.allocate(&state.value_cache, context_size_ * b.value_width() * bytes, cache));
      continue;
    }
    if (b.mixer == MixerType::kLatentAttention) {
      EVOB_TRY(stage.allocate(&state.key_cache, context_size_ * b.latent_rank * bytes, cache));
      continue;
    }
    EVOB_TRY(stage.allocate(&p, b.heads * b.dim * b.value_dim * sizeof(float), cache));
    state.recurrent_state = static_cast<float *>(p);
    if (b.conv_taps > 1)
      EVOB_TRY(stage.allocate(&state.conv_history, (b.conv_taps - 1) * b.gate_column() * bytes, cache));
  }
  return kOk;
}

int Context::decoder_linear(Stage &s, const DecoderProduct &p) {
  if (profile_ == ExecutionProfile::kFloat32) {
    LinearF32Args a;
    a.input = p.input;
    a.weight = p.weight;
    a.rows = p.rows;
    a.in_features = p.in_features;
    a.out_features = p.out_features;
    a.output = p.output_f32 != nullptr ? p.output_f32 : static_cast<float *>(p.output);
    a.accumulate = p.accumulate;
    a.bias = p.bias;
    a.alpha = p.alpha;
    a.softcap = p.softcap;
    return linear_f32(a, s.stream);
  }
  LinearArgs a;
  a.split_workspace = s.split_workspace;
  a.split_workspace_bytes = kSplitWorkspaceBytes;
  a.dependent_launch = decode_dependent_launch_ && p.rows == 1;
  a.input = p.input;
  a.weight = p.weight;
  a.output = p.output;
  a.output_f32 = p.output_f32;
  a.accumulate_f32 = p.accumulate;
  a.bias_f32 = p.bias;
  a.alpha = p.alpha;
  a.softcap = p.softcap;
  a.rows = p.rows;
  a.in_features = p.in_features;
  a.out_features = p.out_features;
  return linear(a, s.stream);
}

int Context::decoder_embed(Stage &s, const std::uint32_t *device_tokens, const std::size_t rows,
                           const std::size_t position) {
  const ModelConfig &c = weights_->config;
  const Activation type = activation_type(profile_);
  if (!c.learned_positions)
    return embed_rows(device_tokens, s.weights->embedding, rows, c.width, c.vocab, static_cast<float *>(s.hidden),
                      type == Activation::kBf16 ? s.normalized : nullptr, type, s.stream);
  return embed_positions(device_tokens, s.weights->embedding, s.weights->positions, s.weights->embedding_norm, rows,
                         c.width, c.vocab, position, c.epsilon, static_cast<float *>(s.hidden), s.stream,
                         dynamic_position_);
}

int Context::decoder_head(Stage &s, const std::size_t rows) {
  const ModelConfig &c = weights_->config;
  if (c.output_norms) {
    LayerNormArgs n;
    n.input = s.hidden;
    n.gain = s.weights->final_norm;
    n.output = s.normalized;
    n.output_type = activation_type(profile_);
    n.rows = rows;
    n.width = c.width;
    n.epsilon = c.epsilon;
    EVOB_OP(kCatNorm, layer_norm(n, s.stream));
  } else {
    EVOB_OP(kCatNorm, rms_norm_residual(static_cast<const float *>(s.hidden), s.weights->final_norm, rows, c.width,
                                        c.epsilon, s.normalized, activation_type(profile_), s.stream));
  }
  DecoderProduct p;
  p.input = s.normalized;
  p.weight = s.weights->head;
  p.rows = rows;
  p.in_features = c.width;
  p.out_features = c.vocab;
  p.output_f32 = static_cast<float *>(s.logits);
  p.alpha = c.logit_scale;
  p.softcap = c.logit_softcap;
  EVOB_OP(kCatGemmBf16, decoder_linear(s, p));
  return kOk;
}

// Latent attention behind the fused input projection: s.mixer_out [rows, heads * value_dim].  A few rows attend to
// the cached latents themselves (one key/value head of width latent_rank); more rows expand the keys and values of
// the tokens that they see and run the ordinary window attention on them.
int Context::latent_mixer(Stage &s, const std::size_t i, const std::size_t rows, const std::size_t position,
                          const int *const dynamic) {
  const ModelConfig &c = weights_->config;
  const Activation type = activation_type(profile_);
  const LayerWeights &w = s.weights->layers[i];
  const DecoderBlock &b = c.blocks[s.weights->layer_begin + i];
  void *const cache = s.layers[i].key_cache;
  cudaStream_t stream = s.stream;
  LatentNormArgs n;
  n.projection = s.projection;
  n.stride = b.projection_width();
  n.latent_column = b.latent_column();
  n.query_gain = w.query_norm;
  n.latent_gain = w.key_norm;
  n.query_latent = s.query_latent;
  n.cache = cache;
  n.rows = rows;
  n.position = position;
  n.capacity = context_size_;
  n.query_rank = b.query_rank;
  n.latent_rank = b.latent_rank;
  n.epsilon = c.epsilon;
  n.type = type;
  n.dynamic_position = dynamic;
  EVOB_OP(kCatNorm, latent_norm_append(n, stream));
  DecoderProduct q;
  q.input = s.query_latent;
  q.weight = w.query_up;
  q.rows = rows;
  q.in_features = b.query_rank;
  q.out_features = b.heads * b.dim;
  q.output = s.query;
  EVOB_OP(kCatGemmBf16, decoder_linear(s, q));
  WindowAttentionArgs a;
  a.rows = rows;
  a.heads = b.heads;
  a.window = b.window;
  a.scale = b.scale;
  a.sink = b.sink;
  a.sink_logit = w.sink_logit;
  a.type = type;
  if (rows <= kLatentRows) {
    EVOB_OP(kCatAttention, absorb_queries(s.query, w.key_up, rows, b.heads, b.dim, b.latent_rank, s.absorbed, type, stream));
    a.query = s.absorbed;
    a.key_cache = a.value_cache = cache;
    a.output = s.latent_mix;
    a.position = position;
    a.capacity = context_size_;
    a.kv_heads = 1;
    a.dim = a.value_dim = b.latent_rank;
    a.dynamic_position = dynamic;
    EVOB_OP(kCatAttention, window_attention(a, stream));
    EVOB_OP(kCatAttention, expand_values(s.latent_mix, w.value_up, rows, b.heads, b.value_dim, b.latent_rank, s.mixer_out,
                                         type, stream));
    return kOk;
  }
  // the oldest token that the first row sees becomes row 0: only distances matter
  const std::size_t oldest = position >= b.window ? position - b.window + 1 : 0, span = position + rows - oldest;
  DecoderProduct up;
  up.input = element(cache, oldest * b.latent_rank, type);
  up.rows = span;
  up.in_features = b.latent_rank;
  up.weight = w.key_up;
  up.out_features = b.heads * b.dim;
  up.output = s.expanded_keys;
  EVOB_OP(kCatGemmBf16, decoder_linear(s, up));
  up.weight = w.value_up;
  up.out_features = b.heads * b.value_dim;
  up.output = s.expanded_values;
  EVOB_OP(kCatGemmBf16, decoder_linear(s, up));
  a.query = s.query;
  a.key_cache = s.expanded_keys;
  a.value_cache = s.expanded_values;
  a.output = s.mixer_out;
  a.position = position - oldest;
  a.capacity = span;
  a.kv_heads = b.heads;
  a.dim = b.dim;
  a.value_dim = b.value_dim;
  EVOB_OP(kCatAttention, window_attention(a, stream));
  return kOk;
}

int Context::gated_feed_forward(Stage &s, const std::size_t i, const std::size_t rows, const void *const input,
                                LayerNormArgs *const norm) {
  const ModelConfig &c = weights_->config;
  const LayerWeights &w = s.weights->layers[i];
  const DecoderBlock &b = c.blocks[s.weights->layer_begin + i];
  const std::size_t I = b.inner_columns();
  if (gate_fusable(profile_, c.width)) {
    LinearArgs a;
    a.split_workspace = s.split_workspace;
    a.split_workspace_bytes = kSplitWorkspaceBytes;
    a.dependent_launch = decode_dependent_launch_ && rows == 1;
    a.input = input;
    a.weight = w.l12;
    a.output = s.gated;
    a.bias_f32 = w.l12_bias;
    a.gate_mode = kGateRelu;
    a.rows = rows;
    a.in_features = c.width;
    a.out_features = 2 * I;
    EVOB_OP(kCatGemmBf16, linear(a, s.stream));
  } else {
    DecoderProduct p;
    p.input = input;
    p.weight = w.l12;
    p.rows = rows;
    p.in_features = c.width;
    p.out_features = 2 * I;
    p.output_f32 = static_cast<float *>(s.gate_products);
    p.bias = w.l12_bias;
    EVOB_OP(kCatGemmBf16, decoder_linear(s, p));
    EVOB_OP(kCatElementwise, gated_activation(static_cast<const float *>(s.gate_products), kGateRelu, 0.0F, rows, I, s.gated,
                                              activation_type(profile_), nullptr, 0, s.stream));
  }
  DecoderProduct down;
  down.input = s.gated;
  down.weight = w.l3;
  down.rows = rows;
  down.in_features = I;
  down.out_features = c.width;
  down.output_f32 = static_cast<float *>(s.sublayer);
  down.bias = w.l3_bias;
  EVOB_OP(kCatGemmBf16, decoder_linear(s, down));
  norm->input = s.sublayer;
  return kOk;
}

// A mixture of experts.  A few rows: each (row, expert) pair streams its expert's weights.  More rows: rows are
// grouped by expert into whole tiles and every expert's products run as row tiles of one launch.  The score
// multiplies the products of the up projections (which are linear in the expert's input); the sum over a row's
// experts is taken by the norm.
int Context::expert_feed_forward(Stage &s, const std::size_t i, const std::size_t rows, const void *const input,
                                 LayerNormArgs *const norm) {
  const ModelConfig &c = weights_->config;
  const Activation type = activation_type(profile_);
  const LayerWeights &w = s.weights->layers[i];
  const DecoderBlock &b = c.blocks[s.weights->layer_begin + i];
  const std::size_t I = b.inner_columns(), D = c.width;
  const bool pairwise = rows <= kPairwiseRows, fused = gate_fusable(profile_, D);
  cudaStream_t stream = s.stream;
  RouteArgs r;
  r.rows = rows;
  r.width = D;
  r.experts = b.experts;
  r.top = b.top;
  r.expert = s.pair_expert;
  r.score = s.pair_score;
  if (pairwise) {
    r.input = input;
    r.type = type;
    r.router = w.router;
  } else {
    DecoderProduct p;
    p.input = input;
    p.weight = w.router;
    p.rows = rows;
    p.in_features = D;
    p.out_features = b.router_rows();
    p.output_f32 = s.router_logits;
    EVOB_OP(kCatRouting, decoder_linear(s, p));
    r.logits = s.router_logits;
    r.logit_stride = b.router_rows();
    r.counts = s.expert_counts;
    r.rank = s.pair_rank;
  }
  EVOB_OP(kCatRouting, route_rows(r, stream));
  const std::size_t tile_rows = rows * b.top >= kPairTileRows * b.experts && D >= kWidestTile ? kWidestTile : 128;
  if (!pairwise) {
    GroupRowsArgs g;
    g.input = input;
    g.type = type;
    g.rows = rows;
    g.width = D;
    g.experts = b.experts;
    g.top = b.top;
    g.tile_rows = tile_rows;
    g.expert = s.pair_expert;
    g.rank = s.pair_rank;
    g.counts = s.expert_counts;
    g.score = s.pair_score;
    g.grouped = s.grouped_rows;
    g.slot_score = s.slot_score;
    g.slot = s.pair_slot;
    g.tile_group = s.tile_group;
    g.tile_count = s.tile_count;
    EVOB_OP(kCatRouting, group_rows(g, stream));
  }
  const std::size_t live = pairwise ? rows * b.top : grouped_tiles(rows, b.top, b.experts, tile_rows) * tile_rows;
  // the members that both kinds of projection share
  const auto grouping = [&](auto &a, const bool first) {
    a.rows = live;
    if (pairwise) {
      a.row_group = s.pair_expert;
      a.row_fanout = first ? b.top : 1;
    } else {
      a.tile_group = s.tile_group;
      a.tile_count = s.tile_count;
      a.tile_rows = tile_rows;
    }
    a.input = first ? (pairwise ? input : s.grouped_rows) : s.gated;
    a.weight = first ? w.l12 : w.l3;
    a.in_features = first ? D : I;
    a.out_features = first ? 2 * I : D;
    if (first) a.row_scale = pairwise ? s.pair_score : s.slot_score;
  };
  if (fused) {
    LinearArgs a;
    grouping(a, true);
    a.groups = b.experts;
    a.dependent_launch = decode_dependent_launch_ && rows == 1;
    a.output = s.gated;
    a.gate_mode = kGateClamped;
    a.gate_limit = b.gate_limit;
    EVOB_OP(kCatGemmGrouped, linear(a, stream));
  } else {
    LinearF32Args a;
    grouping(a, true);
    a.input_type = type;
    a.output = static_cast<float *>(s.gate_products);
    EVOB_OP(kCatGemmGrouped, linear_f32(a, stream));
    EVOB_OP(kCatElementwise, gated_activation(a.output, kGateClamped, b.gate_limit, live, I, s.gated, type, a.tile_count,
                                              tile_rows, stream));
  }
  if (type == Activation::kBf16 && (pairwise || grouped_down(profile_, D))) {
    LinearArgs a;
    grouping(a, false);
    a.groups = b.experts;
    a.dependent_launch = decode_dependent_launch_ && rows == 1;
    a.output = s.expert_out;
    EVOB_OP(kCatGemmGrouped, linear(a, stream));
    norm->input_type = Activation::kBf16;
  } else {
    LinearF32Args a;
    grouping(a, false);
    a.input_type = type;
    a.output = static_cast<float *>(s.expert_out);
    EVOB_OP(kCatGemmGrouped, linear_f32(a, stream));
  }
  norm->input = s.expert_out;
  norm->parts = b.top;
  norm->slots = pairwise ? nullptr : s.pair_slot;
  return kOk;
}

int Context::run_decoder_stage(Stage &s, const std::size_t rows, const Mode mode, const std::size_t position,
                               const long capture_layer, std::vector<float> *captured, const DumpPlan *const dumps) {
  const ModelConfig &c = weights_->config;
  const Activation type = activation_type(profile_);
  const std::size_t D = c.width;
  const bool fresh = mode == Mode::kPrefill || mode == Mode::kStateless || mode == Mode::kCachedPrefill;
  const int *const dynamic = mode == Mode::kDecode ? dynamic_position_ : nullptr;
  float *const hidden = static_cast<float *>(s.hidden);
  cudaStream_t stream = s.stream;
  if (dumps != nullptr)
    for (const DumpPlan::Request &request : dumps->requests)
      if (!decoder_tap(c, request.point))
        return fail(kUnsupported, std::string("a decoder block has no tap named ") +
                                      dump_point_name(static_cast<int>(request.point)));
  // what a sublayer reads where the norms are on the outputs: the stream in the activation type
  const void *const stream_input = type == Activation::kF32 ? s.hidden : s.normalized;
  if (c.output_norms && type == Activation::kBf16 && s.weights->layer_begin != 0)
    EVOB_OP(kCatElementwise, convert_rows(hidden, rows * D, s.normalized, type, stream));  // (the embedding leaves it too)
  const auto product = [&](const void *input, const void *weight, const std::size_t in_features,
                           const std::size_t out_features, void *output, float *output_f32, const bool accumulate) {
    DecoderProduct p;
    p.input = input;
    p.weight = weight;
    p.rows = rows;
    p.in_features = in_features;
    p.out_features = out_features;
    p.output = output;
    p.output_f32 = output_f32;
    p.accumulate = accumulate;
    return decoder_linear(s, p);
  };
  LayerNormArgs behind;  // of a sublayer: added to the residual, which also becomes the next sublayer's input
  behind.residual = hidden;
  behind.output = type == Activation::kBf16 ? s.normalized : nullptr;
  behind.output_type = type;
  behind.rows = rows;
  behind.width = D;
  behind.epsilon = c.epsilon;
  for (std::size_t i = 0; i < s.layers.size(); ++i) {
    const LayerWeights &w = s.weights->layers[i];
    LayerState &state = s.layers[i];
    const std::size_t layer = s.weights->layer_begin + i;
    const DecoderBlock &b = c.blocks[layer];
    const DumpPlan *const tap = dumps != nullptr && dumps->wants_layer(layer) ? dumps : nullptr;
    const void *input = stream_input;
    if (!c.output_norms) {
      EVOB_OP(kCatNorm, rms_norm_residual(hidden, w.pre_norm, rows, D, c.epsilon, s.normalized, type, stream));
      if (tap != nullptr)
        EVOB_TRY(emit_activation(stream, *tap, layer, DumpPoint::kPreNorm, s.normalized, rows, D, type));
      input = s.normalized;
    }
    const std::size_t stride = b.projection_width();
    EVOB_OP(kCatGemmBf16, product(input, w.projection, D, stride, s.projection, nullptr, false));
    if (tap != nullptr)
      EVOB_TRY(emit_activation(stream, *tap, layer, DumpPoint::kMixerInputProjection, s.projection, rows, stride, type));
    if (b.mixer == MixerType::kWindowAttention) {
      HeadNormArgs n;
      n.projection = s.projection;
      n.stride = stride;
      n.key_column = b.key_column();
      n.value_column = b.value_column();
      n.query_gain = w.query_norm;
      n.key_gain = w.key_norm;
      n.query = s.query;
      n.key_cache = state.key_cache;
      n.value_cache = state.value_cache;
      n.rows = rows;
      n.position = position;
      n.capacity = context_size_;
      n.heads = b.heads;
      n.kv_heads = b.kv_heads;
      n.dim = b.dim;
      n.value_dim = b.value_dim;
      n.epsilon = c.epsilon;
      n.type = type;
      n.dynamic_position = dynamic;
      EVOB_OP(kCatAttention, head_norm_append(n, stream));
      WindowAttentionArgs a;
      a.query = s.query;
      a.key_cache = state.key_cache;
      a.value_cache = state.value_cache;
      a.gate = element(s.projection, b.gate_column(), type);
      a.gate_stride = stride;
      a.distance_bias = w.distance_bias;
      a.bias_stride = c.max_seqlen;
      a.output = s.mixer_out;
      a.rows = rows;
      a.position = position;
      a.capacity = context_size_;
      a.heads = b.heads;
      a.kv_heads = b.kv_heads;
      a.dim = b.dim;
      a.value_dim = b.value_dim;
      a.window = b.window;
      a.keep_first = b.keep_first;
      a.scale = b.scale;
      a.softcap = b.softcap;
      a.sink = true;
      a.type = type;
      a.dynamic_position = dynamic;
      EVOB_OP(kCatAttention, window_attention(a, stream));
    } else if (b.mixer == MixerType::kLatentAttention) {
      EVOB_TRY(latent_mixer(s, i, rows, position, dynamic));
    } else {
      RecurrentArgs a;
      a.delta = b.mixer == MixerType::kGatedDelta;
      a.projection = s.projection;
      a.stride = stride;
      a.key_column = b.key_column();
      a.value_column = b.value_column();
      a.gate_column = b.gate_column();
      a.beta_column = b.beta_column();
      a.decay_column = b.decay_column();
      a.rows = rows;
      a.heads = b.heads;
      a.kv_heads = b.kv_heads;
      a.dim = b.dim;
      a.value_dim = b.value_dim;
      a.conv = w.conv;
      a.conv_taps = b.conv_taps;
      a.conv_history = state.conv_history;
      a.decay_rate = w.decay_rate;
      a.decay_shift = w.decay_shift;
      a.decay_weight = w.decay_weight;
      a.decay_bias = w.decay_bias;
      a.decay_rank = b.decay_rank;
      a.tau = b.tau;
      a.output_norm = w.output_norm;
      a.epsilon = c.epsilon;
      a.state = state.recurrent_state;
      a.fresh = fresh;
      a.workspace = s.recurrent_workspace;
      a.output = s.mixer_out;
      a.type = type;
      EVOB_OP(a.delta ? kCatGatedDelta : kCatGatedLinear, recurrent_mixer(a, stream));
    }
    if (tap != nullptr)
      EVOB_TRY(emit_activation(stream, *tap, layer, DumpPoint::kMixerOutput, s.mixer_out, rows, b.output_width(), type));
    float *const sublayer = c.output_norms ? static_cast<float *>(s.sublayer) : hidden;
    EVOB_OP(kCatGemmBf16, product(s.mixer_out, w.out_weight, b.output_width(), D, nullptr, sublayer, !c.output_norms));
    if (c.output_norms) {
      if (tap != nullptr) EVOB_TRY(emit_f32(stream, *tap, layer, DumpPoint::kMixerProjection, sublayer, rows, D, D));
      LayerNormArgs n = behind;
      n.input = sublayer;
      n.gain = w.pre_norm;
      EVOB_OP(kCatNorm, layer_norm(n, stream));
    }
    if (tap != nullptr) EVOB_TRY(emit_f32(stream, *tap, layer, DumpPoint::kMixerResidual, hidden, rows, D, D));
    if (b.feed_forward == FeedForward::kPolyNorm) {
      const std::size_t I = b.inner_width;
      EVOB_OP(kCatNorm, rms_norm_residual(hidden, w.post_norm, rows, D, c.epsilon, s.normalized, type, stream));
      if (tap != nullptr)
        EVOB_TRY(emit_activation(stream, *tap, layer, DumpPoint::kPostNorm, s.normalized, rows, D, type));
      EVOB_OP(kCatGemmBf16, product(s.normalized, w.l1, D, I, s.mlp_first, nullptr, false));
      EVOB_OP(kCatPolyNorm, poly_norm(s.mlp_first, w.activation, rows, I, c.epsilon, s.gated, type, stream));
      if (tap != nullptr) {
        EVOB_TRY(emit_activation(stream, *tap, layer, DumpPoint::kMlpL1, s.mlp_first, rows, I, type));
        EVOB_TRY(emit_activation(stream, *tap, layer, DumpPoint::kMlpActivation, s.gated, rows, I, type));
      }
      EVOB_OP(kCatGemmBf16, product(s.gated, w.l3, I, D, nullptr, hidden, true));
    } else if (b.feed_forward != FeedForward::kNone) {
      LayerNormArgs n = behind;
      n.gain = w.post_norm;
      if (b.feed_forward == FeedForward::kReluGated) EVOB_TRY(gated_feed_forward(s, i, rows, stream_input, &n));
      else EVOB_TRY(expert_feed_forward(s, i, rows, stream_input, &n));
      EVOB_OP(kCatNorm, layer_norm(n, stream));
    }
    if (tap != nullptr) EVOB_TRY(emit_f32(stream, *tap, layer, DumpPoint::kBlockOutput, hidden, rows, D, D));
    if (capture_layer >= 0 && static_cast<std::size_t>(capture_layer) == layer && captured != nullptr) {
      captured->resize(rows * D);
      if (cudaMemcpyAsync(captured->data(), hidden, rows * D * sizeof(float), cudaMemcpyDeviceToHost, stream) !=
              cudaSuccess ||
          cudaStreamSynchronize(stream) != cudaSuccess)
        return fail(kCuda, "layer capture failed");
    }
  }
  return kOk;
}

}  // namespace evob
