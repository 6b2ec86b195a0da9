// The decoder block graph of Context: an F32 residual stream, one mixer and an optional feed-forward per
// block, each with its own sizes (DecoderBlock).  It uses the context's arena, caches, per-operator timing,
// captured decode step and pipeline hand-off like the StripedHyena2 graph; what differs is here.
//
// Per block: norm -> fused input projection -> mixer -> output projection added to the residual;
// norm -> up projection -> polynomial activation -> down projection added to the residual.  In the F32
// profile the activations, caches and products are F32 (linear_f32); otherwise they are BF16 with F32
// accumulation and the residual takes the F32 accumulators directly.
#include <algorithm>

#include "stage.hpp"

namespace evob {
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
bool decoder_tap(const DumpPoint point) {
  switch (point) {
    case DumpPoint::kBlockOutput: case DumpPoint::kPreNorm: case DumpPoint::kMixerInputProjection:
    case DumpPoint::kMixerOutput: case DumpPoint::kMixerResidual: case DumpPoint::kPostNorm:
    case DumpPoint::kMlpL1: case DumpPoint::kMlpActivation:
      return true;
    default: return false;
  }
}

}  // namespace

int Context::allocate_decoder_stage(Stage &stage) {
  const ModelConfig &c = weights_->config;
  const Activation type = activation_type(profile_);
  const std::size_t T = arena_rows_, bytes = activation_bytes(type);
  std::size_t projection = 0, query = 0, output = 0, inner = 0, workspace = 0;
  for (const DecoderBlock &b : c.blocks) {
    projection = std::max(projection, b.projection_width());
    output = std::max(output, b.output_width());
    inner = std::max(inner, b.inner_width);
    if (b.mixer == MixerType::kWindowAttention) query = std::max(query, b.query_width());
    else
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
  EVOB_TRY(stage.allocate(&stage.gated, T * inner * bytes, arena));
  EVOB_TRY(stage.allocate(&stage.recurrent_workspace, workspace, arena));
  void *p = nullptr;
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
    EVOB_TRY(stage.allocate(&p, b.heads * b.dim * b.value_dim * sizeof(float), cache));
    state.recurrent_state = static_cast<float *>(p);
    if (b.conv_taps > 1)
      EVOB_TRY(stage.allocate(&state.conv_history, (b.conv_taps - 1) * b.gate_column() * bytes, cache));
  }
  return kOk;
}

int Context::decoder_linear(Stage &s, const void *input, const void *weight, const std::size_t rows,
                            const std::size_t in_features, const std::size_t out_features, void *output,
                            float *output_f32, const bool accumulate) {
  if (profile_ == ExecutionProfile::kFloat32)
    return linear_f32(static_cast<const float *>(input), weight, rows, in_features, out_features,
                      output_f32 != nullptr ? output_f32 : static_cast<float *>(output), accumulate, s.stream);
  LinearArgs a;
  a.split_workspace = s.split_workspace;
  a.split_workspace_bytes = kSplitWorkspaceBytes;
  a.dependent_launch = decode_dependent_launch_ && rows == 1;
  a.input = input;
  a.weight = weight;
  a.output = output;
  a.output_f32 = output_f32;
  a.accumulate_f32 = accumulate;
  a.rows = rows;
  a.in_features = in_features;
  a.out_features = out_features;
  return linear(a, s.stream);
}

int Context::decoder_embed(Stage &s, const std::uint32_t *device_tokens, const std::size_t rows,
                           const std::size_t position) {
  const ModelConfig &c = weights_->config;
  return embed_positions(device_tokens, s.weights->embedding, s.weights->positions, s.weights->embedding_norm, rows,
                         c.width, c.vocab, position, c.epsilon, static_cast<float *>(s.hidden), s.stream,
                         dynamic_position_);
}

int Context::decoder_head(Stage &s, const std::size_t rows) {
  const ModelConfig &c = weights_->config;
  EVOB_OP(kCatNorm, rms_norm_residual(static_cast<const float *>(s.hidden), s.weights->final_norm, rows, c.width,
                                      c.epsilon, s.normalized, activation_type(profile_), s.stream));
  EVOB_OP(kCatGemmBf16, decoder_linear(s, s.normalized, s.weights->head, rows, c.width, c.vocab, nullptr,
                                       static_cast<float *>(s.logits), false));
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
      if (!decoder_tap(request.point))
        return fail(kUnsupported, std::string("a decoder block has no tap named ") +
                                      dump_point_name(static_cast<int>(request.point)));
  for (std::size_t i = 0; i < s.layers.size(); ++i) {
    const LayerWeights &w = s.weights->layers[i];
    LayerState &state = s.layers[i];
    const std::size_t layer = s.weights->layer_begin + i;
    const DecoderBlock &b = c.blocks[layer];
    const DumpPlan *const tap = dumps != nullptr && dumps->wants_layer(layer) ? dumps : nullptr;
    EVOB_OP(kCatNorm, rms_norm_residual(hidden, w.pre_norm, rows, D, c.epsilon, s.normalized, type, stream));
    if (tap != nullptr) EVOB_TRY(emit_activation(stream, *tap, layer, DumpPoint::kPreNorm, s.normalized, rows, D, type));
    const std::size_t stride = b.projection_width();
    EVOB_OP(kCatGemmBf16, decoder_linear(s, s.normalized, w.projection, rows, D, stride, s.projection, nullptr, false));
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
    EVOB_OP(kCatGemmBf16, decoder_linear(s, s.mixer_out, w.out_weight, rows, b.output_width(), D, nullptr, hidden, true));
    if (tap != nullptr) EVOB_TRY(emit_f32(stream, *tap, layer, DumpPoint::kMixerResidual, hidden, rows, D, D));
    if (b.inner_width != 0) {
      const std::size_t I = b.inner_width;
      EVOB_OP(kCatNorm, rms_norm_residual(hidden, w.post_norm, rows, D, c.epsilon, s.normalized, type, stream));
      if (tap != nullptr)
        EVOB_TRY(emit_activation(stream, *tap, layer, DumpPoint::kPostNorm, s.normalized, rows, D, type));
      EVOB_OP(kCatGemmBf16, decoder_linear(s, s.normalized, w.l1, rows, D, I, s.mlp_first, nullptr, false));
      EVOB_OP(kCatPolyNorm, poly_norm(s.mlp_first, w.activation, rows, I, c.epsilon, s.gated, type, stream));
      if (tap != nullptr) {
        EVOB_TRY(emit_activation(stream, *tap, layer, DumpPoint::kMlpL1, s.mlp_first, rows, I, type));
        EVOB_TRY(emit_activation(stream, *tap, layer, DumpPoint::kMlpActivation, s.gated, rows, I, type));
      }
      EVOB_OP(kCatGemmBf16, decoder_linear(s, s.gated, w.l3, rows, I, D, nullptr, hidden, true));
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
