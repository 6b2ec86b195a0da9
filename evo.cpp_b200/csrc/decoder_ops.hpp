// Host-side launchers of the decoder graph's kernels (runtime/decoder.cu).  Activations between operators
// are BF16 or, in the F32 profile, F32; the residual stream, norms, attention scores, decays, gates of a
// recurrence and recurrent states are F32 in both.  All pointers are device pointers on the current
// device; every function returns an evo_status value.  `dynamic_position` (optional, device int) replaces
// the host's position in launches that are recorded once and replayed.
#pragma once

#include <cuda_runtime.h>

#include <cstddef>
#include <cstdint>

namespace evob {

constexpr std::size_t kDecoderMaxHeadDim = 256;
constexpr std::size_t kDecoderMaxLatent = 1024;  // widest latent of latent attention (row kernel)
constexpr std::size_t kDecoderMaxExperts = 1024;

enum class Activation { kBf16, kF32 };
inline std::size_t activation_bytes(const Activation a) { return a == Activation::kBf16 ? 2 : 4; }

// ---- decoder_rows.cu
// output[r, :] = rms_norm(table[token[r], :] + positions[position + r, :]) * gain, F32.  Ids >= vocabulary:
// see embedding().
int embed_positions(const std::uint32_t *tokens, const void *table, const void *positions, const float *gain,
                    std::size_t rows, std::size_t width, std::size_t vocabulary, std::size_t position, float epsilon,
                    float *output, cudaStream_t stream, const int *dynamic_position = nullptr);
// output[r, :] = input[r, :] / sqrt(mean(input[r, :]^2) + epsilon) * gain.
int rms_norm_residual(const float *input, const float *gain, std::size_t rows, std::size_t width, float epsilon,
                      void *output, Activation type, cudaStream_t stream);
// output = a N(z) + b N(z^2) + c N(z^3) + e with coefficients (a, b, c, e) and N dividing a row by its root
// mean square (epsilon inside the root).  In place allowed.
int poly_norm(const void *input, const float *coefficients, std::size_t rows, std::size_t width, float epsilon,
              void *output, Activation type, cudaStream_t stream);
// table[h, d] = r1[h] ln(1 + r2[h] d), d < distances.
int distance_bias_table(const float *r1, const float *r2, std::size_t heads, std::size_t distances, float *table,
                        cudaStream_t stream);
// [rows, in] (F32 or BF16) x BF16 [out, in]^T in F32 fused multiply-adds.  output = [output +] alpha *
// row_scale[r] * product + bias, then softcap tanh(output / softcap) where softcap > 0.  Grouped weights
// [groups, out, in]: see LinearArgs (row_group / row_fanout, or tile_group / tile_count / tile_rows).
struct LinearF32Args {
  const void *input = nullptr;
  Activation input_type = Activation::kF32;
  const void *weight = nullptr;
  float *output = nullptr;
  std::size_t rows = 0, in_features = 0, out_features = 0;
  bool accumulate = false;
  float alpha = 1.0F, softcap = 0.0F;
  const float *row_scale = nullptr, *bias = nullptr;
  const int *row_group = nullptr;
  std::size_t row_fanout = 1;
  const int *tile_group = nullptr, *tile_count = nullptr;
  std::size_t tile_rows = 128;
};
int linear_f32(const LinearF32Args &args, cudaStream_t stream);
int linear_f32(const float *input, const void *weight, std::size_t rows, std::size_t in_features,
               std::size_t out_features, float *output, bool accumulate, cudaStream_t stream);
// stream[r, :] = table[token[r], :] in F32, and the same row in `copy` (optional).  Ids >= vocabulary: see embedding().
int embed_rows(const std::uint32_t *tokens, const void *table, std::size_t rows, std::size_t width,
               std::size_t vocabulary, float *stream_rows, void *copy, Activation type, cudaStream_t stream);
// Row r of the input is y = the sum of its `parts` rows (row slots[r * parts + k], or r * parts + k without
// slots); n = (y - mean) / sqrt(variance + epsilon) * gain.  With a residual: residual[r, :] += n, and the new
// residual row goes to `output` (optional); without: n goes to `output`.
struct LayerNormArgs {
  const void *input = nullptr;
  Activation input_type = Activation::kF32;
  const int *slots = nullptr;
  std::size_t parts = 1;
  const float *gain = nullptr;
  float *residual = nullptr;
  void *output = nullptr;
  Activation output_type = Activation::kF32;
  std::size_t rows = 0, width = 0;
  float epsilon = 1e-6F;
};
int layer_norm(const LayerNormArgs &args, cudaStream_t stream);
// F32 rows in the activation type.
int convert_rows(const float *input, std::size_t elements, void *output, Activation type, cudaStream_t stream);
// Gated activation of row-interleaved products [rows, 2 * inner] (blocks of 128 gate columns followed by the
// matching 128 up columns), `gate` as LinearArgs::gate_mode 3 and 4; with tile_count only its tiles' rows are live.
int gated_activation(const float *input, int gate, float limit, std::size_t rows, std::size_t inner, void *output,
                     Activation type, const int *tile_count, std::size_t tile_rows, cudaStream_t stream);

// ---- experts.cu
// Router of a mixture of experts: scores sigmoid(x . router[e]) in F32, the `top` largest, best first, ties to
// the lower index.  The products come from `logits` [rows, logit_stride] where given; else the kernel makes
// them itself (few rows).  Results per (row, place): expert id and score.
struct RouteArgs {
  const void *input = nullptr;    // [rows, width], without logits
  Activation type = Activation::kBf16;
  const void *router = nullptr;   // [experts, width] BF16
  const float *logits = nullptr;
  std::size_t logit_stride = 0;
  std::size_t rows = 0, width = 0, experts = 0, top = 0;
  int *expert = nullptr;          // [rows * top]
  float *score = nullptr;         // [rows * top]
  // with counts (zeroed by the launch): counts[e] = rows that chose e, rank = a pair's place among them
  int *counts = nullptr, *rank = nullptr;
};
int route_rows(const RouteArgs &args, cudaStream_t stream);
// Rows grouped by expert: expert e owns whole tiles of tile_rows rows of `grouped`, in the order of the experts.
// grouped[slot[pair], :] = input[pair / top, :], slot_score[slot[pair]] = score[pair]; tile_group[t] = expert of
// tile t, *tile_count = tiles in use (at most grouped_tiles()).  Rows that fill up a tile are left as they are.
struct GroupRowsArgs {
  const void *input = nullptr;
  Activation type = Activation::kBf16;
  std::size_t rows = 0, width = 0, experts = 0, top = 0, tile_rows = 128;
  const int *expert = nullptr, *rank = nullptr, *counts = nullptr;
  const float *score = nullptr;
  void *grouped = nullptr;
  float *slot_score = nullptr;
  int *slot = nullptr, *tile_group = nullptr, *tile_count = nullptr;
};
int group_rows(const GroupRowsArgs &args, cudaStream_t stream);
inline std::size_t grouped_tiles(const std::size_t rows, const std::size_t top, const std::size_t experts,
                                 const std::size_t tile_rows) {
  const std::size_t pairs = rows * top;
  return pairs / tile_rows + (pairs < experts ? pairs : experts);
}

// ---- latent_attention.cu
// Row r of `projection` ([rows, stride]) holds the query latent at column 0 and the key/value latent at
// latent_column.  Both are RMS-normed with their gains: the first goes to query_latent [rows, query_rank], the
// second to row position + r of the cache [capacity, latent_rank].
struct LatentNormArgs {
  const void *projection = nullptr;
  std::size_t stride = 0, latent_column = 0;
  const float *query_gain = nullptr, *latent_gain = nullptr;
  void *query_latent = nullptr, *cache = nullptr;
  std::size_t rows = 0, position = 0, capacity = 0, query_rank = 0, latent_rank = 0;
  float epsilon = 1e-6F;
  Activation type = Activation::kBf16;
  const int *dynamic_position = nullptr;
};
int latent_norm_append(const LatentNormArgs &args, cudaStream_t stream);
// Few rows: the per-head up projections moved to the query and output side, so that attention runs on the
// cached latents themselves.  absorbed[r, h, :] = sum_d query[r, h, d] key_up[h * dim + d, :], and
// output[r, h, d] = value_up[h * value_dim + d, :] . mixed[r, h, :].  At most kLatentRows rows.
constexpr std::size_t kLatentRows = 8;
int absorb_queries(const void *query, const void *key_up, std::size_t rows, std::size_t heads, std::size_t dim,
                   std::size_t latent_rank, void *absorbed, Activation type, cudaStream_t stream);
int expand_values(const void *mixed, const void *value_up, std::size_t rows, std::size_t heads, std::size_t value_dim,
                  std::size_t latent_rank, void *output, Activation type, cudaStream_t stream);

// ---- attention_window.cu
// Row r of `projection` ([rows, stride]) holds query heads at column 0, key heads at key_column, value heads
// at value_column.  Queries and keys are RMS-normed per head with their gains; queries go to
// query [rows, heads, dim], keys and values to row position + r of the caches.
struct HeadNormArgs {
  const void *projection = nullptr;
  std::size_t stride = 0, key_column = 0, value_column = 0;
  const float *query_gain = nullptr, *key_gain = nullptr;
  void *query = nullptr, *key_cache = nullptr, *value_cache = nullptr;
  std::size_t rows = 0, position = 0, capacity = 0, heads = 0, kv_heads = 0, dim = 0, value_dim = 0;
  float epsilon = 1e-6F;
  Activation type = Activation::kBf16;
  const int *dynamic_position = nullptr;
};
int head_norm_append(const HeadNormArgs &args, cudaStream_t stream);

// Softmax attention of `rows` queries at positions position .. against the cached keys.  Query i sees key
// j <= i if i - j < window (window 0: no limit) or j < keep_first.  score = softcap tanh(q.k scale / softcap)
// (softcap 0: plain) - distance_bias[head, i - j] (optional); with `sink` the softmax denominator has one
// more term exp(sink_logit[head]) (exp(0) without sink_logit) that has no value.  Head h uses key/value head h / (heads / kv_heads).  output[r, h, :] is
// multiplied by sigmoid(gate[r * gate_stride + h]) when a gate is given.  Heads above kDecoderMaxHeadDim (up to
// kDecoderMaxLatent) run in the row kernel only.
struct WindowAttentionArgs {
  const void *query = nullptr, *key_cache = nullptr, *value_cache = nullptr;
  const void *gate = nullptr;
  std::size_t gate_stride = 0;
  const float *distance_bias = nullptr;
  std::size_t bias_stride = 0;
  void *output = nullptr;
  std::size_t rows = 0, position = 0, capacity = 0, heads = 0, kv_heads = 0, dim = 0, value_dim = 0;
  std::size_t window = 0, keep_first = 0;
  float scale = 1.0F, softcap = 0.0F;
  bool sink = false;
  const float *sink_logit = nullptr;  // [heads]
  Activation type = Activation::kBf16;
  const int *dynamic_position = nullptr;
  // tests: 1 the row kernel, 2 the tile kernel, 3 the tcgen05 kernel, 4 the latent kernel (refused where it does not apply)
  int force = 0;
};
int window_attention(const WindowAttentionArgs &args, cudaStream_t stream);
// attention_tcgen05_k64.cu: the same contract on the tensor cores (BF16, head sizes up to 128 in steps of 8).
bool window_attention_tcgen05_applicable(const WindowAttentionArgs &args);
int window_attention_tcgen05(const WindowAttentionArgs &args, cudaStream_t stream);
// latent_attention.cu: the same contract for a few BF16 queries of all heads to one shared head whose keys are its
// values (latents of up to 512 columns in steps of 64), plain softmax in a window, with or without sinks.
bool latent_decode_applicable(const WindowAttentionArgs &args);
int latent_decode(const WindowAttentionArgs &args, cudaStream_t stream);

// ---- recurrent_mixers.cu
// Both recurrences keep one F32 state [heads, dim, value_dim] per sequence.  `fresh` starts from zero
// instead of the state (and, for the convolution, from an empty history); the state is always left as it
// is after the last row.
//
// Gated linear attention: S_t = diag(alpha_t) S_{t-1} + k_t v_t^T, o_t = S_t^T q_t dim^-1/2 with
// alpha = sigmoid(bottleneck a2 + a2.b)^(1/tau).  q, k, v, the output gate and the decay bottleneck are
// columns of `projection`.
// Gated delta rule: S <- g S; u = beta (v - S^T k); S <- S + k u^T; o = S^T q, with q, k, v behind a short
// causal convolution per channel and SiLU, q and k made unit vectors per head (q also times dim^-1/2),
// beta = sigmoid(b), g = exp(decay_rate softplus(a + decay_shift)).
// Output of both: rms_norm(o per head) * output_norm * silu(gate), [rows, heads * value_dim].
struct RecurrentArgs {
  bool delta = false;
  const void *projection = nullptr;  // [rows, stride]
  std::size_t stride = 0, key_column = 0, value_column = 0, gate_column = 0, beta_column = 0, decay_column = 0;
  std::size_t rows = 0, heads = 0, kv_heads = 0, dim = 0, value_dim = 0;
  // delta
  const float *conv = nullptr;        // [gate_column, conv_taps]
  std::size_t conv_taps = 0;
  void *conv_history = nullptr;       // [conv_taps - 1, gate_column], type of the activations, oldest first
  const float *decay_rate = nullptr, *decay_shift = nullptr;  // [heads]
  // linear
  const float *decay_weight = nullptr;  // [decay_rank, heads * dim]
  const float *decay_bias = nullptr;    // [heads * dim]
  std::size_t decay_rank = 0;
  float tau = 1.0F;
  const float *output_norm = nullptr;  // [value_dim]
  float epsilon = 1e-6F;
  float *state = nullptr;
  bool fresh = true;
  void *workspace = nullptr;  // recurrent_workspace_bytes
  void *output = nullptr;     // [rows, heads * value_dim]
  Activation type = Activation::kBf16;
};
std::size_t recurrent_workspace_bytes(bool delta, std::size_t rows, std::size_t heads, std::size_t kv_heads,
                                      std::size_t dim, std::size_t value_dim, Activation type);
int recurrent_mixer(const RecurrentArgs &args, cudaStream_t stream);

}  // namespace evob
