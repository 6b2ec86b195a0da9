// State of a context on one GPU (a pipeline stage) and the helpers that the block graphs share: launch and
// error macros, activation taps.  Included by model.cu (the StripedHyena2 graph and the context's public
// calls) and decoder.cu (the decoder graph).
#pragma once

#include <cuda_runtime.h>

#include <cstring>
#include <string>
#include <vector>

#include "../common.cuh"
#include "../decoder_ops.hpp"
#include "../ops_internal.hpp"
#include "model.hpp"

namespace evob {

#define EVOB_TRY(expr)                    \
  do {                                    \
    const int status__ = (expr);          \
    if (status__ != kOk) return status__; \
  } while (0)

// Runs one operator launch; when the stage is profiling, brackets it with CUDA
// events on the stage stream and files the elapsed time under `category`.
#define EVOB_OP(category, expr)           \
  do {                                    \
    s.begin_op(category);                 \
    const int status__ = (expr);          \
    s.end_op();                           \
    if (status__ != kOk) return status__; \
  } while (0)

struct DeviceGuard {
  int previous = 0;
  explicit DeviceGuard(const int device) {
    cudaGetDevice(&previous);
    cudaSetDevice(device);
  }
  ~DeviceGuard() { cudaSetDevice(previous); }
};

// Rows of history kept in front of a continuation chunk inside the activation
// buffers (>= the longest filter's reach of 127 + 2 featurizer rows, and a
// multiple of 16 so the tensor-core FIR tiles keep their alignment).
constexpr std::size_t kHistoryPad = 144;
constexpr std::size_t kSplitWorkspaceBytes = std::size_t{64} << 20;
constexpr std::size_t kQ8PageTokens = 16384;  // upstream src/cuda/model.cu:33

struct LayerState {
  float *short_cache = nullptr;  // [3D, short_taps-1]
  float *inner_cache = nullptr;  // [D, taps-1]
  float *modal_state = nullptr;  // [D, S]
  // [context, D] BF16; decoders: [context, kv_heads, dim] and [context, kv_heads, value_dim], type of the activations;
  // latent attention: [context, latent_rank], keys and values in one
  void *key_cache = nullptr, *value_cache = nullptr;
  // decoders: the last conv_taps - 1 projection rows, oldest first, and the matrix state of a recurrent mixer
  void *conv_history = nullptr;       // [conv_taps - 1, channels], type of the activations
  float *recurrent_state = nullptr;   // [heads, dim, value_dim]
  // Pipelines only: the last projection rows of the previous wavefront chunk
  // ([history_rows, 3D] BF16).  The projection arena is shared by all blocks of
  // a stage, so a block's own history is parked here between chunks.
  void *history = nullptr;
  std::size_t history_rows = 0;
  // fast-q8-kv: page p holds positions [p * kQ8PageTokens, ...); pointers are mirrored in four
  // device arrays (key codes, value codes, key scales, value scales) that the kernels index
  std::vector<void *> q8_pages[4];
  void **q8_tables = nullptr;  // [4][page_count] device
  std::size_t q8_page_count = 0;
  Q8PageTable q8_table() const {
    Q8PageTable t;
    t.key = reinterpret_cast<std::int8_t *const *>(q8_tables);
    t.value = reinterpret_cast<std::int8_t *const *>(q8_tables + q8_page_count);
    t.key_scale = reinterpret_cast<float *const *>(q8_tables + 2 * q8_page_count);
    t.value_scale = reinterpret_cast<float *const *>(q8_tables + 3 * q8_page_count);
    t.page_tokens = kQ8PageTokens;
    return t;
  }
};

struct Context::Stage {
  std::shared_ptr<StageWeights> weights;
  int device = 0;
  cudaStream_t stream = nullptr;
  cudaEvent_t done = nullptr;
  std::vector<void *> allocations;
  std::size_t arena_bytes = 0, cache_bytes = 0;
  // activations
  void *hidden = nullptr, *residual = nullptr, *normalized = nullptr, *mixer_out = nullptr;
  void *codes = nullptr, *projection = nullptr, *query = nullptr, *gated = nullptr;
  void *codes_wide = nullptr;   // [T, I] E4M3 codes of the gated MLP activations (FP8 FFN profile)
  float *row_scale = nullptr;   // [T] dequantisation factor of the row-quantised operand in flight
  void *mlp_first = nullptr, *mlp_second = nullptr;
  void *short_filtered = nullptr, *x2 = nullptr, *x1 = nullptr, *value = nullptr, *pregate = nullptr;
  float *modal_scratch = nullptr;
  // decoders with norms on the sublayers' outputs: what a sublayer adds, F32 [T, width]
  void *sublayer = nullptr;
  // latent attention: normed query latents [T, query_rank]; of up to kLatentRows rows the queries against latents and
  // the mixed latents [rows, heads, latent_rank]; expanded keys and values of the tokens that a pass sees
  void *query_latent = nullptr, *absorbed = nullptr, *latent_mix = nullptr;
  void *expanded_keys = nullptr, *expanded_values = nullptr;
  // gated feed-forwards whose gate is not applied by the projection: F32 [rows, 2 inner_columns]
  void *gate_products = nullptr;
  // mixtures of experts: rows in the experts' tiles and their results, the router's scores, per (row, place) the
  // expert, its score, the place among the expert's rows and the row's slot; the table of tiles
  void *grouped_rows = nullptr, *expert_out = nullptr;
  float *router_logits = nullptr, *pair_score = nullptr, *slot_score = nullptr;
  int *pair_expert = nullptr, *pair_rank = nullptr, *pair_slot = nullptr;
  int *expert_counts = nullptr, *tile_group = nullptr, *tile_count = nullptr;
  void *recurrent_workspace = nullptr;  // decoders: recurrent_workspace_bytes of the largest recurrent block
  void *split_workspace = nullptr;  // F32 partial sums of split-K projections (<= 128 rows)
  // fast-q8-kv: BF16 images [context, D] of the keys and values one attention block at a time
  void *kv_image_key = nullptr, *kv_image_value = nullptr;
  std::uint32_t *tokens = nullptr;
  void *logits = nullptr;
  std::vector<LayerState> layers;

  // ---- optional per-operator timing
  bool profiling = false;
  std::vector<cudaEvent_t> events;    // pairs: start, stop
  std::vector<int> event_category;    // one per pair in use
  double category_ms[kProfileCategories] = {};
  std::uint64_t category_launches[kProfileCategories] = {};

  void begin_op(const int category) {
    if (!profiling) return;
    const std::size_t pair = event_category.size();
    while (events.size() < 2 * (pair + 1)) {
      cudaEvent_t event = nullptr;
      cudaEventCreate(&event);
      events.push_back(event);
    }
    event_category.push_back(category);
    cudaEventRecord(events[2 * pair], stream);
  }
  void end_op() {
    if (!profiling || event_category.empty()) return;
    cudaEventRecord(events[2 * (event_category.size() - 1) + 1], stream);
  }
  // Call after the stream has been synchronised.
  void collect_profile() {
    for (std::size_t pair = 0; pair < event_category.size(); ++pair) {
      float ms = 0.0F;
      if (cudaEventElapsedTime(&ms, events[2 * pair], events[2 * pair + 1]) == cudaSuccess) {
        category_ms[event_category[pair]] += ms;
        ++category_launches[event_category[pair]];
      }
    }
    event_category.clear();
  }

  // Advances (or rewinds) every row-indexed activation pointer by `rows`.
  void shift_rows(const long rows, const std::size_t D, const std::size_t I) {
    const auto move = [rows](void *&pointer, const std::size_t row_bytes) {
      if (pointer != nullptr)
        pointer = static_cast<unsigned char *>(pointer) + rows * static_cast<long>(row_bytes);
    };
    for (void **p : {&hidden, &residual, &normalized, &mixer_out, &query, &x2, &x1, &value, &pregate})
      move(*p, D * 2);
    move(codes, D);
    move(codes_wide, I);
    if (row_scale != nullptr) row_scale += rows;
    move(projection, D * 6);
    move(short_filtered, D * 6);
    for (void **p : {&gated, &mlp_first, &mlp_second}) move(*p, I * 2);
  }

  // Pages of one attention block up to position `tokens_end` (exclusive); new pointers are
  // written into the device tables in stream order.
  int ensure_q8_pages(LayerState &state, const std::size_t tokens_end, const std::size_t heads,
                      const std::size_t head_dim) {
    const std::size_t needed = (tokens_end + kQ8PageTokens - 1) / kQ8PageTokens;
    if (needed > state.q8_page_count) return fail(kInvalidArgument, "quantised KV cache capacity exceeded");
    for (std::size_t page = state.q8_pages[0].size(); page < needed; ++page) {
      for (int which = 0; which < 4; ++which) {
        void *memory = nullptr;
        const std::size_t bytes = which < 2 ? kQ8PageTokens * heads * head_dim : kQ8PageTokens * heads * sizeof(float);
        const int status = allocate(&memory, bytes, &cache_bytes);
        if (status != kOk) return status;
        state.q8_pages[which].push_back(memory);
        if (cudaMemcpyAsync(state.q8_tables + which * state.q8_page_count + page, &state.q8_pages[which][page],
                            sizeof(void *), cudaMemcpyHostToDevice, stream) != cudaSuccess)
          return fail(kCuda, "cannot publish a quantised KV page");
      }
    }
    return kOk;
  }

  int allocate(void **out, const std::size_t bytes, std::size_t *counter) {
    if (cudaMalloc(out, bytes == 0 ? 16 : bytes) != cudaSuccess)
      return fail(kCuda, "cannot allocate " + std::to_string(bytes >> 20) + " MiB on device " +
                             std::to_string(device));
    allocations.push_back(*out);
    *counter += bytes;
    return kOk;
  }
  ~Stage() {
    DeviceGuard guard(device);
    if (stream != nullptr) cudaStreamSynchronize(stream);
    for (void *p : allocations) cudaFree(p);
    for (cudaEvent_t event : events) cudaEventDestroy(event);
    if (done != nullptr) cudaEventDestroy(done);
    if (stream != nullptr) cudaStreamDestroy(stream);
  }
};

// ---- activation taps (upstream dump_matching & friends, src/cuda/model.cu:1583-1742): device rows to F32 on
// the host, handed to every request of the plan that names (layer, point); no-ops for points nobody asked for
int emit_bf16(cudaStream_t stream, const DumpPlan &plan, std::size_t layer, DumpPoint point, const void *device,
              std::size_t rows, std::size_t columns);
// only the last `active` columns of each row are reported (FIR histories are left-padded until they fill)
int emit_f32(cudaStream_t stream, const DumpPlan &plan, std::size_t layer, DumpPoint point, const float *device,
             std::size_t rows, std::size_t columns, std::size_t active);

}  // namespace evob
