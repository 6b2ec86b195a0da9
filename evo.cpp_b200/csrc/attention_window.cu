// Softmax attention of decoder blocks: grouped key/value heads, a sliding window that keeps the first
// tokens, soft-capped scores with a distance bias per head, a sink in the denominator and an output gate
// per head.  Three kernels share the contract (decoder_ops.hpp):
//   * the row kernel (few queries, decode): a cluster of CTAs splits the visible keys of one (row, head),
//     8 lanes per key, partial softmaxes merged through shared and distributed shared memory;
//   * the tile kernel (any head sizes, both activation types): 16 query rows of one head per CTA walk key
//     tiles of 32 through shared memory with F32 multiply-adds;
//   * the tcgen05 kernel (attention_tcgen05_k64.cu) for BF16 prompts.
// A query's visible keys are enumerated as [0, kept) and [low, position], low = position - window + 1 and
// kept = min(keep_first, low): nothing between is read.
#include <cooperative_groups.h>

#include "decoder_types.cuh"
#include "ops_internal.hpp"

namespace evob {
namespace {
namespace cg = cooperative_groups;

// ---------------------------------------------------------------- head norms and cache append
constexpr int kAppendThreads = 256;

// kQuads: head sizes that are multiples of four, all columns at multiples of four; a lane owns runs of four.
template <typename T, bool kQuads>
__global__ void __launch_bounds__(kAppendThreads)
head_norm_append_kernel(const T *__restrict__ projection, const std::size_t stride, const int key_column,
                        const int value_column, const float *__restrict__ query_gain,
                        const float *__restrict__ key_gain, T *__restrict__ query, T *__restrict__ key_cache,
                        T *__restrict__ value_cache, const int static_position,
                        const int *__restrict__ dynamic_position, const int capacity, const int heads,
                        const int kv_heads, const int dim, const int value_dim, const float epsilon) {
  const std::size_t row = blockIdx.x;
  const std::size_t at = (dynamic_position != nullptr ? *dynamic_position : static_position) + row;
  const T *const source = projection + row * stride;
  const int warp = threadIdx.x / 32, lane = threadIdx.x % 32;
  const float inverse_dim = 1.0F / static_cast<float>(dim);
  if (at >= static_cast<std::size_t>(capacity)) return;  // the host checks the capacity; nothing is written past it
  for (int head = warp; head < heads + 2 * kv_heads; head += kAppendThreads / 32) {
    if (head >= heads + kv_heads) {
      const int g = head - heads - kv_heads;
      T *const out = value_cache + (at * kv_heads + g) * value_dim;
      const T *const in = source + value_column + g * value_dim;
      if constexpr (kQuads) {
        for (int i = 4 * lane; i < value_dim; i += 128) {
          float v[4];
          load_quad(in + i, v);
          store_quad(out + i, v);
        }
      } else {
        for (int i = lane; i < value_dim; i += 32) out[i] = in[i];
      }
      continue;
    }
    const bool is_query = head < heads;
    const int local = is_query ? head : head - heads;
    const T *const in = source + (is_query ? 0 : key_column) + local * dim;
    const float *const gain = is_query ? query_gain : key_gain;
    T *const out = is_query ? query + (row * heads + local) * dim : key_cache + (at * kv_heads + local) * dim;
    if constexpr (kQuads) {
      constexpr int kRuns = static_cast<int>(kDecoderMaxHeadDim) / 128;
      float v[kRuns][4] = {}, square = 0.0F;
#pragma unroll
      for (int i = 0; i < kRuns; ++i) {
        const int d = 4 * lane + 128 * i;
        if (d < dim) load_quad(in + d, v[i]);
#pragma unroll
        for (int e = 0; e < 4; ++e) square = fmaf(v[i][e], v[i][e], square);
      }
      const float factor = rsqrtf(fmaf(warp_sum(square), inverse_dim, epsilon));
#pragma unroll
      for (int i = 0; i < kRuns; ++i) {
        const int d = 4 * lane + 128 * i;
        if (d >= dim) continue;
        float w[4], y[4];
        load_quad(gain + d, w);
#pragma unroll
        for (int e = 0; e < 4; ++e) y[e] = v[i][e] * factor * w[e];
        store_quad(out + d, y);
      }
    } else {
      float v[kDecoderMaxHeadDim / 32];
      float square = 0.0F;
#pragma unroll
      for (int i = 0; i < static_cast<int>(kDecoderMaxHeadDim) / 32; ++i) {
        const int d = lane + 32 * i;
        v[i] = d < dim ? to_float(in[d]) : 0.0F;
        square = fmaf(v[i], v[i], square);
      }
      square = warp_sum(square);
      const float factor = 1.0F / sqrtf(square / static_cast<float>(dim) + epsilon);
#pragma unroll
      for (int i = 0; i < static_cast<int>(kDecoderMaxHeadDim) / 32; ++i) {
        const int d = lane + 32 * i;
        if (d < dim) out[d] = from_float<T>(v[i] * factor * gain[d]);
      }
    }
  }
}

// ---------------------------------------------------------------- shared score arithmetic
struct ScoreParams {
  float scale, softcap;
  const float *bias;  // of the head, null: none
};

__device__ __forceinline__ float capped_score(const float dot, const ScoreParams &p, const int distance) {
  float s = dot * p.scale;
  if (p.softcap > 0.0F) s = p.softcap * tanhf(s / p.softcap);
  if (p.bias != nullptr) s -= __ldg(p.bias + distance);
  return s;
}

// Folds (m, l, acc) of another partial softmax into this one.
__device__ __forceinline__ void merge(float &m, float &l, float &acc, const float other_m, const float other_l,
                                      const float other_acc) {
  const float merged = fmaxf(m, other_m);
  const float mine = m == -INFINITY ? 0.0F : expf(m - merged);
  const float theirs = other_m == -INFINITY ? 0.0F : expf(other_m - merged);
  acc = acc * mine + other_acc * theirs;
  l = l * mine + other_l * theirs;
  m = merged;
}

// ---------------------------------------------------------------- row kernel
constexpr int kSplits = 8;  // CTAs per cluster
constexpr int kRowThreads = 256;
constexpr int kRowWarps = kRowThreads / 32;

struct RowParams {
  int position;
  const int *dynamic_position;
  int heads, kv_heads, dim, value_dim, window, keep_first;
  float scale, softcap;
  const float *distance_bias;
  std::size_t bias_stride, gate_stride;
  int sink;
  const float *sink_logit;  // [heads] or null: zeros
};

// Elements of a head that a lane holds: runs of kVec at ((chunk * kLanes + part) * kVec), part = lane % kLanes.
template <typename T, int kVec, int kElements, int kLanes>
__device__ __forceinline__ void load_part(const T *const head, const int part, const int dim, float (&v)[kElements]) {
#pragma unroll
  for (int c = 0; c < kElements / kVec; ++c) {
    const int base = (c * kLanes + part) * kVec;
    if constexpr (kVec == 8) {
      if (base < dim) {
        float w[8];
        load_floats<8>(head + base, w);
#pragma unroll
        for (int i = 0; i < 8; ++i) v[8 * c + i] = w[i];
      } else {
#pragma unroll
        for (int i = 0; i < 8; ++i) v[8 * c + i] = 0.0F;
      }
    } else {
      v[c] = base < dim ? to_float(head[base]) : 0.0F;
    }
  }
}

// kLanes lanes share a key; kElements * kLanes >= max(dim, value_dim)
template <typename T, int kVec, int kElements, int kLanes>
__global__ void __launch_bounds__(kRowThreads)
window_attention_row_kernel(const T *__restrict__ query, const T *__restrict__ key_cache,
                            const T *__restrict__ value_cache, const T *__restrict__ gate, T *__restrict__ output,
                            const RowParams p) {
  // a one-row projection launched with programmatic stream serialisation may start under this kernel
  asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
  constexpr int kWidth = kElements * kLanes, kGroups = 32 / kLanes;  // keys that a warp takes at once
  __shared__ float warp_partials[kRowWarps][kWidth + 2];
  __shared__ float cta_partial[kWidth + 2];
  cg::cluster_group cluster = cg::this_cluster();
  const int split = static_cast<int>(cluster.block_rank());
  const int head = blockIdx.y, row = blockIdx.z;
  const int kv = head / (p.heads / p.kv_heads);
  const int warp = threadIdx.x / 32, lane = threadIdx.x % 32;
  const int group = lane / kLanes, part = lane % kLanes;
  const int position = (p.dynamic_position != nullptr ? *p.dynamic_position : p.position) + row;
  const int low = p.window > 0 ? max(0, position - p.window + 1) : 0;
  const int kept = min(p.keep_first, low);
  const int visible = kept + position + 1 - low;
  const int per_split = (visible + kSplits - 1) / kSplits;
  const int begin = split * per_split, end = min(visible, begin + per_split);
  const ScoreParams score{p.scale, p.softcap,
                          p.distance_bias != nullptr ? p.distance_bias + head * p.bias_stride : nullptr};

  float q[kElements];
  load_part<T, kVec, kElements, kLanes>(query + (static_cast<std::size_t>(row) * p.heads + head) * p.dim, part, p.dim, q);
  float running_max = -INFINITY, running_sum = 0.0F, acc[kElements];
#pragma unroll
  for (int i = 0; i < kElements; ++i) acc[i] = 0.0F;
  for (int n0 = begin + warp * kGroups; n0 < end; n0 += kRowWarps * kGroups) {
    const int n = n0 + group;
    const bool live = n < end;
    const int key = n < kept ? n : low + (n - kept);
    float k[kElements], v[kElements];
    if (live) {
      load_part<T, kVec, kElements, kLanes>(key_cache + (static_cast<std::size_t>(key) * p.kv_heads + kv) * p.dim, part,
                                            p.dim, k);
      load_part<T, kVec, kElements, kLanes>(value_cache + (static_cast<std::size_t>(key) * p.kv_heads + kv) * p.value_dim,
                                            part, p.value_dim, v);
    } else {
#pragma unroll
      for (int i = 0; i < kElements; ++i) k[i] = v[i] = 0.0F;
    }
    float dot = 0.0F;
#pragma unroll
    for (int i = 0; i < kElements; ++i) dot = fmaf(q[i], k[i], dot);
#pragma unroll
    for (int offset = 1; offset < kLanes; offset *= 2) dot += __shfl_xor_sync(0xffffffffU, dot, offset);
    if (live) {
      const float s = capped_score(dot, score, position - key);
      const float next = fmaxf(running_max, s);
      const float correction = expf(running_max - next);  // exp(-inf) = 0 on the first key
      const float weight = expf(s - next);
      running_sum = fmaf(running_sum, correction, weight);
#pragma unroll
      for (int i = 0; i < kElements; ++i) acc[i] = fmaf(acc[i], correction, weight * v[i]);
      running_max = next;
    }
  }
  // the key groups of a warp hold partials over the same elements per part
#pragma unroll
  for (int offset = kLanes; offset <= 16; offset *= 2) {
    const float other_m = __shfl_xor_sync(0xffffffffU, running_max, offset);
    const float other_l = __shfl_xor_sync(0xffffffffU, running_sum, offset);
    const float merged = fmaxf(running_max, other_m);
    const float mine = running_max == -INFINITY ? 0.0F : expf(running_max - merged);
    const float theirs = other_m == -INFINITY ? 0.0F : expf(other_m - merged);
#pragma unroll
    for (int i = 0; i < kElements; ++i)
      acc[i] = acc[i] * mine + __shfl_xor_sync(0xffffffffU, acc[i], offset) * theirs;
    running_sum = running_sum * mine + other_l * theirs;
    running_max = merged;
  }
  if (group == 0) {
#pragma unroll
    for (int i = 0; i < kElements; ++i) warp_partials[warp][((i / kVec) * kLanes + part) * kVec + i % kVec] = acc[i];
    if (part == 0) {
      warp_partials[warp][kWidth] = running_max;
      warp_partials[warp][kWidth + 1] = running_sum;
    }
  }
  __syncthreads();
  for (int i = threadIdx.x; i < kWidth; i += kRowThreads) {
    float m = warp_partials[0][kWidth], l = warp_partials[0][kWidth + 1], a = warp_partials[0][i];
    for (int w = 1; w < kRowWarps; ++w)
      merge(m, l, a, warp_partials[w][kWidth], warp_partials[w][kWidth + 1], warp_partials[w][i]);
    cta_partial[i] = a;
    if (i == 0) {
      cta_partial[kWidth] = m;
      cta_partial[kWidth + 1] = l;
    }
  }
  cluster.sync();
  if (split == 0) {
    for (int i = threadIdx.x; i < p.value_dim; i += kRowThreads) {
      float m = cta_partial[kWidth], l = cta_partial[kWidth + 1], a = cta_partial[i];
      for (int other = 1; other < kSplits; ++other) {
        const float *const remote = cluster.map_shared_rank(cta_partial, other);
        merge(m, l, a, remote[kWidth], remote[kWidth + 1], remote[i]);
      }
      if (p.sink != 0) merge(m, l, a, p.sink_logit != nullptr ? p.sink_logit[head] : 0.0F, 1.0F, 0.0F);
      float y = a / l;
      if (gate != nullptr) y *= sigmoid_f32(to_float(gate[static_cast<std::size_t>(row) * p.gate_stride + head]));
      output[(static_cast<std::size_t>(row) * p.heads + head) * p.value_dim + i] = from_float<T>(y);
    }
  }
  cluster.sync();  // remote shared memory stays alive until rank 0 has read it
}

// ---------------------------------------------------------------- tile kernel
constexpr int kTileRows = 16, kTileKeys = 32, kTileThreads = 256;
// floats of dynamic shared memory: queries, keys (padded rows), values, scores, output
constexpr std::size_t tile_floats(const int dim, const int value_dim) {
  return static_cast<std::size_t>(kTileRows) * dim + static_cast<std::size_t>(kTileKeys) * (dim + 1) +
         static_cast<std::size_t>(kTileKeys) * value_dim + kTileRows * (kTileKeys + 1) +
         static_cast<std::size_t>(kTileRows) * value_dim;
}

template <typename T>
__global__ void __launch_bounds__(kTileThreads)
window_attention_tile_kernel(const T *__restrict__ query, const T *__restrict__ key_cache,
                             const T *__restrict__ value_cache, const T *__restrict__ gate, T *__restrict__ output,
                             const int rows, const RowParams p) {
  extern __shared__ float tile_smem[];
  float *const qs = tile_smem;
  float *const ks = qs + kTileRows * p.dim;
  float *const vs = ks + kTileKeys * (p.dim + 1);
  float *const ps = vs + kTileKeys * p.value_dim;
  float *const os = ps + kTileRows * (kTileKeys + 1);
  __shared__ float row_max[kTileRows], row_sum[kTileRows], row_scale[kTileRows];
  const int head = blockIdx.y, kv = head / (p.heads / p.kv_heads);
  const int row0 = blockIdx.x * kTileRows;
  const int live_rows = min(kTileRows, rows - row0);
  const int first = p.position + row0, last = first + live_rows - 1;  // positions of the tile's queries
  const ScoreParams score{p.scale, p.softcap,
                          p.distance_bias != nullptr ? p.distance_bias + head * p.bias_stride : nullptr};
  for (int i = threadIdx.x; i < kTileRows * p.dim; i += kTileThreads) {
    const int r = i / p.dim, d = i % p.dim;
    qs[i] = r < live_rows ? to_float(query[(static_cast<std::size_t>(row0 + r) * p.heads + head) * p.dim + d]) : 0.0F;
  }
  for (int i = threadIdx.x; i < kTileRows * p.value_dim; i += kTileThreads) os[i] = 0.0F;
  if (threadIdx.x < kTileRows) {
    row_max[threadIdx.x] = p.sink == 0 ? -INFINITY : p.sink_logit != nullptr ? p.sink_logit[head] : 0.0F;
    row_sum[threadIdx.x] = p.sink != 0 ? 1.0F : 0.0F;
  }
  const int low = p.window > 0 ? max(0, first - p.window + 1) : 0;
  const int low_tile = low / kTileKeys;
  const int kept_tiles = min((p.keep_first + kTileKeys - 1) / kTileKeys, low_tile);
  const int tiles = kept_tiles + last / kTileKeys - low_tile + 1;
  for (int t = 0; t < tiles; ++t) {
    const int key0 = (t < kept_tiles ? t : low_tile + (t - kept_tiles)) * kTileKeys;
    __syncthreads();
    for (int i = threadIdx.x; i < kTileKeys * p.dim; i += kTileThreads) {
      const int r = i / p.dim, d = i % p.dim;
      ks[r * (p.dim + 1) + d] =
          key0 + r <= last ? to_float(key_cache[(static_cast<std::size_t>(key0 + r) * p.kv_heads + kv) * p.dim + d]) : 0.0F;
    }
    for (int i = threadIdx.x; i < kTileKeys * p.value_dim; i += kTileThreads) {
      const int r = i / p.value_dim, d = i % p.value_dim;
      vs[i] = key0 + r <= last
                  ? to_float(value_cache[(static_cast<std::size_t>(key0 + r) * p.kv_heads + kv) * p.value_dim + d])
                  : 0.0F;
    }
    __syncthreads();
    // a warp computes rows warp and warp + 8; lane = key
    const int warp = threadIdx.x / 32, lane = threadIdx.x % 32;
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int r = warp + 8 * half, position = first + r, key = key0 + lane;
      const bool seen = r < live_rows && key <= position &&
                        (p.window == 0 || position - key < p.window || key < p.keep_first);
      float s = -INFINITY;
      if (seen) {
        float dot = 0.0F;
        for (int d = 0; d < p.dim; ++d) dot = fmaf(qs[r * p.dim + d], ks[lane * (p.dim + 1) + d], dot);
        s = capped_score(dot, score, position - key);
      }
      float peak = s;
#pragma unroll
      for (int offset = 16; offset > 0; offset /= 2) peak = fmaxf(peak, __shfl_xor_sync(0xffffffffU, peak, offset));
      const float old = row_max[r], next = fmaxf(old, peak);
      const float weight = seen ? expf(s - next) : 0.0F;
      const float total = warp_sum(weight);
      const float scale = next == -INFINITY ? 1.0F : expf(old - next);
      ps[r * (kTileKeys + 1) + lane] = weight;
      __syncwarp();
      if (lane == 0) {
        row_scale[r] = scale;
        row_sum[r] = fmaf(row_sum[r], scale, total);
        row_max[r] = next;
      }
    }
    __syncthreads();
    for (int i = threadIdx.x; i < kTileRows * p.value_dim; i += kTileThreads) {
      const int r = i / p.value_dim, d = i % p.value_dim;
      float o = os[i] * row_scale[r];
#pragma unroll 8
      for (int k = 0; k < kTileKeys; ++k) o = fmaf(ps[r * (kTileKeys + 1) + k], vs[k * p.value_dim + d], o);
      os[i] = o;
    }
  }
  __syncthreads();
  for (int i = threadIdx.x; i < live_rows * p.value_dim; i += kTileThreads) {
    const int r = i / p.value_dim, d = i % p.value_dim;
    float y = os[i] / row_sum[r];
    if (gate != nullptr) y *= sigmoid_f32(to_float(gate[static_cast<std::size_t>(row0 + r) * p.gate_stride + head]));
    output[(static_cast<std::size_t>(row0 + r) * p.heads + head) * p.value_dim + d] = from_float<T>(y);
  }
}

RowParams row_params(const WindowAttentionArgs &a) {
  RowParams p{};
  p.position = static_cast<int>(a.position);
  p.dynamic_position = a.dynamic_position;
  p.heads = static_cast<int>(a.heads);
  p.kv_heads = static_cast<int>(a.kv_heads);
  p.dim = static_cast<int>(a.dim);
  p.value_dim = static_cast<int>(a.value_dim);
  p.window = static_cast<int>(a.window > 0x7fffff00U ? 0 : a.window);  // beyond any position: no limit
  p.keep_first = static_cast<int>(a.keep_first > 0x7fffff00U ? 0x7fffff00U : a.keep_first);
  p.scale = a.scale;
  p.softcap = a.softcap;
  p.distance_bias = a.distance_bias;
  p.bias_stride = a.bias_stride;
  p.gate_stride = a.gate_stride;
  p.sink = a.sink ? 1 : 0;
  p.sink_logit = a.sink ? a.sink_logit : nullptr;
  return p;
}

template <typename T, int kVec, int kElements, int kLanes = 8>
int launch_rows(const WindowAttentionArgs &a, cudaStream_t stream) {
  cudaLaunchAttribute attribute{};
  attribute.id = cudaLaunchAttributeClusterDimension;
  attribute.val.clusterDim.x = kSplits;
  attribute.val.clusterDim.y = attribute.val.clusterDim.z = 1;
  cudaLaunchConfig_t config{};
  config.gridDim = dim3(kSplits, static_cast<unsigned int>(a.heads), static_cast<unsigned int>(a.rows));
  config.blockDim = dim3(kRowThreads);
  config.stream = stream;
  config.attrs = &attribute;
  config.numAttrs = 1;
  if (cudaLaunchKernelEx(&config, window_attention_row_kernel<T, kVec, kElements, kLanes>, static_cast<const T *>(a.query),
                         static_cast<const T *>(a.key_cache), static_cast<const T *>(a.value_cache),
                         static_cast<const T *>(a.gate), static_cast<T *>(a.output), row_params(a)) != cudaSuccess)
    return fail(kCuda, std::string("cannot launch the window attention row kernel: ") +
                           cudaGetErrorString(cudaGetLastError()));
  return check_launch("window attention row kernel");
}

template <typename T>
int dispatch_rows(const WindowAttentionArgs &a, cudaStream_t stream) {
  const std::size_t widest = a.dim > a.value_dim ? a.dim : a.value_dim;
  const bool vector = a.dim % 8 == 0 && a.value_dim % 8 == 0 && aligned16(a.query) && aligned16(a.key_cache) &&
                      aligned16(a.value_cache);
  if (vector) {
    if (widest <= 64) return launch_rows<T, 8, 8>(a, stream);
    if (widest <= 128) return launch_rows<T, 8, 16>(a, stream);
    if (widest <= 256) return launch_rows<T, 8, 32>(a, stream);
    if (widest <= 512) return launch_rows<T, 8, 16, 32>(a, stream);
    return launch_rows<T, 8, 32, 32>(a, stream);
  }
  if (widest <= 64) return launch_rows<T, 1, 8>(a, stream);
  if (widest <= 128) return launch_rows<T, 1, 16>(a, stream);
  if (widest <= 256) return launch_rows<T, 1, 32>(a, stream);
  return launch_rows<T, 1, 32, 32>(a, stream);
}

template <typename T>
int launch_tiles(const WindowAttentionArgs &a, cudaStream_t stream) {
  const std::size_t bytes = tile_floats(static_cast<int>(a.dim), static_cast<int>(a.value_dim)) * sizeof(float);
  if (cudaFuncSetAttribute(window_attention_tile_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                           static_cast<int>(bytes)) != cudaSuccess)
    return fail(kCuda, "cannot raise the window attention shared-memory limit");
  const dim3 grid(ceil_div_u(a.rows, kTileRows), static_cast<unsigned int>(a.heads));
  window_attention_tile_kernel<T><<<grid, kTileThreads, bytes, stream>>>(
      static_cast<const T *>(a.query), static_cast<const T *>(a.key_cache), static_cast<const T *>(a.value_cache),
      static_cast<const T *>(a.gate), static_cast<T *>(a.output), static_cast<int>(a.rows), row_params(a));
  return check_launch("window attention tile kernel");
}

}  // namespace

int head_norm_append(const HeadNormArgs &a, cudaStream_t stream) {
  if (a.projection == nullptr || a.query_gain == nullptr || a.key_gain == nullptr || a.query == nullptr ||
      a.key_cache == nullptr || a.value_cache == nullptr || a.heads == 0 || a.kv_heads == 0 || a.dim == 0 ||
      a.value_dim == 0 || a.dim > kDecoderMaxHeadDim || a.position + a.rows > a.capacity || a.capacity > 0x7fffff00U ||
      a.stride > 0x7fffff00U)
    return fail(kInvalidArgument, "head norm arguments are invalid");
  if (a.rows == 0) return kOk;
  const bool quads = a.dim % 4 == 0 && a.value_dim % 4 == 0 && a.stride % 4 == 0 && a.key_column % 4 == 0 &&
                     a.value_column % 4 == 0 && aligned16(a.projection) && aligned16(a.query) && aligned16(a.key_cache) &&
                     aligned16(a.value_cache) && aligned16(a.query_gain) && aligned16(a.key_gain);
  const auto launch = [&](auto tag) {
    using T = decltype(tag);
    const auto kernel = quads ? head_norm_append_kernel<T, true> : head_norm_append_kernel<T, false>;
    kernel<<<static_cast<unsigned int>(a.rows), kAppendThreads, 0, stream>>>(
        static_cast<const T *>(a.projection), a.stride, static_cast<int>(a.key_column),
        static_cast<int>(a.value_column), a.query_gain, a.key_gain, static_cast<T *>(a.query),
        static_cast<T *>(a.key_cache), static_cast<T *>(a.value_cache), static_cast<int>(a.position),
        a.dynamic_position, static_cast<int>(a.capacity), static_cast<int>(a.heads), static_cast<int>(a.kv_heads),
        static_cast<int>(a.dim), static_cast<int>(a.value_dim), a.epsilon);
  };
  if (a.type == Activation::kBf16) launch(bf16{});
  else launch(float{});
  return check_launch("head norm kernel");
}

int window_attention(const WindowAttentionArgs &a, cudaStream_t stream) {
  if (a.query == nullptr || a.key_cache == nullptr || a.value_cache == nullptr || a.output == nullptr ||
      a.heads == 0 || a.heads > 65535 || a.kv_heads == 0 || a.heads % a.kv_heads != 0 || a.dim == 0 ||
      a.value_dim == 0 || a.dim > kDecoderMaxLatent || a.value_dim > kDecoderMaxLatent ||
      a.position + a.rows > a.capacity || a.capacity > 0x7fffff00U || a.softcap < 0.0F ||
      (a.distance_bias != nullptr && a.bias_stride < a.position + a.rows))
    return fail(kInvalidArgument, "window attention arguments are invalid");
  if (a.rows == 0) return kOk;
  if (a.force == 3 || (a.force == 0 && a.rows >= 32)) {
    if (window_attention_tcgen05_applicable(a)) return window_attention_tcgen05(a, stream);
    if (a.force == 3) return fail(kUnsupported, "the tensor-core attention kernel does not take these sizes");
  }
  if (a.force == 4 || (a.force == 0 && a.rows <= kLatentRows && latent_decode_applicable(a))) return latent_decode(a, stream);
  const bool wide = a.dim > kDecoderMaxHeadDim || a.value_dim > kDecoderMaxHeadDim;
  if (a.force == 1 || (a.force == 0 && (a.rows <= 8 || wide))) {
    if (a.rows > 65535) return fail(kInvalidArgument, "too many rows for the row kernel");
    return a.type == Activation::kBf16 ? dispatch_rows<bf16>(a, stream) : dispatch_rows<float>(a, stream);
  }
  if (a.dynamic_position != nullptr) return fail(kInvalidArgument, "replayed attention launches take few rows");
  if (wide) return fail(kUnsupported, "the tile kernel does not take heads of this size");
  return a.type == Activation::kBf16 ? launch_tiles<bf16>(a, stream) : launch_tiles<float>(a, stream);
}

}  // namespace evob
