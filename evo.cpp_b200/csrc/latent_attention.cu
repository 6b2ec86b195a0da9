// Latent attention around the window attention kernels: the norms of the two latents with the cache append, and,
// for a few rows, the per-head up projections moved to the query and output side - q W_uk against the cached
// latents instead of expanded keys, W_uv behind the attention instead of expanded values - so that a step reads
// each cached token's latent once for all heads' keys and values.  The attention between the two is
// latent_decode_kernel for BF16 latents of whole 64-column blocks, the row kernel of window_attention otherwise.
#include <cooperative_groups.h>

#include "decoder_types.cuh"

namespace evob {
namespace {

namespace cg = cooperative_groups;

constexpr int kThreads = 256;
constexpr int kWarps = kThreads / 32;

// Ranks that are multiples of eight, all rows 16-byte aligned.
template <typename T>
__global__ void __launch_bounds__(kThreads)
latent_norm_vector_kernel(const T *__restrict__ projection, const LatentNormArgs a) {
  // a one-row projection launched with programmatic stream serialisation may start under this kernel
  asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
  // a warp per (row, latent): neither waits for the rest of the CTA
  const std::size_t item = static_cast<std::size_t>(blockIdx.x) * kWarps + threadIdx.x / 32;
  const int lane = threadIdx.x % 32;
  const std::size_t row = item / 2;
  const bool is_query = item % 2 == 0;
  if (row >= a.rows) return;
  const int rank = static_cast<int>(is_query ? a.query_rank : a.latent_rank);
  const T *const in = projection + row * a.stride + (is_query ? 0 : a.latent_column);
  const float *const gain = is_query ? a.query_gain : a.latent_gain;
  const std::size_t at = (a.dynamic_position != nullptr ? static_cast<std::size_t>(*a.dynamic_position) : a.position) + row;
  if (!is_query && at >= a.capacity) return;  // the host checks the capacity; nothing is written past it
  T *const out = is_query ? static_cast<T *>(a.query_latent) + row * rank : static_cast<T *>(a.cache) + at * rank;
  constexpr int kKept = 4;  // groups of eight per lane that stay in registers
  float kept[kKept][8], square = 0.0F;
#pragma unroll
  for (int c = 0; c < kKept; ++c) {
    const int d = 8 * (lane + 32 * c);
    if (d < rank) {
      load_floats<8>(in + d, kept[c]);
#pragma unroll
      for (int i = 0; i < 8; ++i) square = fmaf(kept[c][i], kept[c][i], square);
    }
  }
  for (int d = 8 * (lane + 32 * kKept); d < rank; d += 256) {
    float v[8];
    load_floats<8>(in + d, v);
#pragma unroll
    for (int i = 0; i < 8; ++i) square = fmaf(v[i], v[i], square);
  }
  const float factor = 1.0F / sqrtf(warp_sum(square) / static_cast<float>(rank) + a.epsilon);
  const auto emit = [&](const int d, const float (&v)[8]) {
    float g[8], y[8];
    load_floats<8>(gain + d, g);
#pragma unroll
    for (int i = 0; i < 8; ++i) y[i] = v[i] * factor * g[i];
    store_floats(out + d, y);
  };
#pragma unroll
  for (int c = 0; c < kKept; ++c) {
    const int d = 8 * (lane + 32 * c);
    if (d < rank) emit(d, kept[c]);
  }
  for (int d = 8 * (lane + 32 * kKept); d < rank; d += 256) {
    float v[8];
    load_floats<8>(in + d, v);
    emit(d, v);
  }
}

// Any ranks.  CTA (row, which): the row's query latent or its key/value latent.
template <typename T>
__global__ void __launch_bounds__(kThreads)
latent_norm_kernel(const T *__restrict__ projection, const LatentNormArgs a) {
  // a one-row projection launched with programmatic stream serialisation may start under this kernel
  asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
  __shared__ float scratch[kWarps];
  const std::size_t row = blockIdx.x;
  const bool is_query = blockIdx.y == 0;
  const int rank = static_cast<int>(is_query ? a.query_rank : a.latent_rank);
  const T *const in = projection + row * a.stride + (is_query ? 0 : a.latent_column);
  const float *const gain = is_query ? a.query_gain : a.latent_gain;
  const std::size_t at = (a.dynamic_position != nullptr ? static_cast<std::size_t>(*a.dynamic_position) : a.position) + row;
  if (!is_query && at >= a.capacity) return;  // the host checks the capacity; nothing is written past it
  T *const out = is_query ? static_cast<T *>(a.query_latent) + row * rank : static_cast<T *>(a.cache) + at * rank;
  constexpr int kKept = 8;
  float kept[kKept], square = 0.0F;
#pragma unroll
  for (int i = 0; i < kKept; ++i) {
    const int d = threadIdx.x + i * kThreads;
    kept[i] = d < rank ? to_float(in[d]) : 0.0F;
    square = fmaf(kept[i], kept[i], square);
  }
  for (int d = threadIdx.x + kKept * kThreads; d < rank; d += kThreads) square = fmaf(to_float(in[d]), to_float(in[d]), square);
  const float mean = block_sum<kThreads>(square, scratch) / static_cast<float>(rank);
  const float factor = 1.0F / sqrtf(mean + a.epsilon);
#pragma unroll
  for (int i = 0; i < kKept; ++i) {
    const int d = threadIdx.x + i * kThreads;
    if (d < rank) out[d] = from_float<T>(kept[i] * factor * gain[d]);
  }
  for (int d = threadIdx.x + kKept * kThreads; d < rank; d += kThreads) out[d] = from_float<T>(to_float(in[d]) * factor * gain[d]);
}

// CTA (head, 8 kVec latent columns): eight threads across the columns, 32 down the head's dimensions.
template <typename T, int kVec, int kRows>
__global__ void __launch_bounds__(kThreads)
absorb_kernel(const T *__restrict__ query, const bf16 *__restrict__ key_up, T *__restrict__ absorbed, const int rows,
              const int heads, const int dim, const int rank) {
  constexpr int kColumns = 8 * kVec;
  __shared__ float partial[kWarps][kRows][kColumns];
  const int head = blockIdx.x, part = threadIdx.x % 8, down = threadIdx.x / 8;
  const int column = blockIdx.y * kColumns + part * kVec;
  float acc[kRows][kVec];
#pragma unroll
  for (int r = 0; r < kRows; ++r)
#pragma unroll
    for (int i = 0; i < kVec; ++i) acc[r][i] = 0.0F;
  if (column < rank) {
#pragma unroll 4
    for (int d = down; d < dim; d += 32) {
      const bf16 *const w = key_up + (static_cast<std::size_t>(head) * dim + d) * rank + column;
      float v[kVec];
      if constexpr (kVec == 8) load_floats<8>(w, v);
      else v[0] = bf2f(w[0]);
#pragma unroll
      for (int r = 0; r < kRows; ++r) {
        const float q = r < rows ? to_float(query[(static_cast<std::size_t>(r) * heads + head) * dim + d]) : 0.0F;
#pragma unroll
        for (int i = 0; i < kVec; ++i) acc[r][i] = fmaf(q, v[i], acc[r][i]);
      }
    }
  }
  const int warp = threadIdx.x / 32, lane = threadIdx.x % 32;
#pragma unroll
  for (int r = 0; r < kRows; ++r)
#pragma unroll
    for (int i = 0; i < kVec; ++i) {
      acc[r][i] += __shfl_xor_sync(0xffffffffU, acc[r][i], 8);
      acc[r][i] += __shfl_xor_sync(0xffffffffU, acc[r][i], 16);
      if (lane < 8) partial[warp][r][part * kVec + i] = acc[r][i];
    }
  __syncthreads();
  for (int i = threadIdx.x; i < kRows * kColumns; i += kThreads) {
    const int r = i / kColumns, c = i % kColumns, at = blockIdx.y * kColumns + c;
    if (r >= rows || at >= rank) continue;
    float sum = 0.0F;
#pragma unroll
    for (int w = 0; w < kWarps; ++w) sum += partial[w][r][c];
    absorbed[(static_cast<std::size_t>(r) * heads + head) * rank + at] = from_float<T>(sum);
  }
}

// A warp per (head, value column).
template <typename T, int kVec, int kRows>
__global__ void __launch_bounds__(kThreads)
expand_kernel(const T *__restrict__ mixed, const bf16 *__restrict__ value_up, T *__restrict__ output, const int rows,
              const int heads, const int value_dim, const int rank) {
  // a one-row projection launched with programmatic stream serialisation may start under this kernel
  asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
  const int head = blockIdx.x, column = blockIdx.y * kWarps + threadIdx.x / 32, lane = threadIdx.x % 32;
  if (column >= value_dim) return;
  const bf16 *const w = value_up + (static_cast<std::size_t>(head) * value_dim + column) * rank;
  float acc[kRows];
#pragma unroll
  for (int r = 0; r < kRows; ++r) acc[r] = 0.0F;
#pragma unroll 2
  for (int k = kVec * lane; k < rank; k += 32 * kVec) {
    float v[kVec];
    if constexpr (kVec == 8) load_floats<8>(w + k, v);
    else v[0] = bf2f(w[k]);
#pragma unroll
    for (int r = 0; r < kRows; ++r) {
      if (r >= rows) continue;
      const T *const x = mixed + (static_cast<std::size_t>(r) * heads + head) * rank + k;
      float m[kVec];
      if constexpr (kVec == 8) load_floats<8>(x, m);
      else m[0] = to_float(x[0]);
#pragma unroll
      for (int i = 0; i < kVec; ++i) acc[r] = fmaf(m[i], v[i], acc[r]);
    }
  }
#pragma unroll
  for (int r = 0; r < kRows; ++r) {
    const float sum = warp_sum(acc[r]);
    if (lane == 0 && r < rows)
      output[(static_cast<std::size_t>(r) * heads + head) * value_dim + column] = from_float<T>(sum);
  }
}

// ---------------------------------------------------------------- attention of a few queries to BF16 latents
// A cluster of kSplits CTAs owns one query row and 16 heads; its CTAs split the visible tokens.  Every token's
// latent comes into shared memory once for all 16 heads, as key and as value: scores S [16, 64] = Q C^T and
// O [16, rank] += P C are warp MMAs (m16n8k16) on the same 64-token tile, two tiles in flight.  The partial
// softmaxes are merged through distributed shared memory, every CTA a share of the columns.
constexpr int kSplits = 8;
constexpr int kHeadGroup = 16;
constexpr int kTokens = 64;           // per tile
constexpr int kWidestTile = 512;      // latent columns
constexpr int kScoreStride = kTokens + 4, kWeightStride = kTokens + 8;

struct LatentDecodeParams {
  const bf16 *query, *cache;          // [rows, heads, rank], [*, rank]
  bf16 *output;                       // [rows, heads, rank]
  int heads, rank, window, position;
  const int *dynamic_position;
  float scale;
  const float *sink_logit;
};

__host__ __device__ constexpr int latent_stride(const int rank) { return rank + 8; }  // elements of a row in shared memory
constexpr std::size_t latent_decode_smem(const int rank) {
  return static_cast<std::size_t>(2 * kTokens + kHeadGroup) * latent_stride(rank) * sizeof(bf16) +
         kHeadGroup * kScoreStride * sizeof(float) + kHeadGroup * kWeightStride * sizeof(bf16);
}

__device__ __forceinline__ std::uint32_t shared_address(const void *const p) {
  return static_cast<std::uint32_t>(__cvta_generic_to_shared(p));
}
__device__ __forceinline__ void copy16_async(void *const target, const void *const source) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(shared_address(target)), "l"(source) : "memory");
}
__device__ __forceinline__ void load_matrices(const std::uint32_t address, std::uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(address));
}
__device__ __forceinline__ void load_matrices_transposed(const std::uint32_t address, std::uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(address));
}
__device__ __forceinline__ void mma_bf16(float (&d)[4], const std::uint32_t (&a)[4], const std::uint32_t b0, const std::uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
      : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

// kBlocks = rank / 64: a warp owns 8 kBlocks output columns.
template <int kBlocks>
__global__ void __launch_bounds__(kThreads)
latent_decode_kernel(const LatentDecodeParams p) {
  constexpr int kRank = 64 * kBlocks, kStride = latent_stride(kRank);
  extern __shared__ __align__(16) unsigned char latent_smem[];
  bf16 *const tiles = reinterpret_cast<bf16 *>(latent_smem);                    // [2][kTokens][kStride]
  bf16 *const queries = tiles + 2 * kTokens * kStride;                           // [16][kStride]
  float *const scores = reinterpret_cast<float *>(queries + kHeadGroup * kStride);  // [16][kScoreStride]
  bf16 *const weights = reinterpret_cast<bf16 *>(scores + kHeadGroup * kScoreStride);  // [16][kWeightStride]
  __shared__ float head_max[kHeadGroup], head_sum[kHeadGroup], head_scale[kHeadGroup];
  cg::cluster_group cluster = cg::this_cluster();
  const int split = static_cast<int>(cluster.block_rank());
  const int head0 = blockIdx.y * kHeadGroup, row = blockIdx.z;
  const int warp = threadIdx.x / 32, lane = threadIdx.x % 32;
  const int position = (p.dynamic_position != nullptr ? *p.dynamic_position : p.position) + row;
  const int low = p.window > 0 ? max(0, position - p.window + 1) : 0;
  const int visible = position + 1 - low, per_split = (visible + kSplits - 1) / kSplits;
  const int begin = low + split * per_split, end = min(position + 1, begin + per_split);
  const int count = max(0, (end - begin + kTokens - 1) / kTokens);

  const auto fetch = [&](const int t) {
    bf16 *const target = tiles + (t & 1) * kTokens * kStride;
    const int first = begin + t * kTokens;
    for (int i = threadIdx.x; i < kTokens * (kRank / 8); i += kThreads) {
      const int token = i / (kRank / 8), part = i % (kRank / 8);
      bf16 *const slot = target + token * kStride + 8 * part;
      if (first + token < end)
        copy16_async(slot, p.cache + static_cast<std::size_t>(first + token) * kRank + 8 * part);
      else
        *reinterpret_cast<uint4 *>(slot) = make_uint4(0U, 0U, 0U, 0U);  // (a weight of zero times it stays zero)
    }
  };
  for (int i = threadIdx.x; i < kHeadGroup * (kRank / 8); i += kThreads) {
    const int head = i / (kRank / 8), part = i % (kRank / 8);
    bf16 *const slot = queries + head * kStride + 8 * part;
    if (head0 + head < p.heads)
      copy16_async(slot, p.query + (static_cast<std::size_t>(row) * p.heads + head0 + head) * kRank + 8 * part);
    else
      *reinterpret_cast<uint4 *>(slot) = make_uint4(0U, 0U, 0U, 0U);
  }
  if (count > 0) fetch(0);
  asm volatile("cp.async.commit_group;" ::: "memory");
  if (count > 1) fetch(1);
  asm volatile("cp.async.commit_group;" ::: "memory");
  if (threadIdx.x < kHeadGroup) {
    head_max[threadIdx.x] = -INFINITY;
    head_sum[threadIdx.x] = 0.0F;
  }
  float out[kBlocks][4];
#pragma unroll
  for (int n = 0; n < kBlocks; ++n)
#pragma unroll
    for (int i = 0; i < 4; ++i) out[n][i] = 0.0F;
  // addresses of the ldmatrix rows: lane l gives row l % 8 of matrix l / 8
  const std::uint32_t query_address = shared_address(queries + (lane % 16) * kStride + (lane / 16) * 8);
  const std::uint32_t weight_address = shared_address(weights + (lane % 16) * kWeightStride + (lane / 16) * 8);

  for (int t = 0; t < count; ++t) {
    asm volatile("cp.async.wait_group 1;" ::: "memory");
    __syncthreads();
    const bf16 *const tile = tiles + (t & 1) * kTokens * kStride;
    // scores of tokens 8 warp .. 8 warp + 7
    float s[4] = {0.0F, 0.0F, 0.0F, 0.0F}, s_odd[4] = {0.0F, 0.0F, 0.0F, 0.0F};  // two chains of MMAs
    const std::uint32_t key_address = shared_address(tile + (8 * warp + lane % 8) * kStride + (lane / 8) * 8);
#pragma unroll
    for (int k = 0; k < kRank / 32; ++k) {  // 32 columns: two MMAs
      std::uint32_t b[4], a0[4], a1[4];
      load_matrices(key_address + k * 64U, b);
      load_matrices(query_address + k * 64U, a0);
      load_matrices(query_address + k * 64U + 32U, a1);
      mma_bf16(s, a0, b[0], b[1]);
      mma_bf16(s_odd, a1, b[2], b[3]);
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      s[i] += s_odd[i];
      const int token = 8 * warp + 2 * (lane % 4) + i % 2, head = lane / 4 + 8 * (i / 2);
      scores[head * kScoreStride + token] = begin + t * kTokens + token < end ? s[i] * p.scale : -INFINITY;
    }
    __syncthreads();
    // a warp turns the scores of two heads into weights
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int head = warp + kWarps * half;
      const float2 pair = *reinterpret_cast<const float2 *>(scores + head * kScoreStride + 2 * lane);
      float peak = fmaxf(pair.x, pair.y);
#pragma unroll
      for (int offset = 16; offset > 0; offset /= 2) peak = fmaxf(peak, __shfl_xor_sync(0xffffffffU, peak, offset));
      const float old = head_max[head], next = fmaxf(old, peak);  // (a tile holds a visible token: next is finite)
      const float first = expf(pair.x - next), second = expf(pair.y - next);
      *reinterpret_cast<std::uint32_t *>(weights + head * kWeightStride + 2 * lane) = pack_bf16x2(first, second);
      const float total = warp_sum(first + second);
      __syncwarp();
      if (lane == 0) {
        const float scale = expf(old - next);
        head_scale[head] = scale;
        head_sum[head] = fmaf(head_sum[head], scale, total);
        head_max[head] = next;
      }
    }
    __syncthreads();
    const float scale_low = head_scale[lane / 4], scale_high = head_scale[lane / 4 + 8];
#pragma unroll
    for (int n = 0; n < kBlocks; ++n) {
      out[n][0] *= scale_low;
      out[n][1] *= scale_low;
      out[n][2] *= scale_high;
      out[n][3] *= scale_high;
    }
#pragma unroll
    for (int k = 0; k < kTokens / 16; k += 2) {  // 32 tokens
      std::uint32_t a0[4], a1[4];
      load_matrices(weight_address + k * 32U, a0);
      load_matrices(weight_address + k * 32U + 32U, a1);
#pragma unroll
      for (int n = 0; n < kBlocks; ++n) {
        std::uint32_t b[4];
        load_matrices_transposed(shared_address(tile + (16 * k + lane) * kStride + 8 * (kBlocks * warp + n)), b);
        mma_bf16(out[n], a0, b[0], b[1]);
        mma_bf16(out[n], a1, b[2], b[3]);
      }
    }
    __syncthreads();
    if (t + 2 < count) fetch(t + 2);
    asm volatile("cp.async.commit_group;" ::: "memory");
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");
  __syncthreads();
  // the partial sums replace the tiles
  float *const partial = reinterpret_cast<float *>(latent_smem);  // [16][kRank]
#pragma unroll
  for (int n = 0; n < kBlocks; ++n) {
    const int column = 8 * (kBlocks * warp + n) + 2 * (lane % 4);
    *reinterpret_cast<float2 *>(partial + (lane / 4) * kRank + column) = make_float2(out[n][0], out[n][1]);
    *reinterpret_cast<float2 *>(partial + (lane / 4 + 8) * kRank + column) = make_float2(out[n][2], out[n][3]);
  }
  cluster.sync();
  // this CTA's share of the columns, four at a time
  constexpr int kShare = kRank / kSplits / 4;
  for (int i = threadIdx.x; i < kHeadGroup * kShare; i += kThreads) {
    const int head = i / kShare, column = 4 * (split * kShare + i % kShare);
    if (head0 + head >= p.heads) continue;
    const float sink = p.sink_logit != nullptr ? p.sink_logit[head0 + head] : -INFINITY;
    float maxima[kSplits], sums[kSplits];
    float4 parts[kSplits];
#pragma unroll
    for (int other = 0; other < kSplits; ++other) {
      maxima[other] = cluster.map_shared_rank(head_max, other)[head];
      sums[other] = cluster.map_shared_rank(head_sum, other)[head];
      parts[other] = *reinterpret_cast<const float4 *>(cluster.map_shared_rank(partial, other) + head * kRank + column);
    }
    float peak = sink;
#pragma unroll
    for (int other = 0; other < kSplits; ++other) peak = fmaxf(peak, maxima[other]);
    float total = expf(sink - peak);  // 0 without a sink
    float4 mixed = make_float4(0.0F, 0.0F, 0.0F, 0.0F);
#pragma unroll
    for (int other = 0; other < kSplits; ++other) {
      const float factor = expf(maxima[other] - peak);  // 0 for a CTA without tokens
      total = fmaf(sums[other], factor, total);
      mixed.x = fmaf(parts[other].x, factor, mixed.x);
      mixed.y = fmaf(parts[other].y, factor, mixed.y);
      mixed.z = fmaf(parts[other].z, factor, mixed.z);
      mixed.w = fmaf(parts[other].w, factor, mixed.w);
    }
    const float y[4] = {mixed.x / total, mixed.y / total, mixed.z / total, mixed.w / total};
    store_quad(p.output + (static_cast<std::size_t>(row) * p.heads + head0 + head) * kRank + column, y);
  }
  cluster.sync();  // remote shared memory stays alive until every CTA has read it
}

template <int kBlocks>
int launch_latent_decode(const LatentDecodeParams &p, const std::size_t rows, cudaStream_t stream) {
  constexpr std::size_t kBytes = latent_decode_smem(64 * kBlocks);
  static_assert(kBytes + 1024 <= 227 * 1024, "fits an SM");
  if (cudaFuncSetAttribute(latent_decode_kernel<kBlocks>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                           static_cast<int>(kBytes)) != cudaSuccess)
    return fail(kCuda, "cannot raise the latent attention shared-memory limit");
  cudaLaunchAttribute attribute{};
  attribute.id = cudaLaunchAttributeClusterDimension;
  attribute.val.clusterDim.x = kSplits;
  attribute.val.clusterDim.y = attribute.val.clusterDim.z = 1;
  cudaLaunchConfig_t config{};
  config.gridDim = dim3(kSplits, ceil_div_u(static_cast<std::size_t>(p.heads), kHeadGroup), static_cast<unsigned int>(rows));
  config.blockDim = dim3(kThreads);
  config.dynamicSmemBytes = kBytes;
  config.stream = stream;
  config.attrs = &attribute;
  config.numAttrs = 1;
  if (cudaLaunchKernelEx(&config, latent_decode_kernel<kBlocks>, p) != cudaSuccess)
    return fail(kCuda, std::string("cannot launch the latent attention kernel: ") + cudaGetErrorString(cudaGetLastError()));
  return check_launch("latent attention kernel");
}

// f(T{}, kVec constant, kRows constant) for an activation type, vector width and a bound on the rows.
template <typename F>
void dispatch(const Activation type, const bool vector, const std::size_t rows, const F &f) {
  const auto with_rows = [&](auto tag, auto vec) {
    if (rows <= 1) f(tag, vec, std::integral_constant<int, 1>{});
    else if (rows <= 2) f(tag, vec, std::integral_constant<int, 2>{});
    else if (rows <= 4) f(tag, vec, std::integral_constant<int, 4>{});
    else f(tag, vec, std::integral_constant<int, 8>{});
  };
  const auto with_type = [&](auto tag) {
    if (vector) with_rows(tag, std::integral_constant<int, 8>{});
    else with_rows(tag, std::integral_constant<int, 1>{});
  };
  if (type == Activation::kBf16) with_type(bf16{});
  else with_type(float{});
}

bool sizes_ok(const std::size_t rows, const std::size_t heads, const std::size_t dim, const std::size_t rank) {
  return rows <= kLatentRows && heads > 0 && heads <= 65535 && dim > 0 && dim <= 65535 && rank > 0 &&
         rank <= kDecoderMaxLatent;
}

}  // namespace

int latent_norm_append(const LatentNormArgs &a, cudaStream_t stream) {
  if (a.projection == nullptr || a.query_gain == nullptr || a.latent_gain == nullptr || a.query_latent == nullptr ||
      a.cache == nullptr || a.query_rank == 0 || a.latent_rank == 0 || a.query_rank > 0x7fffff00U ||
      a.latent_rank > 0x7fffff00U || a.position + a.rows > a.capacity || a.rows > 0x7fffffffU)
    return fail(kInvalidArgument, "latent norm arguments are invalid");
  if (a.rows == 0) return kOk;
  const std::size_t size = activation_bytes(a.type);
  if (a.query_rank % 8 == 0 && a.latent_rank % 8 == 0 && a.stride * size % 16 == 0 && a.latent_column * size % 16 == 0 &&
      aligned16(a.projection) && aligned16(a.query_gain) && aligned16(a.latent_gain) && aligned16(a.query_latent) &&
      aligned16(a.cache)) {
    const unsigned int ctas = ceil_div_u(2 * a.rows, kWarps);
    if (a.type == Activation::kBf16)
      latent_norm_vector_kernel<<<ctas, kThreads, 0, stream>>>(static_cast<const bf16 *>(a.projection), a);
    else
      latent_norm_vector_kernel<<<ctas, kThreads, 0, stream>>>(static_cast<const float *>(a.projection), a);
    return check_launch("latent norm kernel");
  }
  const dim3 grid(static_cast<unsigned int>(a.rows), 2);
  if (a.type == Activation::kBf16)
    latent_norm_kernel<<<grid, kThreads, 0, stream>>>(static_cast<const bf16 *>(a.projection), a);
  else
    latent_norm_kernel<<<grid, kThreads, 0, stream>>>(static_cast<const float *>(a.projection), a);
  return check_launch("latent norm kernel");
}

int absorb_queries(const void *query, const void *key_up, const std::size_t rows, const std::size_t heads,
                   const std::size_t dim, const std::size_t latent_rank, void *absorbed, const Activation type,
                   cudaStream_t stream) {
  if (query == nullptr || key_up == nullptr || absorbed == nullptr || !sizes_ok(rows, heads, dim, latent_rank))
    return fail(kInvalidArgument, "query absorption arguments are invalid");
  if (rows == 0) return kOk;
  const bool vector = latent_rank % 8 == 0 && aligned16(key_up);
  dispatch(type, vector, rows, [&](auto tag, auto vec, auto bound) {
    using T = decltype(tag);
    constexpr int kVec = decltype(vec)::value;
    const dim3 grid(static_cast<unsigned int>(heads), ceil_div_u(latent_rank, 8 * kVec));
    absorb_kernel<T, kVec, decltype(bound)::value><<<grid, kThreads, 0, stream>>>(
        static_cast<const T *>(query), static_cast<const bf16 *>(key_up), static_cast<T *>(absorbed),
        static_cast<int>(rows), static_cast<int>(heads), static_cast<int>(dim), static_cast<int>(latent_rank));
  });
  return check_launch("query absorption kernel");
}

int expand_values(const void *mixed, const void *value_up, const std::size_t rows, const std::size_t heads,
                  const std::size_t value_dim, const std::size_t latent_rank, void *output, const Activation type,
                  cudaStream_t stream) {
  if (mixed == nullptr || value_up == nullptr || output == nullptr || !sizes_ok(rows, heads, value_dim, latent_rank))
    return fail(kInvalidArgument, "value expansion arguments are invalid");
  if (rows == 0) return kOk;
  const bool vector = latent_rank % 8 == 0 && aligned16(mixed) && aligned16(value_up);
  dispatch(type, vector, rows, [&](auto tag, auto vec, auto bound) {
    using T = decltype(tag);
    const dim3 grid(static_cast<unsigned int>(heads), ceil_div_u(value_dim, kWarps));
    expand_kernel<T, decltype(vec)::value, decltype(bound)::value><<<grid, kThreads, 0, stream>>>(
        static_cast<const T *>(mixed), static_cast<const bf16 *>(value_up), static_cast<T *>(output),
        static_cast<int>(rows), static_cast<int>(heads), static_cast<int>(value_dim), static_cast<int>(latent_rank));
  });
  return check_launch("value expansion kernel");
}

bool latent_decode_applicable(const WindowAttentionArgs &a) {
  return a.type == Activation::kBf16 && a.kv_heads == 1 && a.key_cache == a.value_cache && a.dim == a.value_dim &&
         a.dim % 64 == 0 && a.dim <= static_cast<std::size_t>(kWidestTile) && a.keep_first == 0 && a.softcap == 0.0F &&
         a.distance_bias == nullptr && a.gate == nullptr && (!a.sink || a.sink_logit != nullptr) && a.rows > 0 &&
         a.rows <= 65535 && a.heads <= 65535 && aligned16(a.query) && aligned16(a.key_cache) && aligned16(a.output) &&
         a.position + a.rows < 0x7fff0000U;
}

int latent_decode(const WindowAttentionArgs &a, cudaStream_t stream) {
  if (!latent_decode_applicable(a)) return fail(kUnsupported, "the latent attention kernel does not take these arguments");
  LatentDecodeParams p{};
  p.query = static_cast<const bf16 *>(a.query);
  p.cache = static_cast<const bf16 *>(a.key_cache);
  p.output = static_cast<bf16 *>(a.output);
  p.heads = static_cast<int>(a.heads);
  p.rank = static_cast<int>(a.dim);
  p.window = static_cast<int>(a.window > 0x7fffff00U ? 0 : a.window);
  p.position = static_cast<int>(a.position);
  p.dynamic_position = a.dynamic_position;
  p.scale = a.scale;
  p.sink_logit = a.sink ? a.sink_logit : nullptr;
  switch (a.dim / 64) {
    case 1: return launch_latent_decode<1>(p, a.rows, stream);
    case 2: return launch_latent_decode<2>(p, a.rows, stream);
    case 3: return launch_latent_decode<3>(p, a.rows, stream);
    case 4: return launch_latent_decode<4>(p, a.rows, stream);
    case 5: return launch_latent_decode<5>(p, a.rows, stream);
    case 6: return launch_latent_decode<6>(p, a.rows, stream);
    case 7: return launch_latent_decode<7>(p, a.rows, stream);
    default: return launch_latent_decode<8>(p, a.rows, stream);
  }
}

}  // namespace evob
