// Latent attention around the window attention kernels: the norms of the two latents with the cache append, and,
// for a few rows, the per-head up projections moved to the query and output side - q W_uk against the cached
// latents instead of expanded keys, W_uv behind the attention instead of expanded values - so that a step reads
// each cached token's latent once for all heads' keys and values.
#include "decoder_types.cuh"

namespace evob {
namespace {

constexpr int kThreads = 256;
constexpr int kWarps = kThreads / 32;

// CTA (row, which): the row's query latent or its key/value latent.
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

}  // namespace evob
