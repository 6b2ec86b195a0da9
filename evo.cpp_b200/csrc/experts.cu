// Mixture of experts around the projections: the router's scores and choice, and the regrouping of rows so that
// every expert owns whole row tiles.  The products themselves are grouped projections (LinearArgs) and the sum
// over a row's experts is taken by the norm behind them (LayerNormArgs::slots).
#include <cooperative_groups.h>

#include "decoder_types.cuh"
#include "ops_internal.hpp"

namespace evob {
namespace {
namespace cg = cooperative_groups;

constexpr int kRouteWarps = 8;
constexpr int kMaxPerLane = static_cast<int>(kDecoderMaxExperts) / 32;
constexpr int kRouterSplits = 8;  // CTAs of a cluster that share one row's products

struct Choice {
  int experts, top;
  int *expert;
  float *score;
  int *counts, *rank;
};

// The warp's row: logits[e] for e = lane, lane + 32, ...; writes the `top` best.  sigmoid is monotonic, so the
// choice is made on the logits.
template <int kPerLane>
__device__ __forceinline__ void choose(float (&logit)[kPerLane], const Choice &c, const std::size_t row, const int lane) {
  for (int place = 0; place < c.top; ++place) {
    float best = -INFINITY;
    int at = 0x7fffffff;
#pragma unroll
    for (int i = 0; i < kPerLane; ++i) {
      const int e = lane + 32 * i;
      // (also the first one: an index below `experts` whatever the values are)
      if (e < c.experts && (logit[i] > best || (at == 0x7fffffff && !(logit[i] <= -INFINITY)))) {
        best = logit[i];
        at = e;
      }
    }
#pragma unroll
    for (int offset = 16; offset > 0; offset /= 2) {
      const float other = __shfl_xor_sync(0xffffffffU, best, offset);
      const int other_at = __shfl_xor_sync(0xffffffffU, at, offset);
      if (other > best || (other == best && other_at < at)) {
        best = other;
        at = other_at;
      }
    }
    at = __shfl_sync(0xffffffffU, at, 0);
    best = __shfl_sync(0xffffffffU, best, 0);
    at = min(at, c.experts - 1);
#pragma unroll
    for (int i = 0; i < kPerLane; ++i)
      if (lane + 32 * i == at) logit[i] = -INFINITY;
    if (lane == 0) {
      const std::size_t pair = row * c.top + place;
      c.expert[pair] = at;
      c.score[pair] = sigmoid_f32(best);
      if (c.counts != nullptr) c.rank[pair] = atomicAdd(c.counts + at, 1);
    }
  }
}

template <int kPerLane>
__global__ void __launch_bounds__(32 * kRouteWarps)
route_logits_kernel(const float *__restrict__ logits, const std::size_t stride, const int rows, const Choice c) {
  const int row = blockIdx.x * kRouteWarps + threadIdx.x / 32, lane = threadIdx.x % 32;
  if (row >= rows) return;
  float logit[kPerLane];
#pragma unroll
  for (int i = 0; i < kPerLane; ++i) {
    const int e = lane + 32 * i;
    logit[i] = e < c.experts ? logits[static_cast<std::size_t>(row) * stride + e] : -INFINITY;
  }
  choose<kPerLane>(logit, c, static_cast<std::size_t>(row), lane);
}

// A cluster per row: every CTA makes its share of the products, rank 0 chooses.
template <typename T, bool kVector, int kPerLane>
__global__ void __launch_bounds__(32 * kRouteWarps)
route_rows_kernel(const T *__restrict__ input, const bf16 *__restrict__ router, const int width, const Choice c) {
  // a grouped projection launched with programmatic stream serialisation may start under this kernel
  asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
  __shared__ float logits[kDecoderMaxExperts / kRouterSplits + kRouteWarps];  // of this CTA's experts
  cg::cluster_group cluster = cg::this_cluster();
  const int split = static_cast<int>(cluster.block_rank()), warp = threadIdx.x / 32, lane = threadIdx.x % 32;
  const std::size_t row = blockIdx.y;
  const T *const x = input + row * width;
  // expert e is the CTA's number e / kRouterSplits
  for (int e = split + kRouterSplits * warp; e < c.experts; e += kRouterSplits * kRouteWarps) {
    const bf16 *const w = router + static_cast<std::size_t>(e) * width;
    float sum = 0.0F;
    if constexpr (kVector) {
#pragma unroll 4
      for (int k = 8 * lane; k < width; k += 256) {
        float a[8], b[8];
        load_floats<8>(x + k, a);
        load_floats<8>(w + k, b);
#pragma unroll
        for (int i = 0; i < 8; ++i) sum = fmaf(a[i], b[i], sum);
      }
    } else {
      for (int k = lane; k < width; k += 32) sum = fmaf(to_float(x[k]), bf2f(w[k]), sum);
    }
    sum = warp_sum(sum);
    if (lane == 0) logits[e / kRouterSplits] = sum;
  }
  cluster.sync();
  float logit[kPerLane];
  if (split == 0 && warp == 0) {
#pragma unroll
    for (int i = 0; i < kPerLane; ++i) {
      const int e = lane + 32 * i;
      logit[i] = e < c.experts ? cluster.map_shared_rank(logits, e % kRouterSplits)[e / kRouterSplits] : -INFINITY;
    }
  }
  cluster.sync();  // remote shared memory stays alive until rank 0 has read it
  if (split != 0 || warp != 0) return;
  choose<kPerLane>(logit, c, row, lane);
}

constexpr int kGroupThreads = 256;

// One CTA per pair (row, place).  Every CTA finds the first tile of each expert for itself; CTA 0 also writes the
// table of tiles.
template <typename T, bool kVector>
__global__ void __launch_bounds__(kGroupThreads)
group_rows_kernel(const T *__restrict__ input, T *__restrict__ grouped, const int width, const int experts,
                  const int top, const int tile_rows, const std::size_t pairs, const int *__restrict__ expert,
                  const int *__restrict__ rank, const int *__restrict__ counts, const float *__restrict__ score,
                  float *__restrict__ slot_score, int *__restrict__ slot, int *__restrict__ tile_group,
                  int *__restrict__ tile_count) {
  __shared__ int first_tile[kDecoderMaxExperts + 1];
  if (threadIdx.x < 32) {
    const int lane = threadIdx.x;
    int before = 0;
    for (int e0 = 0; e0 < experts; e0 += 32) {
      const int tiles = e0 + lane < experts ? (counts[e0 + lane] + tile_rows - 1) / tile_rows : 0;
      int inclusive = tiles;
#pragma unroll
      for (int offset = 1; offset < 32; offset *= 2) {
        const int other = __shfl_up_sync(0xffffffffU, inclusive, offset);
        if (lane >= offset) inclusive += other;
      }
      if (e0 + lane < experts) first_tile[e0 + lane] = before + inclusive - tiles;
      before += __shfl_sync(0xffffffffU, inclusive, 31);
    }
    if (lane == 0) first_tile[experts] = before;
  }
  __syncthreads();
  if (blockIdx.x == 0) {
    for (int e = threadIdx.x; e < experts; e += kGroupThreads)
      for (int t = first_tile[e]; t < first_tile[e + 1]; ++t) tile_group[t] = e;
    if (threadIdx.x == 0) *tile_count = first_tile[experts];
  }
  for (std::size_t pair = blockIdx.x; pair < pairs; pair += gridDim.x) {
    const std::size_t at = static_cast<std::size_t>(first_tile[expert[pair]]) * tile_rows + rank[pair];
    const T *const source = input + pair / top * width;
    T *const target = grouped + at * width;
    if constexpr (kVector) {
      constexpr int kPerWord = 16 / sizeof(T);
      for (int i = threadIdx.x; i < width / kPerWord; i += kGroupThreads)
        reinterpret_cast<uint4 *>(target)[i] = reinterpret_cast<const uint4 *>(source)[i];
    } else {
      for (int i = threadIdx.x; i < width; i += kGroupThreads) target[i] = source[i];
    }
    if (threadIdx.x == 0) {
      slot[pair] = static_cast<int>(at);
      slot_score[at] = score[pair];
    }
  }
}

template <typename T>
int launch_route_rows(const RouteArgs &a, const Choice &c, cudaStream_t stream) {
  const bool vector = a.width % 8 == 0 && aligned16(a.input) && aligned16(a.router);
  cudaLaunchAttribute attribute{};
  attribute.id = cudaLaunchAttributeClusterDimension;
  attribute.val.clusterDim.x = kRouterSplits;
  attribute.val.clusterDim.y = attribute.val.clusterDim.z = 1;
  cudaLaunchConfig_t config{};
  config.gridDim = dim3(kRouterSplits, static_cast<unsigned int>(a.rows));
  config.blockDim = dim3(32 * kRouteWarps);
  config.stream = stream;
  config.attrs = &attribute;
  config.numAttrs = 1;
  const auto kernel = a.experts <= 64 ? (vector ? route_rows_kernel<T, true, 2> : route_rows_kernel<T, false, 2>)
                                      : (vector ? route_rows_kernel<T, true, kMaxPerLane>
                                                : route_rows_kernel<T, false, kMaxPerLane>);
  if (cudaLaunchKernelEx(&config, kernel,
                         static_cast<const T *>(a.input), static_cast<const bf16 *>(a.router), static_cast<int>(a.width),
                         c) != cudaSuccess)
    return fail(kCuda, std::string("cannot launch the router kernel: ") + cudaGetErrorString(cudaGetLastError()));
  return check_launch("router kernel");
}

}  // namespace

int route_rows(const RouteArgs &a, cudaStream_t stream) {
  if ((a.logits == nullptr && (a.input == nullptr || a.router == nullptr || a.width == 0 || a.width > 0x7fffff00U)) ||
      (a.logits != nullptr && a.logit_stride < a.experts) || a.expert == nullptr || a.score == nullptr || a.experts == 0 ||
      a.experts > kDecoderMaxExperts || a.top == 0 || a.top > a.experts || a.rows > 0x7fffffffU / a.top ||
      (a.counts != nullptr && a.rank == nullptr))
    return fail(kInvalidArgument, "router arguments are invalid");
  if (a.rows == 0) return kOk;
  if (a.counts != nullptr && cudaMemsetAsync(a.counts, 0, a.experts * sizeof(int), stream) != cudaSuccess)
    return fail(kCuda, "cannot clear the router's counts");
  const Choice c{static_cast<int>(a.experts), static_cast<int>(a.top), a.expert, a.score, a.counts, a.rank};
  if (a.logits == nullptr) {
    if (a.rows > 65535) return fail(kInvalidArgument, "too many rows for the router's own products");
    return a.type == Activation::kBf16 ? launch_route_rows<bf16>(a, c, stream) : launch_route_rows<float>(a, c, stream);
  }
  const auto launch = [&](auto per_lane) {
    route_logits_kernel<decltype(per_lane)::value><<<ceil_div_u(a.rows, kRouteWarps), 32 * kRouteWarps, 0, stream>>>(
        a.logits, a.logit_stride, static_cast<int>(a.rows), c);
    return check_launch("router choice kernel");
  };
  if (a.experts <= 64) return launch(std::integral_constant<int, 2>{});
  if (a.experts <= 256) return launch(std::integral_constant<int, 8>{});
  return launch(std::integral_constant<int, kMaxPerLane>{});
}

int group_rows(const GroupRowsArgs &a, cudaStream_t stream) {
  if (a.input == nullptr || a.expert == nullptr || a.rank == nullptr || a.counts == nullptr || a.score == nullptr ||
      a.grouped == nullptr || a.slot_score == nullptr || a.slot == nullptr || a.tile_group == nullptr ||
      a.tile_count == nullptr || a.width == 0 || a.width > 0x7fffff00U || a.experts == 0 ||
      a.experts > kDecoderMaxExperts || a.top == 0 || a.tile_rows == 0 ||
      grouped_tiles(a.rows, a.top, a.experts, a.tile_rows) * a.tile_rows > 0x7fffffffU)
    return fail(kInvalidArgument, "row grouping arguments are invalid");
  if (a.rows == 0) return kOk;
  const std::size_t pairs = a.rows * a.top;
  const unsigned int grid = static_cast<unsigned int>(pairs < 16 * kSmCount ? pairs : 16 * kSmCount);
  const auto launch = [&](auto tag) {
    using T = decltype(tag);
    const bool vector = a.width * sizeof(T) % 16 == 0 && aligned16(a.input) && aligned16(a.grouped);
    const auto kernel = vector ? group_rows_kernel<T, true> : group_rows_kernel<T, false>;
    kernel<<<grid, kGroupThreads, 0, stream>>>(static_cast<const T *>(a.input), static_cast<T *>(a.grouped),
                                               static_cast<int>(a.width), static_cast<int>(a.experts),
                                               static_cast<int>(a.top), static_cast<int>(a.tile_rows), pairs, a.expert,
                                               a.rank, a.counts, a.score, a.slot_score, a.slot, a.tile_group,
                                               a.tile_count);
  };
  if (a.type == Activation::kBf16) launch(bf16{});
  else launch(float{});
  return check_launch("row grouping kernel");
}

}  // namespace evob
