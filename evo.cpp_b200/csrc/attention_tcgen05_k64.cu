// Causal prefill attention for head size 128 on the 5th-generation tensor
// cores, two CTAs per SM: softmax(Q K^T / sqrt(128)) V with query i seeing keys
// 0 .. prefix + i (the contract of upstream's FlashAttention-2 call,
// src/cuda/flash_attention.cu:199-441).
//
// The one-CTA-per-SM kernel (attention_tcgen05.cu) is a latency chain: its eight
// softmax warps walk TMEM load -> row maximum -> exchange -> exp2 -> P store in
// lock-step and the tensor core waits for them.  Here a CTA still owns 128 query
// rows of one head but
//   * walks 64-key tiles, so Q (32 KiB), two K stages and two V stages
//     (16 KiB each) are 96 KiB and two CTAs share an SM: while one CTA's
//     softmax runs, the other's MMAs do;
//   * keeps P in TMEM: the BF16 probabilities overwrite the first half of the
//     row's scores (tcgen05.st) and are the A operand of P_j V_j from there, so P
//     costs no shared-memory write, read or proxy fence - shared-memory bandwidth
//     (Q and K_j for the scores, V_j, the TMA writes) is what bounds the kernel;
//   * keeps O in TMEM for the whole walk: P_j V_j accumulates in place, and the
//     accumulator is rescaled (TMEM load, multiply, TMEM store) only when a
//     row's reference maximum moves up by more than 2^8 - rows whose reference
//     holds multiply by one.  A thread therefore carries no output accumulator
//     (the other kernel spends 64 registers and 64 FMAs per tile on it);
//   * the row's reference, not its running maximum, is what the probabilities
//     are taken against: p = 2^((s - ref) / sqrt(128) * log2 e) <= 2^8, the same
//     value after the final division by the row sum.
// Warp roles: warp 0 TMA producer (K and V two stages deep), warp 1 MMA issuer (one
// lane each), warps 2-5 softmax: a thread owns one query row - its TMEM lane -
// so the row maximum and the row sum are its own (no exchange between warps),
// with the scale-and-shift and the sums as packed F32 pairs.  Every wait is
// time-bounded and raises the sticky error word of the projection kernels.
//
// The same walk with kWindow is the window attention of decoder blocks (window_attention, decoder_ops.hpp):
// head sizes 64 .. 128 in steps of 8 (the tensor maps are [rows, heads, dim], so a box that reaches past a
// head's end reads zeros), grouped key/value heads, only the key tiles that the window and the kept first
// tokens touch, scores capped by tanh and lowered by a distance table, a sink in the row sum and a sigmoid
// gate per row and head on the output.
#include <cuda.h>

#include "common.cuh"
#include "decoder_types.cuh"
#include "ops_internal.hpp"
#include "projection_featurizer.cuh"  // round_pair_bf16
#include "tcgen05.cuh"

namespace evob {
namespace {
using namespace tc;

constexpr int kRows = 128;                      // query rows per CTA = head dimensions
constexpr int kKeys = 64;                       // keys per tile
constexpr int kThreads = 64 + 128;              // TMA warp, MMA warp, four softmax warps (a thread = a query row)
constexpr int kQHalfBytes = kRows * 128;        // one 64-column box of Q: 128 rows x 128 bytes
constexpr int kQBytes = 2 * kQHalfBytes;
constexpr int kKvHalfBytes = kKeys * 128;       // one 64-column box of K or V: 64 keys x 128 bytes
constexpr int kKvBytes = 2 * kKvHalfBytes;
constexpr int kQOffset = 0;
constexpr int kKOffset = kQOffset + kQBytes;    // two stages
constexpr int kVOffset = kKOffset + 2 * kKvBytes;  // two stages
constexpr int kBarrierOffset = kVOffset + 2 * kKvBytes;
enum Barrier : int {
  kQFull = 0, kKFull = 1, kKEmpty = 3, kVFull = 5, kVEmpty = 7, kSFull = 9, kPFull = 11, kOFull = 12, kBarriers = 13
};
constexpr int kTmemPtrOffset = kBarrierOffset + kBarriers * 8;
constexpr int kAbortOffset = kTmemPtrOffset + 8;
constexpr int kSmemBytes = kAbortOffset + 16;  // no slack: the kernel checks the 1024-byte alignment it asked for
static_assert(2 * (kSmemBytes + 1024) <= 228 * 1024, "two CTAs per SM");
constexpr std::uint32_t kTmemColumns = 256;  // S0 | S1 (64 each; P_j replaces the first 32 columns of S_j) | O (128)
constexpr std::uint32_t kScoreColumns = kKeys;
// A reference maximum is replaced only when the tile's maximum exceeds it by this many doublings.
constexpr float kLazyDoublings = 8.0F;

// V tile as the B operand of O += P V: N (head dimension) is the contiguous
// direction.  64-column boxes are one box apart (leading offset), groups of
// eight keys 1 KiB apart (stride offset).
__device__ __forceinline__ std::uint64_t v_descriptor(const std::uint32_t address) {
  std::uint64_t desc = 0;
  desc |= static_cast<std::uint64_t>((address & 0x3ffffU) >> 4U);
  desc |= static_cast<std::uint64_t>(kKvHalfBytes >> 4U) << 16U;  // LBO
  desc |= static_cast<std::uint64_t>(1024U >> 4U) << 32U;         // SBO
  desc |= static_cast<std::uint64_t>(1U) << 46U;                  // version
  desc |= static_cast<std::uint64_t>(2U) << 61U;                  // SWIZZLE_128B
  return desc;
}

__host__ __device__ constexpr std::uint32_t instruction_descriptor(const int n, const bool b_mn_major) {
  std::uint32_t d = 0;
  d |= 1U << 4U;                       // accumulator F32
  d |= 1U << 7U;                       // A BF16
  d |= 1U << 10U;                      // B BF16
  d |= (b_mn_major ? 1U : 0U) << 16U;  // B major
  d |= static_cast<std::uint32_t>(n >> 3) << 17U;
  d |= static_cast<std::uint32_t>(kRows >> 4) << 24U;  // M = 128
  return d;
}

__device__ __forceinline__ float max3(const float a, const float b, const float c) {
  float d;
  asm("max.f32 %0, %1, %2, %3;" : "=f"(d) : "f"(a), "f"(b), "f"(c));
  return d;
}
__device__ __forceinline__ float fast_exp2(const float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// D[tmem] (+)= A[tmem] * B[smem]: the A operand (M x 16 BF16, two per 32-bit column) is read from
// tensor memory.
__device__ __forceinline__ void tc_mma_a_tmem(const std::uint32_t tmem_d, const std::uint32_t tmem_a,
                                              const std::uint64_t desc_b, const std::uint32_t idesc,
                                              const std::uint32_t accumulate) {
  asm volatile(
      "{\n\t.reg .pred p;\n\tsetp.ne.b32 p, %4, 0;\n\t"
      "tcgen05.mma.cta_group::1.kind::f16 [%0], [%1], %2, %3, p;\n\t}" ::"r"(tmem_d),
      "r"(tmem_a), "l"(desc_b), "r"(idesc), "r"(accumulate)
      : "memory");
}
__device__ __forceinline__ void tmem_store_32(const std::uint32_t taddr, const std::uint32_t (&v)[32]) {
  asm volatile(
      "tcgen05.st.sync.aligned.32x32b.x32.b32 [%0], "
      "{%1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15, %16, "
      "%17, %18, %19, %20, %21, %22, %23, %24, %25, %26, %27, %28, %29, %30, %31, %32};" ::"r"(taddr),
      "r"(v[0]), "r"(v[1]), "r"(v[2]), "r"(v[3]), "r"(v[4]), "r"(v[5]), "r"(v[6]), "r"(v[7]), "r"(v[8]), "r"(v[9]),
      "r"(v[10]), "r"(v[11]), "r"(v[12]), "r"(v[13]), "r"(v[14]), "r"(v[15]), "r"(v[16]), "r"(v[17]), "r"(v[18]),
      "r"(v[19]), "r"(v[20]), "r"(v[21]), "r"(v[22]), "r"(v[23]), "r"(v[24]), "r"(v[25]), "r"(v[26]), "r"(v[27]),
      "r"(v[28]), "r"(v[29]), "r"(v[30]), "r"(v[31])
      : "memory");
}
// Packed F32 pairs: one instruction for two lanes of F32 arithmetic.
__device__ __forceinline__ unsigned long long pack_f32x2(const float low, const float high) {
  unsigned long long d;
  asm("mov.b64 %0, {%1, %2};" : "=l"(d) : "f"(low), "f"(high));
  return d;
}
__device__ __forceinline__ void unpack_f32x2(const unsigned long long pair, float &low, float &high) {
  asm("mov.b64 {%0, %1}, %2;" : "=f"(low), "=f"(high) : "l"(pair));
}
__device__ __forceinline__ unsigned long long fma_f32x2(const unsigned long long a, const unsigned long long b,
                                                        const unsigned long long c) {
  unsigned long long d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
  return d;
}
__device__ __forceinline__ unsigned long long add_f32x2(const unsigned long long a, const unsigned long long b) {
  unsigned long long d;
  asm("add.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
  return d;
}
__device__ __forceinline__ void tmem_load_16(const std::uint32_t taddr, std::uint32_t (&v)[16]) {
  asm volatile(
      "tcgen05.ld.sync.aligned.32x32b.x16.b32 "
      "{%0, %1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15}, [%16];"
      : "=r"(v[0]), "=r"(v[1]), "=r"(v[2]), "=r"(v[3]), "=r"(v[4]), "=r"(v[5]), "=r"(v[6]), "=r"(v[7]), "=r"(v[8]),
        "=r"(v[9]), "=r"(v[10]), "=r"(v[11]), "=r"(v[12]), "=r"(v[13]), "=r"(v[14]), "=r"(v[15])
      : "r"(taddr)
      : "memory");
}
__device__ __forceinline__ void tmem_store_16(const std::uint32_t taddr, const std::uint32_t (&v)[16]) {
  asm volatile(
      "tcgen05.st.sync.aligned.32x32b.x16.b32 [%0], "
      "{%1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15, %16};" ::"r"(taddr),
      "r"(v[0]), "r"(v[1]), "r"(v[2]), "r"(v[3]), "r"(v[4]), "r"(v[5]), "r"(v[6]), "r"(v[7]), "r"(v[8]), "r"(v[9]),
      "r"(v[10]), "r"(v[11]), "r"(v[12]), "r"(v[13]), "r"(v[14]), "r"(v[15])
      : "memory");
}
__device__ __forceinline__ void tmem_store_wait() { asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory"); }

struct WindowParams {
  int kv_heads, dim, value_dim, window, keep_first;
  float scale, softcap;
  const float *distance_bias;  // [heads, bias_stride] or null
  std::size_t bias_stride;
  const bf16 *gate;            // [rows, gate_stride] or null
  std::size_t gate_stride;
  int sink;
  const float *sink_logit;     // [heads] or null: zeros
};

__device__ __forceinline__ float fast_reciprocal(const float x) {
  float y;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// kCausal: plain softmax over every earlier key.  kWindow: window attention with the running row maximum.
// kCapped: window attention whose scores a soft cap keeps inside +-kMaxCap in base-2 units: F32 sums and BF16
// probabilities hold 2^score as it is, so there is no row maximum, no reference and no rescaling of O.
enum class Form { kCausal, kWindow, kCapped };
constexpr float kMaxCap = 100.0F;

// tanh for |x| <= 1/2 by its Taylor series up to x^11 (the next term is below 5e-7), two at a time; cap is
// multiplied in.
constexpr float kSeriesLimit = 0.5F;
__device__ __forceinline__ unsigned long long mul_f32x2(const unsigned long long a, const unsigned long long b) {
  unsigned long long d;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
  return d;
}

template <Form kForm>
__global__ void __launch_bounds__(kThreads, 2)
flash_tcgen05_k64_kernel(const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_k,
                         const __grid_constant__ CUtensorMap map_v, bf16 *const output, const int rows,
                         const int total_keys, const int heads, const WindowParams w, int *const error_word) {
  constexpr bool kWindow = kForm != Form::kCausal;
  extern __shared__ __align__(1024) unsigned char smem[];
  const std::uint32_t smem_base = smem_u32(smem);
  auto bar = [&](const int index) { return smem_base + kBarrierOffset + 8U * index; };
  volatile std::uint32_t *const tmem_ptr = reinterpret_cast<volatile std::uint32_t *>(smem + kTmemPtrOffset);
  volatile int *const abort_flag = reinterpret_cast<volatile int *>(smem + kAbortOffset);
  const int warp = threadIdx.x / 32, lane = threadIdx.x % 32;

  // heaviest query blocks first
  const int q_block = static_cast<int>(gridDim.x) - 1 - static_cast<int>(blockIdx.x);
  const int head = blockIdx.y;
  const int q0 = q_block * kRows;
  const int prefix = total_keys - rows;
  // keys this block may see: 0 .. prefix + q0 + 127, inside the cache
  const int visible = min(total_keys, prefix + q0 + kRows);
  int tiles = (visible + kKeys - 1) / kKeys;
  // window form: tiles with kept first tokens, then the tiles from the first row's window on
  int kept_tiles = 0, low_tile = 0;
  if constexpr (kWindow) {
    low_tile = w.window > 0 ? max(0, prefix + q0 - w.window + 1) / kKeys : 0;
    kept_tiles = min((w.keep_first + kKeys - 1) / kKeys, low_tile);
    tiles += kept_tiles - low_tile;
  }
  const auto first_key = [&](const int j) {
    if constexpr (kWindow) return (j < kept_tiles ? j : low_tile + (j - kept_tiles)) * kKeys;
    else return j * kKeys;
  };

  if (threadIdx.x == 0) {
    mbar_init(bar(kQFull), 1);
    for (int s = 0; s < 2; ++s) {
      mbar_init(bar(kKFull + s), 1);
      mbar_init(bar(kKEmpty + s), 1);
      mbar_init(bar(kVFull + s), 1);
      mbar_init(bar(kVEmpty + s), 1);
      mbar_init(bar(kSFull + s), 1);
    }
    mbar_init(bar(kPFull), 4);
    mbar_init(bar(kOFull), 1);
    *abort_flag = (smem_base & 1023U) != 0U ? 1 : 0;  // the tiles need the alignment the declaration asks for
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
  }
  if (warp == 1) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(
                     smem_u32(const_cast<std::uint32_t *>(tmem_ptr))),
                 "r"(kTmemColumns)
                 : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const std::uint32_t tmem_base = *tmem_ptr;
  const std::uint32_t tmem_o = tmem_base + 2 * kScoreColumns;
  const bool aligned = *abort_flag == 0;

  if (!aligned) {
    // nothing is issued; the error word is raised below
  } else if (warp == 0) {
    if (lane == 0) {
      const int column = head * kRows;
      int kv_head = 0;
      if constexpr (kWindow) kv_head = head / (heads / w.kv_heads);
      const auto load_tile = [&](const std::uint32_t dst, const CUtensorMap *const map, const std::uint32_t full,
                                 const int half_bytes, const int map_head, const int row) {
        if constexpr (kWindow) {
          tma_load_3d(dst, map, full, 0, map_head, row);
          tma_load_3d(dst + half_bytes, map, full, 64, map_head, row);
        } else {
          tma_load_2d(dst, map, full, column, row);
          tma_load_2d(dst + half_bytes, map, full, column + 64, row);
        }
      };
      mbar_expect_tx(bar(kQFull), kQBytes);
      load_tile(smem_base + kQOffset, &map_q, bar(kQFull), kQHalfBytes, head, q0);
      for (int j = 0; j < tiles; ++j) {
        const int s = j & 1;
        const std::uint32_t phase = (j >> 1) & 1U;
        if (!mbar_wait(bar(kKEmpty + s), phase ^ 1U, abort_flag)) break;
        const std::uint32_t k_dst = smem_base + kKOffset + s * kKvBytes;
        mbar_expect_tx(bar(kKFull + s), kKvBytes);
        load_tile(k_dst, &map_k, bar(kKFull + s), kKvHalfBytes, kv_head, first_key(j));
        if (!mbar_wait(bar(kVEmpty + s), phase ^ 1U, abort_flag)) break;
        const std::uint32_t v_dst = smem_base + kVOffset + s * kKvBytes;
        mbar_expect_tx(bar(kVFull + s), kKvBytes);
        load_tile(v_dst, &map_v, bar(kVFull + s), kKvHalfBytes, kv_head, first_key(j));
      }
    }
  } else if (warp == 1) {
    if (lane == 0) {
      constexpr std::uint32_t idesc_scores = instruction_descriptor(kKeys, false);
      constexpr std::uint32_t idesc_output = instruction_descriptor(kRows, true);
      bool ok = mbar_wait(bar(kQFull), 0U, abort_flag);
      // S_j = Q K_j^T (M128 N64, K = 128 dimensions in eight k16 steps) into score buffer j & 1.
      // P_{j-2} sat in that buffer: its P V must have finished (which also means the scores of
      // tile j - 2 were read long ago).
      auto issue_scores = [&](const int j) -> bool {
        const int s = j & 1;
        if (!mbar_wait(bar(kKFull + s), (j >> 1) & 1U, abort_flag)) return false;
        if (j >= 2 && !mbar_wait(bar(kOFull), (j - 2) & 1U, abort_flag)) return false;
        tc_fence_after();
        const std::uint32_t k_base = smem_base + kKOffset + s * kKvBytes;
#pragma unroll
        for (int k = 0; k < 8; ++k)
          tc_mma<false>(tmem_base + s * kScoreColumns,
                        smem_descriptor(smem_base + kQOffset + (k / 4) * kQHalfBytes + (k % 4) * 32),
                        smem_descriptor(k_base + (k / 4) * kKvHalfBytes + (k % 4) * 32), idesc_scores,
                        k != 0 ? 1U : 0U);
        tc_commit(bar(kKEmpty + s));
        tc_commit(bar(kSFull + s));
        return true;
      };
      if (ok) ok = issue_scores(0);
      for (int j = 0; j < tiles && ok; ++j) {
        if (j + 1 < tiles && !issue_scores(j + 1)) break;
        const int s = j & 1;
        if (!mbar_wait(bar(kVFull + s), (j >> 1) & 1U, abort_flag)) break;
        // P_j is in tensor memory, and O is rescaled where a row needed it
        if (!mbar_wait(bar(kPFull), j & 1U, abort_flag)) break;
        tc_fence_after();
        const std::uint32_t v_base = smem_base + kVOffset + s * kKvBytes;
#pragma unroll
        for (int k = 0; k < kKeys / 16; ++k)
          // A: 16 keys of P (eight 32-bit columns of tensor memory); B: 16 key rows of V
          tc_mma_a_tmem(tmem_o, tmem_base + s * kScoreColumns + k * 8, v_descriptor(v_base + k * 16 * 128),
                        idesc_output, (j | k) != 0 ? 1U : 0U);
        tc_commit(bar(kVEmpty + s));
        tc_commit(bar(kOFull));
      }
    }
  } else {
    const int quarter = warp % 4;
    const int row = quarter * 32 + lane;  // query row inside the block = TMEM lane
    const std::uint32_t lane_base = static_cast<std::uint32_t>(quarter * 32) << 16U;
    const int position = prefix + q0 + row;  // last key this row may see
    constexpr float kLog2e = 1.4426950408889634F;
    // window form: the scores are final and in base-2 units before the maximum is taken
    const float scale_log2 = kWindow ? 1.0F : kLog2e * rsqrtf(static_cast<float>(kRows));
    const float slack = kLazyDoublings / scale_log2;  // in score units
    const unsigned long long scale_pair = pack_f32x2(scale_log2, scale_log2);
    float reference = -INFINITY, running_sum = 0.0F;
    float cap_log2 = 0.0F, score_scale = 0.0F;
    unsigned long long ratio_pair = 0ULL, minus_log2e_pair = 0ULL, series[6] = {};
    float series_scale = 0.0F;
    const float *bias_row = nullptr;
    if constexpr (kWindow) {
      if (w.sink != 0) {  // the sink is a score without a value
        reference = w.sink_logit != nullptr ? w.sink_logit[head] * kLog2e : 0.0F;
        running_sum = 1.0F;
      } else {
        reference = -3.0e38F;  // finite: a tile may hide every key from a row
      }
      cap_log2 = w.softcap * kLog2e;
      // with a cap: exponent of e^(2 s / cap) in base 2; without: the score in base 2
      score_scale = w.softcap > 0.0F ? w.scale * 2.0F * kLog2e / w.softcap : w.scale * kLog2e;
      // (rows past the last query compute on table entries inside the table and are not stored)
      if constexpr (kForm == Form::kCapped) {
        running_sum = w.sink != 0 ? 1.0F : 0.0F;
        const float ratio = w.scale / w.softcap;
        ratio_pair = pack_f32x2(ratio, ratio);
        series_scale = fabsf(ratio);
        minus_log2e_pair = pack_f32x2(-kLog2e, -kLog2e);
        const float coefficients[6] = {1.0F, -1.0F / 3.0F, 2.0F / 15.0F, -17.0F / 315.0F, 62.0F / 2835.0F, -1382.0F / 155925.0F};
#pragma unroll
        for (int i = 0; i < 6; ++i) series[i] = pack_f32x2(cap_log2 * coefficients[i], cap_log2 * coefficients[i]);
      }
      if (w.distance_bias != nullptr) bias_row = w.distance_bias + head * w.bias_stride + min(position, total_keys - 1);
    }
    bool ok = true;

    for (int j = 0; j < tiles; ++j) {
      const int s = j & 1;
      // capped form: what the distance takes off, infinity for a key that the row does not see; fetched while the
      // scores are still being multiplied
      float lowered[kForm == Form::kCapped ? kKeys : 1];
      if constexpr (kForm == Form::kCapped) {
        const int key0 = first_key(j);
        const bool partial = key0 + kKeys - 1 > prefix + q0 ||
                             (w.window > 0 && prefix + q0 + kRows - 1 - key0 >= w.window && key0 + kKeys > w.keep_first);
        const float *const bias = bias_row - key0;
        if (partial) {
          // seen: key <= position, and in the window or kept
          const int own = position - key0, oldest = w.window > 0 ? own - w.window : -1, kept = w.keep_first - key0;
          const int distance0 = min(position, total_keys - 1) - key0;
#pragma unroll
          for (int i = 0; i < kKeys; ++i) {
            const float value = bias_row != nullptr ? __ldg(bias - min(i, distance0)) : 0.0F;
            lowered[i] = i <= own && (i > oldest || i < kept) ? value : INFINITY;
          }
        } else if (bias_row != nullptr) {
#pragma unroll
          for (int i = 0; i < kKeys; ++i) lowered[i] = __ldg(bias - i);
        } else {
#pragma unroll
          for (int i = 0; i < kKeys; ++i) lowered[i] = 0.0F;
        }
      }
      if (!mbar_wait(bar(kSFull + s), (j >> 1) & 1U, abort_flag)) {
        ok = false;
        break;
      }
      tc_fence_after();
      std::uint32_t v[kKeys];
      {
        std::uint32_t chunk[2][32];
        tmem_load_32(tmem_base + s * kScoreColumns + lane_base, chunk[0]);
        tmem_load_32(tmem_base + s * kScoreColumns + lane_base + 32, chunk[1]);
        tmem_load_wait();
#pragma unroll
        for (int i = 0; i < kKeys; ++i) v[i] = chunk[i / 32][i % 32];
      }
      std::uint32_t packed[kKeys / 2];
      bool moved = false;
      float alpha = 1.0F;
      if constexpr (kForm == Form::kCapped) {
        unsigned long long partial_sum[2] = {0ULL, 0ULL};
        float largest[4] = {};
#pragma unroll
        for (int i = 0; i < kKeys; i += 2)
          largest[(i / 2) % 4] = max3(largest[(i / 2) % 4], fabsf(__uint_as_float(v[i])), fabsf(__uint_as_float(v[i + 1])));
        const bool wide = fmaxf(fmaxf(largest[0], largest[1]), fmaxf(largest[2], largest[3])) * series_scale > kSeriesLimit;
        const auto finish = [&](const int i, const unsigned long long capped) {
          float low, high;
          unpack_f32x2(fma_f32x2(pack_f32x2(lowered[i], lowered[i + 1]), minus_log2e_pair, capped), low, high);
          low = fast_exp2(low);
          high = fast_exp2(high);
          partial_sum[(i / 2) % 2] = add_f32x2(partial_sum[(i / 2) % 2], pack_f32x2(low, high));
          packed[i / 2] = round_pair_bf16(low, high);
        };
        if (__any_sync(0xffffffffU, wide)) {
#pragma unroll
          for (int i = 0; i < kKeys; i += 2) {
            float y[2];
#pragma unroll
            for (int h = 0; h < 2; ++h) {
              const float e = fast_exp2(__uint_as_float(v[i + h]) * score_scale);  // e^(2 s / cap)
              y[h] = fmaf(-2.0F * cap_log2, fast_reciprocal(e + 1.0F), cap_log2);
            }
            finish(i, pack_f32x2(y[0], y[1]));
          }
        } else {
#pragma unroll
          for (int i = 0; i < kKeys; i += 2) {
            const unsigned long long x =
                mul_f32x2(pack_f32x2(__uint_as_float(v[i]), __uint_as_float(v[i + 1])), ratio_pair);
            const unsigned long long square = mul_f32x2(x, x);
            unsigned long long y = fma_f32x2(square, series[5], series[4]);
            y = fma_f32x2(y, square, series[3]);
            y = fma_f32x2(y, square, series[2]);
            y = fma_f32x2(y, square, series[1]);
            y = fma_f32x2(y, square, series[0]);
            finish(i, mul_f32x2(y, x));
          }
        }
        float even, odd;
        unpack_f32x2(add_f32x2(partial_sum[0], partial_sum[1]), even, odd);
        running_sum += even + odd;
      } else {
        if constexpr (kWindow) {
          const int key0 = first_key(j);
          const bool partial = key0 + kKeys - 1 > prefix + q0 ||
                               (w.window > 0 && prefix + q0 + kRows - 1 - key0 >= w.window && key0 + kKeys > w.keep_first);
          if (w.softcap > 0.0F) {
#pragma unroll
            for (int i = 0; i < kKeys; ++i) {
              const float e = fast_exp2(__uint_as_float(v[i]) * score_scale);
              v[i] = __float_as_uint(fmaf(-2.0F * cap_log2, fast_reciprocal(e + 1.0F), cap_log2));  // cap tanh(s / cap)
            }
          } else {
#pragma unroll
            for (int i = 0; i < kKeys; ++i) v[i] = __float_as_uint(__uint_as_float(v[i]) * score_scale);
          }
          if (bias_row != nullptr) {
            const int distance0 = min(position, total_keys - 1) - key0;
            const float *const bias = bias_row - key0;
            if (partial) {
#pragma unroll
              for (int i = 0; i < kKeys; ++i)
                v[i] = __float_as_uint(fmaf(-kLog2e, __ldg(bias - min(i, distance0)), __uint_as_float(v[i])));
            } else {
#pragma unroll
              for (int i = 0; i < kKeys; ++i)
                v[i] = __float_as_uint(fmaf(-kLog2e, __ldg(bias - i), __uint_as_float(v[i])));
            }
          }
          if (partial) {
#pragma unroll
            for (int i = 0; i < kKeys; ++i) {
              const int key = key0 + i;
              const bool seen = key <= position && (w.window == 0 || position - key < w.window || key < w.keep_first);
              if (!seen) v[i] = 0xff800000U;  // -inf
            }
          }
        } else if (j * kKeys + kKeys - 1 > prefix + q0) {     // some key hidden from some row
#pragma unroll
          for (int i = 0; i < kKeys; ++i)
            if (j * kKeys + i > position) v[i] = 0xff800000U;  // -inf
        }
        float partial_max[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll
        for (int i = 0; i < kKeys; i += 2)
          partial_max[(i / 2) % 4] = max3(partial_max[(i / 2) % 4], __uint_as_float(v[i]), __uint_as_float(v[i + 1]));
        const float tile_max = fmaxf(fmaxf(partial_max[0], partial_max[1]), fmaxf(partial_max[2], partial_max[3]));
        moved = tile_max > reference + slack;  // true on the first tile: reference = -inf
        alpha = moved ? fast_exp2((reference - tile_max) * scale_log2) : 1.0F;
        if (moved) reference = tile_max;
        const float bias = -reference * scale_log2;
        const unsigned long long bias_pair = pack_f32x2(bias, bias);
        // probabilities and the row sum first: they need nothing from the previous tile's P V
        unsigned long long partial_sum[4] = {0ULL, 0ULL, 0ULL, 0ULL};  // (even key, odd key) pairs of F32 sums
        // in three sweeps, so that no instruction waits for the one before it
        float t[kKeys];
#pragma unroll
        for (int i = 0; i < kKeys; i += 2)
          unpack_f32x2(fma_f32x2(pack_f32x2(__uint_as_float(v[i]), __uint_as_float(v[i + 1])), scale_pair, bias_pair),
                       t[i], t[i + 1]);
#pragma unroll
        for (int i = 0; i < kKeys; ++i) t[i] = fast_exp2(t[i]);
#pragma unroll
        for (int i = 0; i < kKeys; i += 2) {
          partial_sum[(i / 2) % 4] = add_f32x2(partial_sum[(i / 2) % 4], pack_f32x2(t[i], t[i + 1]));
          packed[i / 2] = round_pair_bf16(t[i], t[i + 1]);
        }
        partial_sum[0] = add_f32x2(partial_sum[0], partial_sum[2]);
        partial_sum[1] = add_f32x2(partial_sum[1], partial_sum[3]);
        float sum_even, sum_odd, sum_even_b, sum_odd_b;
        unpack_f32x2(partial_sum[0], sum_even, sum_odd);
        unpack_f32x2(partial_sum[1], sum_even_b, sum_odd_b);
        running_sum = fmaf(running_sum, alpha, (sum_even + sum_odd) + (sum_even_b + sum_odd_b));
      }
      if (j > 0) {
        // Every warp follows the O-ready barrier tile by tile, whether it has to rescale or not: a parity
        // wait cannot tell a phase from the one two before or two after it, so a waiter that skipped
        // phases would either run ahead of a P V that has not finished or wait for one that finished
        // long ago.  Having seen P V of tile j - 1 finish also means every warp has stored its
        // probabilities of tile j - 1 (an mbarrier does not know which tile an arrival belongs to: no
        // warp may arrive for tile j while the phase of tile j - 1 is still open).
        if (!mbar_wait(bar(kOFull), (j - 1) & 1U, abort_flag)) {
          ok = false;
          break;
        }
        tc_fence_after();
        if (kForm != Form::kCapped && __any_sync(0xffffffffU, moved)) {
#pragma unroll
          for (int c = 0; c < kRows / 16; ++c) {
            std::uint32_t o[16];
            const std::uint32_t address = tmem_o + lane_base + c * 16;
            tmem_load_16(address, o);
            tmem_load_wait();
#pragma unroll
            for (int i = 0; i < 16; ++i) o[i] = __float_as_uint(__uint_as_float(o[i]) * alpha);
            tmem_store_16(address, o);
          }
        }
      }
      // BF16 P over the first 32 columns of this row's scores (all 64 are in registers by now)
      tmem_store_32(tmem_base + s * kScoreColumns + lane_base, packed);
      tmem_store_wait();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(bar(kPFull));
    }
    if (kWindow && ok && tiles > 0 && mbar_wait(bar(kOFull), (tiles - 1) & 1U, abort_flag)) {
      tc_fence_after();
      float factor = 1.0F / running_sum;
      if (w.gate != nullptr && q0 + row < rows)
        factor *= sigmoid_f32(bf2f(w.gate[static_cast<std::size_t>(q0 + row) * w.gate_stride + head]));
      bf16 *const out = output + (static_cast<std::size_t>(q0 + row) * heads + head) * w.value_dim;
#pragma unroll
      for (int c = 0; c < kRows / 32; ++c) {
        std::uint32_t o[32];
        tmem_load_32(tmem_o + lane_base + c * 32, o);  // warp-wide: before the row test
        tmem_load_wait();
#pragma unroll
        for (int q = 0; q < 4; ++q) {
          if (q0 + row < rows && c * 32 + 8 * q < w.value_dim) {
            uint4 word;
            word.x = round_pair_bf16(__uint_as_float(o[8 * q]) * factor, __uint_as_float(o[8 * q + 1]) * factor);
            word.y = round_pair_bf16(__uint_as_float(o[8 * q + 2]) * factor, __uint_as_float(o[8 * q + 3]) * factor);
            word.z = round_pair_bf16(__uint_as_float(o[8 * q + 4]) * factor, __uint_as_float(o[8 * q + 5]) * factor);
            word.w = round_pair_bf16(__uint_as_float(o[8 * q + 6]) * factor, __uint_as_float(o[8 * q + 7]) * factor);
            *reinterpret_cast<uint4 *>(out + c * 32 + 8 * q) = word;
          }
        }
      }
    }
    if (!kWindow && ok && tiles > 0 && mbar_wait(bar(kOFull), (tiles - 1) & 1U, abort_flag)) {
      tc_fence_after();
      const float inverse = 1.0F / running_sum;
      bf16 *const out = output + static_cast<std::size_t>(q0 + row) * (static_cast<std::size_t>(heads) * kRows) +
                        static_cast<std::size_t>(head) * kRows;
#pragma unroll
      for (int c = 0; c < kRows / 32; ++c) {
        std::uint32_t o[32];
        tmem_load_32(tmem_o + lane_base + c * 32, o);  // warp-wide: before the row test
        tmem_load_wait();
        if (q0 + row < rows) {
#pragma unroll
          for (int q = 0; q < 4; ++q) {
            uint4 word;
            word.x = round_pair_bf16(__uint_as_float(o[8 * q]) * inverse, __uint_as_float(o[8 * q + 1]) * inverse);
            word.y = round_pair_bf16(__uint_as_float(o[8 * q + 2]) * inverse, __uint_as_float(o[8 * q + 3]) * inverse);
            word.z = round_pair_bf16(__uint_as_float(o[8 * q + 4]) * inverse, __uint_as_float(o[8 * q + 5]) * inverse);
            word.w = round_pair_bf16(__uint_as_float(o[8 * q + 6]) * inverse, __uint_as_float(o[8 * q + 7]) * inverse);
            *reinterpret_cast<uint4 *>(out + c * 32 + 8 * q) = word;
          }
        }
      }
    }
  }

  __syncwarp();
  tc_fence_before();
  __syncthreads();
  if (*abort_flag != 0) {
    // let copies that may still be in flight land before the shared memory is recycled
    // (also reached when the dynamic shared memory did not start on a 1024-byte boundary)
    const unsigned long long start = global_timer_ns();
    while (global_timer_ns() - start < 200000ULL) __nanosleep(1000);
    if (threadIdx.x == 0) atomicOr(error_word, 1 | 8);  // bit 3: this kernel
  }
  if (warp == 1) {
    tc_fence_after();
    asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem_base), "r"(kTmemColumns)
                 : "memory");
  }
}

}  // namespace

int flash_tcgen05_attention_k64(const void *query, const void *key_cache, const void *value_cache,
                                const std::size_t rows, const std::size_t total_keys, const std::size_t heads,
                                void *output, cudaStream_t stream) {
  int status = kOk;
  int *const error = tc::error_word(&status, nullptr);
  if (error == nullptr) return status;
  const std::size_t width = heads * kRows;
  CUtensorMap map_q, map_k, map_v;
  if ((status = tc::make_bf16_tile_map(&map_q, query, rows, width, kRows)) != kOk ||
      (status = tc::make_bf16_tile_map(&map_k, key_cache, total_keys, width, kKeys)) != kOk ||
      (status = tc::make_bf16_tile_map(&map_v, value_cache, total_keys, width, kKeys)) != kOk)
    return status;
  if (cudaFuncSetAttribute(flash_tcgen05_k64_kernel<Form::kCausal>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                           kSmemBytes) != cudaSuccess ||
      cudaFuncSetAttribute(flash_tcgen05_k64_kernel<Form::kCausal>, cudaFuncAttributePreferredSharedMemoryCarveout,
                           cudaSharedmemCarveoutMaxShared) != cudaSuccess)
    return fail(kCuda, "cannot raise the attention shared-memory limit");
  const dim3 grid(ceil_div_u(rows, kRows), static_cast<unsigned int>(heads));
  flash_tcgen05_k64_kernel<Form::kCausal><<<grid, kThreads, kSmemBytes, stream>>>(
      map_q, map_k, map_v, static_cast<bf16 *>(output), static_cast<int>(rows), static_cast<int>(total_keys),
      static_cast<int>(heads), WindowParams{}, error);
  return check_launch("tcgen05 attention kernel (64-key tiles)");
}

bool window_attention_tcgen05_applicable(const WindowAttentionArgs &a) {
  const auto takes = [](const std::size_t dim) { return dim >= 64 && dim <= static_cast<std::size_t>(kRows) && dim % 8 == 0; };
  return a.type == Activation::kBf16 && a.dynamic_position == nullptr && takes(a.dim) && takes(a.value_dim) &&
         a.rows > 0 && a.position + a.rows < 0x7fff0000U && aligned16(a.query) && aligned16(a.key_cache) &&
         aligned16(a.value_cache) && aligned16(a.output);
}

int window_attention_tcgen05(const WindowAttentionArgs &a, cudaStream_t stream) {
  int status = kOk;
  int *const error = tc::error_word(&status, nullptr);
  if (error == nullptr) return status;
  const std::size_t total_keys = a.position + a.rows;
  CUtensorMap map_q, map_k, map_v;
  if ((status = tc::make_bf16_head_map(&map_q, a.query, a.rows, a.heads, a.dim, kRows)) != kOk ||
      (status = tc::make_bf16_head_map(&map_k, a.key_cache, total_keys, a.kv_heads, a.dim, kKeys)) != kOk ||
      (status = tc::make_bf16_head_map(&map_v, a.value_cache, total_keys, a.kv_heads, a.value_dim, kKeys)) != kOk)
    return status;
  // (a sink of any size needs the running reference)
  const bool capped = a.softcap > 0.0F && a.softcap * 1.4426950408889634F <= kMaxCap &&
                      !(a.sink && a.sink_logit != nullptr);
  const auto kernel = capped ? flash_tcgen05_k64_kernel<Form::kCapped> : flash_tcgen05_k64_kernel<Form::kWindow>;
  if (cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, kSmemBytes) != cudaSuccess ||
      cudaFuncSetAttribute(kernel, cudaFuncAttributePreferredSharedMemoryCarveout, cudaSharedmemCarveoutMaxShared) !=
          cudaSuccess)
    return fail(kCuda, "cannot raise the attention shared-memory limit");
  WindowParams w{};
  w.kv_heads = static_cast<int>(a.kv_heads);
  w.dim = static_cast<int>(a.dim);
  w.value_dim = static_cast<int>(a.value_dim);
  w.window = static_cast<int>(a.window >= total_keys ? 0 : a.window);  // nothing is hidden: no limit
  w.keep_first = static_cast<int>(a.keep_first > total_keys ? total_keys : a.keep_first);
  w.scale = a.scale;
  w.softcap = a.softcap;
  w.distance_bias = a.distance_bias;
  w.bias_stride = a.bias_stride;
  w.gate = static_cast<const bf16 *>(a.gate);
  w.gate_stride = a.gate_stride;
  w.sink = a.sink ? 1 : 0;
  w.sink_logit = a.sink ? a.sink_logit : nullptr;
  const dim3 grid(ceil_div_u(a.rows, kRows), static_cast<unsigned int>(a.heads));
  kernel<<<grid, kThreads, kSmemBytes, stream>>>(
      map_q, map_k, map_v, static_cast<bf16 *>(a.output), static_cast<int>(a.rows), static_cast<int>(total_keys),
      static_cast<int>(a.heads), w, error);
  return check_launch("tcgen05 window attention kernel");
}

}  // namespace evob
