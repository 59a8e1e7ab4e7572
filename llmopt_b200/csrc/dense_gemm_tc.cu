// Prompt rows of the dense bfloat16 linear layer on the 5th-generation tensor cores:
//   y[m, n] = x[m, k] . w[n, k]^T, fp32 accumulation in tensor memory.
// With a plan the rows are sorted by expert and a tile multiplies with its expert's n rows of w [experts n, k];
// the rows of a box that belong to the next expert are computed and dropped.
//
// A persistent CTA walks over 128 x BN output tiles.  Warp 0 brings the x tile [128 x 64] and the w
// tile [BN x 64] of every k-block into a shared-memory ring by TMA (128-byte swizzle); one thread of
// warp 1 issues four tcgen05.mma (K = 16) per k-block into one of two accumulators in tensor memory;
// warps 2-9 read the finished accumulator (each its quarter of the lanes = output rows), apply bias
// and activation and store, while the next tile accumulates in the other one.  Rows, columns and k
// beyond the matrices are zero-filled by TMA.
//
// Every wait on an mbarrier is bounded; a wait that runs out raises the context's device error word,
// and the CTA lets its copies land, frees its tensor memory and returns.
#include <cuda.h>

#include <initializer_list>

#include "dense_linear.cuh"
#include "w4a16_tc_device.cuh"

namespace llmopt {
using namespace tc;

uint32_t* context_device_error(Context* ctx);

namespace {

constexpr uint32_t kRows = kExpertTile, kDepth = 64;
constexpr uint32_t kEpilogueWarps = 8;
constexpr uint32_t kThreads = (2 + kEpilogueWarps) * 32;  // TMA, MMA, epilogue
constexpr uint32_t kStagingRow = 20;  // words of a lane's values on their way out: sixteen and four of padding
// per epilogue warp; the others keep the shared memory as cache for what their writeback reads
template <DenseStore STORE>
constexpr uint32_t kStagingBytes = STORE == kStoreResidual || STORE == kStoreCached ? 32u * kStagingRow * 4u : 0u;
constexpr uint32_t kXTileBytes = kRows * kDepth * 2;

template <uint32_t BN>
struct Shape {
  static constexpr uint32_t kWTileBytes = BN * kDepth * 2;
  // 64-wide k-blocks per ring stage: a commit costs the issuing thread as much as several narrow MMAs
  static constexpr uint32_t kBlocks = BN == 256 ? 1 : 2;
  static constexpr uint32_t kStageBytes = (kXTileBytes + kWTileBytes) * kBlocks;
  static constexpr uint32_t kStages = BN == 128 ? 3 : 4;
  static constexpr uint32_t kTmemColumns = 2 * BN;
  static constexpr uint32_t kBarriers = kStages * kStageBytes;
  static constexpr uint32_t kHolder = kBarriers + (2 * kStages + 4) * 8;
  static constexpr uint32_t kAbort = kHolder + 4;
  static constexpr uint32_t kStaging = (kAbort + 4 + 15) / 16 * 16;
  static constexpr uint32_t kSharedBytes = kStaging + 1024;  // without the staging; slack: 1024-byte alignment of the tiles
};

// kind::f16 with bfloat16 A and B (format 1), fp32 accumulator, both K-major.
__host__ __device__ constexpr uint32_t bf16_instruction(uint32_t m, uint32_t n) {
  return (1u << 4) | (1u << 7) | (1u << 10) | ((n >> 3) << 17) | ((m >> 4) << 24);
}

// 32 neighbouring sums of each of a warp's 32 rows on their way out, and what they need besides, requested ahead of them.
// The sums lie a row per lane.  Plain rows leave in that order; where as much is read as written (the residual) or the target
// rows lie apart (the cache) values change places through shared memory first, so that four lanes share 64 bytes of a row.

// Sixteen words per lane -> what lane / 4 of eight rows at a time stores: take(row of the warp, four words, their place).
template <typename Take>
__device__ __forceinline__ void exchange(float* staging, const uint4 (&words)[4], Take take) {
  const uint32_t lane = threadIdx.x & 31u;
#pragma unroll
  for (int j = 0; j < 4; ++j) *reinterpret_cast<uint4*>(staging + lane * kStagingRow + j * 4) = words[j];
  __syncwarp();
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const uint32_t row = i * 8u + (lane >> 2);
    take(i, row, *reinterpret_cast<const uint4*>(staging + row * kStagingRow + (lane & 3u) * 4u), lane & 3u);
  }
  __syncwarp();  // read before the next exchange
}

template <DenseStore STORE>
struct Piece {
  __device__ __forceinline__ void fetch(const DenseTask<STORE>&, uint32_t, uint32_t, uint32_t) {}
  __device__ __forceinline__ void store(const DenseTask<STORE>& p, uint32_t first_row, uint32_t row_end, uint32_t column,
                                        const uint32_t (&raw)[32], float* staging) const {
    const uint32_t row = first_row + (threadIdx.x & 31u), kept = dense_kept(p);
    if constexpr (STORE == kStoreCached) {
      if (column >= p.split && column + 32u <= p.split + kept) {
        bf16* const cached = row < row_end ? dense_cache_row<bf16>(p, row) : nullptr;
        const uint32_t at = column - p.split, offset = dense_cache_offset(p, at);
        if ((at + 32u <= p.key_columns || at >= p.key_columns) && offset % 8u == 0 && p.token_stride % 8u == 0) {
          uint4 words[4];
#pragma unroll
          for (int j = 0; j < 4; ++j) {
            uint32_t packed[4];
#pragma unroll
            for (int e = 0; e < 4; ++e) {
              const int i = j * 8 + e * 2;
              const __nv_bfloat162 pair = __floats2bfloat162_rn(dense_biased(p, column + i, __uint_as_float(raw[i])),
                                                                dense_biased(p, column + i + 1, __uint_as_float(raw[i + 1])));
              packed[e] = *reinterpret_cast<const uint32_t*>(&pair);
            }
            words[j] = make_uint4(packed[0], packed[1], packed[2], packed[3]);
          }
          exchange(staging, words, [&](int, uint32_t r, const uint4& v, uint32_t place) {
            const unsigned long long target = __shfl_sync(0xffffffffu, (unsigned long long)(uintptr_t)cached, r);
            if (target) *reinterpret_cast<uint4*>(reinterpret_cast<bf16*>((uintptr_t)target) + offset + place * 8u) = v;
          });
          return;
        }
        if (!cached) return;
#pragma unroll
        for (int i = 0; i < 32; ++i)
          cached[dense_cache_offset(p, at + i)] = __float2bfloat16_rn(dense_biased(p, column + i, __uint_as_float(raw[i])));
        return;
      }
    }
    if (row >= row_end || column >= p.n) return;
    const size_t at = (size_t)row * p.split + column;
    const size_t at32 = (size_t)row * (p.n - p.split - kept) + (column - p.split - kept);
    auto value = [&](int i) {
      return STORE == kStoreCached ? dense_biased(p, column + i, __uint_as_float(raw[i]))
                                   : dense_finish<bf16>(p, row, column + i, __uint_as_float(raw[i]));
    };
    if (column + 32u <= p.split && (at & 7u) == 0) {
      uint4* target = reinterpret_cast<uint4*>(reinterpret_cast<bf16*>(p.out) + at);
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        uint32_t packed[4];
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const __nv_bfloat162 pair = __floats2bfloat162_rn(value(i * 8 + j * 2), value(i * 8 + j * 2 + 1));
          packed[j] = *reinterpret_cast<const uint32_t*>(&pair);
        }
        target[i] = make_uint4(packed[0], packed[1], packed[2], packed[3]);
      }
      return;
    }
    if (column >= p.split + kept && column + 32u <= p.n && (at32 & 3u) == 0) {
      float4* target = reinterpret_cast<float4*>(p.out32 + at32);
#pragma unroll
      for (int i = 0; i < 8; ++i) target[i] = make_float4(value(i * 4), value(i * 4 + 1), value(i * 4 + 2), value(i * 4 + 3));
      return;
    }
#pragma unroll
    for (int i = 0; i < 32; ++i)
      if (column + i < p.n) dense_store<bf16>(p, row, column + i, __uint_as_float(raw[i]));
  }
};

template <>
struct Piece<kStorePair> {
  __device__ __forceinline__ void fetch(const DenseTask<kStorePair>&, uint32_t, uint32_t, uint32_t) {}
  __device__ __forceinline__ void store(const DenseTask<kStorePair>& p, uint32_t first_row, uint32_t row_end, uint32_t column,
                                        const uint32_t (&raw)[32], float*) const {
    const uint32_t row = first_row + (threadIdx.x & 31u);
    if (row >= row_end || column >= p.n) return;
    bf16* target = reinterpret_cast<bf16*>(p.out) + (size_t)row * (p.n / 2u) + column / 2u;
    const bool whole = column + 32u <= p.n && ((uintptr_t)target & 15u) == 0;
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      uint32_t packed[4];
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int e = i * 16 + j * 4;
        float pair[2];
#pragma unroll
        for (int h = 0; h < 2; ++h)
          pair[h] = column + e + 2 * h < p.n ? dense_pair(p, row, column + e + 2 * h, __uint_as_float(raw[e + 2 * h]),
                                                          __uint_as_float(raw[e + 2 * h + 1]))
                                             : 0.0f;
        const __nv_bfloat162 both = __floats2bfloat162_rn(pair[0], pair[1]);
        packed[j] = *reinterpret_cast<const uint32_t*>(&both);
        if (!whole) {
          if (column + e < p.n) target[i * 8 + j * 2] = both.x;
          if (column + e + 2 < p.n) target[i * 8 + j * 2 + 1] = both.y;
        }
      }
      if (whole) reinterpret_cast<uint4*>(target)[i] = make_uint4(packed[0], packed[1], packed[2], packed[3]);
    }
  }
};

template <>
struct Piece<kStoreResidual> {
  float4 x[8];  // in the order of the exchange
  static __device__ __forceinline__ uint32_t row_of(uint32_t first_row, int i) { return first_row + (i & 3) * 8u + ((threadIdx.x & 31u) >> 2); }
  static __device__ __forceinline__ uint32_t column_of(uint32_t column, int i) { return column + (i >> 2) * 16u + (threadIdx.x & 3u) * 4u; }
  __device__ __forceinline__ void fetch(const DenseTask<kStoreResidual>& p, uint32_t first_row, uint32_t row_end, uint32_t column) {
    if (p.n % 4u != 0) return;
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      const uint32_t row = row_of(first_row, i), c = column_of(column, i);
      if (row < row_end && c < p.n) x[i] = *reinterpret_cast<const float4*>(p.residual + (size_t)row * p.n + c);
    }
  }
  __device__ __forceinline__ void store(const DenseTask<kStoreResidual>& p, uint32_t first_row, uint32_t row_end, uint32_t column,
                                        const uint32_t (&raw)[32], float* staging) const {
    const uint32_t lane = threadIdx.x & 31u;
    if (p.n % 4u != 0) {
#pragma unroll
      for (int i = 0; i < 32; ++i)
        if (first_row + lane < row_end && column + i < p.n) dense_store<bf16>(p, first_row + lane, column + i, __uint_as_float(raw[i]));
      return;
    }
    const TanhNorm post(p.post_norm, p.n), next(p.next_norm, p.n);
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      uint4 words[4];
#pragma unroll
      for (int j = 0; j < 4; ++j)
        words[j] = make_uint4(raw[half * 16 + j * 4], raw[half * 16 + j * 4 + 1], raw[half * 16 + j * 4 + 2], raw[half * 16 + j * 4 + 3]);
      exchange(staging, words, [&](int i, uint32_t r, const uint4& sums, uint32_t place) {
        const uint32_t row = first_row + r, c = column + half * 16 + place * 4u;
        if (row >= row_end || c >= p.n) return;
        float4 v = make_float4(__uint_as_float(sums.x), __uint_as_float(sums.y), __uint_as_float(sums.z), __uint_as_float(sums.w));
        if (p.has_bias) {
          const float4 bias = __ldg(reinterpret_cast<const float4*>(p.bias + c));
          v.x += bias.x, v.y += bias.y, v.z += bias.z, v.w += bias.w;
        }
        const float4 y = post.four_short(v, c), &held = x[half * 4 + i];
        const float4 sum = make_float4(held.x + y.x, held.y + y.y, held.z + y.z, held.w + y.w);
        *reinterpret_cast<float4*>(p.residual + (size_t)row * p.n + c) = sum;
        store_four(reinterpret_cast<bf16*>(p.out) + (size_t)row * p.n + c, next.four_short(sum, c));
      });
    }
  }
};

template <uint32_t BN, DenseStore STORE>
__global__ void __launch_bounds__(kThreads, 1)
dense_gemm_tc_kernel(const __grid_constant__ CUtensorMap map_x, const __grid_constant__ CUtensorMap map_w,
                     const __grid_constant__ DenseTask<STORE> p, const DensePlan plan, uint32_t most_tiles,
                     uint32_t* error_word) {
  using S = Shape<BN>;
  extern __shared__ unsigned char shared_raw[];
  grid_chain_prologue();
  const uint32_t base = (smem_u32(shared_raw) + 1023u) & ~1023u;
  unsigned char* base_pointer = shared_raw + (base - smem_u32(shared_raw));
  const uint32_t full = base + S::kBarriers, empty = full + S::kStages * 8;
  const uint32_t sums_full = empty + S::kStages * 8, sums_empty = sums_full + 16;
  volatile uint32_t* holder = reinterpret_cast<volatile uint32_t*>(base_pointer + S::kHolder);
  volatile uint32_t* abort_flag = reinterpret_cast<volatile uint32_t*>(base_pointer + S::kAbort);
  const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31u;
  const uint32_t m_tiles = plan.tiles ? min(plan.tiles[0], most_tiles) : (p.m + kRows - 1u) / kRows;
  const uint32_t n_tiles = (p.n + BN - 1u) / BN, tiles = m_tiles * n_tiles;
  // first row, row end, and first row of the weights (column of the output) of a tile
  auto place = [&](uint32_t tile) -> DenseTile {
    const uint32_t m_tile = tile % m_tiles, n0 = tile / m_tiles * BN;
    if (!plan.tiles) return {n0, m_tile * kRows, p.m};
    const DenseTile rows = dense_tile(plan, m_tile);
    return {rows.expert * p.n + n0, rows.first, min(rows.end, p.m)};
  };
  const uint32_t k_stages = (p.k + kDepth * S::kBlocks - 1u) / (kDepth * S::kBlocks);

  if (threadIdx.x == 0) {
    for (uint32_t s = 0; s < S::kStages; ++s) {
      barrier_init(full + s * 8, 1);   // the producer's expect_tx arrival; completes by byte count
      barrier_init(empty + s * 8, 1);  // one tcgen05.commit
    }
    for (uint32_t s = 0; s < 2; ++s) {
      barrier_init(sums_full + s * 8, 1);   // one tcgen05.commit
      barrier_init(sums_empty + s * 8, kEpilogueWarps);  // one arrival per epilogue warp
    }
    *abort_flag = 0u;
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  if (warp == 1) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(base + S::kHolder),
                 "r"(S::kTmemColumns)
                 : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
  }
  asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
  __syncthreads();
  asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
  const uint32_t tmem_base = *holder;
  auto give_up = [&]() {
    *abort_flag = 1u;
    if (error_word) atomicExch(error_word, 1u);
  };

  if (warp == 0) {
    if (lane == 0) {
      uint32_t issued = 0;  // k-blocks over all tiles of this CTA
      bool ok = true;
      for (uint32_t tile = blockIdx.x; tile < tiles && ok; tile += gridDim.x) {
        const DenseTile at = place(tile);
        for (uint32_t ks = 0; ks < k_stages; ++ks, ++issued) {
          const uint32_t s = issued % S::kStages;
          ok = !*abort_flag && barrier_wait(empty + s * 8, ((issued / S::kStages) & 1u) ^ 1u);
          if (!ok) {
            give_up();
            break;
          }
          barrier_expect_tx(full + s * 8, S::kStageBytes);
          const uint32_t stage = base + s * S::kStageBytes;
#pragma unroll
          for (uint32_t block = 0; block < S::kBlocks; ++block) {
            const int32_t k0 = (int32_t)((ks * S::kBlocks + block) * kDepth);
            tma_load_2d(stage + block * kXTileBytes, &map_x, k0, (int32_t)at.first, full + s * 8);
            tma_load_2d(stage + S::kBlocks * kXTileBytes + block * S::kWTileBytes, &map_w, k0, (int32_t)at.expert, full + s * 8);
          }
        }
      }
      // on the way out after a failure the copies already started must land first
      if (!ok || *abort_flag)
        for (uint32_t i = issued > S::kStages ? issued - S::kStages : 0u; i < issued; ++i)
          barrier_wait(full + (i % S::kStages) * 8, (i / S::kStages) & 1u);
    }
  } else if (warp == 1) {
    if (lane == 0) {
      uint32_t consumed = 0, turn = 0;
      bool ok = true;
      for (uint32_t tile = blockIdx.x; tile < tiles && ok; tile += gridDim.x, ++turn) {
        const uint32_t half = turn & 1u, sums = tmem_base + half * BN;
        ok = !*abort_flag && barrier_wait(sums_empty + half * 8, ((turn >> 1) & 1u) ^ 1u);
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        for (uint32_t ks = 0; ks < k_stages && ok; ++ks, ++consumed) {
          const uint32_t s = consumed % S::kStages;
          ok = !*abort_flag && barrier_wait(full + s * 8, (consumed / S::kStages) & 1u);
          if (!ok) break;
          asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
          const uint32_t x_tile = base + s * S::kStageBytes, w_tile = x_tile + S::kBlocks * kXTileBytes;
#pragma unroll
          for (uint32_t j = 0; j < S::kBlocks * kDepth / 16; ++j) {
            const uint32_t block = j / (kDepth / 16), at = j % (kDepth / 16) * 32;
            mma_f16(sums, operand_descriptor(x_tile + block * kXTileBytes + at),
                    operand_descriptor(w_tile + block * S::kWTileBytes + at), (ks > 0 || j > 0) ? 1u : 0u,
                    bf16_instruction(kRows, BN));
          }
          mma_commit(empty + s * 8);
        }
        if (ok) mma_commit(sums_full + half * 8);
      }
      if (!ok) give_up();
    }
  } else {
    const uint32_t quarter = warp & 3u, side = (warp - 2u) >> 2;  // lanes of tensor memory; every other piece of the columns
    float* staging = reinterpret_cast<float*>(base_pointer + S::kStaging) + (warp - 2u) * (kStagingBytes<STORE> / 4u);
    uint32_t turn = 0;
    bool ok = true;
    for (uint32_t tile = blockIdx.x; tile < tiles && ok; tile += gridDim.x, ++turn) {
      const uint32_t half = turn & 1u;
      const DenseTile rows = place(tile);
      const uint32_t first_row = rows.first + quarter * 32u, n0 = (tile / m_tiles) * BN;  // of this warp
      Piece<STORE> ahead;
      ahead.fetch(p, first_row, rows.end, n0 + side * 32u);
      ok = !*abort_flag && barrier_wait(sums_full + half * 8, (turn >> 1) & 1u);
      ok = __all_sync(0xffffffffu, ok);
      if (!ok) {
        give_up();
        break;
      }
      asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
      const uint32_t address = tmem_base + half * BN + ((quarter * 32u) << 16);
#pragma unroll 1
      for (uint32_t piece = side; piece < BN / 32u; piece += kEpilogueWarps / 4u) {
        uint32_t raw[32];
        tmem_load_32(address + piece * 32u, raw);
        asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
        const uint32_t column = n0 + piece * 32u, following = piece + kEpilogueWarps / 4u;
        Piece<STORE> held = ahead;
        if (following < BN / 32u) ahead.fetch(p, first_row, rows.end, n0 + following * 32u);
        held.store(p, first_row, rows.end, column, raw, staging);
        __syncwarp();  // tcgen05.ld needs the whole warp
      }
      asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
      __syncwarp();
      if (lane == 0) barrier_arrive(sums_empty + half * 8);
    }
  }

  __syncthreads();
  if (warp == 1) {
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem_base), "r"(S::kTmemColumns)
                 : "memory");
  }
}

// cuTensorMapEncodeTiled, resolved through the runtime so that the library does not link libcuda.
typedef CUresult (*EncodeTiled)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*,
                                const cuuint64_t*, const cuuint32_t*, const cuuint32_t*, CUtensorMapInterleave,
                                CUtensorMapSwizzle, CUtensorMapL2promotion, CUtensorMapFloatOOBfill);

// Row-major bf16 matrix [outer, inner] read in boxes of 64 x `box_rows` with the 128-byte swizzle.
bool make_map(CUtensorMap* map, const void* base, uint64_t inner, uint64_t outer, uint32_t box_rows) {
  static EncodeTiled encode = []() -> EncodeTiled {
    void* pointer = nullptr;
    cudaDriverEntryPointQueryResult result;
    if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &pointer, cudaEnableDefault, &result) != cudaSuccess ||
        result != cudaDriverEntryPointSuccess)
      return nullptr;
    return reinterpret_cast<EncodeTiled>(pointer);
  }();
  if (encode == nullptr) return false;
  const cuuint64_t dims[2] = {inner, outer}, strides[1] = {inner * 2};
  const cuuint32_t box[2] = {kDepth, box_rows}, element_strides[2] = {1, 1};
  return encode(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(base), dims, strides, box, element_strides,
                CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
}

// Row tiles; of rows sorted by expert, the most there can be.
uint32_t most_tiles(const DenseProblem& p) {
  if (!p.plan.tiles) return (p.m + kRows - 1u) / kRows;
  return p.m / kRows + (p.plan.experts < p.m ? p.plan.experts : p.m);
}

template <uint32_t BN, DenseStore STORE>
int run(const KernelArgs& args, const DenseProblem& p, uint32_t sms) {
  using S = Shape<BN>;
  CUtensorMap map_x, map_w;
  if (!make_map(&map_x, p.x, p.k, p.m, kRows) ||
      !make_map(&map_w, p.w, p.k, (uint64_t)p.n * (p.plan.tiles ? p.plan.experts : 1u), BN))
    return -1;
  auto kernel = dense_gemm_tc_kernel<BN, STORE>;
  constexpr uint32_t shared = S::kSharedBytes + kEpilogueWarps * kStagingBytes<STORE>;
  if (cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, shared) != cudaSuccess) {
    cudaGetLastError();
    return -1;
  }
  const uint32_t most = most_tiles(p), tiles = most * ((p.n + BN - 1u) / BN);
  launch_kernel(args, kernel, dim3(tiles < sms ? tiles : sms), dim3(kThreads), shared, map_x, map_w, DenseTask<STORE>(p), p.plan, most,
                context_device_error(args.ctx));
  return check_launch(args);
}

template <DenseStore STORE>
int run_tiles(const KernelArgs& args, const DenseProblem& p) {
  if (args.ctx == nullptr || p.k % 8u != 0) return -1;
  for (const void* pointer : {p.x, p.w, (const void*)p.out, (const void*)p.out32, (const void*)p.pool})
    if ((uintptr_t)pointer & 15u) return -1;
  const uint32_t sms = (uint32_t)context_sm_count(args.ctx);
  // waves times the cost of one MMA (an MMA of up to 128 columns costs about two thirds of one of 256)
  const uint32_t m_tiles = most_tiles(p);
  auto cost = [&](uint32_t columns, uint32_t mma) {
    const uint32_t tiles = m_tiles * ((p.n + columns - 1u) / columns);
    return (tiles + sms - 1u) / sms * mma;
  };
  const uint32_t wide = cost(256, 128), middle = cost(128, 85), narrow = cost(64, 80);
  if (narrow < middle && narrow < wide) return run<64, STORE>(args, p, sms);
  if (middle < wide) return run<128, STORE>(args, p, sms);
  return run<256, STORE>(args, p, sms);
}

}  // namespace

int launch_dense_gemm_tc(const KernelArgs& args, const DenseProblem& p, DenseStore store) {
  switch (store) {
    case kStoreCached: return run_tiles<kStoreCached>(args, p);
    case kStorePair: return run_tiles<kStorePair>(args, p);
    case kStoreResidual: return run_tiles<kStoreResidual>(args, p);
    default: return run_tiles<kStorePlain>(args, p);
  }
}

}  // namespace llmopt
