// Dense linear layer y = x . w^T (+ bias, + activation) in bfloat16 or fp32, fp32 accumulation:
//   llmopt_dense_linear_{bf16,f32}     outputs in the element type and in fp32
//   llmopt_dense_cached_{bf16,f32}     key and value columns go straight into the tokens' cache rows
//   llmopt_dense_residual_{bf16,f32}   the product that ends a sublayer: tanh norm of the sum, residual add in
//                                      place, the following sublayer's tanh norm, all in the writeback
//
// Kernels behind the names:
//  * bf16, up to 64 rows (decode): dense_gemv_kernel, weights streamed once from HBM straight into
//    mma.sync fragments.  The order of the contraction is free, so a lane takes 16 contiguous bytes of
//    a weight row (eight k) as the A words of two MMAs and the same eight k of an activation row
//    as their B words: no shared-memory staging and full 128-byte lines.  Eight warps split K and
//    add their sums in warp order.
//  * bf16, more rows: dense_gemm_tc.cu (tcgen05).
//  * fp32, and bf16 rows that are no whole 16-byte vectors: CUDA-core kernels (a warp per column for
//    few rows, 64 x 64 tiles otherwise).
#include <type_traits>

#include "dense_stream.cuh"

namespace llmopt {
namespace {

// NT: 8-row batch tiles.  16 weight rows per cluster of `cluster` CTAs, which share out the k-blocks (narrow
// matrices would leave most SMs without a stream otherwise) and add their sums through distributed shared memory.
template <int NT, DenseStore STORE>
__global__ void __launch_bounds__(kGemvWarps * 32, NT <= 4 ? 2 : 1) dense_gemv_kernel(const DenseTask<STORE> p) {
  const uint32_t cluster = p.cluster;
  grid_launch_dependents();
  const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31u, g = lane >> 2, t = lane & 3u;
  const uint32_t n0 = blockIdx.x / cluster * 16u, rank = blockIdx.x % cluster, stride = kGemvWarps * cluster;
  const bf16* w = reinterpret_cast<const bf16*>(p.w);
  const bf16* w_low = w + (size_t)min(n0 + g, p.n - 1u) * p.k;
  const bf16* w_high = w + (size_t)min(n0 + g + 8u, p.n - 1u) * p.k;
  const uint32_t blocks = (p.k + 63u) / 64u;
  const uint4 zero = make_uint4(0u, 0u, 0u, 0u);
  uint4 a[kGemvStages][4];  // rows g / g + 8, low / high 32 of the k-block
  auto fetch = [&](uint4 (&stage)[4], uint32_t block) {
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const uint32_t k = block * 64u + half * 32u + t * 8u;
      const bool present = block < blocks && k < p.k;
      stage[half] = present ? load_stream(w_low + k) : zero;
      stage[2 + half] = present ? load_stream(w_high + k) : zero;
    }
  };
  // the weights are nobody's output: their first blocks may be requested before the predecessor ends
#pragma unroll
  for (int s = 0; s < kGemvStages; ++s) fetch(a[s], rank * kGemvWarps + warp + s * stride);
  grid_dependency_wait();

  const bf16* x = reinterpret_cast<const bf16*>(p.x);
  float sum[NT][4];
#pragma unroll
  for (int nt = 0; nt < NT; ++nt)
#pragma unroll
    for (int i = 0; i < 4; ++i) sum[nt][i] = 0.0f;
  for (uint32_t first = rank * kGemvWarps + warp; first < blocks; first += kGemvStages * stride) {
#pragma unroll
    for (int s = 0; s < kGemvStages; ++s) {
      const uint32_t block = first + s * stride;
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const uint32_t k = block * 64u + half * 32u + t * 8u;
        const uint4 low = a[s][half], high = a[s][2 + half];
#pragma unroll
        for (int nt = 0; nt < NT; ++nt) {
          const uint32_t row = nt * 8u + g;
          const uint4 b = (row < p.m && k < p.k) ? *reinterpret_cast<const uint4*>(x + (size_t)row * p.k + k) : zero;
          mma_bf16(sum[nt], low.x, high.x, low.y, high.y, b.x, b.y);
          mma_bf16(sum[nt], low.z, high.z, low.w, high.w, b.z, b.w);
        }
      }
      fetch(a[s], block + kGemvStages * stride);
    }
  }

  __shared__ float partial[kGemvWarps][NT * 8][17];
  stream_collect<NT>(sum, partial[warp]);
  stream_finish<NT>(p, partial, n0, rank, cluster);
}

// One warp per output column (pairs: per two columns), up to eight rows.
template <typename T, DenseStore STORE>
__global__ void __launch_bounds__(256) dense_columns_kernel(const DenseTask<STORE> p, uint32_t row0) {
  constexpr bool PAIR = STORE == kStorePair;
  grid_chain_prologue();
  const uint32_t column = (blockIdx.x * 8u + (threadIdx.x >> 5)) * (PAIR ? 2u : 1u), lane = threadIdx.x & 31u;
  if (column >= p.n) return;
  const T* w = reinterpret_cast<const T*>(p.w) + (size_t)column * p.k;
  const T* x = reinterpret_cast<const T*>(p.x) + (size_t)row0 * p.k;
  const uint32_t rows = min(p.m - row0, 8u);
  float sum[8], second[8];
#pragma unroll
  for (int r = 0; r < 8; ++r) sum[r] = second[r] = 0.0f;
  for (uint32_t k = lane; k < p.k; k += 32u) {
    const float weight = as_float(w[k]), other = PAIR ? as_float(w[p.k + k]) : 0.0f;
#pragma unroll
    for (int r = 0; r < 8; ++r)
      if (r < rows) {
        const float value = as_float(x[(size_t)r * p.k + k]);
        sum[r] = fmaf(weight, value, sum[r]);
        if (PAIR) second[r] = fmaf(other, value, second[r]);
      }
  }
#pragma unroll
  for (int r = 0; r < 8; ++r) {
    const float total = warp_sum(sum[r]), other = PAIR ? warp_sum(second[r]) : 0.0f;
    if (r >= rows || lane != 0) continue;
    if constexpr (PAIR) dense_store_pair<T>(p, row0 + r, column, total, other);
    else dense_store<T>(p, row0 + r, column, total);
  }
}

// 64 x 64 output tiles, 4 x 4 per thread; rows sorted by expert: half a plan's tile each.
template <typename T, DenseStore STORE>
__global__ void __launch_bounds__(256) dense_tile_kernel(const DenseTask<STORE> p, const DensePlan plan) {
  grid_chain_prologue();
  constexpr int kTile = 64, kDepth = 16;
  __shared__ float x_tile[kDepth][kTile + 4], w_tile[kDepth][kTile + 4];
  const uint32_t n0 = blockIdx.x * kTile;
  uint32_t m0 = blockIdx.y * kTile, row_end = p.m;
  const uint32_t tx = threadIdx.x & 15u, ty = threadIdx.x >> 4;
  const T* x = reinterpret_cast<const T*>(p.x);
  const T* w = reinterpret_cast<const T*>(p.w);
  if (plan.tiles) {
    const uint32_t index = blockIdx.y / (kExpertTile / kTile);
    if (index >= plan.tiles[0]) return;
    const DenseTile tile = dense_tile(plan, index);
    m0 = tile.first + blockIdx.y % (kExpertTile / kTile) * kTile;
    row_end = min(tile.end, p.m);
    if (m0 >= row_end || tile.expert >= plan.experts) return;
    w += (size_t)tile.expert * p.n * p.k;
  }
  float sum[4][4] = {};
  for (uint32_t k0 = 0; k0 < p.k; k0 += kDepth) {
    for (uint32_t index = threadIdx.x; index < kTile * kDepth; index += 256u) {
      const uint32_t k = index % kDepth, row = index / kDepth;
      const bool k_present = k0 + k < p.k;
      x_tile[k][row] = k_present && m0 + row < row_end ? as_float(x[(size_t)(m0 + row) * p.k + k0 + k]) : 0.0f;
      w_tile[k][row] = k_present && n0 + row < p.n ? as_float(w[(size_t)(n0 + row) * p.k + k0 + k]) : 0.0f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < kDepth; ++k) {
      const float4 xa = *reinterpret_cast<const float4*>(&x_tile[k][ty * 4]);
      const float4 wb = *reinterpret_cast<const float4*>(&w_tile[k][tx * 4]);
      const float xs[4] = {xa.x, xa.y, xa.z, xa.w}, ws[4] = {wb.x, wb.y, wb.z, wb.w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) sum[i][j] = fmaf(xs[i], ws[j], sum[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const uint32_t row = m0 + ty * 4 + i, column = n0 + tx * 4 + j;
      if (row >= row_end || column >= p.n) continue;
      if constexpr (STORE == kStorePair) {
        if (j % 2 == 0) dense_store_pair<T>(p, row, column, sum[i][j], sum[i][(j + 1) % 4]);
      } else {
        dense_store<T>(p, row, column, sum[i][j]);
      }
    }
}

// `run` with the store as a constant.
template <typename Run>
int with_store(DenseStore store, Run run) {
  switch (store) {
    case kStoreCached: return run(std::integral_constant<DenseStore, kStoreCached>());
    case kStorePair: return run(std::integral_constant<DenseStore, kStorePair>());
    case kStoreResidual: return run(std::integral_constant<DenseStore, kStoreResidual>());
    default: return run(std::integral_constant<DenseStore, kStorePlain>());
  }
}

template <typename T>
int run_cuda_cores(const KernelArgs& args, const DenseProblem& p, DenseStore store) {
  return with_store(store, [&](auto constant) {
    constexpr DenseStore STORE = decltype(constant)::value;
    if (p.m <= 32u) {
      const uint32_t warps = STORE == kStorePair ? p.n / 2u : p.n;
      for (uint32_t row0 = 0; row0 < p.m; row0 += 8u)
        launch_kernel(args, dense_columns_kernel<T, STORE>, dim3((warps + 7u) / 8u), dim3(256), 0, DenseTask<STORE>(p), row0);
    } else {
      launch_kernel(args, dense_tile_kernel<T, STORE>, dim3((p.n + 63u) / 64u, (p.m + 63u) / 64u), dim3(256), 0,
                    DenseTask<STORE>(p), p.plan);
    }
    return check_launch(args);
  });
}

int run_gemv(const KernelArgs& args, DenseProblem p, DenseStore store) {
  const uint32_t tiles = (p.n + 15u) / 16u;
  p.cluster = stream_cluster(args, tiles, (p.k + 63u) / 64u);
  return with_store(store, [&](auto constant) {
    constexpr DenseStore STORE = decltype(constant)::value;
    auto run = [&](auto kernel) {
      const DenseTask<STORE> task(p);
      if (p.cluster == 1u) launch_kernel(args, kernel, dim3(tiles), dim3(kGemvWarps * 32), 0, task);
      else launch_cluster_kernel(args, kernel, dim3(tiles * p.cluster), dim3(kGemvWarps * 32), 0, p.cluster, task);
      return check_launch(args);
    };
    if (p.m <= 8u) return run(dense_gemv_kernel<1, STORE>);
    if (p.m <= 16u) return run(dense_gemv_kernel<2, STORE>);
    if (p.m <= 32u) return run(dense_gemv_kernel<4, STORE>);
    return run(dense_gemv_kernel<8, STORE>);
  });
}

template <typename T>
int run_dense(const KernelArgs& args, const DenseProblem& p, DenseStore store) {
  if (p.m == 0) return 0;
  if (sizeof(T) == 4) return run_cuda_cores<T>(args, p, store);
  const bool vectors = p.k % 8u == 0 && ((uintptr_t)p.x & 15u) == 0 && ((uintptr_t)p.w & 15u) == 0;
  if (!vectors) return run_cuda_cores<T>(args, p, store);
  if (p.m > 64u) {
    const int status = launch_dense_gemm_tc(args, p, store);
    return status >= 0 ? status : run_cuda_cores<T>(args, p, store);
  }
  return run_gemv(args, p, store);
}

// Common part of a problem: buffers x and w, {m, n, k} at the start of the parameters.
template <typename T>
int read_problem(const KernelArgs& args, DenseProblem& p) {
  p = {};
  p.m = param_u32(args, 0), p.n = param_u32(args, 1), p.k = param_u32(args, 2);
  p.scale = 1.0f;
  p.x = args.buffers[0], p.w = args.buffers[1], p.bias = (const float*)args.buffers[2];
  LLMOPT_REQUIRE(p.n > 0 && p.k > 0, "needs n > 0 and k > 0");
  LLMOPT_REQUIRE(args.lengths[0] >= (size_t)p.m * p.k * sizeof(T), "activation buffer is too short");
  LLMOPT_REQUIRE(args.lengths[1] >= (size_t)p.n * p.k * sizeof(T), "weight buffer is too short");
  return 0;
}

// Buffers [x, w, bias, out, out32, ids, table] (an absent one repeats another); params
// {m, n, k, split, has_bias, epilogue, table_rows, table_stride, table_offset, scale f32}.
template <typename T>
int launch_dense_linear(const KernelArgs& args) {
  LLMOPT_REQUIRE(args.buffer_count == 7 && args.param_bytes == 40,
                 "expects buffers [x, w, bias, out, out32, ids, table] and 40 parameter bytes");
  DenseProblem p;
  if (const int status = read_problem<T>(args, p)) return status;
  p.split = param_u32(args, 3);
  p.has_bias = param_u32(args, 4), p.epilogue = param_u32(args, 5), p.table_rows = param_u32(args, 6);
  p.table_stride = param_u32(args, 7), p.table_offset = param_u32(args, 8), p.scale = param_f32(args, 9);
  p.out = args.buffers[3];
  p.out32 = (float*)args.buffers[4], p.ids = (const long long*)args.buffers[5], p.table = args.buffers[6];
  LLMOPT_REQUIRE(p.split <= p.n, "needs split <= n");
  LLMOPT_REQUIRE(!p.has_bias || args.lengths[2] >= (size_t)p.n * 4, "bias buffer is too short");
  LLMOPT_REQUIRE(p.epilogue <= kDenseSiluPair, "unknown epilogue");
  LLMOPT_REQUIRE(p.epilogue != kDenseSiluPair || (p.split == p.n && p.n % 2u == 0), "pairs of columns leave in the element type");
  const size_t columns = p.epilogue == kDenseSiluPair ? p.n / 2u : p.split;
  LLMOPT_REQUIRE(p.split == 0 || args.lengths[3] >= (size_t)p.m * columns * sizeof(T), "output buffer is too short");
  LLMOPT_REQUIRE(p.split == p.n || args.lengths[4] >= (size_t)p.m * (p.n - p.split) * 4, "fp32 output buffer is too short");
  if (p.epilogue == kDenseTokenGate) {
    LLMOPT_REQUIRE(args.lengths[5] >= (size_t)p.m * 8, "token buffer is too short");
    LLMOPT_REQUIRE(p.table_rows > 0 && (size_t)p.table_offset + p.n <= p.table_stride &&
                       args.lengths[6] >= (size_t)p.table_rows * p.table_stride * sizeof(T),
                   "token table is too short");
  }
  return run_dense<T>(args, p, p.epilogue == kDenseSiluPair ? kStorePair : kStorePlain);
}

}  // namespace
uint32_t* context_device_error(Context* ctx);
namespace {

// Buffers [x, w, bias, out, out32, pool, slot table, past, sequence rows]; params {m, n, k, split, has_bias, tokens,
// key_columns, value_columns, token_stride, key_offset, value_offset, table_stride, table_rows, pool_rows}.
template <typename T>
int launch_dense_cached(const KernelArgs& args) {
  LLMOPT_REQUIRE(args.buffer_count == 9 && args.param_bytes == 56, "expects 9 buffers and 56 parameter bytes");
  DenseProblem p;
  if (const int status = read_problem<T>(args, p)) return status;
  p.split = param_u32(args, 3), p.has_bias = param_u32(args, 4);
  p.out = args.buffers[3], p.out32 = (float*)args.buffers[4];
  DenseCacheRows& c = p;
  c.pool = args.buffers[5], c.slots = (const uint32_t*)args.buffers[6], c.past = (const uint32_t*)args.buffers[7];
  c.sequence_rows = (const uint32_t*)args.buffers[8], c.error_word = context_device_error(args.ctx);
  c.tokens = param_u32(args, 5), c.key_columns = param_u32(args, 6), c.value_columns = param_u32(args, 7);
  c.token_stride = param_u32(args, 8), c.key_offset = param_u32(args, 9), c.value_offset = param_u32(args, 10);
  c.slots_stride = param_u32(args, 11), c.slots_rows = param_u32(args, 12), c.pool_rows = param_u32(args, 13);
  const size_t kept = (size_t)c.key_columns + c.value_columns, sequences = c.tokens ? p.m / c.tokens : 0;
  LLMOPT_REQUIRE(c.tokens > 0 && p.m % c.tokens == 0, "needs whole sequences of rows");
  LLMOPT_REQUIRE(p.split + kept <= p.n, "columns lie outside the product");
  LLMOPT_REQUIRE((size_t)c.key_offset + c.key_columns <= c.token_stride && (size_t)c.value_offset + c.value_columns <= c.token_stride,
                 "key or value segment lies outside the cache row");
  LLMOPT_REQUIRE(!p.has_bias || args.lengths[2] >= (size_t)p.n * 4, "bias buffer is too short");
  LLMOPT_REQUIRE(args.lengths[3] >= (size_t)p.m * p.split * sizeof(T) && args.lengths[4] >= (size_t)p.m * (p.n - p.split - kept) * 4,
                 "output buffer is too short");
  LLMOPT_REQUIRE(args.lengths[5] >= (size_t)c.pool_rows * c.token_stride * sizeof(T) &&
                     args.lengths[6] >= (size_t)c.slots_rows * c.slots_stride * 4 && args.lengths[7] >= sequences * 4 &&
                     args.lengths[8] >= sequences * 4,
                 "cache buffer is too short");
  return run_dense<T>(args, p, kStoreCached);
}

// Buffers [x, w, bias, norm of the sum, following norm, residual, out]; params {m, n, k, has_bias}.
template <typename T>
int launch_dense_residual(const KernelArgs& args) {
  LLMOPT_REQUIRE(args.buffer_count == 7 && args.param_bytes == 16, "expects 7 buffers and 16 parameter bytes");
  DenseProblem p;
  if (const int status = read_problem<T>(args, p)) return status;
  p.has_bias = param_u32(args, 3), p.epilogue = kDenseResidualTanh, p.split = p.n;
  p.post_norm = (const float*)args.buffers[3], p.next_norm = (const float*)args.buffers[4];
  p.residual = (float*)args.buffers[5], p.out = args.buffers[6];
  LLMOPT_REQUIRE(!p.has_bias || args.lengths[2] >= (size_t)p.n * 4, "bias buffer is too short");
  LLMOPT_REQUIRE(args.lengths[3] >= (2 * (size_t)p.n + 1) * 4 && args.lengths[4] >= (2 * (size_t)p.n + 1) * 4, "norm is too short");
  LLMOPT_REQUIRE(args.lengths[5] >= (size_t)p.m * p.n * 4 && args.lengths[6] >= (size_t)p.m * p.n * sizeof(T),
                 "output buffer is too short");
  LLMOPT_REQUIRE(p.out != p.x, "the product cannot overwrite its input");
  for (int i = 2; i < 7; ++i) LLMOPT_REQUIRE(((uintptr_t)args.buffers[i] & 15u) == 0, "buffers must be 16-byte aligned");
  return run_dense<T>(args, p, kStoreResidual);
}

}  // namespace

template <typename T>
int run_expert_rows(const KernelArgs& args, const DenseProblem& p, DenseStore store, uint32_t tiles) {
  if (sizeof(T) == 2) {
    const int status = launch_dense_gemm_tc(args, p, store);
    if (status >= 0) return status;
  }
  constexpr uint32_t kHalves = kExpertTile / 64u;
  LLMOPT_REQUIRE(tiles * kHalves <= 65535u, "too many tiles");
  const dim3 grid((p.n + 63u) / 64u, tiles * kHalves);
  return with_store(store, [&](auto constant) {
    constexpr DenseStore STORE = decltype(constant)::value;
    launch_kernel(args, dense_tile_kernel<T, STORE>, grid, dim3(256), 0, DenseTask<STORE>(p), p.plan);
    return check_launch(args);
  });
}
template int run_expert_rows<bf16>(const KernelArgs&, const DenseProblem&, DenseStore, uint32_t);
template int run_expert_rows<float>(const KernelArgs&, const DenseProblem&, DenseStore, uint32_t);

const NamedLauncher* dense_linear_launchers(size_t* count) {
  static const NamedLauncher table[] = {
      {"llmopt_dense_linear_bf16", launch_dense_linear<bf16>},
      {"llmopt_dense_linear_f32", launch_dense_linear<float>},
      {"llmopt_dense_cached_bf16", launch_dense_cached<bf16>},
      {"llmopt_dense_cached_f32", launch_dense_cached<float>},
      {"llmopt_dense_residual_bf16", launch_dense_residual<bf16>},
      {"llmopt_dense_residual_f32", launch_dense_residual<float>},
  };
  *count = sizeof(table) / sizeof(table[0]);
  return table;
}

}  // namespace llmopt
