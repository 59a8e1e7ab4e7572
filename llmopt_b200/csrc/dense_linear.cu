// Dense linear layer y = x . w^T (+ bias, + activation) in bfloat16 or fp32, fp32 accumulation:
//   llmopt_dense_linear_{bf16,f32}
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
#include "dense_linear.cuh"

namespace llmopt {
namespace {

constexpr int kGemvWarps = 8;
constexpr int kGemvStages = 3;  // 64-wide k-blocks a warp keeps in flight

__device__ __forceinline__ void mma_bf16(float (&d)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0,
                                         uint32_t b1) {
  asm("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
      : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
      : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}

__device__ __forceinline__ uint4 load_stream(const bf16* source) {
  uint4 v;
  asm volatile("ld.global.nc.L1::no_allocate.v4.u32 {%0,%1,%2,%3}, [%4];"
               : "=r"(v.x), "=r"(v.y), "=r"(v.z), "=r"(v.w)
               : "l"(source));
  return v;
}

// NT: 8-row batch tiles.  16 weight rows per cluster of `cluster` CTAs, which share out the k-blocks (narrow
// matrices would leave most SMs without a stream otherwise) and add their sums through distributed shared memory.
template <int NT>
__global__ void __launch_bounds__(kGemvWarps * 32) dense_gemv_kernel(const DenseProblem p, uint32_t cluster) {
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
#pragma unroll
  for (int nt = 0; nt < NT; ++nt)
#pragma unroll
    for (int i = 0; i < 4; ++i) partial[warp][nt * 8 + 2 * t + (i & 1)][g + (i >> 1) * 8] = sum[nt][i];
  __syncthreads();
  for (uint32_t index = threadIdx.x; index < NT * 8u * 16u; index += kGemvWarps * 32) {
    const uint32_t column = index & 15u, row = index >> 4;
    if (row >= p.m || n0 + column >= p.n) continue;
    float value = 0.0f;
#pragma unroll
    for (int part = 0; part < kGemvWarps; ++part) value += partial[part][row][column];
    if (cluster == 1u) dense_store<bf16>(p, row, n0 + column, value);
    else partial[0][row][column] = value;  // read and written by this thread only
  }
  if (cluster == 1u) return;
  cluster_sync();
  // the cluster's CTAs share out the outputs; sums in rank order
  for (uint32_t index = rank * kGemvWarps * 32 + threadIdx.x; index < NT * 8u * 16u; index += stride * 32u) {
    const uint32_t column = index & 15u, row = index >> 4;
    if (row >= p.m || n0 + column >= p.n) continue;
    float value = 0.0f;
    for (uint32_t other = 0; other < cluster; ++other) value += cluster_load(&partial[0][row][column], other);
    dense_store<bf16>(p, row, n0 + column, value);
  }
  cluster_sync();  // nobody leaves while its sums may be read
}

// One warp per output column, up to eight rows.
template <typename T>
__global__ void __launch_bounds__(256) dense_columns_kernel(const DenseProblem p, uint32_t row0) {
  grid_chain_prologue();
  const uint32_t column = blockIdx.x * 8u + (threadIdx.x >> 5), lane = threadIdx.x & 31u;
  if (column >= p.n) return;
  const T* w = reinterpret_cast<const T*>(p.w) + (size_t)column * p.k;
  const T* x = reinterpret_cast<const T*>(p.x) + (size_t)row0 * p.k;
  const uint32_t rows = min(p.m - row0, 8u);
  float sum[8];
#pragma unroll
  for (int r = 0; r < 8; ++r) sum[r] = 0.0f;
  for (uint32_t k = lane; k < p.k; k += 32u) {
    const float weight = as_float(w[k]);
#pragma unroll
    for (int r = 0; r < 8; ++r)
      if (r < rows) sum[r] = fmaf(weight, as_float(x[(size_t)r * p.k + k]), sum[r]);
  }
#pragma unroll
  for (int r = 0; r < 8; ++r) {
    const float total = warp_sum(sum[r]);
    if (r < rows && lane == 0) dense_store<T>(p, row0 + r, column, total);
  }
}

// 64 x 64 output tiles, 4 x 4 per thread.
template <typename T>
__global__ void __launch_bounds__(256) dense_tile_kernel(const DenseProblem p) {
  grid_chain_prologue();
  constexpr int kTile = 64, kDepth = 16;
  __shared__ float x_tile[kDepth][kTile + 4], w_tile[kDepth][kTile + 4];
  const uint32_t n0 = blockIdx.x * kTile, m0 = blockIdx.y * kTile;
  const uint32_t tx = threadIdx.x & 15u, ty = threadIdx.x >> 4;
  const T* x = reinterpret_cast<const T*>(p.x);
  const T* w = reinterpret_cast<const T*>(p.w);
  float sum[4][4] = {};
  for (uint32_t k0 = 0; k0 < p.k; k0 += kDepth) {
    for (uint32_t index = threadIdx.x; index < kTile * kDepth; index += 256u) {
      const uint32_t k = index % kDepth, row = index / kDepth;
      const bool k_present = k0 + k < p.k;
      x_tile[k][row] = k_present && m0 + row < p.m ? as_float(x[(size_t)(m0 + row) * p.k + k0 + k]) : 0.0f;
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
      if (row < p.m && column < p.n) dense_store<T>(p, row, column, sum[i][j]);
    }
}

template <typename T>
int run_cuda_cores(const KernelArgs& args, const DenseProblem& p) {
  if (p.m <= 32u) {
    for (uint32_t row0 = 0; row0 < p.m; row0 += 8u)
      launch_kernel(args, dense_columns_kernel<T>, dim3((p.n + 7u) / 8u), dim3(256), 0, p, row0);
  } else {
    launch_kernel(args, dense_tile_kernel<T>, dim3((p.n + 63u) / 64u, (p.m + 63u) / 64u), dim3(256), 0, p);
  }
  return check_launch(args);
}

int run_gemv(const KernelArgs& args, const DenseProblem& p) {
  const uint32_t tiles = (p.n + 15u) / 16u, blocks = (p.k + 63u) / 64u;
  // at least one CTA per SM; a warp of a split keeps at least one k-block
  const uint32_t wanted = (uint32_t)context_sm_count(args.ctx);
  uint32_t cluster = 1;
  while (cluster < 8u && tiles * cluster < wanted && blocks >= 2u * cluster * kGemvWarps) cluster *= 2u;
  auto run = [&](auto kernel) {
    if (cluster == 1u) launch_kernel(args, kernel, dim3(tiles), dim3(kGemvWarps * 32), 0, p, cluster);
    else launch_cluster_kernel(args, kernel, dim3(tiles * cluster), dim3(kGemvWarps * 32), 0, cluster, p, cluster);
    return check_launch(args);
  };
  if (p.m <= 8u) return run(dense_gemv_kernel<1>);
  if (p.m <= 16u) return run(dense_gemv_kernel<2>);
  if (p.m <= 32u) return run(dense_gemv_kernel<4>);
  return run(dense_gemv_kernel<8>);
}

// Buffers [x, w, bias, out, out32, ids, table] (an absent one repeats another); params
// {m, n, k, split, has_bias, epilogue, table_rows, table_stride, table_offset}.
template <typename T>
int launch_dense_linear(const KernelArgs& args) {
  LLMOPT_REQUIRE(args.buffer_count == 7 && args.param_bytes == 36,
                 "expects buffers [x, w, bias, out, out32, ids, table] and 36 parameter bytes");
  DenseProblem p = {};
  p.m = param_u32(args, 0), p.n = param_u32(args, 1), p.k = param_u32(args, 2), p.split = param_u32(args, 3);
  p.has_bias = param_u32(args, 4), p.epilogue = param_u32(args, 5), p.table_rows = param_u32(args, 6);
  p.table_stride = param_u32(args, 7), p.table_offset = param_u32(args, 8);
  p.x = args.buffers[0], p.w = args.buffers[1], p.bias = (const float*)args.buffers[2], p.out = args.buffers[3];
  p.out32 = (float*)args.buffers[4], p.ids = (const long long*)args.buffers[5], p.table = args.buffers[6];
  LLMOPT_REQUIRE(p.n > 0 && p.k > 0 && p.split <= p.n, "needs n > 0, k > 0 and split <= n");
  if (p.m == 0) return 0;
  LLMOPT_REQUIRE(args.lengths[0] >= (size_t)p.m * p.k * sizeof(T), "activation buffer is too short");
  LLMOPT_REQUIRE(args.lengths[1] >= (size_t)p.n * p.k * sizeof(T), "weight buffer is too short");
  LLMOPT_REQUIRE(!p.has_bias || args.lengths[2] >= (size_t)p.n * 4, "bias buffer is too short");
  LLMOPT_REQUIRE(p.split == 0 || args.lengths[3] >= (size_t)p.m * p.split * sizeof(T), "output buffer is too short");
  LLMOPT_REQUIRE(p.split == p.n || args.lengths[4] >= (size_t)p.m * (p.n - p.split) * 4, "fp32 output buffer is too short");
  LLMOPT_REQUIRE(p.epilogue <= kDenseTokenGate, "unknown epilogue");
  if (p.epilogue == kDenseTokenGate) {
    LLMOPT_REQUIRE(args.lengths[5] >= (size_t)p.m * 8, "token buffer is too short");
    LLMOPT_REQUIRE(p.table_rows > 0 && (size_t)p.table_offset + p.n <= p.table_stride &&
                       args.lengths[6] >= (size_t)p.table_rows * p.table_stride * sizeof(T),
                   "token table is too short");
  }
  if (sizeof(T) == 4) return run_cuda_cores<T>(args, p);
  const bool vectors = p.k % 8u == 0 && ((uintptr_t)p.x & 15u) == 0 && ((uintptr_t)p.w & 15u) == 0;
  if (!vectors) return run_cuda_cores<T>(args, p);
  if (p.m > 64u) {
    const int status = launch_dense_gemm_tc(args, p);
    return status >= 0 ? status : run_cuda_cores<T>(args, p);
  }
  return run_gemv(args, p);
}

}  // namespace

const NamedLauncher* dense_linear_launchers(size_t* count) {
  static const NamedLauncher table[] = {
      {"llmopt_dense_linear_bf16", launch_dense_linear<bf16>},
      {"llmopt_dense_linear_f32", launch_dense_linear<float>},
  };
  *count = sizeof(table) / sizeof(table[0]);
  return table;
}

}  // namespace llmopt
