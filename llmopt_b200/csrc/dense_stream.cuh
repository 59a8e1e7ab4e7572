// Pieces of the kernels that stream bfloat16 weight rows from HBM straight into mma.sync fragments, for few
// activation rows: a warp holds 16 weight rows against NT tiles of eight activation rows.
#pragma once
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

// A 64-wide k-block of the lane's two weight rows: low / high 32 k of each; zeros from `width` on.
__device__ __forceinline__ void stream_fetch(uint4 (&stage)[4], const bf16* w_low, const bf16* w_high, uint32_t width,
                                             uint32_t block) {
  const uint32_t t = threadIdx.x & 3u;
#pragma unroll
  for (int half = 0; half < 2; ++half) {
    const uint32_t k = block * 64u + half * 32u + t * 8u;
    const uint4 zero = make_uint4(0u, 0u, 0u, 0u);
    stage[half] = k < width ? load_stream(w_low + k) : zero;
    stage[2 + half] = k < width ? load_stream(w_high + k) : zero;
  }
}

// sum += a half (32 k) of a k-block of the weights times the same k of a tile's rows.
__device__ __forceinline__ void stream_multiply(float (&sum)[4], const uint4& low, const uint4& high, const uint4& x) {
  mma_bf16(sum, low.x, high.x, low.y, high.y, x.x, x.y);
  mma_bf16(sum, low.z, high.z, low.w, high.w, x.z, x.w);
}

// A warp's sums, [activation row][weight row].
template <int NT>
__device__ __forceinline__ void stream_collect(const float (&sum)[NT][4], float (&mine)[NT * 8][17]) {
  const uint32_t lane = threadIdx.x & 31u, g = lane >> 2, t = lane & 3u;
#pragma unroll
  for (int nt = 0; nt < NT; ++nt)
#pragma unroll
    for (int i = 0; i < 4; ++i) mine[nt * 8 + 2 * t + (i & 1)][g + (i >> 1) * 8] = sum[nt][i];
}

template <DenseStore STORE, int N>
__device__ __forceinline__ void stream_store(const DenseTask<STORE>& p, uint32_t row, uint32_t column, const float (&value)[N]) {
  if constexpr (STORE == kStorePair) dense_store_pair<bf16>(p, row, column, value[0], value[N - 1]);
  else dense_store<bf16>(p, row, column, value[0]);
}

// Adds the warps' sums of the 16 columns from n0 on (and those of the cluster's CTAs) and stores them.
template <int NT, DenseStore STORE>
__device__ __forceinline__ void stream_finish(const DenseTask<STORE>& p, float (&partial)[kGemvWarps][NT * 8][17], uint32_t n0,
                                              uint32_t rank, uint32_t cluster) {
  const uint32_t stride = kGemvWarps * cluster;
  __syncthreads();
  constexpr uint32_t kStep = STORE == kStorePair ? 2u : 1u;  // columns a thread stores together
  for (uint32_t index = threadIdx.x * kStep; index < NT * 8u * 16u; index += kGemvWarps * 32 * kStep) {
    const uint32_t column = index & 15u, row = index >> 4;
    if (row >= p.m || n0 + column >= p.n) continue;
    float value[kStep];
#pragma unroll
    for (uint32_t i = 0; i < kStep; ++i) {
      value[i] = 0.0f;
#pragma unroll
      for (int part = 0; part < kGemvWarps; ++part) value[i] += partial[part][row][column + i];
      if (cluster > 1u) partial[0][row][column + i] = value[i];  // read and written by this thread only
    }
    if (cluster == 1u) stream_store(p, row, n0 + column, value);
  }
  if (cluster == 1u) return;
  cluster_sync();
  // the cluster's CTAs share out the outputs; sums in rank order
  for (uint32_t index = (rank * kGemvWarps * 32 + threadIdx.x) * kStep; index < NT * 8u * 16u; index += stride * 32u * kStep) {
    const uint32_t column = index & 15u, row = index >> 4;
    if (row >= p.m || n0 + column >= p.n) continue;
    float value[kStep];
#pragma unroll
    for (uint32_t i = 0; i < kStep; ++i) {
      value[i] = 0.0f;
      for (uint32_t other = 0; other < cluster; ++other) value[i] += cluster_load(&partial[0][row][column + i], other);
    }
    stream_store(p, row, n0 + column, value);
  }
  cluster_sync();  // nobody leaves while its sums may be read
}

// CTAs per cluster that share out the k-blocks of `tiles` 16-row tiles: at least one CTA per SM, and a warp of a
// split keeps at least one of the `blocks`.
inline uint32_t stream_cluster(const KernelArgs& args, uint32_t tiles, uint32_t blocks) {
  const uint32_t wanted = (uint32_t)context_sm_count(args.ctx);
  uint32_t cluster = 1;
  while (cluster < 8u && tiles * cluster < wanted && blocks >= 2u * cluster * kGemvWarps) cluster *= 2u;
  return cluster;
}

}  // namespace
}  // namespace llmopt
