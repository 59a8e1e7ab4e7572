// Feed-forward layers with routed experts.  A token's `top` experts are those with the largest router scores, a score
// is the sigmoid of its logit, and it multiplies the expert's input; an expert's weights are the gate and up rows
// interleaved ([2 width, k]: neighbouring rows are one pair) and the down rows, all experts' one after the other.
//
// Few rows, bfloat16 (decode): a chosen expert's weights are streamed once against the rows that chose it.
//   llmopt_route_step_f32             the chosen experts in order, their rows and scores
//   llmopt_expert_step_bf16           silu(s gate) (s up) of every (row, choice) pair
//   llmopt_expert_step_residual_bf16  down products of all chosen experts as one contraction, then (tanh norm, residual
//                                     add, next tanh norm) as in llmopt_dense_residual_*
// Any number of rows:
//   llmopt_route_rows_f32             (expert, score) of every (row, choice) pair
//   llmopt_route_plan                 the pairs sorted by expert, and the tiles of at most 128 of them
//   llmopt_expert_rows_{bf16,f32}     product of sorted rows with their experts' matrices (tcgen05 in bfloat16)
//   llmopt_expert_combine_{bf16,f32}  sum of a row's pairs, tanh norm, residual add, next tanh norm
#include "dense_stream.cuh"

namespace llmopt {
namespace {

constexpr uint32_t kMostExperts = 1024, kMostStreamed = 64, kMostPairs = 4096;  // of a step

// Next choice of a row after the one ranked `last`; the warp works together.
__device__ __forceinline__ unsigned long long next_choice(const float* logits, uint32_t experts, unsigned long long last) {
  unsigned long long best = 0;
  for (uint32_t e = threadIdx.x & 31u; e < experts; e += 32u) {
    const unsigned long long key = ranked(logits[e], e);
    if (key < last) best = max(best, key);
  }
  for (int offset = 16; offset > 0; offset >>= 1) best = max(best, __shfl_xor_sync(0xffffffffu, best, offset));
  return best;
}
__device__ __forceinline__ uint32_t ranked_column(unsigned long long key) { return 0xffffffffu - (uint32_t)key; }

// ---- few rows ------------------------------------------------------------------------------------
// Route of a step, in words: the number of chosen experts, three unused, the experts, the first slot of each (and the end),
// then per slot its row and per slot its score (fp32).
struct Route {
  uint32_t first, row, score, words;
  __host__ __device__ Route(uint32_t rows, uint32_t experts, uint32_t top) {
    first = 4u + (experts + 3u) / 4u * 4u;
    row = first + (experts + 4u) / 4u * 4u;
    score = row + rows * top;
    words = score + rows * top;
  }
};

__global__ void __launch_bounds__(1024) route_step_kernel(const float* logits, uint32_t* route, uint32_t rows, uint32_t experts,
                                                          uint32_t top, Route at) {
  grid_chain_prologue();
  extern __shared__ uint32_t route_shared[];
  uint32_t* counts = route_shared;                                  // [experts]
  uint32_t* active = counts + experts;                              // [experts] chosen ones in order
  uint32_t* first = active + experts;                               // [experts + 1]
  uint32_t* chosen = first + experts + 1u;                          // [rows * top]
  float* scores = reinterpret_cast<float*>(chosen + rows * top);    // [rows * top]
  __shared__ uint32_t used;
  const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31u, pairs = rows * top;
  for (uint32_t e = threadIdx.x; e < experts; e += blockDim.x) counts[e] = 0u;
  __syncthreads();
  for (uint32_t row = warp; row < rows; row += blockDim.x / 32u) {
    const float* z = logits + (size_t)row * experts;
    unsigned long long last = ~0ull;
    for (uint32_t j = 0; j < top; ++j) {
      last = next_choice(z, experts, last);
      const uint32_t expert = min(ranked_column(last), experts - 1u);
      if (lane == 0) {
        chosen[row * top + j] = expert;
        scores[row * top + j] = sigmoid_f32(z[expert]);
        atomicAdd(&counts[expert], 1u);
      }
    }
  }
  __syncthreads();
  if (warp == 0) {
    uint32_t place = 0, slot = 0;
    for (uint32_t e0 = 0; e0 < experts; e0 += 32u) {
      const uint32_t e = e0 + lane, count = e < experts ? counts[e] : 0u;
      const uint32_t all = __ballot_sync(0xffffffffu, count > 0u), mine = place + __popc(all & ((1u << lane) - 1u));
      uint32_t through = count;  // inclusive sum
#pragma unroll
      for (int offset = 1; offset < 32; offset <<= 1) {
        const uint32_t other = __shfl_up_sync(0xffffffffu, through, offset);
        if (lane >= (uint32_t)offset) through += other;
      }
      if (count > 0u) {
        active[mine] = route[4 + mine] = e;
        first[mine] = route[at.first + mine] = slot + through - count;
      }
      place += __popc(all);
      slot += __shfl_sync(0xffffffffu, through, 31);
    }
    if (lane == 0) {
      used = route[0] = place;
      route[at.first + place] = slot;
    }
  }
  __syncthreads();
  for (uint32_t a = warp; a < used; a += blockDim.x / 32u) {
    uint32_t slot = first[a];
    for (uint32_t p0 = 0; p0 < pairs; p0 += 32u) {
      const uint32_t pair = p0 + lane;
      const bool hit = pair < pairs && chosen[pair] == active[a];
      const uint32_t all = __ballot_sync(0xffffffffu, hit), here = slot + __popc(all & ((1u << lane) - 1u));
      if (hit) {
        route[at.row + here] = pair / top;
        route[at.score + here] = __float_as_uint(scores[pair]);
      }
      slot += __popc(all);
    }
  }
}

uint32_t most_chosen(uint32_t rows, uint32_t experts, uint32_t top) {
  const size_t pairs = (size_t)rows * top;
  return pairs < experts ? (uint32_t)pairs : experts;
}

// Buffers [logits f32, route]; params {rows, experts, top}.
int launch_route_step(const KernelArgs& args) {
  LLMOPT_REQUIRE(args.buffer_count == 2 && args.param_bytes == 12, "expects 2 buffers and 12 parameter bytes");
  const uint32_t rows = param_u32(args, 0), experts = param_u32(args, 1), top = param_u32(args, 2);
  LLMOPT_REQUIRE(experts > 0 && experts <= kMostExperts && top > 0 && top <= experts, "needs experts, at most 1024, and a choice of them");
  LLMOPT_REQUIRE(rows <= kMostStreamed, "at most 64 rows");
  const Route at(rows, experts, top);
  LLMOPT_REQUIRE(args.lengths[0] >= (size_t)rows * experts * 4 &&
                     args.lengths[1] >= (size_t)at.words * 4,
                 "buffer is too short");
  const size_t shared = (3 * (size_t)experts + 1 + 2 * (size_t)rows * top) * 4;
  LLMOPT_REQUIRE(shared <= 48 * 1024, "too many choices for one step");
  if (rows == 0) return 0;
  launch_kernel(args, route_step_kernel, dim3(1), dim3(1024), shared, (const float*)args.buffers[0], (uint32_t*)args.buffers[1],
                rows, experts, top, at);
  return check_launch(args);
}

// DOWN: x holds [slot][k], an expert's rows one after the other, and the k-blocks of all chosen experts form one
// contraction: a warp adds an expert's sums to those of the rows that chose it when it goes on to the next.  Otherwise x
// is [row][k] and blockIdx.y picks the expert.
// The first eight rows of an expert travel through the stages with the weights, further ones are loaded when it is their turn.
template <int NT, bool DOWN>
__global__ void __launch_bounds__(kGemvWarps * 32, NT <= 4 ? 2 : 1) expert_step_kernel(DenseTask<DOWN ? kStoreResidual : kStorePair> p, uint32_t experts, const uint32_t* route, Route at, uint32_t pairs) {
  const uint32_t cluster = p.cluster;
  grid_chain_prologue();
  __shared__ uint32_t chosen[DOWN ? kMostExperts : 1], firsts[DOWN ? kMostExperts + 1 : 1];
  __shared__ uint8_t row_of_slot[DOWN ? kMostPairs : 1];
  __shared__ float partial[kGemvWarps][NT * 8][17];
  const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31u, g = lane >> 2, t = lane & 3u;
  const uint32_t n0 = blockIdx.x / cluster * 16u, rank = blockIdx.x % cluster, stride = kGemvWarps * cluster;
  const uint32_t used = min(route[0], experts), rows = p.m;
  if (!DOWN && blockIdx.y >= used) return;  // the whole cluster: it lies along x
  if (DOWN) {
    for (uint32_t i = threadIdx.x; i <= used; i += kGemvWarps * 32) {
      if (i < used) chosen[i] = min(route[4 + i], experts - 1u);
      firsts[i] = min(route[at.first + i], pairs);
    }
    for (uint32_t i = threadIdx.x; i < pairs; i += kGemvWarps * 32) row_of_slot[i] = (uint8_t)min(route[at.row + i], rows - 1u);
    for (uint32_t i = lane; i < NT * 8u * 17u; i += 32u) (&partial[warp][0][0])[i] = 0.0f;
    __syncthreads();
  }
  const uint32_t low = min(n0 + g, p.n - 1u), high = min(n0 + g + 8u, p.n - 1u);
  const uint32_t per_expert = (p.k + 63u) / 64u, blocks = DOWN ? used * per_expert : per_expert;
  const bf16* w = reinterpret_cast<const bf16*>(p.w);
  const bf16* x = reinterpret_cast<const bf16*>(p.x);
  const bf16* own[DOWN ? 1 : NT];  // the lane's rows of this expert
  uint32_t mine = 0;
  if (!DOWN) {
    const uint32_t first = min(route[at.first + blockIdx.y], pairs);
    mine = min(route[at.first + blockIdx.y + 1u] - first, rows);
    w += (size_t)min(route[4 + blockIdx.y], experts - 1u) * p.n * p.k;
#pragma unroll
    for (int nt = 0; nt < (DOWN ? 1 : NT); ++nt) {
      const uint32_t place = nt * 8u + g;
      own[nt] = place < mine ? x + (size_t)min(route[at.row + first + place], rows - 1u) * p.k : nullptr;
    }
    p.m = mine;
    if constexpr (!DOWN) p.row_scale = reinterpret_cast<const float*>(route) + at.score + first;
    p.out = reinterpret_cast<bf16*>(p.out) + (size_t)first * (p.n / 2u);
  }
  // rows of the expert at `place`, and the lane's row of tile nt
  auto count_of = [&](uint32_t place) { return DOWN ? min(firsts[place + 1u] - firsts[place], rows) : mine; };
  auto row_of = [&](uint32_t place, int nt) -> const bf16* {
    if (!DOWN) return own[DOWN ? 0 : nt];
    return nt * 8u + g < count_of(place) ? x + (size_t)min(firsts[place] + nt * 8u + g, pairs - 1u) * p.k : nullptr;
  };
  const uint4 zero = make_uint4(0u, 0u, 0u, 0u);
  uint4 a[kGemvStages][4], b[kGemvStages][2];
  auto fetch = [&](int stage, uint32_t index) {
    const bool present = index < blocks;
    const uint32_t place = DOWN && present ? index / per_expert : 0u, block = index - place * per_expert;
    const bf16* matrix = DOWN && present ? w + (size_t)chosen[place] * p.n * p.k : w;
    stream_fetch(a[stage], matrix + (size_t)low * p.k, matrix + (size_t)high * p.k, present ? p.k : 0u, block);
    const bf16* row = present ? row_of(place, 0) : nullptr;
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const uint32_t k = block * 64u + half * 32u + t * 8u;
      b[stage][half] = row != nullptr && k < p.k ? *reinterpret_cast<const uint4*>(row + k) : zero;
    }
  };
#pragma unroll
  for (int s = 0; s < kGemvStages; ++s) fetch(s, rank * kGemvWarps + warp + s * stride);
  float sum[NT][4];
  auto clear = [&]() {
#pragma unroll
    for (int nt = 0; nt < NT; ++nt)
#pragma unroll
      for (int i = 0; i < 4; ++i) sum[nt][i] = 0.0f;
  };
  // the finished expert's sums to the rows that chose it
  auto flush = [&](uint32_t place) {
    const uint32_t first = firsts[DOWN ? place : 0], count = count_of(place);
#pragma unroll
    for (int nt = 0; nt < NT; ++nt)
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const uint32_t c = nt * 8u + 2u * t + (i & 1);
        if (c < count) partial[warp][row_of_slot[DOWN ? first + c : 0]][g + (i >> 1) * 8] += sum[nt][i];
      }
    __syncwarp();
    clear();
  };
  clear();
  uint32_t current = 0;
  for (uint32_t first = rank * kGemvWarps + warp; first < blocks; first += kGemvStages * stride) {
#pragma unroll
    for (int s = 0; s < kGemvStages; ++s) {
      const uint32_t index = first + s * stride;
      if (index < blocks) {
        const uint32_t place = DOWN ? index / per_expert : 0u, block = index - place * per_expert;
        if (DOWN && place != current) {
          flush(current);
          current = place;
        }
#pragma unroll
        for (int half = 0; half < 2; ++half) stream_multiply(sum[0], a[s][half], a[s][2 + half], b[s][half]);
        const uint32_t count = count_of(place);
#pragma unroll
        for (int nt = 1; nt < NT; ++nt) {
          if (nt * 8u >= count) break;
          const bf16* row = row_of(place, nt);
#pragma unroll
          for (int half = 0; half < 2; ++half) {
            const uint32_t k = block * 64u + half * 32u + t * 8u;
            stream_multiply(sum[nt], a[s][half], a[s][2 + half],
                            row != nullptr && k < p.k ? *reinterpret_cast<const uint4*>(row + k) : zero);
          }
        }
      }
      fetch(s, index + kGemvStages * stride);
    }
  }
  if (!DOWN) stream_collect<NT>(sum, partial[warp]);
  else if (used > 0) flush(current);
  stream_finish<NT>(p, partial, n0, rank, cluster);
}

template <bool DOWN>
int run_step(const KernelArgs& args, DenseProblem p, const uint32_t* route, const Route& at, uint32_t most, uint32_t top) {
  if (p.m == 0) return 0;
  const uint32_t tiles = (p.n + 15u) / 16u, blocks = (p.k + 63u) / 64u;
  p.cluster = stream_cluster(args, DOWN ? tiles : tiles * most, DOWN ? blocks * most : blocks);
  auto run = [&](auto kernel) {
    const dim3 grid(tiles * p.cluster, DOWN ? 1u : most);
    const DenseTask<DOWN ? kStoreResidual : kStorePair> task(p);
    const uint32_t experts = p.plan.experts, pairs = p.m * top;
    if (p.cluster == 1u) launch_kernel(args, kernel, grid, dim3(kGemvWarps * 32), 0, task, experts, route, at, pairs);
    else launch_cluster_kernel(args, kernel, grid, dim3(kGemvWarps * 32), 0, p.cluster, task, experts, route, at, pairs);
    return check_launch(args);
  };
  if (p.m <= 8u) return run(expert_step_kernel<1, DOWN>);
  if (p.m <= 16u) return run(expert_step_kernel<2, DOWN>);
  if (p.m <= 32u) return run(expert_step_kernel<4, DOWN>);
  return run(expert_step_kernel<8, DOWN>);
}

// Params {rows, n, k, experts, top} (both forms), the route at buffer 2.
int read_step(const KernelArgs& args, DenseProblem& p, uint32_t& top) {
  LLMOPT_REQUIRE(args.param_bytes == 20, "expects 20 parameter bytes");
  p = {};
  p.m = param_u32(args, 0), p.n = param_u32(args, 1), p.k = param_u32(args, 2), p.plan.experts = param_u32(args, 3);
  top = param_u32(args, 4);
  p.scale = 1.0f, p.x = args.buffers[0], p.w = args.buffers[1], p.split = p.n;
  LLMOPT_REQUIRE(p.n > 0 && p.k > 0 && p.k % 8u == 0 && p.plan.experts > 0 && p.plan.experts <= kMostExperts && top > 0 && top <= p.plan.experts &&
                     p.m <= kMostStreamed && p.m * top <= kMostPairs,
                 "needs experts, k in whole vectors of eight, at most 64 rows and 4096 choices");
  LLMOPT_REQUIRE(args.lengths[1] >= (size_t)p.plan.experts * p.n * p.k * 2 &&
                     args.lengths[2] >= (size_t)Route(p.m, p.plan.experts, top).words * 4,
                 "buffer is too short");
  LLMOPT_REQUIRE(((uintptr_t)p.x & 15u) == 0 && ((uintptr_t)p.w & 15u) == 0, "buffers must be 16-byte aligned");
  return 0;
}

// Buffers [x, gate and up rows, route, out [slot][n / 2]].
int launch_expert_step(const KernelArgs& args) {
  LLMOPT_REQUIRE(args.buffer_count == 4, "expects 4 buffers");
  DenseProblem p;
  uint32_t top;
  if (const int status = read_step(args, p, top)) return status;
  p.epilogue = kDenseSiluPair, p.out = args.buffers[3];
  LLMOPT_REQUIRE(p.n % 2u == 0 && args.lengths[0] >= (size_t)p.m * p.k * 2 && args.lengths[3] >= (size_t)p.m * top * (p.n / 2u) * 2,
                 "buffer is too short");
  const uint32_t most = most_chosen(p.m, p.plan.experts, top);
  return run_step<false>(args, p, (const uint32_t*)args.buffers[2], Route(p.m, p.plan.experts, top), most, top);
}

// Buffers [x [slot][k], down rows, route, norm of the sum, following norm, residual, out].
int launch_expert_step_residual(const KernelArgs& args) {
  LLMOPT_REQUIRE(args.buffer_count == 7, "expects 7 buffers");
  DenseProblem p;
  uint32_t top;
  if (const int status = read_step(args, p, top)) return status;
  p.epilogue = kDenseResidualTanh;
  p.post_norm = (const float*)args.buffers[3], p.next_norm = (const float*)args.buffers[4];
  p.residual = (float*)args.buffers[5], p.out = args.buffers[6];
  LLMOPT_REQUIRE(args.lengths[0] >= (size_t)p.m * top * p.k * 2 && args.lengths[3] >= (2 * (size_t)p.n + 1) * 4 &&
                     args.lengths[4] >= (2 * (size_t)p.n + 1) * 4 && args.lengths[5] >= (size_t)p.m * p.n * 4 &&
                     args.lengths[6] >= (size_t)p.m * p.n * 2,
                 "buffer is too short");
  const uint32_t most = most_chosen(p.m, p.plan.experts, top);
  return run_step<true>(args, p, (const uint32_t*)args.buffers[2], Route(p.m, p.plan.experts, top), most, top);
}

// ---- any number of rows ----------------------------------------------------------------------------
__global__ void __launch_bounds__(128) route_rows_kernel(const float* logits, uint32_t* chosen, float* scores, uint32_t rows,
                                                         uint32_t experts, uint32_t top) {
  grid_chain_prologue();
  const uint32_t row = blockIdx.x * 4u + (threadIdx.x >> 5);
  if (row >= rows) return;
  const float* z = logits + (size_t)row * experts;
  unsigned long long last = ~0ull;
  for (uint32_t j = 0; j < top; ++j) {
    last = next_choice(z, experts, last);
    const uint32_t expert = min(ranked_column(last), experts - 1u);
    if ((threadIdx.x & 31u) == 0u) {
      chosen[(size_t)row * top + j] = expert;
      scores[(size_t)row * top + j] = sigmoid_f32(z[expert]);
    }
  }
}

// Buffers [logits f32, chosen u32 [rows, top], scores f32 [rows, top]]; params {rows, experts, top}.
int launch_route_rows(const KernelArgs& args) {
  LLMOPT_REQUIRE(args.buffer_count == 3 && args.param_bytes == 12, "expects 3 buffers and 12 parameter bytes");
  const uint32_t rows = param_u32(args, 0), experts = param_u32(args, 1), top = param_u32(args, 2);
  LLMOPT_REQUIRE(experts > 0 && top > 0 && top <= experts, "needs experts and a choice of them");
  LLMOPT_REQUIRE(args.lengths[0] >= (size_t)rows * experts * 4 && args.lengths[1] >= (size_t)rows * top * 4 &&
                     args.lengths[2] >= (size_t)rows * top * 4,
                 "buffer is too short");
  if (rows == 0) return 0;
  launch_kernel(args, route_rows_kernel, dim3((rows + 3u) / 4u), dim3(128), 0, (const float*)args.buffers[0],
                (uint32_t*)args.buffers[1], (float*)args.buffers[2], rows, experts, top);
  return check_launch(args);
}

__device__ __forceinline__ uint32_t block_total(uint32_t v, uint32_t* scratch) {
#pragma unroll
  for (int offset = 16; offset > 0; offset >>= 1) v += __shfl_xor_sync(0xffffffffu, v, offset);
  __syncthreads();  // the previous use of the scratch is over
  if ((threadIdx.x & 31u) == 0u) scratch[threadIdx.x >> 5] = v;
  __syncthreads();
  v = 0;
  for (uint32_t w = 0; w < blockDim.x / 32u; ++w) v += scratch[w];
  return v;
}

// One CTA per expert: counts all pairs, finds its first slot and tile, and lists its own pairs in their order.
__global__ void __launch_bounds__(1024) route_plan_kernel(const uint32_t* chosen, const float* scores, uint32_t* plan,
                                                         uint32_t* row_of_slot, float* score_of_slot, uint32_t* slot_of_pair,
                                                         uint32_t pairs, uint32_t experts, uint32_t top) {
  grid_chain_prologue();
  extern __shared__ uint32_t counts[];
  __shared__ uint32_t scratch[32], hits_of_warp[32];
  const uint32_t expert = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31u;
  for (uint32_t e = threadIdx.x; e < experts; e += 1024u) counts[e] = 0u;
  __syncthreads();
  for (uint32_t i = threadIdx.x; i < pairs; i += 1024u) atomicAdd(&counts[min(chosen[i], experts - 1u)], 1u);
  __syncthreads();
  uint32_t before = 0, tiles_before = 0, all_tiles = 0;
  for (uint32_t e = threadIdx.x; e < experts; e += 1024u) {
    const uint32_t tiles = (counts[e] + kExpertTile - 1u) / kExpertTile;
    all_tiles += tiles;
    if (e < expert) {
      before += counts[e];
      tiles_before += tiles;
    }
  }
  before = block_total(before, scratch);
  tiles_before = block_total(tiles_before, scratch);
  all_tiles = block_total(all_tiles, scratch);
  const uint32_t mine = counts[expert];
  if (expert == 0 && threadIdx.x == 0) plan[0] = all_tiles;
  for (uint32_t t = threadIdx.x; t * kExpertTile < mine; t += 1024u)
    reinterpret_cast<uint4*>(plan)[1 + tiles_before + t] =
        make_uint4(expert, before + t * kExpertTile, before + min(mine, (t + 1u) * kExpertTile), 0u);
  uint32_t slot = before;
  for (uint32_t first = 0; first < pairs; first += 1024u) {
    const uint32_t pair = first + threadIdx.x;
    const bool hit = pair < pairs && min(chosen[pair], experts - 1u) == expert;
    const uint32_t all = __ballot_sync(0xffffffffu, hit);
    __syncthreads();
    if (lane == 0) hits_of_warp[warp] = __popc(all);
    __syncthreads();
    uint32_t here = slot + __popc(all & ((1u << lane) - 1u));
    for (uint32_t w = 0; w < 32u; ++w) {
      if (w < warp) here += hits_of_warp[w];
      slot += hits_of_warp[w];
    }
    if (hit) {
      row_of_slot[here] = pair / top;
      score_of_slot[here] = scores[pair];
      slot_of_pair[pair] = here;
    }
  }
}

uint32_t most_plan_tiles(uint32_t pairs, uint32_t experts) { return pairs / kExpertTile + (pairs < experts ? pairs : experts); }

// Buffers [chosen, scores, plan, row of slot u32, score of slot f32, slot of pair u32]; params {rows, experts, top}.
int launch_route_plan(const KernelArgs& args) {
  LLMOPT_REQUIRE(args.buffer_count == 6 && args.param_bytes == 12, "expects 6 buffers and 12 parameter bytes");
  const uint32_t rows = param_u32(args, 0), experts = param_u32(args, 1), top = param_u32(args, 2);
  LLMOPT_REQUIRE(experts > 0 && experts <= 8192u && top > 0 && top <= experts && (size_t)rows * top < (1u << 30),
                 "needs experts and a choice of them");
  const uint32_t pairs = rows * top;
  for (int i : {0, 1, 3, 4, 5}) LLMOPT_REQUIRE(args.lengths[i] >= (size_t)pairs * 4, "buffer is too short");
  LLMOPT_REQUIRE(args.lengths[2] >= 16 * (1 + (size_t)most_plan_tiles(pairs, experts)), "plan is too short");
  LLMOPT_REQUIRE(((uintptr_t)args.buffers[2] & 15u) == 0, "the plan must be 16-byte aligned");
  if (rows == 0) return 0;
  launch_kernel(args, route_plan_kernel, dim3(experts), dim3(1024), experts * 4, (const uint32_t*)args.buffers[0],
                (const float*)args.buffers[1], (uint32_t*)args.buffers[2], (uint32_t*)args.buffers[3], (float*)args.buffers[4],
                (uint32_t*)args.buffers[5], pairs, experts, top);
  return check_launch(args);
}

// Buffers [x sorted, w, plan, score of slot, out]; params {pairs, n, k, experts, paired}.  paired: n gate and up rows, out
// [pairs, n / 2] in the element type; otherwise out is fp32 [pairs, n].
template <typename T>
int launch_expert_rows(const KernelArgs& args) {
  LLMOPT_REQUIRE(args.buffer_count == 5 && args.param_bytes == 20, "expects 5 buffers and 20 parameter bytes");
  DenseProblem p = {};
  p.m = param_u32(args, 0), p.n = param_u32(args, 1), p.k = param_u32(args, 2), p.plan.experts = param_u32(args, 3);
  const bool paired = param_u32(args, 4) != 0;
  p.scale = 1.0f, p.x = args.buffers[0], p.w = args.buffers[1], p.plan.tiles = (const uint32_t*)args.buffers[2];
  if (paired) p.epilogue = kDenseSiluPair, p.split = p.n, p.row_scale = (const float*)args.buffers[3], p.out = args.buffers[4];
  else p.out32 = (float*)args.buffers[4];
  LLMOPT_REQUIRE(p.n > 0 && p.k > 0 && p.plan.experts > 0 && (!paired || p.n % 2u == 0), "needs n > 0, k > 0 and experts");
  const uint32_t tiles = most_plan_tiles(p.m, p.plan.experts);
  LLMOPT_REQUIRE(args.lengths[0] >= (size_t)p.m * p.k * sizeof(T) && args.lengths[1] >= (size_t)p.plan.experts * p.n * p.k * sizeof(T) &&
                     args.lengths[2] >= 16 * (1 + (size_t)tiles) && args.lengths[3] >= (size_t)p.m * 4 &&
                     args.lengths[4] >= (paired ? (size_t)p.m * (p.n / 2u) * sizeof(T) : (size_t)p.m * p.n * 4),
                 "buffer is too short");
  LLMOPT_REQUIRE((size_t)p.plan.experts * p.n < (1u << 31), "too many weight rows");
  if (p.m == 0) return 0;
  return run_expert_rows<T>(args, p, paired ? kStorePair : kStorePlain, tiles);
}

// One CTA per row.
template <typename T>
__global__ void __launch_bounds__(256) expert_combine_kernel(const float* y, const uint32_t* slot_of_pair, const float* post_norm,
                                                             const float* next_norm, float* residual, T* out, uint32_t rows,
                                                             uint32_t width, uint32_t top, uint32_t vectors) {
  grid_chain_prologue();
  const uint32_t pairs = rows * top;
  const uint32_t* slots = slot_of_pair + (size_t)blockIdx.x * top;
  const size_t base = (size_t)blockIdx.x * width;
  const TanhNorm post(post_norm, width), next(next_norm, width);
  if (vectors) {
    for (uint32_t c = threadIdx.x * 4u; c < width; c += 1024u) {
      float4 sum = make_float4(0.f, 0.f, 0.f, 0.f);
      for (uint32_t j = 0; j < top; ++j) {
        const float4 v = *reinterpret_cast<const float4*>(y + (size_t)min(slots[j], pairs - 1u) * width + c);
        sum.x += v.x, sum.y += v.y, sum.z += v.z, sum.w += v.w;
      }
      float4 x = *reinterpret_cast<const float4*>(residual + base + c);
      const float4 add = post.four(sum, c);
      x.x += add.x, x.y += add.y, x.z += add.z, x.w += add.w;
      *reinterpret_cast<float4*>(residual + base + c) = x;
      store_four(out + base + c, next.four(x, c));
    }
    return;
  }
  for (uint32_t c = threadIdx.x; c < width; c += 256u) {
    float sum = 0.0f;
    for (uint32_t j = 0; j < top; ++j) sum += y[(size_t)min(slots[j], pairs - 1u) * width + c];
    const float x = residual[base + c] + post(sum, c);
    residual[base + c] = x;
    out[base + c] = from_float<T>(next(x, c));
  }
}

// Buffers [y f32 [pairs, width], slot of pair, norm of the sum, following norm, residual, out]; params {rows, width, top}.
template <typename T>
int launch_expert_combine(const KernelArgs& args) {
  LLMOPT_REQUIRE(args.buffer_count == 6 && args.param_bytes == 12, "expects 6 buffers and 12 parameter bytes");
  const uint32_t rows = param_u32(args, 0), width = param_u32(args, 1), top = param_u32(args, 2);
  const size_t pairs = (size_t)rows * top;
  LLMOPT_REQUIRE(width > 0 && top > 0, "needs a width and choices");
  LLMOPT_REQUIRE(args.lengths[0] >= pairs * width * 4 && args.lengths[1] >= pairs * 4 &&
                     args.lengths[2] >= (2 * (size_t)width + 1) * 4 && args.lengths[3] >= (2 * (size_t)width + 1) * 4 &&
                     args.lengths[4] >= (size_t)rows * width * 4 && args.lengths[5] >= (size_t)rows * width * sizeof(T),
                 "buffer is too short");
  if (rows == 0) return 0;
  uint32_t vectors = width % 4u == 0;
  for (int i : {0, 2, 3, 4, 5})
    if ((uintptr_t)args.buffers[i] & 15u) vectors = 0;
  launch_kernel(args, expert_combine_kernel<T>, dim3(rows), dim3(256), 0, (const float*)args.buffers[0],
                (const uint32_t*)args.buffers[1], (const float*)args.buffers[2], (const float*)args.buffers[3],
                (float*)args.buffers[4], (T*)args.buffers[5], rows, width, top, vectors);
  return check_launch(args);
}

}  // namespace

const NamedLauncher* expert_launchers(size_t* count) {
  static const NamedLauncher table[] = {
      {"llmopt_route_step_f32", launch_route_step},
      {"llmopt_expert_step_bf16", launch_expert_step},
      {"llmopt_expert_step_residual_bf16", launch_expert_step_residual},
      {"llmopt_route_rows_f32", launch_route_rows},
      {"llmopt_route_plan", launch_route_plan},
      {"llmopt_expert_rows_bf16", launch_expert_rows<bf16>},
      {"llmopt_expert_rows_f32", launch_expert_rows<float>},
      {"llmopt_expert_combine_bf16", launch_expert_combine<bf16>},
      {"llmopt_expert_combine_f32", launch_expert_combine<float>},
  };
  *count = sizeof(table) / sizeof(table[0]);
  return table;
}

}  // namespace llmopt
