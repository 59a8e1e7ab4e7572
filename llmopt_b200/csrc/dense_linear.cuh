// Dense (unquantised) linear layer: problem description and writeback shared by its kernels.
#pragma once
#include "element.cuh"

namespace llmopt {

enum DenseEpilogue : uint32_t {
  kDenseNone = 0,
  kDenseGeluErf = 1,       // erf gelu of the sum
  kDenseTokenGate = 2,     // tanh gelu of the sum times table[token of the row][offset + column]
  kDenseSiluPair = 3,      // columns 2j, 2j + 1 are a gate and a value: out column j = silu(gate) * value, n / 2 columns
  kDenseResidualTanh = 4,  // residual += tanh norm of the sum; out = the next sublayer's tanh norm of the new residual
};

// What a kernel does with its sums, fixed at compile time (the code of the others would cost every launch).
enum DenseStore : uint32_t {
  kStorePlain = 0,     // rows in T and in fp32: kDenseNone, kDenseGeluErf, kDenseTokenGate
  kStoreCached = 1,    // the same, and key and value columns in the cache
  kStorePair = 2,      // kDenseSiluPair
  kStoreResidual = 3,  // kDenseResidualTanh
};

// y = scale * x . w^T (+ bias), x [m, k], w [n, k].  Columns below `split` go to `out` (T, row stride split), the next
// cache columns (if any) to the cache, the others to `out32` (fp32): one product serves projections that are read
// in T, that are kept, and that feed fp32 arithmetic.
struct DenseCore {
  const void* x;
  const void* w;
  uint32_t m, n, k, cluster;  // cluster: CTAs that share a tile's k-blocks, in the kernels that stream the weights
  uint32_t split, has_bias, epilogue;
  float scale;
  const float* bias;  // [n], read when has_bias
  void* out;
  float* out32;
  const long long* ids;  // kDenseTokenGate: token of every row
  const void* table;     // kDenseTokenGate: T [table_rows, table_stride]
  uint32_t table_rows, table_stride, table_offset;
};

// What only one kind of store reads.  A kernel gets no more than its own: a launch that streams few weights feels the
// size of its parameters.
struct DenseCacheRows {  // where the key and value columns go: the cache row of their token
  void* pool;
  const uint32_t* slots;  // [slots_rows, slots_stride]
  const uint32_t* past;
  const uint32_t* sequence_rows;
  uint32_t* error_word;
  uint32_t tokens;  // rows per sequence
  uint32_t key_columns, value_columns;
  uint32_t token_stride, key_offset, value_offset;  // in elements
  uint32_t slots_stride, slots_rows, pool_rows;
};
struct DenseRowScale {
  const float* row_scale;  // per row, multiplies the input; null: none
};
struct DenseResidual {
  const float* post_norm;  // norm of the sum, and of the sublayer that follows
  const float* next_norm;
  float* residual;  // [m, n], updated in place
};

// Rows sorted by expert, every expert with its own n rows of the weight matrix.  The plan holds the number of tiles,
// three unused words, and {expert, first row, row end, unused} per tile of at most kExpertTile rows.
constexpr uint32_t kExpertTile = 128;
struct DensePlan {
  const uint32_t* tiles;  // null: one matrix for all rows
  uint32_t experts;
};
struct DenseTile {
  uint32_t expert, first, end;
};
__device__ __forceinline__ DenseTile dense_tile(const DensePlan& plan, uint32_t index) {
  const uint4 entry = reinterpret_cast<const uint4*>(plan.tiles)[1 + index];
  return {entry.x, entry.y, entry.z};
}

// What a launch is described by, and what its kernel takes of that.
struct DenseProblem : DenseCore, DenseCacheRows, DenseRowScale, DenseResidual {
  DensePlan plan;
};
template <DenseStore STORE>
struct DenseTask : DenseCore {
  explicit DenseTask(const DenseProblem& p) : DenseCore(p) {}
};
template <>
struct DenseTask<kStoreCached> : DenseCore, DenseCacheRows {
  explicit DenseTask(const DenseProblem& p) : DenseCore(p), DenseCacheRows(p) {}
};
template <>
struct DenseTask<kStorePair> : DenseCore, DenseRowScale {
  explicit DenseTask(const DenseProblem& p) : DenseCore(p), DenseRowScale(p) {}
};
template <>
struct DenseTask<kStoreResidual> : DenseCore, DenseResidual {
  explicit DenseTask(const DenseProblem& p) : DenseCore(p), DenseResidual(p) {}
};

template <typename T>
__device__ __forceinline__ float dense_finish(const DenseCore& p, uint32_t row, uint32_t column, float value) {
  value *= p.scale;
  if (p.has_bias) value += __ldg(p.bias + column);
  if (p.epilogue == kDenseGeluErf) {
    value = gelu_erf_f32(value);
  } else if (p.epilogue == kDenseTokenGate) {
    const size_t token = min((unsigned long long)p.ids[row], (unsigned long long)(p.table_rows - 1u));
    value = gelu_tanh_f32(value) *
            as_float(reinterpret_cast<const T*>(p.table)[token * p.table_stride + p.table_offset + column]);
  }
  return value;
}
__device__ __forceinline__ float dense_biased(const DenseCore& p, uint32_t column, float value) {
  return p.has_bias ? value + __ldg(p.bias + column) : value;
}

// Cache row of the row's token; null (and the error word raised) when there is none.
template <typename T>
__device__ __forceinline__ T* dense_cache_row(const DenseCacheRows& c, uint32_t row) {
  const uint32_t sequence = row / c.tokens, position = c.past[sequence] + row % c.tokens, table_row = c.sequence_rows[sequence];
  uint32_t slot = c.pool_rows;
  if (table_row < c.slots_rows && position < c.slots_stride) slot = c.slots[(size_t)table_row * c.slots_stride + position];
  if (slot < c.pool_rows) return reinterpret_cast<T*>(c.pool) + (size_t)slot * c.token_stride;
  if (c.error_word) atomicExch(c.error_word, 1u);
  return nullptr;
}
// Offset in the cache row of column `at` of the cache columns.
__device__ __forceinline__ uint32_t dense_cache_offset(const DenseCacheRows& c, uint32_t at) {
  return at < c.key_columns ? c.key_offset + at : c.value_offset + at - c.key_columns;
}
// Columns that go to the cache.
template <DenseStore STORE>
__device__ __forceinline__ uint32_t dense_kept(const DenseTask<STORE>& p) {
  if constexpr (STORE == kStoreCached) return p.key_columns + p.value_columns;
  else return 0u;
}

template <typename T, DenseStore STORE>
__device__ __forceinline__ void dense_store(const DenseTask<STORE>& p, uint32_t row, uint32_t column, float value) {
  if constexpr (STORE == kStoreResidual) {
    const size_t at = (size_t)row * p.n + column;
    const float x = p.residual[at] + TanhNorm(p.post_norm, p.n)(dense_biased(p, column, value), column);
    p.residual[at] = x;
    reinterpret_cast<T*>(p.out)[at] = from_float<T>(TanhNorm(p.next_norm, p.n)(x, column));
  } else {
    value = STORE == kStoreCached ? dense_biased(p, column, value) : dense_finish<T>(p, row, column, value);
    const uint32_t kept = dense_kept(p);
    if (column < p.split) {
      reinterpret_cast<T*>(p.out)[(size_t)row * p.split + column] = from_float<T>(value);
      return;
    }
    if constexpr (STORE == kStoreCached) {
      if (column < p.split + kept) {
        T* const cached = dense_cache_row<T>(p, row);
        if (cached) cached[dense_cache_offset(p, column - p.split)] = from_float<T>(value);
        return;
      }
    }
    p.out32[(size_t)row * (p.n - p.split - kept) + (column - p.split - kept)] = value;
  }
}

// kDenseSiluPair: `column` is even; the row's scale (of its input) is linear in both sums.
__device__ __forceinline__ float dense_pair(const DenseTask<kStorePair>& p, uint32_t row, uint32_t column, float gate, float value) {
  const float scale = p.row_scale ? p.scale * p.row_scale[row] : p.scale;
  gate *= scale, value *= scale;
  if (p.has_bias) gate += __ldg(p.bias + column), value += __ldg(p.bias + column + 1u);
  return silu_f32(gate) * value;
}
template <typename T>
__device__ __forceinline__ void dense_store_pair(const DenseTask<kStorePair>& p, uint32_t row, uint32_t column, float gate,
                                                 float value) {
  reinterpret_cast<T*>(p.out)[(size_t)row * (p.n / 2u) + column / 2u] = from_float<T>(dense_pair(p, row, column, gate, value));
}

// Prompt rows on tcgen05 (bf16); -1 when the shape or the pointers are outside its domain.
int launch_dense_gemm_tc(const KernelArgs& args, const DenseProblem& problem, DenseStore store);

// Rows of at most `tiles` tiles of a plan, each with its expert's matrix.
template <typename T>
int run_expert_rows(const KernelArgs& args, const DenseProblem& problem, DenseStore store, uint32_t tiles);

}  // namespace llmopt
