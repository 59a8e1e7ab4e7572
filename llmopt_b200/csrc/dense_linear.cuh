// Dense (unquantised) linear layer: problem description and writeback shared by its kernels.
#pragma once
#include "element.cuh"

namespace llmopt {

enum DenseEpilogue : uint32_t {
  kDenseNone = 0,
  kDenseGeluErf = 1,    // erf gelu of the sum
  kDenseTokenGate = 2,  // tanh gelu of the sum times table[token of the row][offset + column]
};

// y = x . w^T (+ bias), x [m, k], w [n, k].  Columns below `split` go to `out` (T, row stride split),
// the others to `out32` (fp32, row stride n - split): one product serves projections that are read
// in T and projections that feed fp32 arithmetic.
struct DenseProblem {
  const void* x;
  const void* w;
  const float* bias;  // [n], read when has_bias
  void* out;
  float* out32;
  const long long* ids;  // kDenseTokenGate: token of every row
  const void* table;     // kDenseTokenGate: T [table_rows, table_stride]
  uint32_t m, n, k, split, has_bias, epilogue, table_rows, table_stride, table_offset;
};

template <typename T>
__device__ __forceinline__ float dense_finish(const DenseProblem& p, uint32_t row, uint32_t column, float value) {
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

template <typename T>
__device__ __forceinline__ void dense_store(const DenseProblem& p, uint32_t row, uint32_t column, float value) {
  value = dense_finish<T>(p, row, column, value);
  if (column < p.split)
    reinterpret_cast<T*>(p.out)[(size_t)row * p.split + column] = from_float<T>(value);
  else
    p.out32[(size_t)row * (p.n - p.split) + (column - p.split)] = value;
}

// Prompt rows on tcgen05 (bf16); -1 when the shape or the pointers are outside its domain.
int launch_dense_gemm_tc(const KernelArgs& args, const DenseProblem& problem);

}  // namespace llmopt
