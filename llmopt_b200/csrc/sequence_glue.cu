// Row-wise kernels of decoders whose residual stream is kept in fp32 and whose sublayers read it
// directly (T: bfloat16 or float, the element of activations and weights):
//   llmopt_embedding_residual_{bf16,f32}   x = table[token], with a T copy for the next product
//   llmopt_embedding_sinusoid_{bf16,f32}   x = table[token] + sinusoidal position, with its tanh norm for the next product
//   llmopt_gather_rows_{bf16,f32}          chosen rows in a new order
//   llmopt_residual_norm_{bf16,f32}        x += norm(y), or of the mean of two normed branches
//   llmopt_gather_norm_{bf16,f32}          norm of chosen rows (input of the output projection)
//   llmopt_row_attention_prepare_{bf16,f32} head norm + rotary of q and k, k and v into the cache
//   llmopt_head_norm_gate_{bf16,f32}       per-head norm of a mixer's read-out times its gate
//   llmopt_argmax_f32, llmopt_advance_tokens   greedy pick and the step's bookkeeping on the device
#include "element.cuh"

namespace llmopt {
namespace {

// ---- embedding ---------------------------------------------------------------------------------
template <typename T>
__global__ void __launch_bounds__(256) embedding_residual_kernel(const long long* ids, const T* __restrict__ table,
                                                                 float* x, T* x_copy, uint32_t rows, uint32_t vocabulary,
                                                                 uint32_t width) {
  grid_chain_prologue();
  const uint32_t row = blockIdx.x;
  const size_t token = min((unsigned long long)ids[row], (unsigned long long)(vocabulary - 1u));
  constexpr uint32_t kVector = 16 / sizeof(T);
  if (width % kVector == 0) {  // 16 bytes of the table at a time (buffers are 16-byte aligned: checked at launch)
    for (uint32_t c = threadIdx.x * kVector; c < width; c += blockDim.x * kVector) {
      const uint4 raw = *reinterpret_cast<const uint4*>(table + token * width + c);
      const T* values = reinterpret_cast<const T*>(&raw);
      float4* target = reinterpret_cast<float4*>(x + (size_t)row * width + c);
#pragma unroll
      for (uint32_t i = 0; i < kVector / 4; ++i)
        target[i] = make_float4(as_float(values[4 * i]), as_float(values[4 * i + 1]), as_float(values[4 * i + 2]),
                                as_float(values[4 * i + 3]));
      if (sizeof(T) != 4) *reinterpret_cast<uint4*>(x_copy + (size_t)row * width + c) = raw;
    }
    return;
  }
  for (uint32_t c = threadIdx.x; c < width; c += blockDim.x) {
    const T value = table[token * width + c];
    x[(size_t)row * width + c] = as_float(value);
    if (sizeof(T) != 4) x_copy[(size_t)row * width + c] = value;
  }
}

template <typename T>
int launch_embedding_residual(const KernelArgs& args) {
  LLMOPT_REQUIRE(args.buffer_count == 4 && args.param_bytes == 12,
                 "expects buffers [ids, table, x, x copy] and 12 parameter bytes {rows, vocabulary, width}");
  const uint32_t rows = param_u32(args, 0), vocabulary = param_u32(args, 1), width = param_u32(args, 2);
  LLMOPT_REQUIRE(vocabulary > 0 && width > 0, "needs a vocabulary and a width");
  LLMOPT_REQUIRE(args.lengths[0] >= (size_t)rows * 8 && args.lengths[1] >= (size_t)vocabulary * width * sizeof(T) &&
                     args.lengths[2] >= (size_t)rows * width * 4 && args.lengths[3] >= (size_t)rows * width * sizeof(T),
                 "buffer is too short");
  for (int i = 1; i < 4; ++i) LLMOPT_REQUIRE(((uintptr_t)args.buffers[i] & 15u) == 0, "buffers must be 16-byte aligned");
  if (rows == 0) return 0;
  launch_kernel(args, embedding_residual_kernel<T>, dim3(rows), dim3(256), 0, (const long long*)args.buffers[0],
                (const T*)args.buffers[1], (float*)args.buffers[2], (T*)args.buffers[3], rows, vocabulary, width);
  return check_launch(args);
}

// ---- embedding with absolute positions -----------------------------------------------------------
// Columns 2i, 2i + 1 take sine and cosine of a full turn times position * turns[i].  The turns are formed and reduced to
// less than one in double precision, so that late positions lose nothing.
__device__ __forceinline__ float2 sinusoid(double position, double turns) {
  const double angle = position * turns;
  float2 value;
  sincospif(2.0f * (float)(angle - rint(angle)), &value.x, &value.y);
  return value;
}

template <typename T>
__global__ void __launch_bounds__(256) embedding_sinusoid_kernel(const long long* ids, const T* __restrict__ table,
                                                                 const uint32_t* past, const double* __restrict__ turns,
                                                                 const float* __restrict__ norm, float* x, T* normed,
                                                                 uint32_t tokens, uint32_t vocabulary, uint32_t width,
                                                                 uint32_t vectors) {
  grid_chain_prologue();
  const uint32_t row = blockIdx.y;
  const size_t token = min((unsigned long long)ids[row], (unsigned long long)(vocabulary - 1u));
  const double position = (double)(past[row / tokens] + row % tokens);
  const TanhNorm next(norm, width);
  const uint32_t thread = blockIdx.x * 256u + threadIdx.x;
  if (vectors) {  // two pairs together
    const uint32_t column = thread * 4u;
    if (column >= width) return;
    struct alignas(4 * sizeof(T)) Four {
      T v[4];
    };
    const size_t at = (size_t)row * width + column;
    const Four e = *reinterpret_cast<const Four*>(table + token * width + column);
    const float2 low = sinusoid(position, turns[column / 2u]), high = sinusoid(position, turns[column / 2u + 1u]);
    const float4 sum = make_float4(as_float(e.v[0]) + low.x, as_float(e.v[1]) + low.y, as_float(e.v[2]) + high.x, as_float(e.v[3]) + high.y);
    *reinterpret_cast<float4*>(x + at) = sum;
    store_four(normed + at, next.four(sum, column));
    return;
  }
  const uint32_t column = thread * 2u;
  if (column >= width) return;
  const size_t at = (size_t)row * width + column;
  const float2 pair = sinusoid(position, turns[thread]);
  const float first = as_float(table[token * width + column]) + pair.x;
  x[at] = first;
  normed[at] = from_float<T>(next(first, column));
  if (column + 1u < width) {
    const float second = as_float(table[token * width + column + 1u]) + pair.y;
    x[at + 1] = second;
    normed[at + 1] = from_float<T>(next(second, column + 1u));
  }
}

// Buffers [ids, table, past, turns per position f64, following norm, x, normed]; params {rows, tokens per sequence, vocabulary, width}.
template <typename T>
int launch_embedding_sinusoid(const KernelArgs& args) {
  LLMOPT_REQUIRE(args.buffer_count == 7 && args.param_bytes == 16, "expects 7 buffers and 16 parameter bytes");
  const uint32_t rows = param_u32(args, 0), tokens = param_u32(args, 1), vocabulary = param_u32(args, 2), width = param_u32(args, 3);
  LLMOPT_REQUIRE(vocabulary > 0 && width > 0 && tokens > 0 && rows % tokens == 0 && rows <= 65535u,
                 "needs a vocabulary, a width and whole sequences of at most 65535 rows");
  const uint32_t pairs = (width + 1u) / 2u;
  LLMOPT_REQUIRE(args.lengths[0] >= (size_t)rows * 8 && args.lengths[1] >= (size_t)vocabulary * width * sizeof(T) &&
                     args.lengths[2] >= (size_t)(rows / tokens) * 4 && args.lengths[3] >= (size_t)pairs * 8 &&
                     args.lengths[4] >= (2 * (size_t)width + 1) * 4 && args.lengths[5] >= (size_t)rows * width * 4 &&
                     args.lengths[6] >= (size_t)rows * width * sizeof(T),
                 "buffer is too short");
  if (rows == 0) return 0;
  uint32_t vectors = width % 4u == 0;
  for (int i : {1, 4, 5, 6})
    if ((uintptr_t)args.buffers[i] & 15u) vectors = 0;
  const uint32_t threads = vectors ? width / 4u : pairs;
  launch_kernel(args, embedding_sinusoid_kernel<T>, dim3((threads + 255u) / 256u, rows), dim3(256), 0,
                (const long long*)args.buffers[0], (const T*)args.buffers[1], (const uint32_t*)args.buffers[2],
                (const double*)args.buffers[3], (const float*)args.buffers[4], (float*)args.buffers[5], (T*)args.buffers[6],
                tokens, vocabulary, width, vectors);
  return check_launch(args);
}

// ---- rows in a new order -------------------------------------------------------------------------
template <typename T>
__global__ void __launch_bounds__(256) gather_rows_kernel(const T* x, const uint32_t* rows, T* out, uint32_t source_rows,
                                                          uint32_t width, uint32_t vectors) {
  grid_chain_prologue();
  const T* source = x + (size_t)min(rows[blockIdx.x], source_rows - 1u) * width;
  T* target = out + (size_t)blockIdx.x * width;
  if (vectors) {
    for (uint32_t c = threadIdx.x; c < vectors; c += blockDim.x)
      reinterpret_cast<uint4*>(target)[c] = reinterpret_cast<const uint4*>(source)[c];
  } else {
    for (uint32_t c = threadIdx.x; c < width; c += blockDim.x) target[c] = source[c];
  }
}

// Buffers [x, rows u32, out]; params {count, source rows, width}.
template <typename T>
int launch_gather_rows(const KernelArgs& args) {
  LLMOPT_REQUIRE(args.buffer_count == 3 && args.param_bytes == 12, "expects 3 buffers and 12 parameter bytes");
  const uint32_t count = param_u32(args, 0), source_rows = param_u32(args, 1), width = param_u32(args, 2);
  LLMOPT_REQUIRE(source_rows > 0 && width > 0, "needs source rows and a width");
  LLMOPT_REQUIRE(args.lengths[0] >= (size_t)source_rows * width * sizeof(T) && args.lengths[1] >= (size_t)count * 4 &&
                     args.lengths[2] >= (size_t)count * width * sizeof(T),
                 "buffer is too short");
  if (count == 0) return 0;
  const bool aligned = width * sizeof(T) % 16u == 0 && ((uintptr_t)args.buffers[0] & 15u) == 0 && ((uintptr_t)args.buffers[2] & 15u) == 0;
  launch_kernel(args, gather_rows_kernel<T>, dim3(count), dim3(256), 0, (const T*)args.buffers[0], (const uint32_t*)args.buffers[1],
                (T*)args.buffers[2], source_rows, width, aligned ? (uint32_t)(width * sizeof(T) / 16u) : 0u);
  return check_launch(args);
}

// ---- residual + norm ---------------------------------------------------------------------------
struct ResidualNormParams {
  uint32_t rows, width;
  float epsilon, weight_offset;  // the norm multiplies by weight_offset + weight
  uint32_t pair;                 // 1: y is the mean of two branches, each RMS-normed with its own weight
};

// One CTA per row; a thread keeps up to V float4 of the row in registers between the passes.
template <typename T, int V>
__global__ void __launch_bounds__(256) residual_norm_kernel(const float* x_in, const float* y, const float* __restrict__ w,
                                                            const float* y2, const float* __restrict__ w_left,
                                                            const float* __restrict__ w_right, float* x_out, T* x_copy,
                                                            ResidualNormParams p) {
  grid_chain_prologue();
  __shared__ float scratch[8];
  const size_t base = (size_t)blockIdx.x * p.width;
  const uint32_t vectors = p.width / 4u;
  float4 value[V];
  auto square = [](const float4& v) { return v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w; };
  float sum = 0.0f;
#pragma unroll
  for (int i = 0; i < V; ++i) {
    const uint32_t at = threadIdx.x + i * 256u;
    value[i] = at < vectors ? reinterpret_cast<const float4*>(y + base)[at] : make_float4(0.f, 0.f, 0.f, 0.f);
    sum += square(value[i]);
  }
  if (p.pair) {
    float4 other[V];
    float other_sum = 0.0f;
#pragma unroll
    for (int i = 0; i < V; ++i) {
      const uint32_t at = threadIdx.x + i * 256u;
      other[i] = at < vectors ? reinterpret_cast<const float4*>(y2 + base)[at] : make_float4(0.f, 0.f, 0.f, 0.f);
      other_sum += square(other[i]);
    }
    const float left = 0.5f / sqrtf(block_sum(sum, scratch) / (float)p.width + p.epsilon);
    const float right = 0.5f / sqrtf(block_sum(other_sum, scratch) / (float)p.width + p.epsilon);
    sum = 0.0f;
#pragma unroll
    for (int i = 0; i < V; ++i) {
      const uint32_t at = threadIdx.x + i * 256u;
      if (at < vectors) {
        const float4 wl = reinterpret_cast<const float4*>(w_left)[at], wr = reinterpret_cast<const float4*>(w_right)[at];
        value[i].x = value[i].x * left * wl.x + other[i].x * right * wr.x;
        value[i].y = value[i].y * left * wl.y + other[i].y * right * wr.y;
        value[i].z = value[i].z * left * wl.z + other[i].z * right * wr.z;
        value[i].w = value[i].w * left * wl.w + other[i].w * right * wr.w;
      }
      sum += square(value[i]);
    }
  }
  const float scale = 1.0f / sqrtf(block_sum(sum, scratch) / (float)p.width + p.epsilon);
#pragma unroll
  for (int i = 0; i < V; ++i) {
    const uint32_t at = threadIdx.x + i * 256u;
    if (at >= vectors) continue;
    const float4 weight = reinterpret_cast<const float4*>(w)[at];
    float4 x = reinterpret_cast<const float4*>(x_in + base)[at];
    x.x += value[i].x * scale * (p.weight_offset + weight.x);
    x.y += value[i].y * scale * (p.weight_offset + weight.y);
    x.z += value[i].z * scale * (p.weight_offset + weight.z);
    x.w += value[i].w * scale * (p.weight_offset + weight.w);
    reinterpret_cast<float4*>(x_out + base)[at] = x;
    if (sizeof(T) != 4) {
      const __nv_bfloat162 low = __floats2bfloat162_rn(x.x, x.y), high = __floats2bfloat162_rn(x.z, x.w);
      uint2 packed = make_uint2(*reinterpret_cast<const uint32_t*>(&low), *reinterpret_cast<const uint32_t*>(&high));
      reinterpret_cast<uint2*>(x_copy + base)[at] = packed;
    }
  }
}

// Any width: the row is read again in every pass.
template <typename T>
__global__ void __launch_bounds__(256) residual_norm_any_kernel(const float* x_in, const float* y,
                                                                const float* __restrict__ w, const float* y2,
                                                                const float* __restrict__ w_left,
                                                                const float* __restrict__ w_right, float* x_out, T* x_copy,
                                                                ResidualNormParams p) {
  grid_chain_prologue();
  __shared__ float scratch[8];
  const size_t base = (size_t)blockIdx.x * p.width;
  float left = 0.0f, right = 0.0f;
  auto at = [&](uint32_t c) {
    return p.pair ? y[base + c] * left * w_left[c] + y2[base + c] * right * w_right[c] : y[base + c];
  };
  if (p.pair) {
    float a = 0.0f, b = 0.0f;
    for (uint32_t c = threadIdx.x; c < p.width; c += 256u) {
      a += y[base + c] * y[base + c];
      b += y2[base + c] * y2[base + c];
    }
    left = 0.5f / sqrtf(block_sum(a, scratch) / (float)p.width + p.epsilon);
    right = 0.5f / sqrtf(block_sum(b, scratch) / (float)p.width + p.epsilon);
  }
  float sum = 0.0f;
  for (uint32_t c = threadIdx.x; c < p.width; c += 256u) {
    const float v = at(c);
    sum += v * v;
  }
  const float scale = 1.0f / sqrtf(block_sum(sum, scratch) / (float)p.width + p.epsilon);
  for (uint32_t c = threadIdx.x; c < p.width; c += 256u) {
    const float x = x_in[base + c] + at(c) * scale * (p.weight_offset + w[c]);
    x_out[base + c] = x;
    if (sizeof(T) != 4) x_copy[base + c] = from_float<T>(x);
  }
}

// Buffers [x in, y, weight, y of the second branch, left weight, right weight, x out, x copy].
template <typename T>
int launch_residual_norm(const KernelArgs& args) {
  ResidualNormParams p;
  LLMOPT_REQUIRE(args.buffer_count == 8 && args.param_bytes == sizeof(p), "expects 8 buffers and 20 parameter bytes");
  memcpy(&p, args.params, sizeof(p));
  const size_t row_bytes = (size_t)p.rows * p.width * 4;
  LLMOPT_REQUIRE(p.width > 0, "needs a width");
  LLMOPT_REQUIRE(args.lengths[0] >= row_bytes && args.lengths[1] >= row_bytes && args.lengths[6] >= row_bytes &&
                     args.lengths[7] >= row_bytes / 4 * sizeof(T) && args.lengths[2] >= (size_t)p.width * 4,
                 "buffer is too short");
  LLMOPT_REQUIRE(!p.pair || (args.lengths[3] >= row_bytes && args.lengths[4] >= (size_t)p.width * 4 &&
                             args.lengths[5] >= (size_t)p.width * 4),
                 "branch buffer is too short");
  if (p.rows == 0) return 0;
  auto run = [&](auto kernel) {
    launch_kernel(args, kernel, dim3(p.rows), dim3(256), 0, (const float*)args.buffers[0], (const float*)args.buffers[1],
                  (const float*)args.buffers[2], (const float*)args.buffers[3], (const float*)args.buffers[4],
                  (const float*)args.buffers[5], (float*)args.buffers[6], (T*)args.buffers[7], p);
  };
  bool vectors = p.width % 4u == 0 && p.width <= 8192u;
  for (int i = 0; i < 8; ++i)
    if ((uintptr_t)args.buffers[i] & 15u) vectors = false;
  if (!vectors) run(residual_norm_any_kernel<T>);
  else if (p.width <= 1024u) run(residual_norm_kernel<T, 1>);
  else if (p.width <= 2048u) run(residual_norm_kernel<T, 2>);
  else if (p.width <= 4096u) run(residual_norm_kernel<T, 4>);
  else run(residual_norm_kernel<T, 8>);
  return check_launch(args);
}

// ---- norm of chosen rows -----------------------------------------------------------------------
template <typename T>
__global__ void __launch_bounds__(256) gather_norm_kernel(const float* x, const uint32_t* rows, const float* __restrict__ w,
                                                          T* out, uint32_t source_rows, uint32_t width, float epsilon,
                                                          float weight_offset) {
  grid_chain_prologue();
  __shared__ float scratch[8];
  const float* source = x + (size_t)min(rows[blockIdx.x], source_rows - 1u) * width;
  T* target = out + (size_t)blockIdx.x * width;
  constexpr int kVectors = 4;  // float4 of a row a thread keeps between the passes
  if (width % 4u == 0 && width <= 1024u * kVectors) {
    float4 value[kVectors];
    float sum = 0.0f;
#pragma unroll
    for (int i = 0; i < kVectors; ++i) {
      const uint32_t c = (threadIdx.x + i * 256u) * 4u;
      value[i] = *reinterpret_cast<const float4*>(source + min(c, width - 4u));
      if (c < width)
        sum += value[i].x * value[i].x + value[i].y * value[i].y + value[i].z * value[i].z + value[i].w * value[i].w;
    }
    const float scale = 1.0f / sqrtf(block_sum(sum, scratch) / (float)width + epsilon);
#pragma unroll
    for (int i = 0; i < kVectors; ++i) {
      const uint32_t c = (threadIdx.x + i * 256u) * 4u;
      if (c >= width) continue;
      const float4 weight = *reinterpret_cast<const float4*>(w + c);
      target[c] = from_float<T>(value[i].x * scale * (weight_offset + weight.x));
      target[c + 1] = from_float<T>(value[i].y * scale * (weight_offset + weight.y));
      target[c + 2] = from_float<T>(value[i].z * scale * (weight_offset + weight.z));
      target[c + 3] = from_float<T>(value[i].w * scale * (weight_offset + weight.w));
    }
    return;
  }
  float sum = 0.0f;
  for (uint32_t c = threadIdx.x; c < width; c += 256u) sum += source[c] * source[c];
  const float scale = 1.0f / sqrtf(block_sum(sum, scratch) / (float)width + epsilon);
  for (uint32_t c = threadIdx.x; c < width; c += 256u) target[c] = from_float<T>(source[c] * scale * (weight_offset + w[c]));
}

// Buffers [x, rows u32, weight, out]; params {count, source rows, width, epsilon, weight offset}.
template <typename T>
int launch_gather_norm(const KernelArgs& args) {
  LLMOPT_REQUIRE(args.buffer_count == 4 && args.param_bytes == 20, "expects 4 buffers and 20 parameter bytes");
  const uint32_t count = param_u32(args, 0), source_rows = param_u32(args, 1), width = param_u32(args, 2);
  LLMOPT_REQUIRE(source_rows > 0 && width > 0, "needs source rows and a width");
  LLMOPT_REQUIRE(args.lengths[0] >= (size_t)source_rows * width * 4 && args.lengths[1] >= (size_t)count * 4 &&
                     args.lengths[2] >= (size_t)width * 4 && args.lengths[3] >= (size_t)count * width * sizeof(T),
                 "buffer is too short");
  for (int i : {0, 2, 3}) LLMOPT_REQUIRE(((uintptr_t)args.buffers[i] & 15u) == 0, "buffers must be 16-byte aligned");
  if (count == 0) return 0;
  launch_kernel(args, gather_norm_kernel<T>, dim3(count), dim3(256), 0, (const float*)args.buffers[0],
                (const uint32_t*)args.buffers[1], (const float*)args.buffers[2], (T*)args.buffers[3], source_rows, width,
                param_f32(args, 3), param_f32(args, 4));
  return check_launch(args);
}

// ---- attention inputs --------------------------------------------------------------------------
struct AttentionPrepareParams {
  uint32_t sequences, tokens, heads, kv_heads, dim, vdim;
  uint32_t stride;                        // elements per row of the projections
  uint32_t q_column, k_column, v_column;  // first column of each
  uint32_t rotary_dims, trig_rows;
  uint32_t token_stride, key_offset, value_offset;  // cache row, in elements
  uint32_t table_stride, table_rows, pool_rows;
  uint32_t head_norm;
  float epsilon;
  uint32_t own_keys;  // 0: only the queries (the layer reads another layer's keys and values)
  uint32_t pairs;  // set by the launcher: every head starts at an even element
};

// One CTA per row (or, with few rows, several that share its heads), its warps take the heads in turn: query heads are
// normed, rotated and stored; key heads too, into the cache row of the token; value heads are copied there.
// Dimensions 2i, 2i + 1 turn together; `trig` holds [positions][dims / 2] pairs (cos, sin).
template <typename T>
__global__ void __launch_bounds__(256) attention_prepare_kernel(const T* projected, const float* __restrict__ q_weight,
                                                                const float* __restrict__ k_weight,
                                                                const float2* __restrict__ trig, T* q_out, T* pool,
                                                                const uint32_t* slots, const uint32_t* past,
                                                                const uint32_t* sequence_rows, AttentionPrepareParams p,
                                                                uint32_t* error_word) {
  grid_chain_prologue();
  const uint32_t lane = threadIdx.x & 31u, row = blockIdx.x, sequence = row / p.tokens;
  const uint32_t position = past[sequence] + row % p.tokens, table_row = sequence_rows[sequence];
  uint32_t slot = p.pool_rows;
  if (table_row < p.table_rows && position < p.table_stride) slot = slots[(size_t)table_row * p.table_stride + position];
  if (slot >= p.pool_rows && error_word && threadIdx.x == 0) atomicExch(error_word, 1u);
  T* const cached = pool + (size_t)(slot < p.pool_rows ? slot : 0u) * p.token_stride;
  const uint32_t trig_row = min(position, p.trig_rows - 1u);
  const float2* turns = trig + (size_t)trig_row * (p.rotary_dims / 2u);
  const uint32_t per_row = p.heads + (p.own_keys ? 2u * p.kv_heads : 0u);
  for (uint32_t head = blockIdx.y * 8u + (threadIdx.x >> 5); head < per_row; head += 8u * gridDim.y) {
    const T* source = projected + (size_t)row * p.stride;
    if (head < p.heads) source += p.q_column + head * p.dim;
    else if (head < p.heads + p.kv_heads) source += p.k_column + (head - p.heads) * p.dim;
    else source += p.v_column + (head - p.heads - p.kv_heads) * p.vdim;

    T* target;
    if (head < p.heads) {
      target = q_out + ((size_t)row * p.heads + head) * p.dim;
    } else {
      if (slot >= p.pool_rows) continue;  // never write outside the pool
      target = cached;
      if (head >= p.heads + p.kv_heads) {
        target += p.value_offset + (head - p.heads - p.kv_heads) * p.vdim;
        for (uint32_t c = lane; c < p.vdim; c += 32u) target[c] = source[c];
        continue;
      }
      target += p.key_offset + (head - p.heads) * p.dim;
    }
    const float* weight = head < p.heads ? q_weight : k_weight;
    if (p.pairs) {  // neighbours travel together, the head in registers between the passes
      constexpr int kPairs = 4;  // dim <= 256
      struct alignas(2 * sizeof(T)) Two {
        T u, v;
      };
      Two raw[kPairs];
      float sum = 0.0f;
#pragma unroll
      for (int i = 0; i < kPairs; ++i)
        if (i * 64u < p.dim) raw[i] = *reinterpret_cast<const Two*>(source + min((lane + i * 32u) * 2u, p.dim - 2u));
#pragma unroll
      for (int i = 0; i < kPairs; ++i)
        if ((lane + i * 32u) * 2u < p.dim) sum += as_float(raw[i].u) * as_float(raw[i].u) + as_float(raw[i].v) * as_float(raw[i].v);
      const float scale = p.head_norm ? 1.0f / sqrtf(warp_sum(sum) / (float)p.dim + p.epsilon) : 1.0f;
#pragma unroll
      for (int i = 0; i < kPairs; ++i) {
        const uint32_t pair = lane + i * 32u, c = pair * 2u;
        if (c >= p.dim) continue;
        float u = as_float(raw[i].u) * scale, v = as_float(raw[i].v) * scale;
        if (p.head_norm) {
          const float2 w = *reinterpret_cast<const float2*>(weight + c);
          u *= w.x;
          v *= w.y;
        }
        if (c < p.rotary_dims) {
          const float2 turn = turns[pair];
          const float rotated = u * turn.x - v * turn.y;
          v = v * turn.x + u * turn.y;
          u = rotated;
        }
        Two result;
        result.u = from_float<T>(u);
        result.v = from_float<T>(v);
        *reinterpret_cast<Two*>(target + c) = result;
      }
      continue;
    }
    float scale = 1.0f;
    if (p.head_norm) {
      float sum = 0.0f;
      for (uint32_t c = lane; c < p.dim; c += 32u) {
        const float v = as_float(source[c]);
        sum += v * v;
      }
      scale = 1.0f / sqrtf(warp_sum(sum) / (float)p.dim + p.epsilon);
    }
    for (uint32_t pair = lane; pair * 2u < p.dim; pair += 32u) {
      const uint32_t c = pair * 2u;
      float u = as_float(source[c]) * scale, v = c + 1u < p.dim ? as_float(source[c + 1u]) * scale : 0.0f;
      if (p.head_norm) {
        u *= weight[c];
        if (c + 1u < p.dim) v *= weight[c + 1u];
      }
      if (c + 1u < p.rotary_dims) {
        const float2 turn = turns[pair];
        const float rotated = u * turn.x - v * turn.y;
        v = v * turn.x + u * turn.y;
        u = rotated;
      }
      target[c] = from_float<T>(u);
      if (c + 1u < p.dim) target[c + 1u] = from_float<T>(v);
    }
  }
}

}  // namespace
uint32_t* context_device_error(Context* ctx);
namespace {

// Buffers [projected, q weight, k weight, trig, q out, pool, slot table, past, sequence rows].
template <typename T>
int launch_attention_prepare(const KernelArgs& args) {
  AttentionPrepareParams p;
  LLMOPT_REQUIRE(args.buffer_count == 9 && args.param_bytes == 84, "expects 9 buffers and 84 parameter bytes");
  memcpy(&p, args.params, 84);
  p.pairs = p.dim % 2u == 0 && p.dim <= 256u && p.stride % 2u == 0 && p.q_column % 2u == 0 && p.k_column % 2u == 0 &&
            p.token_stride % 2u == 0 && p.key_offset % 2u == 0;
  for (int i : {0, 1, 2, 4, 5})
    if ((uintptr_t)args.buffers[i] & 7u) p.pairs = 0;
  const size_t rows = (size_t)p.sequences * p.tokens, e = sizeof(T);
  LLMOPT_REQUIRE(p.heads > 0 && p.kv_heads > 0 && p.heads % p.kv_heads == 0 && p.dim > 0 && p.vdim > 0,
                 "needs whole groups of query heads");
  LLMOPT_REQUIRE(p.rotary_dims <= p.dim && p.rotary_dims % 2u == 0, "rotated dimensions come in pairs inside the head");
  LLMOPT_REQUIRE(p.q_column + p.heads * p.dim <= p.stride &&
                     (!p.own_keys || (p.k_column + p.kv_heads * p.dim <= p.stride && p.v_column + p.kv_heads * p.vdim <= p.stride)),
                 "projection columns lie outside the row");
  LLMOPT_REQUIRE(p.key_offset + p.kv_heads * p.dim <= p.token_stride && p.value_offset + p.kv_heads * p.vdim <= p.token_stride,
                 "key or value segment lies outside the cache row");
  LLMOPT_REQUIRE(args.lengths[0] >= rows * p.stride * e && args.lengths[4] >= rows * p.heads * p.dim * e, "buffer is too short");
  LLMOPT_REQUIRE(!p.head_norm || (args.lengths[1] >= (size_t)p.dim * 4 && args.lengths[2] >= (size_t)p.dim * 4),
                 "head norm weight is too short");
  LLMOPT_REQUIRE(p.rotary_dims == 0 || (p.trig_rows > 0 && args.lengths[3] >= (size_t)p.trig_rows * p.rotary_dims * 4),
                 "trig table is too short");
  LLMOPT_REQUIRE(args.lengths[5] >= (size_t)p.pool_rows * p.token_stride * e &&
                     args.lengths[6] >= (size_t)p.table_rows * p.table_stride * 4 &&
                     args.lengths[7] >= (size_t)p.sequences * 4 && args.lengths[8] >= (size_t)p.sequences * 4,
                 "cache buffer is too short");
  if (rows == 0) return 0;
  // few rows: a row's heads are spread over several CTAs
  const uint32_t spread = rows < 256 ? (p.heads + 2u * p.kv_heads + 7u) / 8u : 1u;
  launch_kernel(args, attention_prepare_kernel<T>, dim3((uint32_t)rows, spread), dim3(256), 0,
                (const T*)args.buffers[0], (const float*)args.buffers[1], (const float*)args.buffers[2],
                (const float2*)args.buffers[3], (T*)args.buffers[4], (T*)args.buffers[5], (const uint32_t*)args.buffers[6],
                (const uint32_t*)args.buffers[7], (const uint32_t*)args.buffers[8], p, context_device_error(args.ctx));
  return check_launch(args);
}

// ---- per-head norm and gate of a mixer's read-out ---------------------------------------------
struct HeadNormGateParams {
  uint32_t rows, heads, dim;
  uint32_t gate_stride, gate_column;
  uint32_t weight_per_head;  // 1: weight [heads * dim]; 0: weight [dim] shared by the heads
  uint32_t gate_sigmoid;     // 1: sigmoid, 0: silu
  float epsilon;
  uint32_t vectors;  // set by the launcher: all rows start at whole vectors of four
};

template <typename T>
__global__ void __launch_bounds__(128) head_norm_gate_kernel(const float* o, const T* gate, const float* __restrict__ weight,
                                                             T* out, HeadNormGateParams p) {
  grid_chain_prologue();
  const uint32_t lane = threadIdx.x & 31u, item = blockIdx.x * 4u + (threadIdx.x >> 5);
  if (item >= p.rows * p.heads) return;
  const uint32_t row = item / p.heads, head = item % p.heads;
  const float* source = o + (size_t)item * p.dim;
  const T* gate_row = gate + (size_t)row * p.gate_stride + p.gate_column + head * p.dim;
  const float* weight_row = weight + (p.weight_per_head ? head * p.dim : 0u);
  if (p.vectors) {  // four columns at a time, the row in registers between the passes
    constexpr int kVectors = 4;
    float4 value[kVectors];
    float sum = 0.0f;
#pragma unroll
    for (int i = 0; i < kVectors; ++i) {
      const uint32_t c = (lane + i * 32u) * 4u;
      value[i] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (i * 128u < p.dim) value[i] = *reinterpret_cast<const float4*>(source + min(c, p.dim - 4u));
      if (c < p.dim) sum += value[i].x * value[i].x + value[i].y * value[i].y + value[i].z * value[i].z + value[i].w * value[i].w;
    }
    const float scale = 1.0f / sqrtf(warp_sum(sum) / (float)p.dim + p.epsilon);
#pragma unroll
    for (int i = 0; i < kVectors; ++i) {
      const uint32_t c = (lane + i * 32u) * 4u;
      if (c >= p.dim) continue;
      struct alignas(4 * sizeof(T)) Four {
        T v[4];
      };
      const Four z = *reinterpret_cast<const Four*>(gate_row + c);
      const float4 w = *reinterpret_cast<const float4*>(weight_row + c);
      const float values[4] = {value[i].x * w.x, value[i].y * w.y, value[i].z * w.z, value[i].w * w.w};
      Four result;
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const float g = as_float(z.v[e]);
        result.v[e] = from_float<T>(values[e] * scale * (p.gate_sigmoid ? sigmoid_f32(g) : silu_f32(g)));
      }
      *reinterpret_cast<Four*>(out + (size_t)item * p.dim + c) = result;
    }
    return;
  }
  float sum = 0.0f;
  for (uint32_t c = lane; c < p.dim; c += 32u) sum += source[c] * source[c];
  const float scale = 1.0f / sqrtf(warp_sum(sum) / (float)p.dim + p.epsilon);
  for (uint32_t c = lane; c < p.dim; c += 32u) {
    const float z = as_float(gate_row[c]);
    out[(size_t)item * p.dim + c] = from_float<T>(source[c] * scale * weight_row[c] * (p.gate_sigmoid ? sigmoid_f32(z) : silu_f32(z)));
  }
}

// Buffers [o f32, gate, weight, out].
template <typename T>
int launch_head_norm_gate(const KernelArgs& args) {
  HeadNormGateParams p;
  LLMOPT_REQUIRE(args.buffer_count == 4 && args.param_bytes == 32, "expects 4 buffers and 32 parameter bytes");
  memcpy(&p, args.params, 32);
  p.vectors = p.dim % 4u == 0 && p.dim <= 512u && p.gate_stride % 4u == 0 && p.gate_column % 4u == 0;
  for (int i = 0; i < 4; ++i)
    if ((uintptr_t)args.buffers[i] & 15u) p.vectors = 0;
  const size_t items = (size_t)p.rows * p.heads;
  LLMOPT_REQUIRE(p.gate_column + p.heads * p.dim <= p.gate_stride, "gate columns lie outside the row");
  LLMOPT_REQUIRE(args.lengths[0] >= items * p.dim * 4 && args.lengths[1] >= (size_t)p.rows * p.gate_stride * sizeof(T) &&
                     args.lengths[2] >= (size_t)p.dim * (p.weight_per_head ? p.heads : 1u) * 4 &&
                     args.lengths[3] >= items * p.dim * sizeof(T),
                 "buffer is too short");
  if (items == 0) return 0;
  launch_kernel(args, head_norm_gate_kernel<T>, dim3((uint32_t)((items + 3) / 4)), dim3(128), 0,
                (const float*)args.buffers[0], (const T*)args.buffers[1], (const float*)args.buffers[2],
                (T*)args.buffers[3], p);
  return check_launch(args);
}

// ---- greedy pick and bookkeeping ----------------------------------------------------------------
__global__ void __launch_bounds__(256) argmax_kernel(const float* logits, unsigned long long* best, uint32_t columns,
                                                     uint32_t parts) {
  grid_chain_prologue();
  __shared__ unsigned long long warp_best[8];
  const float* row = logits + (size_t)blockIdx.y * columns;
  unsigned long long top = 0;
  for (uint32_t c = blockIdx.x * 256u + threadIdx.x; c < columns; c += parts * 256u) top = max(top, ranked(row[c], c));
  for (int offset = 16; offset > 0; offset >>= 1) top = max(top, __shfl_xor_sync(0xffffffffu, top, offset));
  if ((threadIdx.x & 31u) == 0u) warp_best[threadIdx.x >> 5] = top;
  __syncthreads();
  if (threadIdx.x == 0) {
    for (int w = 1; w < 8; ++w) top = max(top, warp_best[w]);
    best[(size_t)blockIdx.y * parts + blockIdx.x] = top;
  }
}

// Buffers [logits f32, candidates u64 [rows, parts]]; params {rows, columns, parts}.
int launch_argmax_f32(const KernelArgs& args) {
  LLMOPT_REQUIRE(args.buffer_count == 2 && args.param_bytes == 12, "expects 2 buffers and 12 parameter bytes");
  const uint32_t rows = param_u32(args, 0), columns = param_u32(args, 1), parts = param_u32(args, 2);
  LLMOPT_REQUIRE(columns > 0 && parts > 0 && rows <= 65535u, "needs columns, parts and at most 65535 rows");
  LLMOPT_REQUIRE(args.lengths[0] >= (size_t)rows * columns * 4 && args.lengths[1] >= (size_t)rows * parts * 8,
                 "buffer is too short");
  if (rows == 0) return 0;
  launch_kernel(args, argmax_kernel, dim3(parts, rows), dim3(256), 0, (const float*)args.buffers[0],
                (unsigned long long*)args.buffers[1], columns, parts);
  return check_launch(args);
}

__global__ void __launch_bounds__(32) advance_kernel(const unsigned long long* best, int* picked, long long* ids,
                                                     uint32_t* past, uint32_t parts, uint32_t step) {
  grid_chain_prologue();
  unsigned long long top = 0;
  for (uint32_t i = threadIdx.x; i < parts; i += 32u) top = max(top, best[(size_t)blockIdx.x * parts + i]);
  for (int offset = 16; offset > 0; offset >>= 1) top = max(top, __shfl_xor_sync(0xffffffffu, top, offset));
  if (threadIdx.x != 0) return;
  const uint32_t token = 0xffffffffu - (uint32_t)top;
  picked[blockIdx.x] = (int)token;
  ids[blockIdx.x] = (long long)token;
  past[blockIdx.x] += step;
}

// Ends a step of one row per sequence: the picked token becomes the next input and the sequence has `step`
// more tokens behind it.  Buffers [candidates, picked i32, ids i64, past u32]; params {rows, parts, step}.
int launch_advance_tokens(const KernelArgs& args) {
  LLMOPT_REQUIRE(args.buffer_count == 4 && args.param_bytes == 12, "expects 4 buffers and 12 parameter bytes");
  const uint32_t rows = param_u32(args, 0), parts = param_u32(args, 1), step = param_u32(args, 2);
  LLMOPT_REQUIRE(args.lengths[0] >= (size_t)rows * parts * 8 && args.lengths[1] >= (size_t)rows * 4 &&
                     args.lengths[2] >= (size_t)rows * 8 && args.lengths[3] >= (size_t)rows * 4,
                 "buffer is too short");
  if (rows == 0) return 0;
  launch_kernel(args, advance_kernel, dim3(rows), dim3(32), 0, (const unsigned long long*)args.buffers[0],
                (int*)args.buffers[1], (long long*)args.buffers[2], (uint32_t*)args.buffers[3], parts, step);
  return check_launch(args);
}

}  // namespace

const NamedLauncher* sequence_glue_launchers(size_t* count) {
  static const NamedLauncher table[] = {
      {"llmopt_embedding_residual_bf16", launch_embedding_residual<bf16>},
      {"llmopt_embedding_residual_f32", launch_embedding_residual<float>},
      {"llmopt_embedding_sinusoid_bf16", launch_embedding_sinusoid<bf16>},
      {"llmopt_embedding_sinusoid_f32", launch_embedding_sinusoid<float>},
      {"llmopt_gather_rows_bf16", launch_gather_rows<bf16>},
      {"llmopt_gather_rows_f32", launch_gather_rows<float>},
      {"llmopt_residual_norm_bf16", launch_residual_norm<bf16>},
      {"llmopt_residual_norm_f32", launch_residual_norm<float>},
      {"llmopt_gather_norm_bf16", launch_gather_norm<bf16>},
      {"llmopt_gather_norm_f32", launch_gather_norm<float>},
      {"llmopt_row_attention_prepare_bf16", launch_attention_prepare<bf16>},
      {"llmopt_row_attention_prepare_f32", launch_attention_prepare<float>},
      {"llmopt_head_norm_gate_bf16", launch_head_norm_gate<bf16>},
      {"llmopt_head_norm_gate_f32", launch_head_norm_gate<float>},
      {"llmopt_argmax_f32", launch_argmax_f32},
      {"llmopt_advance_tokens", launch_advance_tokens},
  };
  *count = sizeof(table) / sizeof(table[0]);
  return table;
}

}  // namespace llmopt
