// Recurrent mixers with a matrix state per head, carried in fp32 from token to token:
//   llmopt_delta_prepare_{bf16,f32}    short convolutions, unit q and k, decay and step size of a gated delta rule
//   llmopt_conv_state_{bf16,f32}       the convolutions' last inputs
//   llmopt_delta_step_{bf16,f32}, llmopt_memory_step_{bf16,f32}   one token per sequence, everything between the input
//                                      projections and the output projection in one launch
//   llmopt_delta_scan_f32              S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q
//   llmopt_memory_scan_{bf16,f32}      stabilised exponential gating (mLSTM): S <- a S + b k v^T, n <- a n + b k,
//                                      o = S^T q / (max(|n . q|, exp(-m)) + 1e-6)
//
// State of a sequence lives in row `sequence_rows[i]` of a state pool.  A row holds, per head, the
// transposed matrix [vdim][dim]; the matrix-memory form adds n [dim] and m once per slice of kSlice value
// columns, because every slice's CTA needs them and keeps a copy of its own.  A sequence with nothing
// behind it (past = 0) starts from zero whatever its pool row holds.
//
// Scan: a CTA owns kSlice value columns of one head of one sequence and walks over the tokens.  Sixteen lanes
// share two columns of S (each lane dim / 16 rows of them, in registers).  Compute warps work on a chunk of tokens in
// shared memory while producer warps bring in the next chunk (converted to fp32, with the per-token
// scalars) and write out the previous one's results.  The read-out of the delta rule uses
// S_new^T q = g S_old^T q + u (k . q), so that its sum and the one of S_old^T k are reduced at the same time.
#include <type_traits>

#include "element.cuh"

namespace llmopt {
namespace {

constexpr uint32_t kSlice = 32;   // value columns per CTA
constexpr uint32_t kLanes = 16;   // lanes per column
constexpr uint32_t kColumns = 2;  // columns per thread
constexpr uint32_t kColumnWarps = kSlice / kColumns * kLanes / 32;  // 4
constexpr uint32_t kProducerWarps = 4;

__host__ __device__ constexpr uint32_t slices_of(uint32_t vdim) { return (vdim + kSlice - 1u) / kSlice; }

// ---- gated delta rule: inputs ----------------------------------------------------------------------
struct DeltaPrepareParams {
  uint32_t sequences, tokens, heads, kv_heads, dim, vdim, taps;
  uint32_t stride, q_column, k_column, v_column;  // projections, T [rows, stride]
  uint32_t scalar_stride, beta_column, decay_column;  // projections, fp32 [rows, scalar_stride]
  uint32_t state_rows;
};

// Input of channel `channel` (counted over q, k, v; column `column` of the projections) at `token` of the step,
// which may lie before it.  Earlier inputs are kept in a ring [taps][channels]: position p in row p % taps, so that
// a step of one token overwrites what no kernel of that step reads.
template <typename T>
struct ConvInputs {
  const T* projected;  // first row of the sequence
  const T* ring;
  uint32_t stride, taps, channels, past;
  __device__ __forceinline__ float at(uint32_t column, uint32_t channel, int token) const {
    if (token >= 0) return as_float(projected[(size_t)token * stride + column]);
    const int position = (int)past + token;
    return position >= 0 ? as_float(ring[(size_t)((uint32_t)position % taps) * channels + channel]) : 0.0f;
  }
  // The convolution's value before its activation.
  __device__ __forceinline__ float convolve(const float* __restrict__ weight, uint32_t column, uint32_t channel, int token) const {
    const float* w = weight + (size_t)channel * taps;
    float sum = 0.0f;
    if (taps == 4u) {  // the usual length: all loads in flight at once
      float x[4];
#pragma unroll
      for (int tap = 0; tap < 4; ++tap) x[tap] = at(column, channel, token - 3 + tap);
#pragma unroll
      for (int tap = 0; tap < 4; ++tap) sum = fmaf(__ldg(w + tap), x[tap], sum);
      return sum;
    }
    for (uint32_t tap = 0; tap < taps; ++tap)
      sum = fmaf(__ldg(w + tap), at(column, channel, token - (int)(taps - 1u - tap)), sum);
    return sum;
  }
};

template <typename T>
__global__ void __launch_bounds__(128) delta_prepare_kernel(const T* projected, const float* scalars,
                                                            const float* __restrict__ conv_weight, const T* conv_state,
                                                            const uint32_t* past, const uint32_t* sequence_rows,
                                                            const float* __restrict__ a_log,
                                                            const float* __restrict__ dt_bias, float* q_out, float* k_out,
                                                            float* v_out, float* decay, float* beta, DeltaPrepareParams p) {
  grid_chain_prologue();
  const uint32_t lane = threadIdx.x & 31u, item = blockIdx.x * 4u + (threadIdx.x >> 5);
  const uint32_t per_row = 2u * p.kv_heads + p.heads + 1u;
  if (item >= p.sequences * p.tokens * per_row) return;
  const uint32_t row = item / per_row, part = item % per_row, sequence = row / p.tokens, token = row % p.tokens;
  if (part == per_row - 1u) {  // the row's scalars
    for (uint32_t h = lane; h < p.heads; h += 32u) {
      const float* source = scalars + (size_t)row * p.scalar_stride;
      beta[(size_t)row * p.heads + h] = sigmoid_f32(source[p.beta_column + h]);
      decay[(size_t)row * p.heads + h] = expf(-expf(a_log[h]) * softplus_f32(source[p.decay_column + h] + dt_bias[h]));
    }
    return;
  }
  const uint32_t qk = p.kv_heads * p.dim, channels = 2u * qk + p.heads * p.vdim;
  const bool is_value = part >= 2u * p.kv_heads;
  const uint32_t size = is_value ? p.vdim : p.dim;
  uint32_t channel0, column0;
  float* target;
  if (part < p.kv_heads) {
    channel0 = part * p.dim, column0 = p.q_column + part * p.dim;
    target = q_out + (size_t)row * qk + part * p.dim;
  } else if (!is_value) {
    const uint32_t head = part - p.kv_heads;
    channel0 = qk + head * p.dim, column0 = p.k_column + head * p.dim;
    target = k_out + (size_t)row * qk + head * p.dim;
  } else {
    const uint32_t head = part - 2u * p.kv_heads;
    channel0 = 2u * qk + head * p.vdim, column0 = p.v_column + head * p.vdim;
    target = v_out + (size_t)row * p.heads * p.vdim + head * p.vdim;
  }
  const uint32_t state_row = min(sequence_rows[sequence], p.state_rows - 1u);
  const ConvInputs<T> inputs = {projected + (size_t)sequence * p.tokens * p.stride,
                                conv_state + (size_t)state_row * channels * p.taps, p.stride, p.taps, channels,
                                past[sequence]};
  auto convolved = [&](uint32_t c) { return silu_f32(inputs.convolve(conv_weight, column0 + c, channel0 + c, (int)token)); };
  if (is_value) {
    for (uint32_t c = lane; c < size; c += 32u) target[c] = convolved(c);
    return;
  }
  constexpr int kMost = 8;  // dim <= 256
  float value[kMost];
  float squares = 0.0f;
#pragma unroll
  for (int i = 0; i < kMost; ++i) {
    const uint32_t c = lane + i * 32u;
    value[i] = c < size ? convolved(c) : 0.0f;
    squares += value[i] * value[i];
  }
  float scale = 1.0f / sqrtf(warp_sum(squares) + 1e-6f);
  if (part < p.kv_heads) scale *= 1.0f / sqrtf((float)p.dim);
#pragma unroll
  for (int i = 0; i < kMost; ++i) {
    const uint32_t c = lane + i * 32u;
    if (c < size) target[c] = value[i] * scale;
  }
}

// Prompts, four taps, heads of at most 128: a warp walks over kStretch tokens of one head with the taps and the last
// inputs in registers, so that every input is read once.
constexpr uint32_t kStretch = 16;

template <typename T>
__global__ void __launch_bounds__(128) delta_prepare_stream_kernel(const T* projected, const float* scalars,
                                                                   const float* __restrict__ conv_weight,
                                                                   const T* conv_state, const uint32_t* past,
                                                                   const uint32_t* sequence_rows,
                                                                   const float* __restrict__ a_log,
                                                                   const float* __restrict__ dt_bias, float* q_out,
                                                                   float* k_out, float* v_out, float* decay, float* beta,
                                                                   DeltaPrepareParams p) {
  grid_chain_prologue();
  const uint32_t lane = threadIdx.x & 31u, item = blockIdx.x * 4u + (threadIdx.x >> 5);
  const uint32_t parts = 2u * p.kv_heads + p.heads + 1u, stretches = (p.tokens + kStretch - 1u) / kStretch;
  if (item >= p.sequences * stretches * parts) return;
  const uint32_t part = item % parts, sequence = item / parts / stretches, t0 = item / parts % stretches * kStretch;
  const uint32_t count = min(kStretch, p.tokens - t0);
  const size_t row0 = (size_t)sequence * p.tokens + t0;
  if (part == parts - 1u) {
    for (uint32_t index = lane; index < count * p.heads; index += 32u) {
      const uint32_t h = index % p.heads;
      const size_t row = row0 + index / p.heads;
      const float* source = scalars + row * p.scalar_stride;
      beta[row * p.heads + h] = sigmoid_f32(source[p.beta_column + h]);
      decay[row * p.heads + h] = expf(-expf(a_log[h]) * softplus_f32(source[p.decay_column + h] + dt_bias[h]));
    }
    return;
  }
  const uint32_t qk = p.kv_heads * p.dim, channels = 2u * qk + p.heads * p.vdim;
  const bool is_value = part >= 2u * p.kv_heads, is_query = part < p.kv_heads;
  const uint32_t head = is_query ? part : is_value ? part - 2u * p.kv_heads : part - p.kv_heads;
  const uint32_t size = is_value ? p.vdim : p.dim, width = is_value ? p.heads * p.vdim : qk;
  const uint32_t column0 = (is_query ? p.q_column : is_value ? p.v_column : p.k_column) + head * size;
  const uint32_t channel0 = (is_query ? 0u : is_value ? 2u * qk : qk) + head * size;
  float* target = (is_query ? q_out : is_value ? v_out : k_out) + row0 * width + head * size;
  const uint32_t state_row = min(sequence_rows[sequence], p.state_rows - 1u);
  const ConvInputs<T> inputs = {projected + (size_t)sequence * p.tokens * p.stride,
                                conv_state + (size_t)state_row * channels * 4u, p.stride, 4u, channels, past[sequence]};
  constexpr int kMost = 4;  // channels per lane
  float4 w[kMost];
  float last[kMost][3];
#pragma unroll
  for (int i = 0; i < kMost; ++i) {
    const uint32_t c = min(lane + i * 32u, size - 1u);
    w[i] = *reinterpret_cast<const float4*>(conv_weight + (size_t)(channel0 + c) * 4u);
#pragma unroll
    for (int back = 0; back < 3; ++back) last[i][back] = inputs.at(column0 + c, channel0 + c, (int)t0 - 3 + back);
  }
  const float extra = is_query ? 1.0f / sqrtf((float)p.dim) : 1.0f;
  const T* source = inputs.projected + (size_t)t0 * p.stride + column0;
  constexpr uint32_t kAhead = 4;  // tokens whose inputs are in flight together
  for (uint32_t t = 0; t < count; t += kAhead) {
    T raw[kAhead][kMost];
#pragma unroll
    for (uint32_t ahead = 0; ahead < kAhead; ++ahead)
#pragma unroll
      for (int i = 0; i < kMost; ++i)
        raw[ahead][i] = source[(size_t)min(t + ahead, count - 1u) * p.stride + min(lane + i * 32u, size - 1u)];
#pragma unroll
    for (uint32_t ahead = 0; ahead < kAhead; ++ahead) {
      if (t + ahead >= count) break;
      float value[kMost], squares = 0.0f;
#pragma unroll
      for (int i = 0; i < kMost; ++i) {
        const float now = as_float(raw[ahead][i]);
        value[i] = silu_f32(fmaf(w[i].w, now, fmaf(w[i].z, last[i][2], fmaf(w[i].y, last[i][1], w[i].x * last[i][0]))));
        last[i][0] = last[i][1];
        last[i][1] = last[i][2];
        last[i][2] = now;
        if (lane + i * 32u < size) squares += value[i] * value[i];
      }
      const float scale = is_value ? 1.0f : extra / sqrtf(warp_sum(squares) + 1e-6f);
#pragma unroll
      for (int i = 0; i < kMost; ++i)
        if (lane + i * 32u < size) target[(size_t)(t + ahead) * width + lane + i * 32u] = value[i] * scale;
    }
  }
}

bool delta_prepare_params(const KernelArgs& args, DeltaPrepareParams* p) {
  memcpy(p, args.params, sizeof(*p));
  return p->heads > 0 && p->kv_heads > 0 && p->heads % p->kv_heads == 0 && p->dim > 0 && p->dim <= 256u && p->vdim > 0 &&
         p->taps > 0 && p->state_rows > 0 && p->q_column + p->kv_heads * p->dim <= p->stride &&
         p->k_column + p->kv_heads * p->dim <= p->stride && p->v_column + p->heads * p->vdim <= p->stride;
}

// Buffers [projected, scalars, conv weight, conv state, past, sequence rows, A_log, dt_bias, q, k, v, decay, beta].
template <typename T>
int launch_delta_prepare(const KernelArgs& args) {
  DeltaPrepareParams p;
  LLMOPT_REQUIRE(args.buffer_count == 13 && args.param_bytes == sizeof(p), "expects 13 buffers and 60 parameter bytes");
  LLMOPT_REQUIRE(delta_prepare_params(args, &p), "head sizes or projection columns are inconsistent");
  const size_t rows = (size_t)p.sequences * p.tokens, qk = (size_t)p.kv_heads * p.dim, vs = (size_t)p.heads * p.vdim;
  const size_t channels = 2 * qk + vs;
  LLMOPT_REQUIRE(p.beta_column + p.heads <= p.scalar_stride && p.decay_column + p.heads <= p.scalar_stride,
                 "scalar columns lie outside the row");
  LLMOPT_REQUIRE(args.lengths[0] >= rows * p.stride * sizeof(T) && args.lengths[1] >= rows * p.scalar_stride * 4 &&
                     args.lengths[2] >= channels * p.taps * 4 &&
                     args.lengths[3] >= p.state_rows * channels * p.taps * sizeof(T) &&
                     args.lengths[4] >= (size_t)p.sequences * 4 && args.lengths[5] >= (size_t)p.sequences * 4 &&
                     args.lengths[6] >= (size_t)p.heads * 4 && args.lengths[7] >= (size_t)p.heads * 4 &&
                     args.lengths[8] >= rows * qk * 4 && args.lengths[9] >= rows * qk * 4 && args.lengths[10] >= rows * vs * 4 &&
                     args.lengths[11] >= rows * p.heads * 4 && args.lengths[12] >= rows * p.heads * 4,
                 "buffer is too short");
  if (rows == 0) return 0;
  const size_t parts = 2 * p.kv_heads + p.heads + 1;
  auto run = [&](auto kernel, size_t items) {
    launch_kernel(args, kernel, dim3((uint32_t)((items + 3) / 4)), dim3(128), 0, (const T*)args.buffers[0],
                  (const float*)args.buffers[1], (const float*)args.buffers[2], (const T*)args.buffers[3],
                  (const uint32_t*)args.buffers[4], (const uint32_t*)args.buffers[5], (const float*)args.buffers[6],
                  (const float*)args.buffers[7], (float*)args.buffers[8], (float*)args.buffers[9], (float*)args.buffers[10],
                  (float*)args.buffers[11], (float*)args.buffers[12], p);
    return check_launch(args);
  };
  if (p.taps == 4u && p.dim <= 128u && p.vdim <= 128u && p.tokens >= 8u && ((uintptr_t)args.buffers[2] & 15u) == 0)
    return run(delta_prepare_stream_kernel<T>, (size_t)p.sequences * ((p.tokens + kStretch - 1u) / kStretch) * parts);
  return run(delta_prepare_kernel<T>, rows * parts);
}

// ---- the convolutions' stored inputs ---------------------------------------------------------------
template <typename T>
__global__ void __launch_bounds__(128) conv_state_kernel(const T* projected, T* conv_state, const uint32_t* past,
                                                         const uint32_t* sequence_rows, DeltaPrepareParams p) {
  grid_chain_prologue();
  const uint32_t qk = p.kv_heads * p.dim, channels = 2u * qk + p.heads * p.vdim;
  const uint32_t channel = blockIdx.x * 128u + threadIdx.x, sequence = blockIdx.y;
  if (channel >= channels) return;
  const uint32_t column = channel < qk ? p.q_column + channel
                          : channel < 2u * qk ? p.k_column + channel - qk
                                              : p.v_column + channel - 2u * qk;
  T* ring = conv_state + (size_t)min(sequence_rows[sequence], p.state_rows - 1u) * channels * p.taps;
  const T* rows = projected + (size_t)sequence * p.tokens * p.stride;
  for (uint32_t back = 1; back <= min(p.taps, p.tokens); ++back) {
    const uint32_t token = p.tokens - back;
    ring[(size_t)((past[sequence] + token) % p.taps) * channels + channel] = rows[(size_t)token * p.stride + column];
  }
}

// Buffers [projected, conv state, past, sequence rows]; the parameter block of llmopt_delta_prepare.
template <typename T>
int launch_conv_state(const KernelArgs& args) {
  DeltaPrepareParams p;
  LLMOPT_REQUIRE(args.buffer_count == 4 && args.param_bytes == sizeof(p), "expects 4 buffers and 60 parameter bytes");
  LLMOPT_REQUIRE(delta_prepare_params(args, &p), "head sizes or projection columns are inconsistent");
  const size_t channels = 2 * (size_t)p.kv_heads * p.dim + (size_t)p.heads * p.vdim;
  LLMOPT_REQUIRE(args.lengths[0] >= (size_t)p.sequences * p.tokens * p.stride * sizeof(T) &&
                     args.lengths[1] >= p.state_rows * channels * p.taps * sizeof(T) &&
                     args.lengths[2] >= (size_t)p.sequences * 4 && args.lengths[3] >= (size_t)p.sequences * 4,
                 "buffer is too short");
  if (p.sequences == 0 || p.tokens == 0) return 0;
  launch_kernel(args, conv_state_kernel<T>, dim3((uint32_t)((channels + 127) / 128), p.sequences), dim3(128), 0,
                (const T*)args.buffers[0], (T*)args.buffers[1], (const uint32_t*)args.buffers[2],
                (const uint32_t*)args.buffers[3], p);
  return check_launch(args);
}

// ---- scan ------------------------------------------------------------------------------------------
struct ScanParams {
  uint32_t sequences, tokens, heads, kv_heads, dim, vdim;
  uint32_t q_stride, q_column, k_stride, k_column, v_stride, v_column;
  uint32_t scalar_stride, first_column, second_column;  // delta: decay, beta; memory: input gate, forget gate
  uint32_t state_rows, state_stride;                    // fp32 elements per pool row
  float gate_cap;
};

// Where a head's pieces are in a pool row.
struct StateRow {
  uint32_t heads, dim, vdim;
  __host__ __device__ size_t matrix(uint32_t head) const { return (size_t)head * vdim * dim; }
  __host__ __device__ size_t norm(uint32_t head, uint32_t slice) const {
    return (size_t)heads * vdim * dim + ((size_t)head * slices_of(vdim) + slice) * dim;
  }
  __host__ __device__ size_t top(uint32_t head, uint32_t slice) const {
    return (size_t)heads * (vdim + slices_of(vdim)) * dim + (size_t)head * slices_of(vdim) + slice;
  }
  __host__ __device__ size_t elements(bool memory) const {
    return (size_t)heads * vdim * dim + (memory ? (size_t)heads * slices_of(vdim) * (dim + 1u) : 0u);
  }
};

// One chunk's inputs and results in shared memory.
template <int R4, int CHUNK>
struct ScanChunk {
  float q[CHUNK][R4 * kLanes * 4], k[CHUNK][R4 * kLanes * 4];
  float v[CHUNK][kSlice];
  float out[CHUNK][kSlice];
  float4 scalar[CHUNK];   // delta: decay, beta, k . q; memory: keep, write, exp(-m)
  float norm_dot[CHUNK];  // memory: n . q
};

// Tokens whose read-outs are reduced together (a chunk's tokens are padded to a whole group with tokens that
// leave the state as it is).
template <int CHUNK> struct ScanGroup { static constexpr uint32_t kTokens = CHUNK >= 8 ? 4 : 1; };

template <bool MEMORY> struct ScanThreads {
  static constexpr uint32_t kCompute = (kColumnWarps + (MEMORY ? 1u : 0u)) * 32u;  // one more warp carries n
  static constexpr uint32_t kAll = kCompute + kProducerWarps * 32u;
};

// Two fp32 numbers in one register pair (Blackwell's packed fp32 arithmetic).
typedef unsigned long long Pair;
__device__ __forceinline__ Pair pair_of(float low, float high) {
  Pair d;
  asm("mov.b64 %0, {%1, %2};" : "=l"(d) : "f"(low), "f"(high));
  return d;
}
__device__ __forceinline__ Pair pair_fma(Pair a, Pair b, Pair c) {
  Pair d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
  return d;
}
__device__ __forceinline__ Pair pair_mul(Pair a, Pair b) {
  Pair d;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
  return d;
}
__device__ __forceinline__ float pair_sum(Pair a) {
  float low, high;
  asm("mov.b64 {%0, %1}, %2;" : "=f"(low), "=f"(high) : "l"(a));
  return low + high;
}

// A lane's share of kColumns columns of a state: four rows every kLanes * 4.  Rows beyond dim hold some finite
// value, which meets only zeros of q and k and is not stored.
template <int R4>
struct StateColumns {
  float* home[kColumns];
  bool active[kColumns];
  Pair s[kColumns][R4 * 2];
  __device__ __forceinline__ void load(uint32_t part, uint32_t dim, bool vectors, bool fresh) {
    if (fresh) {
#pragma unroll
      for (int j = 0; j < (int)kColumns; ++j)
#pragma unroll
        for (int i = 0; i < R4 * 2; ++i) s[j][i] = 0ull;
    } else if (vectors) {
#pragma unroll
      for (int j = 0; j < (int)kColumns; ++j)
#pragma unroll
        for (int i = 0; i < R4; ++i) {
          const ulonglong2 four = *reinterpret_cast<const ulonglong2*>(home[j] + min(i * kLanes * 4u + part * 4u, dim - 4u));
          s[j][2 * i] = four.x;
          s[j][2 * i + 1] = four.y;
        }
    } else {
#pragma unroll
      for (int j = 0; j < (int)kColumns; ++j)
#pragma unroll
        for (int i = 0; i < R4 * 2; ++i) {
          const uint32_t c = (i >> 1) * (kLanes * 4u) + part * 4u + (i & 1) * 2u;
          s[j][i] = pair_of(home[j][min(c, dim - 1u)], home[j][min(c + 1u, dim - 1u)]);
        }
    }
  }
  __device__ __forceinline__ void store(uint32_t part, uint32_t dim, bool vectors) const {
#pragma unroll
    for (int j = 0; j < (int)kColumns; ++j) {
      if (!active[j]) continue;
#pragma unroll
      for (int i = 0; i < R4; ++i) {
        const uint32_t c = i * kLanes * 4u + part * 4u;
        if (vectors) {
          if (c < dim) *reinterpret_cast<ulonglong2*>(home[j] + c) = make_ulonglong2(s[j][2 * i], s[j][2 * i + 1]);
        } else {
#pragma unroll
          for (int h = 0; h < 2; ++h) {
            float low, high;
            asm("mov.b64 {%0, %1}, %2;" : "=f"(low), "=f"(high) : "l"(s[j][2 * i + h]));
            if (c + 2u * h < dim) home[j][c + 2u * h] = low;
            if (c + 2u * h + 1u < dim) home[j][c + 2u * h + 1u] = high;
          }
        }
      }
    }
  }
};

// TQ: element of q, k, v (fp32 for the delta rule, whose unit vectors are fp32).
template <typename TQ, bool MEMORY, int R4, int CHUNK>
__global__ void __launch_bounds__(ScanThreads<MEMORY>::kAll) scan_kernel(const TQ* query, const TQ* key, const TQ* value,
                                                                         const float* first, const float* second,
                                                                         float* state_pool, const uint32_t* past,
                                                                         const uint32_t* sequence_rows, float* out,
                                                                         ScanParams p) {
  grid_chain_prologue();
  extern __shared__ __align__(16) unsigned char scan_shared[];
  typedef ScanChunk<R4, CHUNK> Chunk;
  Chunk* chunks = reinterpret_cast<Chunk*>(scan_shared);
  constexpr uint32_t kCompute = ScanThreads<MEMORY>::kCompute;
  const uint32_t slice = blockIdx.x, head = blockIdx.y, sequence = blockIdx.z;
  const uint32_t kv_head = head / (p.heads / p.kv_heads);
  const size_t row0 = (size_t)sequence * p.tokens;
  const bool fresh = past[sequence] == 0;
  float* state = state_pool + (size_t)min(sequence_rows[sequence], p.state_rows - 1u) * p.state_stride;
  const StateRow layout = {p.heads, p.dim, p.vdim};
  const uint32_t chunk_count = (p.tokens + CHUNK - 1u) / CHUNK;

  if (threadIdx.x >= kCompute) {
    // ------------------------------ producers ------------------------------
    const uint32_t thread = threadIdx.x - kCompute, warp = thread >> 5, lane = thread & 31u;
    const float q_scale = MEMORY ? 1.0f / sqrtf((float)p.dim) : 1.0f;
    float top = 0.0f;  // memory form: running maximum (warp 0)
    if (MEMORY && !fresh) top = state[layout.top(head, slice)];
    const uint32_t value_column = slice * kSlice + lane;
    auto produce = [&](uint32_t index) {
      Chunk& chunk = chunks[index & 1u];
      const uint32_t t0 = index * CHUNK, count = min((uint32_t)CHUNK, p.tokens - t0);
      constexpr int kSteps = R4 * (int)kLanes / 8;  // 32-wide pieces of a row
      constexpr uint32_t kBatch = kSteps <= 4 ? 4 : 2;  // tokens whose loads are in flight together
      constexpr uint32_t kGroup = ScanGroup<CHUNK>::kTokens;
      const uint32_t padded = (count + kGroup - 1u) / kGroup * kGroup;
      for (uint32_t begin = warp; begin < padded; begin += kProducerWarps * kBatch) {
        // loads without branches (absent elements read a present one), so that all of them are in flight at once
        TQ q_raw[kBatch][kSteps], k_raw[kBatch][kSteps], v_raw[kBatch];
#pragma unroll
        for (uint32_t b = 0; b < kBatch; ++b) {
          const size_t row = row0 + t0 + min(begin + b * kProducerWarps, count - 1u);
          const TQ* q = query + row * p.q_stride + p.q_column + kv_head * p.dim;
          const TQ* k = key + row * p.k_stride + p.k_column + kv_head * p.dim;
#pragma unroll
          for (int i = 0; i < kSteps; ++i) {
            const uint32_t c = min(lane + i * 32u, p.dim - 1u);
            q_raw[b][i] = q[c];
            k_raw[b][i] = k[c];
          }
          v_raw[b] = value[row * p.v_stride + p.v_column + head * p.vdim + min(value_column, p.vdim - 1u)];
        }
        float qs[kBatch][kSteps], ks[kBatch][kSteps], vs[kBatch];
#pragma unroll
        for (uint32_t b = 0; b < kBatch; ++b) {
#pragma unroll
          for (int i = 0; i < kSteps; ++i) {
            const bool present = lane + i * 32u < p.dim && begin + b * kProducerWarps < count;
            qs[b][i] = present ? as_float(q_raw[b][i]) * q_scale : 0.0f;
            ks[b][i] = present ? as_float(k_raw[b][i]) : 0.0f;
          }
          vs[b] = value_column < p.vdim ? as_float(v_raw[b]) : 0.0f;
        }
#pragma unroll
        for (uint32_t b = 0; b < kBatch; ++b) {
          const uint32_t t = begin + b * kProducerWarps;
          if (t >= padded) break;
          float dot = 0.0f;
#pragma unroll
          for (int i = 0; i < kSteps; ++i) {
            chunk.q[t][lane + i * 32u] = qs[b][i];
            chunk.k[t][lane + i * 32u] = ks[b][i];
            dot = fmaf(qs[b][i], ks[b][i], dot);
          }
          chunk.v[t][lane] = vs[b];
          if (!MEMORY) {
            dot = warp_sum(dot);
            if (lane == 0) chunk.scalar[t].z = dot;
          }
        }
      }
      if (warp == 0) {
        const bool present = lane < count;
        const size_t scalar_row = (row0 + t0 + (present ? lane : 0u)) * p.scalar_stride;
        float a = present ? first[scalar_row + p.first_column + head] : 0.0f;
        float b = present ? second[scalar_row + p.second_column + head] : 0.0f;
        if (MEMORY) {
          const float log_input = p.gate_cap * tanhf(a / p.gate_cap);
          const float log_forget = -softplus_f32(-p.gate_cap * tanhf(b / p.gate_cap));
          // m_t = max(f_t + m_(t-1), i_t): composition (f1, i1) then (f2, i2) = (f1 + f2, max(i1 + f2, i2))
          float sum = present ? log_forget : 0.0f, best = present ? log_input : -INFINITY;
#pragma unroll
          for (int offset = 1; offset < 32; offset <<= 1) {
            const float earlier_sum = __shfl_up_sync(0xffffffffu, sum, offset);
            const float earlier_best = __shfl_up_sync(0xffffffffu, best, offset);
            if (lane >= (uint32_t)offset) {
              best = fmaxf(earlier_best + sum, best);
              sum += earlier_sum;
            }
          }
          const float m = fmaxf(sum + top, best);
          float before = __shfl_up_sync(0xffffffffu, m, 1);
          if (lane == 0) before = top;
          a = expf(log_forget + before - m);
          b = expf(log_input - m);
          if (present) chunk.scalar[lane].z = expf(-m);
          top = __shfl_sync(0xffffffffu, m, count - 1u);
        }
        if (lane < padded) {
          chunk.scalar[lane].x = present ? a : 1.0f;
          chunk.scalar[lane].y = present ? b : 0.0f;
        }
      }
    };
    auto write_out = [&](uint32_t index) {
      const Chunk& chunk = chunks[index & 1u];
      const uint32_t t0 = index * CHUNK, count = min((uint32_t)CHUNK, p.tokens - t0);
      for (uint32_t t = warp; t < count; t += kProducerWarps) {
        float o = chunk.out[t][lane];
        if (MEMORY) o /= fmaxf(fabsf(chunk.norm_dot[t]), chunk.scalar[t].z) + 1e-6f;
        if (value_column < p.vdim) out[((row0 + t0 + t) * p.heads + head) * p.vdim + value_column] = o;
      }
    };
    produce(0);
    __syncthreads();
    for (uint32_t index = 0; index < chunk_count; ++index) {
      if (index > 0) {
        write_out(index - 1u);  // before its buffer is filled again
        asm volatile("bar.sync 1, %0;" ::"n"(kProducerWarps * 32) : "memory");
      }
      if (index + 1u < chunk_count) produce(index + 1u);
      __syncthreads();
    }
    write_out(chunk_count - 1u);
    if (MEMORY && thread == 0) state[layout.top(head, slice)] = top;
  } else {
    // ------------------------------ state ------------------------------
    const uint32_t column0 = threadIdx.x / kLanes * kColumns, part = threadIdx.x % kLanes;
    const bool is_norm = MEMORY && column0 >= kSlice;  // the extra warp: the first column of its first lanes carries n
    StateColumns<R4> columns;
    auto& active = columns.active;
    auto& s = columns.s;
#pragma unroll
    for (int j = 0; j < (int)kColumns; ++j) {
      const uint32_t column = slice * kSlice + column0 + j;
      active[j] = is_norm ? column0 + j == kSlice : column < p.vdim;
      columns.home[j] = state + (is_norm ? layout.norm(head, slice) : layout.matrix(head) + (size_t)(active[j] ? column : 0u) * p.dim);
    }
    const bool vectors = p.dim % 4u == 0 && p.state_stride % 4u == 0;
    columns.load(part, p.dim, vectors, fresh);
    __syncthreads();
    for (uint32_t index = 0; index < chunk_count; ++index) {
      Chunk& chunk = chunks[index & 1u];
      const uint32_t count = min((uint32_t)CHUNK, p.tokens - index * CHUNK);
      constexpr int G = ScanGroup<CHUNK>::kTokens;
#pragma unroll 1
      for (uint32_t t0 = 0; t0 < count; t0 += G) {
        float partial[G][kColumns];  // this lane's share of the tokens' read-outs
        float update[G][kColumns];   // delta rule
#pragma unroll
        for (int g = 0; g < G; ++g) {
          const uint32_t t = t0 + g;
          const ulonglong2* q = reinterpret_cast<const ulonglong2*>(chunk.q[t]) + part;
          const ulonglong2* k = reinterpret_cast<const ulonglong2*>(chunk.k[t]) + part;
          const float4 scalar = chunk.scalar[t];
          const float2 values = *reinterpret_cast<const float2*>(&chunk.v[t][column0 % kSlice]);
          const Pair keep2 = pair_of(scalar.x, scalar.x);
          Pair kk[R4 * 2];
#pragma unroll
          for (int i = 0; i < R4; ++i) {
            const ulonglong2 four = k[i * kLanes];
            kk[2 * i] = four.x;
            kk[2 * i + 1] = four.y;
          }
          Pair sums[kColumns][2];
#pragma unroll
          for (int j = 0; j < (int)kColumns; ++j) sums[j][0] = sums[j][1] = 0ull;
          if (MEMORY) {
            const float write = scalar.y;
            const float target[kColumns] = {is_norm ? write : write * values.x, write * values.y};
#pragma unroll
            for (int i = 0; i < R4; ++i) {
              const ulonglong2 qq = q[i * kLanes];
#pragma unroll
              for (int j = 0; j < (int)kColumns; ++j) {
                const Pair write2 = pair_of(target[j], target[j]);
                s[j][2 * i] = pair_fma(kk[2 * i], write2, pair_mul(s[j][2 * i], keep2));
                s[j][2 * i + 1] = pair_fma(kk[2 * i + 1], write2, pair_mul(s[j][2 * i + 1], keep2));
                sums[j][0] = pair_fma(s[j][2 * i], qq.x, sums[j][0]);
                sums[j][1] = pair_fma(s[j][2 * i + 1], qq.y, sums[j][1]);
              }
            }
#pragma unroll
            for (int j = 0; j < (int)kColumns; ++j) partial[g][j] = pair_sum(sums[j][0]) + pair_sum(sums[j][1]);
          } else {
            float with_key[kColumns];
#pragma unroll
            for (int i = 0; i < R4; ++i)
#pragma unroll
              for (int j = 0; j < (int)kColumns; ++j) {
                sums[j][0] = pair_fma(s[j][2 * i], kk[2 * i], sums[j][0]);
                sums[j][1] = pair_fma(s[j][2 * i + 1], kk[2 * i + 1], sums[j][1]);
              }
#pragma unroll
            for (int j = 0; j < (int)kColumns; ++j) {
              with_key[j] = pair_sum(sums[j][0]) + pair_sum(sums[j][1]);
              sums[j][0] = sums[j][1] = 0ull;
            }
#pragma unroll
            for (int offset = 1; offset < (int)kLanes; offset <<= 1)
#pragma unroll
              for (int j = 0; j < (int)kColumns; ++j) with_key[j] += __shfl_xor_sync(0xffffffffu, with_key[j], offset);
#pragma unroll
            for (int i = 0; i < R4; ++i) {
              const ulonglong2 qq = q[i * kLanes];
#pragma unroll
              for (int j = 0; j < (int)kColumns; ++j) {
                sums[j][0] = pair_fma(s[j][2 * i], qq.x, sums[j][0]);
                sums[j][1] = pair_fma(s[j][2 * i + 1], qq.y, sums[j][1]);
              }
            }
            update[g][0] = scalar.y * (values.x - scalar.x * with_key[0]);
            update[g][1] = scalar.y * (values.y - scalar.x * with_key[1]);
#pragma unroll
            for (int j = 0; j < (int)kColumns; ++j) {
              partial[g][j] = pair_sum(sums[j][0]) + pair_sum(sums[j][1]);
              const Pair update2 = pair_of(update[g][j], update[g][j]);
#pragma unroll
              for (int i = 0; i < R4 * 2; ++i) s[j][i] = pair_fma(kk[i], update2, pair_mul(s[j][i], keep2));
            }
          }
        }
        if (G == 4) {
          // eight sums over a column's lanes: each exchange halves what a lane keeps, so that lane `part` ends with
          // value part / (kLanes / 8); the lanes that hold the same value then add what they have
          float v[8], u[8];
#pragma unroll
          for (int i = 0; i < 8; ++i) {
            v[i] = partial[i / 2 % G][i % 2];
            u[i] = MEMORY ? 0.0f : update[i / 2 % G][i % 2];
          }
#pragma unroll
          for (int half = 4; half > 0; half >>= 1) {
            const uint32_t distance = half * (kLanes / 8u);
            const bool upper = (part & distance) != 0;
#pragma unroll
            for (int i = 0; i < half; ++i) {
              const float sent = upper ? v[i] : v[i + half], kept = upper ? v[i + half] : v[i];
              v[i] = kept + __shfl_xor_sync(0xffffffffu, sent, distance);
              if (!MEMORY) u[i] = upper ? u[i + half] : u[i];
            }
          }
#pragma unroll
          for (uint32_t distance = kLanes / 16u; distance > 0; distance >>= 1)
            v[0] += __shfl_xor_sync(0xffffffffu, v[0], distance);
          const uint32_t which = part / (kLanes / 8u), t = t0 + which / 2u, j = which % 2u;
          if (part % (kLanes / 8u) != 0) {
            // another lane writes this value
          } else if (MEMORY) {
            if (!is_norm) chunk.out[t][column0 + j] = v[0];
            else if (active[0] && j == 0u) chunk.norm_dot[t] = v[0];
          } else {
            const float4 scalar = chunk.scalar[t];
            chunk.out[t][column0 + j] = fmaf(u[0], scalar.z, scalar.x * v[0]);
          }
        } else {
#pragma unroll
          for (int j = 0; j < (int)kColumns; ++j)
#pragma unroll
            for (int offset = 1; offset < (int)kLanes; offset <<= 1)
              partial[0][j] += __shfl_xor_sync(0xffffffffu, partial[0][j], offset);
          if (part == 0) {
            if (MEMORY) {
              if (!is_norm) *reinterpret_cast<float2*>(&chunk.out[t0][column0]) = make_float2(partial[0][0], partial[0][1]);
              else if (active[0]) chunk.norm_dot[t0] = partial[0][0];
            } else {
              const float4 scalar = chunk.scalar[t0];
              *reinterpret_cast<float2*>(&chunk.out[t0][column0]) =
                  make_float2(fmaf(update[0][0], scalar.z, scalar.x * partial[0][0]),
                              fmaf(update[0][1], scalar.z, scalar.x * partial[0][1]));
            }
          }
        }
      }
      __syncthreads();
    }
    columns.store(part, p.dim, vectors);
  }
}

// Buffers [q, k, v, first scalar, second scalar, state pool, past, sequence rows, out f32].
template <typename TQ, bool MEMORY>
int launch_scan(const KernelArgs& args) {
  ScanParams p;
  LLMOPT_REQUIRE(args.buffer_count == 9 && args.param_bytes == sizeof(p), "expects 9 buffers and 72 parameter bytes");
  memcpy(&p, args.params, sizeof(p));
  const size_t rows = (size_t)p.sequences * p.tokens, e = sizeof(TQ);
  LLMOPT_REQUIRE(p.heads > 0 && p.kv_heads > 0 && p.heads % p.kv_heads == 0 && p.vdim > 0 && p.dim > 0 && p.dim <= 256u,
                 "needs whole groups of heads and a key size of at most 256");
  LLMOPT_REQUIRE(!MEMORY || p.gate_cap > 0.0f, "the gate cap must be positive");
  const StateRow layout = {p.heads, p.dim, p.vdim};
  LLMOPT_REQUIRE(p.state_rows > 0 && p.state_stride >= layout.elements(MEMORY) &&
                     args.lengths[5] >= (size_t)p.state_rows * p.state_stride * 4,
                 "state pool is too short");
  LLMOPT_REQUIRE(p.q_column + p.kv_heads * p.dim <= p.q_stride && p.k_column + p.kv_heads * p.dim <= p.k_stride &&
                     p.v_column + p.heads * p.vdim <= p.v_stride && p.first_column + p.heads <= p.scalar_stride &&
                     p.second_column + p.heads <= p.scalar_stride,
                 "columns lie outside their rows");
  LLMOPT_REQUIRE(args.lengths[0] >= rows * p.q_stride * e && args.lengths[1] >= rows * p.k_stride * e &&
                     args.lengths[2] >= rows * p.v_stride * e && args.lengths[3] >= rows * p.scalar_stride * 4 &&
                     args.lengths[4] >= rows * p.scalar_stride * 4 && args.lengths[6] >= (size_t)p.sequences * 4 &&
                     args.lengths[7] >= (size_t)p.sequences * 4 && args.lengths[8] >= rows * p.heads * p.vdim * 4,
                 "buffer is too short");
  LLMOPT_REQUIRE(p.sequences <= 65535u && p.heads <= 65535u, "too many sequences or heads");
  if (rows == 0) return 0;
  auto run = [&](auto kernel, size_t shared) {
    if (cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)shared) != cudaSuccess) {
      cudaGetLastError();
      return fail(args, "shared memory request was refused");
    }
    launch_kernel(args, kernel, dim3(slices_of(p.vdim), p.heads, p.sequences), dim3(ScanThreads<MEMORY>::kAll), shared,
                  (const TQ*)args.buffers[0], (const TQ*)args.buffers[1], (const TQ*)args.buffers[2],
                  (const float*)args.buffers[3], (const float*)args.buffers[4], (float*)args.buffers[5],
                  (const uint32_t*)args.buffers[6], (const uint32_t*)args.buffers[7], (float*)args.buffers[8], p);
    return check_launch(args);
  };
  const uint32_t quads = (p.dim + kLanes * 4u - 1u) / (kLanes * 4u);
  // few tokens: small chunks, so that more CTAs fit on an SM
  auto sized = [&](auto r4) {
    constexpr int R4 = decltype(r4)::value;
    if (p.tokens <= 4u) return run(scan_kernel<TQ, MEMORY, R4, 4>, 2 * sizeof(ScanChunk<R4, 4>));
    return run(scan_kernel<TQ, MEMORY, R4, 32>, 2 * sizeof(ScanChunk<R4, 32>));
  };
  if (quads <= 1u) return sized(std::integral_constant<int, 1>());
  if (quads <= 2u) return sized(std::integral_constant<int, 2>());
  if (quads <= 3u) return sized(std::integral_constant<int, 3>());
  return sized(std::integral_constant<int, 4>());
}

// ---- one token per sequence, fused -----------------------------------------------------------------
struct StepParams {
  uint32_t sequences, tokens /* 1 */, heads, kv_heads, dim, vdim, taps;
  uint32_t stride, q_column, k_column, v_column, gate_column;  // projections, T [sequences, stride]
  uint32_t scalar_stride, first_column, second_column;         // delta: beta, decay; memory: input gate, forget gate
  uint32_t state_rows, state_stride;
  float gate_cap, epsilon;
};
struct StepBuffers {
  const void* projected;
  const float* scalars;
  const float* conv_weight;
  void* conv_state;
  const float* a_log;
  const float* dt_bias;
  const float* norm;  // delta: [vdim]; memory: [heads * vdim]
  float* state;
  const uint32_t* past;
  const uint32_t* sequence_rows;
  void* out;  // T [sequences, heads * vdim]
};

template <bool MEMORY> __host__ __device__ constexpr uint32_t step_threads() {
  return (kColumnWarps + (MEMORY ? 1u : 0u)) * 32u;
}

// A CTA owns kSlice value columns of one head of one sequence, the CTAs of a head are one cluster: the
// head's norm needs every column's square.  Lanes and columns as in the scan.
template <typename T, bool MEMORY, int R4>
__global__ void __launch_bounds__(step_threads<MEMORY>()) state_step_kernel(const StepBuffers b, const StepParams p) {
  grid_chain_prologue();
  constexpr uint32_t kRow = R4 * kLanes * 4u, kThreads = step_threads<MEMORY>();
  __shared__ __align__(16) float q_row[kRow], k_row[kRow];
  __shared__ float v_row[kSlice], o_row[kSlice];
  __shared__ float norm_dot, cta_square;
  const uint32_t slices = slices_of(p.vdim);
  const uint32_t slice = blockIdx.x, head = blockIdx.y, sequence = blockIdx.z;
  const uint32_t kv_head = head / (p.heads / p.kv_heads), warp = threadIdx.x >> 5, lane = threadIdx.x & 31u;
  const uint32_t past = b.past[sequence], state_row = min(b.sequence_rows[sequence], p.state_rows - 1u);
  float* state = b.state + (size_t)state_row * p.state_stride;
  const StateRow layout = {p.heads, p.dim, p.vdim};
  const T* projected = reinterpret_cast<const T*>(b.projected) + (size_t)sequence * p.stride;
  const float* scalars = b.scalars + (size_t)sequence * p.scalar_stride;

  // the state is requested first; everything else is computed while it is on its way
  const uint32_t column0 = threadIdx.x / kLanes * kColumns, part = threadIdx.x % kLanes;
  const bool is_norm = MEMORY && column0 >= kSlice;
  StateColumns<R4> columns;
  auto& active = columns.active;
  auto& s = columns.s;
#pragma unroll
  for (int j = 0; j < (int)kColumns; ++j) {
    const uint32_t column = slice * kSlice + column0 + j;
    active[j] = is_norm ? column0 + j == kSlice : column < p.vdim;
    columns.home[j] = state + (is_norm ? layout.norm(head, slice) : layout.matrix(head) + (size_t)(active[j] ? column : 0u) * p.dim);
  }
  const bool vectors = p.dim % 4u == 0 && p.state_stride % 4u == 0;
  columns.load(part, p.dim, vectors, past == 0);
  float old_top = 0.0f;
  if (MEMORY && past > 0) old_top = state[layout.top(head, slice)];
  float keep, write, floor_value = 0.0f, new_top = 0.0f;
  if (MEMORY) {
    const float log_input = p.gate_cap * tanhf(scalars[p.first_column + head] / p.gate_cap);
    const float log_forget = -softplus_f32(-p.gate_cap * tanhf(scalars[p.second_column + head] / p.gate_cap));
    new_top = fmaxf(log_forget + old_top, log_input);
    keep = expf(log_forget + old_top - new_top);
    write = expf(log_input - new_top);
    floor_value = expf(-new_top);
  } else {
    write = sigmoid_f32(scalars[p.first_column + head]);
    keep = expf(-expf(b.a_log[head]) * softplus_f32(scalars[p.second_column + head] + b.dt_bias[head]));
  }

  // q, k and this slice's v
  const uint32_t qk = p.kv_heads * p.dim, channels = 2u * qk + p.heads * p.vdim;
  T* ring = MEMORY ? nullptr : reinterpret_cast<T*>(b.conv_state) + (size_t)state_row * channels * p.taps;
  for (uint32_t index = threadIdx.x; index < 2u * kRow + kSlice; index += kThreads) {
    const bool is_value = index >= 2u * kRow, is_key = !is_value && index >= kRow;
    const uint32_t c = is_value ? slice * kSlice + index - 2u * kRow : index % kRow;
    float value = 0.0f;
    if (c < (is_value ? p.vdim : p.dim)) {
      const uint32_t column = is_value ? p.v_column + head * p.vdim + c : (is_key ? p.k_column : p.q_column) + kv_head * p.dim + c;
      if (MEMORY) {
        value = as_float(projected[column]);
        if (!is_value && !is_key) value *= 1.0f / sqrtf((float)p.dim);
      } else {
        const uint32_t channel = is_value ? 2u * qk + head * p.vdim + c : (is_key ? qk : 0u) + kv_head * p.dim + c;
        const ConvInputs<T> inputs = {projected, ring, p.stride, p.taps, channels, past};
        value = silu_f32(inputs.convolve(b.conv_weight, column, channel, 0));
        // keep the input: once per channel, in a ring row that this step does not read
        if (is_value || (slice == 0u && head % (p.heads / p.kv_heads) == 0u))
          ring[(size_t)(past % p.taps) * channels + channel] = projected[column];
      }
    }
    if (is_value) v_row[index - 2u * kRow] = value;
    else (is_key ? k_row : q_row)[c] = value;
  }
  __syncthreads();
  if (!MEMORY) {  // unit vectors
    if (warp < 2u) {
      float* row = warp == 0u ? q_row : k_row;
      float sum = 0.0f;
      for (uint32_t c = lane; c < kRow; c += 32u) sum += row[c] * row[c];
      float scale = 1.0f / sqrtf(warp_sum(sum) + 1e-6f);
      if (warp == 0u) scale *= 1.0f / sqrtf((float)p.dim);
      for (uint32_t c = lane; c < kRow; c += 32u) row[c] *= scale;
    }
    __syncthreads();
  }

  const ulonglong2* q = reinterpret_cast<const ulonglong2*>(q_row) + part;
  const ulonglong2* k = reinterpret_cast<const ulonglong2*>(k_row) + part;
  const Pair keep2 = pair_of(keep, keep);
#pragma unroll
  for (int j = 0; j < (int)kColumns; ++j) {
    const float value = is_norm ? 1.0f : v_row[(column0 + j) % kSlice];
    float change = write * value;
    if (!MEMORY) {
      Pair sum = 0ull;
#pragma unroll
      for (int i = 0; i < R4; ++i) {
        const ulonglong2 kk = k[i * kLanes];
        sum = pair_fma(s[j][2 * i], kk.x, sum);
        sum = pair_fma(s[j][2 * i + 1], kk.y, sum);
      }
      float with_key = pair_sum(sum);
#pragma unroll
      for (int offset = 1; offset < (int)kLanes; offset <<= 1) with_key += __shfl_xor_sync(0xffffffffu, with_key, offset);
      change = write * (value - keep * with_key);
    }
    const Pair change2 = pair_of(change, change);
    Pair sum = 0ull;
#pragma unroll
    for (int i = 0; i < R4; ++i) {
      const ulonglong2 kk = k[i * kLanes], qq = q[i * kLanes];
      s[j][2 * i] = pair_fma(kk.x, change2, pair_mul(s[j][2 * i], keep2));
      s[j][2 * i + 1] = pair_fma(kk.y, change2, pair_mul(s[j][2 * i + 1], keep2));
      sum = pair_fma(s[j][2 * i], qq.x, sum);
      sum = pair_fma(s[j][2 * i + 1], qq.y, sum);
    }
    float o = pair_sum(sum);
#pragma unroll
    for (int offset = 1; offset < (int)kLanes; offset <<= 1) o += __shfl_xor_sync(0xffffffffu, o, offset);
    if (part == 0) {
      if (is_norm) {
        if (active[j]) norm_dot = o;
      } else {
        o_row[column0 + j] = o;
      }
    }
  }
  columns.store(part, p.dim, vectors);
  if (MEMORY && threadIdx.x == 0) state[layout.top(head, slice)] = new_top;
  __syncthreads();
  float value = 0.0f;
  const uint32_t column = slice * kSlice + threadIdx.x;  // of the first warp's threads
  if (warp == 0u) {
    value = column < p.vdim ? o_row[threadIdx.x] : 0.0f;
    if (MEMORY) value /= fmaxf(fabsf(norm_dot), floor_value) + 1e-6f;
    const float sum = warp_sum(value * value);
    if (lane == 0) cta_square = sum;
  }
  cluster_sync();
  if (warp == 0u) {
    float total = 0.0f;
    for (uint32_t other = 0; other < slices; ++other) total += cluster_load(&cta_square, other);
    const float scale = 1.0f / sqrtf(total / (float)p.vdim + p.epsilon);
    if (column < p.vdim) {
      const float z = as_float(projected[p.gate_column + head * p.vdim + column]);
      const float weight = b.norm[MEMORY ? head * p.vdim + column : column];
      reinterpret_cast<T*>(b.out)[((size_t)sequence * p.heads + head) * p.vdim + column] =
          from_float<T>(value * scale * weight * (MEMORY ? sigmoid_f32(z) : silu_f32(z)));
    }
  }
  cluster_sync();  // nobody leaves while its sum may be read
}

// Memory: buffers [projected, scalars, norm, state, past, sequence rows, out]; delta: [projected, scalars, conv weight,
// conv state, A_log, dt_bias, norm, state, past, sequence rows, out].
template <typename T, bool MEMORY>
int launch_state_step(const KernelArgs& args) {
  StepParams p;
  constexpr int kCount = MEMORY ? 7 : 11;
  LLMOPT_REQUIRE(args.buffer_count == kCount && args.param_bytes == sizeof(p),
                 "expects 7 (memory) or 11 (delta) buffers and 76 parameter bytes");
  memcpy(&p, args.params, sizeof(p));
  LLMOPT_REQUIRE(p.tokens == 1u && p.heads > 0 && p.kv_heads > 0 && p.heads % p.kv_heads == 0 && p.dim > 0 && p.dim <= 256u &&
                     p.vdim > 0,
                 "needs one token, whole groups of heads and a key size of at most 256");
  const uint32_t slices = slices_of(p.vdim);
  LLMOPT_REQUIRE(slices <= 8u, "a value size of at most 256");
  const StateRow layout = {p.heads, p.dim, p.vdim};
  const size_t qk = (size_t)p.kv_heads * p.dim, vs = (size_t)p.heads * p.vdim, rows = p.sequences;
  LLMOPT_REQUIRE(p.q_column + qk <= p.stride && p.k_column + qk <= p.stride && p.v_column + vs <= p.stride &&
                     p.gate_column + vs <= p.stride && p.first_column + p.heads <= p.scalar_stride &&
                     p.second_column + p.heads <= p.scalar_stride,
                 "columns lie outside their rows");
  LLMOPT_REQUIRE(p.state_rows > 0 && p.state_stride >= layout.elements(MEMORY), "state rows are too short");
  LLMOPT_REQUIRE(!MEMORY || p.gate_cap > 0.0f, "the gate cap must be positive");
  LLMOPT_REQUIRE(MEMORY || p.taps > 0, "a convolution needs taps");
  StepBuffers b = {};
  int next = 0;
  bool ok = true;
  auto take = [&](auto& target, size_t bytes) {
    ok = ok && args.lengths[next] >= bytes;
    target = reinterpret_cast<std::remove_reference_t<decltype(target)>>(args.buffers[next]);
    ++next;
  };
  take(b.projected, rows * p.stride * sizeof(T));
  take(b.scalars, rows * p.scalar_stride * 4);
  if (!MEMORY) {
    take(b.conv_weight, (2 * qk + vs) * p.taps * 4);
    take(b.conv_state, p.state_rows * (2 * qk + vs) * p.taps * sizeof(T));
    take(b.a_log, (size_t)p.heads * 4);
    take(b.dt_bias, (size_t)p.heads * 4);
  }
  take(b.norm, (MEMORY ? vs : (size_t)p.vdim) * 4);
  take(b.state, (size_t)p.state_rows * p.state_stride * 4);
  take(b.past, rows * 4);
  take(b.sequence_rows, rows * 4);
  take(b.out, rows * vs * sizeof(T));
  LLMOPT_REQUIRE(ok, "buffer is too short");
  LLMOPT_REQUIRE(p.sequences <= 65535u && p.heads <= 65535u, "too many sequences or heads");
  if (rows == 0) return 0;
  auto run = [&](auto kernel) {
    launch_cluster_kernel(args, kernel, dim3(slices, p.heads, p.sequences), dim3(step_threads<MEMORY>()), 0, slices, b, p);
    return check_launch(args);
  };
  const uint32_t quads = (p.dim + kLanes * 4u - 1u) / (kLanes * 4u);
  if (quads <= 1u) return run(state_step_kernel<T, MEMORY, 1>);
  if (quads <= 2u) return run(state_step_kernel<T, MEMORY, 2>);
  if (quads <= 3u) return run(state_step_kernel<T, MEMORY, 3>);
  return run(state_step_kernel<T, MEMORY, 4>);
}

}  // namespace

const NamedLauncher* matrix_state_launchers(size_t* count) {
  static const NamedLauncher table[] = {
      {"llmopt_delta_prepare_bf16", launch_delta_prepare<bf16>},
      {"llmopt_delta_prepare_f32", launch_delta_prepare<float>},
      {"llmopt_conv_state_bf16", launch_conv_state<bf16>},
      {"llmopt_conv_state_f32", launch_conv_state<float>},
      {"llmopt_delta_scan_f32", launch_scan<float, false>},
      {"llmopt_memory_scan_bf16", launch_scan<bf16, true>},
      {"llmopt_memory_scan_f32", launch_scan<float, true>},
      {"llmopt_delta_step_bf16", launch_state_step<bf16, false>},
      {"llmopt_delta_step_f32", launch_state_step<float, false>},
      {"llmopt_memory_step_bf16", launch_state_step<bf16, true>},
      {"llmopt_memory_step_f32", launch_state_step<float, true>},
  };
  *count = sizeof(table) / sizeof(table[0]);
  return table;
}

}  // namespace llmopt
