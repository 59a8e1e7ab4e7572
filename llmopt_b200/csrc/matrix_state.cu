// Recurrent mixers with a matrix state per head, carried in fp32 from token to token:
//   llmopt_delta_prepare_{bf16,f32}    short convolutions, unit q and k, decay and step size of a gated delta rule
//   llmopt_conv_state_{bf16,f32}       the convolutions' last inputs
//   llmopt_delta_scan_f32              S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q
//   llmopt_memory_scan_{bf16,f32}      stabilised exponential gating (mLSTM): S <- a S + b k v^T, n <- a n + b k,
//                                      o = S^T q / (max(|n . q|, exp(-m)) + 1e-6)
//
// State of a sequence lives in row `sequence_rows[i]` of a state pool.  A row holds, per head, the
// transposed matrix [vdim][dim]; the matrix-memory form adds n [dim] and m once per slice of kSlice value
// columns, because every slice's CTA needs them and keeps a copy of its own.  A sequence with nothing
// behind it (past = 0) starts from zero whatever its pool row holds.
//
// Scan: a CTA owns kSlice value columns of one head of one sequence and walks over the tokens.  Eight lanes
// share a column of S (each dim / 8 rows of it, in registers).  Compute warps work on a chunk of tokens in
// shared memory while producer warps bring in the next chunk (converted to fp32, with the per-token
// scalars) and write out the previous one's results.  The read-out of the delta rule uses
// S_new^T q = g S_old^T q + u (k . q), so that its sum and the one of S_old^T k are reduced at the same time.
#include "element.cuh"

namespace llmopt {
namespace {

constexpr uint32_t kSlice = 16;        // value columns per CTA
constexpr uint32_t kLanes = 8;         // lanes per column
constexpr uint32_t kChunk = 32;        // tokens per chunk
constexpr uint32_t kColumnWarps = kSlice * kLanes / 32;  // 4
constexpr uint32_t kProducerWarps = 4;

__host__ __device__ constexpr uint32_t slices_of(uint32_t vdim) { return (vdim + kSlice - 1u) / kSlice; }

// ---- gated delta rule: inputs ----------------------------------------------------------------------
struct DeltaPrepareParams {
  uint32_t sequences, tokens, heads, kv_heads, dim, vdim, taps;
  uint32_t stride, q_column, k_column, v_column;  // projections, T [rows, stride]
  uint32_t scalar_stride, beta_column, decay_column;  // projections, fp32 [rows, scalar_stride]
  uint32_t state_rows;
};

// Input of channel `channel` (counted over q, k, v) at `token` - `back`, from the projections or, before
// the step's first token, from the sequence's stored inputs [channels][taps - 1], oldest first.
template <typename T>
struct ConvInputs {
  const T* projected;  // first row of the sequence
  const T* stored;     // or null: nothing before the step
  uint32_t stride, taps;
  __device__ __forceinline__ float at(uint32_t column, uint32_t channel, int token) const {
    if (token >= 0) return as_float(projected[(size_t)token * stride + column]);
    const int kept = (int)taps - 1 + token;
    return stored != nullptr ? as_float(stored[(size_t)channel * (taps - 1u) + kept]) : 0.0f;
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
                                past[sequence] > 0 ? conv_state + (size_t)state_row * channels * (p.taps - 1u) : nullptr,
                                p.stride, p.taps};
  auto convolved = [&](uint32_t c) {
    float sum = 0.0f;
    for (uint32_t tap = 0; tap < p.taps; ++tap)
      sum = fmaf(__ldg(conv_weight + (size_t)(channel0 + c) * p.taps + tap),
                 inputs.at(column0 + c, channel0 + c, (int)token - (int)(p.taps - 1u - tap)), sum);
    return silu_f32(sum);
  };
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
                     args.lengths[3] >= p.state_rows * channels * (p.taps - 1) * sizeof(T) &&
                     args.lengths[4] >= (size_t)p.sequences * 4 && args.lengths[5] >= (size_t)p.sequences * 4 &&
                     args.lengths[6] >= (size_t)p.heads * 4 && args.lengths[7] >= (size_t)p.heads * 4 &&
                     args.lengths[8] >= rows * qk * 4 && args.lengths[9] >= rows * qk * 4 && args.lengths[10] >= rows * vs * 4 &&
                     args.lengths[11] >= rows * p.heads * 4 && args.lengths[12] >= rows * p.heads * 4,
                 "buffer is too short");
  if (rows == 0) return 0;
  const size_t items = rows * (2 * p.kv_heads + p.heads + 1);
  launch_kernel(args, delta_prepare_kernel<T>, dim3((uint32_t)((items + 3) / 4)), dim3(128), 0, (const T*)args.buffers[0],
                (const float*)args.buffers[1], (const float*)args.buffers[2], (const T*)args.buffers[3],
                (const uint32_t*)args.buffers[4], (const uint32_t*)args.buffers[5], (const float*)args.buffers[6],
                (const float*)args.buffers[7], (float*)args.buffers[8], (float*)args.buffers[9], (float*)args.buffers[10],
                (float*)args.buffers[11], (float*)args.buffers[12], p);
  return check_launch(args);
}

// ---- the convolutions' stored inputs ---------------------------------------------------------------
constexpr uint32_t kMostTaps = 16;

template <typename T>
__global__ void __launch_bounds__(128) conv_state_kernel(const T* projected, T* conv_state, const uint32_t* past,
                                                         const uint32_t* sequence_rows, DeltaPrepareParams p) {
  grid_chain_prologue();
  const uint32_t qk = p.kv_heads * p.dim, channels = 2u * qk + p.heads * p.vdim, kept = p.taps - 1u;
  const uint32_t channel = blockIdx.x * 128u + threadIdx.x, sequence = blockIdx.y;
  if (channel >= channels) return;
  const uint32_t column = channel < qk ? p.q_column + channel
                          : channel < 2u * qk ? p.k_column + channel - qk
                                              : p.v_column + channel - 2u * qk;
  T* stored = conv_state + (size_t)min(sequence_rows[sequence], p.state_rows - 1u) * channels * kept;
  const ConvInputs<T> inputs = {projected + (size_t)sequence * p.tokens * p.stride, past[sequence] > 0 ? stored : nullptr,
                                p.stride, p.taps};
  float next[kMostTaps];
#pragma unroll
  for (uint32_t i = 0; i < kMostTaps; ++i)
    if (i < kept) next[i] = inputs.at(column, channel, (int)p.tokens - (int)kept + (int)i);
#pragma unroll
  for (uint32_t i = 0; i < kMostTaps; ++i)
    if (i < kept) stored[(size_t)channel * kept + i] = from_float<T>(next[i]);
}

// Buffers [projected, conv state, past, sequence rows]; the parameter block of llmopt_delta_prepare.
template <typename T>
int launch_conv_state(const KernelArgs& args) {
  DeltaPrepareParams p;
  LLMOPT_REQUIRE(args.buffer_count == 4 && args.param_bytes == sizeof(p), "expects 4 buffers and 60 parameter bytes");
  LLMOPT_REQUIRE(delta_prepare_params(args, &p), "head sizes or projection columns are inconsistent");
  LLMOPT_REQUIRE(p.taps <= kMostTaps + 1u, "at most 17 taps");
  const size_t channels = 2 * (size_t)p.kv_heads * p.dim + (size_t)p.heads * p.vdim;
  LLMOPT_REQUIRE(args.lengths[0] >= (size_t)p.sequences * p.tokens * p.stride * sizeof(T) &&
                     args.lengths[1] >= p.state_rows * channels * (p.taps - 1) * sizeof(T) &&
                     args.lengths[2] >= (size_t)p.sequences * 4 && args.lengths[3] >= (size_t)p.sequences * 4,
                 "buffer is too short");
  if (p.sequences == 0 || p.tokens == 0 || p.taps == 1u) return 0;
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
template <int R4>
struct ScanChunk {
  float q[kChunk][R4 * 32], k[kChunk][R4 * 32];
  float v[kChunk][kSlice];
  float out[kChunk][kSlice];
  float first[kChunk], second[kChunk];  // delta: decay, beta; memory: keep, write
  float extra[kChunk];                  // delta: k . q; memory: exp(-m)
  float norm_dot[kChunk];               // memory: n . q
};

template <bool MEMORY> struct ScanThreads {
  static constexpr uint32_t kCompute = (kColumnWarps + (MEMORY ? 1u : 0u)) * 32u;  // one more warp carries n
  static constexpr uint32_t kAll = kCompute + kProducerWarps * 32u;
};

// TQ: element of q, k, v (fp32 for the delta rule, whose unit vectors are fp32).
template <typename TQ, bool MEMORY, int R4>
__global__ void __launch_bounds__(ScanThreads<MEMORY>::kAll) scan_kernel(const TQ* query, const TQ* key, const TQ* value,
                                                                         const float* first, const float* second,
                                                                         float* state_pool, const uint32_t* past,
                                                                         const uint32_t* sequence_rows, float* out,
                                                                         ScanParams p) {
  grid_chain_prologue();
  extern __shared__ __align__(16) unsigned char scan_shared[];
  ScanChunk<R4>* chunks = reinterpret_cast<ScanChunk<R4>*>(scan_shared);
  constexpr uint32_t kCompute = ScanThreads<MEMORY>::kCompute;
  const uint32_t slice = blockIdx.x, head = blockIdx.y, sequence = blockIdx.z;
  const uint32_t kv_head = head / (p.heads / p.kv_heads);
  const size_t row0 = (size_t)sequence * p.tokens;
  const bool fresh = past[sequence] == 0;
  float* state = state_pool + (size_t)min(sequence_rows[sequence], p.state_rows - 1u) * p.state_stride;
  const StateRow layout = {p.heads, p.dim, p.vdim};
  const uint32_t chunk_count = (p.tokens + kChunk - 1u) / kChunk;

  if (threadIdx.x >= kCompute) {
    // ------------------------------ producers ------------------------------
    const uint32_t thread = threadIdx.x - kCompute, warp = thread >> 5, lane = thread & 31u;
    const float q_scale = MEMORY ? 1.0f / sqrtf((float)p.dim) : 1.0f;
    float top = 0.0f;  // memory form: running maximum (warp 0)
    if (MEMORY && !fresh) top = state[layout.top(head, slice)];
    auto produce = [&](uint32_t index) {
      ScanChunk<R4>& chunk = chunks[index & 1u];
      const uint32_t t0 = index * kChunk, count = min(kChunk, p.tokens - t0);
      for (uint32_t t = warp; t < count; t += kProducerWarps) {
        const size_t row = row0 + t0 + t;
        const TQ* q = query + row * p.q_stride + p.q_column + kv_head * p.dim;
        const TQ* k = key + row * p.k_stride + p.k_column + kv_head * p.dim;
        float dot = 0.0f;
#pragma unroll
        for (int i = 0; i < R4; ++i) {
          const uint32_t c = lane + i * 32u;
          const float qv = c < p.dim ? as_float(q[c]) * q_scale : 0.0f, kv = c < p.dim ? as_float(k[c]) : 0.0f;
          chunk.q[t][c] = qv;
          chunk.k[t][c] = kv;
          dot = fmaf(qv, kv, dot);
        }
        if (!MEMORY) {
          dot = warp_sum(dot);
          if (lane == 0) chunk.extra[t] = dot;
        }
        if (lane < kSlice) {
          const uint32_t column = slice * kSlice + lane;
          chunk.v[t][lane] = column < p.vdim ? as_float(value[row * p.v_stride + p.v_column + head * p.vdim + column]) : 0.0f;
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
          if (present) chunk.extra[lane] = expf(-m);
          top = __shfl_sync(0xffffffffu, m, count - 1u);
        }
        if (present) {
          chunk.first[lane] = a;
          chunk.second[lane] = b;
        }
      }
    };
    auto write_out = [&](uint32_t index) {
      const ScanChunk<R4>& chunk = chunks[index & 1u];
      const uint32_t t0 = index * kChunk, count = min(kChunk, p.tokens - t0);
      for (uint32_t i = thread; i < count * kSlice; i += kProducerWarps * 32u) {
        const uint32_t t = i / kSlice, column = slice * kSlice + i % kSlice;
        float o = chunk.out[t][i % kSlice];
        if (MEMORY) o /= fmaxf(fabsf(chunk.norm_dot[t]), chunk.extra[t]) + 1e-6f;
        if (column < p.vdim) out[((row0 + t0 + t) * p.heads + head) * p.vdim + column] = o;
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
    const uint32_t column = threadIdx.x / kLanes, part = threadIdx.x % kLanes;
    const bool is_norm = MEMORY && column >= kSlice;  // the extra warp: its first eight lanes carry n
    const bool active = is_norm ? column == kSlice : slice * kSlice + column < p.vdim;
    float* home = state + (is_norm ? layout.norm(head, slice)
                                   : layout.matrix(head) + (size_t)(active ? slice * kSlice + column : 0u) * p.dim);
    float4 s[R4];
#pragma unroll
    for (int i = 0; i < R4; ++i) {
      const uint32_t c = i * 32u + part * 4u;
      s[i] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (active && !fresh) {
        if (c < p.dim) s[i].x = home[c];
        if (c + 1u < p.dim) s[i].y = home[c + 1u];
        if (c + 2u < p.dim) s[i].z = home[c + 2u];
        if (c + 3u < p.dim) s[i].w = home[c + 3u];
      }
    }
    __syncthreads();
    for (uint32_t index = 0; index < chunk_count; ++index) {
      ScanChunk<R4>& chunk = chunks[index & 1u];
      const uint32_t count = min(kChunk, p.tokens - index * kChunk);
#pragma unroll 2
      for (uint32_t t = 0; t < count; ++t) {
        const float4* q = reinterpret_cast<const float4*>(chunk.q[t]) + part;
        const float4* k = reinterpret_cast<const float4*>(chunk.k[t]) + part;
        const float keep = chunk.first[t];
        if (MEMORY) {
          const float write = chunk.second[t] * (is_norm ? 1.0f : chunk.v[t][column % kSlice]);
          float o = 0.0f, o2 = 0.0f;
#pragma unroll
          for (int i = 0; i < R4; ++i) {
            const float4 kk = k[i * 8], qq = q[i * 8];
            s[i].x = fmaf(kk.x, write, s[i].x * keep);
            s[i].y = fmaf(kk.y, write, s[i].y * keep);
            s[i].z = fmaf(kk.z, write, s[i].z * keep);
            s[i].w = fmaf(kk.w, write, s[i].w * keep);
            o = fmaf(s[i].x, qq.x, o);
            o2 = fmaf(s[i].y, qq.y, o2);
            o = fmaf(s[i].z, qq.z, o);
            o2 = fmaf(s[i].w, qq.w, o2);
          }
          o += o2;
          o += __shfl_xor_sync(0xffffffffu, o, 1);
          o += __shfl_xor_sync(0xffffffffu, o, 2);
          o += __shfl_xor_sync(0xffffffffu, o, 4);
          if (part == 0) {
            if (!is_norm) chunk.out[t][column] = o;
            else if (active) chunk.norm_dot[t] = o;
          }
        } else {
          float4 kk[R4];
          float with_key = 0.0f, with_key2 = 0.0f, with_query = 0.0f, with_query2 = 0.0f;
#pragma unroll
          for (int i = 0; i < R4; ++i) {
            kk[i] = k[i * 8];
            with_key = fmaf(s[i].x, kk[i].x, with_key);
            with_key2 = fmaf(s[i].y, kk[i].y, with_key2);
            with_key = fmaf(s[i].z, kk[i].z, with_key);
            with_key2 = fmaf(s[i].w, kk[i].w, with_key2);
          }
#pragma unroll
          for (int i = 0; i < R4; ++i) {
            const float4 qq = q[i * 8];
            with_query = fmaf(s[i].x, qq.x, with_query);
            with_query2 = fmaf(s[i].y, qq.y, with_query2);
            with_query = fmaf(s[i].z, qq.z, with_query);
            with_query2 = fmaf(s[i].w, qq.w, with_query2);
          }
          with_key += with_key2;
          with_query += with_query2;
#pragma unroll
          for (int offset = 1; offset < (int)kLanes; offset <<= 1) {
            with_key += __shfl_xor_sync(0xffffffffu, with_key, offset);
            with_query += __shfl_xor_sync(0xffffffffu, with_query, offset);
          }
          const float update = chunk.second[t] * (chunk.v[t][column] - keep * with_key);
#pragma unroll
          for (int i = 0; i < R4; ++i) {
            s[i].x = fmaf(kk[i].x, update, s[i].x * keep);
            s[i].y = fmaf(kk[i].y, update, s[i].y * keep);
            s[i].z = fmaf(kk[i].z, update, s[i].z * keep);
            s[i].w = fmaf(kk[i].w, update, s[i].w * keep);
          }
          if (part == 0) chunk.out[t][column] = fmaf(update, chunk.extra[t], keep * with_query);
        }
      }
      __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < R4; ++i) {
      const uint32_t c = i * 32u + part * 4u;
      if (!active) continue;
      if (c < p.dim) home[c] = s[i].x;
      if (c + 1u < p.dim) home[c + 1u] = s[i].y;
      if (c + 2u < p.dim) home[c + 2u] = s[i].z;
      if (c + 3u < p.dim) home[c + 3u] = s[i].w;
    }
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
  const uint32_t quads = (p.dim + 31u) / 32u;
  if (quads <= 1u) return run(scan_kernel<TQ, MEMORY, 1>, 2 * sizeof(ScanChunk<1>));
  if (quads <= 2u) return run(scan_kernel<TQ, MEMORY, 2>, 2 * sizeof(ScanChunk<2>));
  if (quads <= 3u) return run(scan_kernel<TQ, MEMORY, 3>, 2 * sizeof(ScanChunk<3>));
  if (quads <= 4u) return run(scan_kernel<TQ, MEMORY, 4>, 2 * sizeof(ScanChunk<4>));
  if (quads <= 6u) return run(scan_kernel<TQ, MEMORY, 6>, 2 * sizeof(ScanChunk<6>));
  return run(scan_kernel<TQ, MEMORY, 8>, 2 * sizeof(ScanChunk<8>));
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
  };
  *count = sizeof(table) / sizeof(table[0]);
  return table;
}

}  // namespace llmopt
