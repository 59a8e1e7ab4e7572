// Causal attention over a cache of unquantised rows (T: bfloat16 or float):
//   llmopt_row_attention_{bf16,f32}
// A sequence's token p sits in pool row slots[sequence row][p]; a pool row holds, per attention layer, the
// kv_heads key vectors (size dim) and value vectors (size vdim, which may differ).  The rows of the step's
// own tokens are in the pool already.  Row t of a sequence sees keys 0 .. past + t; with a `window` only the
// last `window` of them (its own included) and the first `keep_first` of the sequence.  With `softcap` a score
// becomes softcap * tanh(score / softcap).  With `sink` the softmax denominator counts one more score of zero that
// has no value.  With `gate_stride` the read-out is multiplied by the sigmoid of the row's gate columns.
// Queries and gates are read where the projections left them: row stride, first column.
//
// Kernels behind the names:
//  * bf16, at most 16 (query head, token) rows per key/value head (decode): split over the keys;
//    the query heads of a group ride in the 16 rows of one MMA tile, four warps walk over 16-key tiles
//    with private cp.async rings.  The last CTA of a (sequence, key/value head) to arrive merges the
//    splits in split order.
//  * bf16, more rows (prompts): 64 query tokens of one head per CTA, 64-key tiles double-buffered with
//    cp.async, online softmax in fp32, P rounded to bfloat16 for P V.
//  * fp32, and head sizes that are no whole 16-byte vectors: one warp per (row, head).
#include "element.cuh"

namespace llmopt {

uint32_t* context_device_error(Context* ctx);

namespace {

struct RowAttentionParams {
  uint32_t sequences, tokens, heads, kv_heads, dim, vdim;
  uint32_t token_stride, key_offset, value_offset;  // in elements
  uint32_t table_stride, table_rows, pool_rows;
  uint32_t sink, splits;
  float scale, softcap;        // 0: scores are not capped
  uint32_t window, keep_first; // 0: no window
  uint32_t query_stride, query_column, gate_stride, gate_column;  // in elements; gate_stride 0: no gate
  uint32_t weights32;  // softmax weights meet the values in 32 bits (two bfloat16 parts), not rounded to bfloat16
  bool extended() const { return weights32 || window || softcap > 0.0f || gate_stride; }
};

constexpr float kLog2e = 1.4426950408889634f;
constexpr float kLowest = -1.0e30f;
constexpr float kBoundedCap = 40.0f;  // e^40 and e^-40, and sums of many of them, are ordinary fp32 numbers

struct KeyRows {  // rows of one sequence
  const uint32_t* slots;
  uint32_t limit, pool_rows;
  // pool row of key `position`; an index outside the table or the pool reads row 0 and is reported
  __device__ __forceinline__ uint32_t operator()(uint32_t position, uint32_t* error_word) const {
    const uint32_t slot = position < limit ? slots[position] : pool_rows;
    if (slot < pool_rows) return slot;
    if (error_word) atomicExch(error_word, 1u);
    return 0u;
  }
};
__device__ __forceinline__ KeyRows key_rows(const RowAttentionParams& p, const uint32_t* table, uint32_t row) {
  const bool present = row < p.table_rows;
  return {table + (present ? (size_t)row * p.table_stride : 0u), present ? p.table_stride : 0u, p.pool_rows};
}

// EXTENDED kernels know windows, caps and gates, and keep the softmax weights in 32 bits; the others compile without.

// The keys a run of rows sees, positions first .. last of them: the kept ones, then those from `begin` on.
template <bool EXTENDED>
struct Visible {
  uint32_t kept, begin, end;
  __device__ __forceinline__ Visible(const RowAttentionParams& p, uint32_t first, uint32_t last) {
    end = last + 1u;
    begin = EXTENDED && p.window && first + 1u > p.window ? first + 1u - p.window : 0u;
    kept = EXTENDED && p.window ? min(p.keep_first, begin) : 0u;
  }
  __device__ __forceinline__ uint32_t count() const { return kept + end - begin; }
  __device__ __forceinline__ uint32_t position(uint32_t index) const { return index < kept ? index : index - kept + begin; }
};
template <bool EXTENDED>
__device__ __forceinline__ bool sees(const RowAttentionParams& p, uint32_t position, uint32_t key) {
  return key <= position && (!EXTENDED || !p.window || position - key < p.window || key < p.keep_first);
}

// Factor of a read-out.
template <bool EXTENDED, typename T>
__device__ __forceinline__ float gate_of(const RowAttentionParams& p, const T* gate, size_t row, uint32_t head, uint32_t column) {
  return EXTENDED && p.gate_stride ? sigmoid_f32(as_float(gate[row * p.gate_stride + p.gate_column + head * p.vdim + column])) : 1.0f;
}

// ---- one warp per (row, head) --------------------------------------------------------------------
template <typename T, int SEGMENTS>
__global__ void __launch_bounds__(128) attention_rows_kernel(const T* query, const T* pool, const uint32_t* table,
                                                             const uint32_t* past, const uint32_t* sequence_rows, T* out,
                                                             const T* gate, RowAttentionParams p, uint32_t* error_word) {
  grid_chain_prologue();
  const uint32_t lane = threadIdx.x & 31u, item = blockIdx.x * 4u + (threadIdx.x >> 5);
  if (item >= p.sequences * p.tokens * p.heads) return;
  const uint32_t row = item / p.heads, head = item % p.heads, sequence = row / p.tokens;
  const uint32_t kv_head = head / (p.heads / p.kv_heads);
  const uint32_t position = past[sequence] + row % p.tokens;
  const Visible<true> visible(p, position, position);
  const KeyRows rows = key_rows(p, table, sequence_rows[sequence]);
  float q[SEGMENTS], o[SEGMENTS];
#pragma unroll
  for (int s = 0; s < SEGMENTS; ++s) {
    const uint32_t c = lane + s * 32u;
    q[s] = c < p.dim ? as_float(query[(size_t)row * p.query_stride + p.query_column + head * p.dim + c]) : 0.0f;
    o[s] = 0.0f;
  }
  float top = p.sink ? 0.0f : kLowest, total = p.sink ? 1.0f : 0.0f;
  for (uint32_t index = 0; index < visible.count(); ++index) {
    const T* cached = pool + (size_t)rows(visible.position(index), error_word) * p.token_stride;
    const T* k = cached + p.key_offset + kv_head * p.dim;
    const T* v = cached + p.value_offset + kv_head * p.vdim;
    float score = 0.0f;
#pragma unroll
    for (int s = 0; s < SEGMENTS; ++s) {
      const uint32_t c = lane + s * 32u;
      if (c < p.dim) score = fmaf(q[s], as_float(k[c]), score);
    }
    score = warp_sum(score) * p.scale;
    if (p.softcap > 0.0f) score = p.softcap * tanhf(score / p.softcap);
    const float next = fmaxf(top, score), keep = expf(top - next), weight = expf(score - next);
    top = next;
    total = total * keep + weight;
#pragma unroll
    for (int s = 0; s < SEGMENTS; ++s) {
      const uint32_t c = lane + s * 32u;
      if (c < p.vdim) o[s] = o[s] * keep + weight * as_float(v[c]);
    }
  }
#pragma unroll
  for (int s = 0; s < SEGMENTS; ++s) {
    const uint32_t c = lane + s * 32u;
    if (c < p.vdim) out[(size_t)item * p.vdim + c] = from_float<T>(o[s] / total * gate_of<true>(p, gate, row, head, c));
  }
}

// ---- tensor-core pieces --------------------------------------------------------------------------
__device__ __forceinline__ void ldmatrix_x4(uint32_t (&r)[4], const void* shared_address) {
  const uint32_t address = (uint32_t)__cvta_generic_to_shared(shared_address);
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(address)
               : "memory");
}
__device__ __forceinline__ void ldmatrix_x4_trans(uint32_t (&r)[4], const void* shared_address) {
  const uint32_t address = (uint32_t)__cvta_generic_to_shared(shared_address);
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(address)
               : "memory");
}
__device__ __forceinline__ void mma_bf16(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
      : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void copy_async_16(void* shared_target, const void* source, uint32_t bytes) {
  const uint32_t address = (uint32_t)__cvta_generic_to_shared(shared_target);
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(address), "l"(source), "r"(bytes) : "memory");
}
__device__ __forceinline__ float exp2_approx(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__host__ __device__ constexpr uint32_t round16(uint32_t v) { return (v + 15u) & ~15u; }

// Online softmax of one warp's 16 rows (this lane: rows r and r + 8) over KEYS keys, scores already in units
// of log2 e with invisible ones at -inf; then O += P V from the value tile at `v_tile` (row stride v_stride).
// EXTENDED: P enters the product as its bfloat16 rounding plus the bfloat16 rounding of what that leaves.
template <int KEYS, int DV, bool EXTENDED>
struct Softmax {
  float top[2], total[2], out[DV / 8][4];
  bool bounded;  // capped scores: no maximum has to be taken off
  __device__ __forceinline__ explicit Softmax(const RowAttentionParams& p)
      : bounded(EXTENDED && p.softcap > 0.0f && p.softcap <= kBoundedCap) {
    top[0] = top[1] = bounded ? 0.0f : kLowest;
    total[0] = total[1] = 0.0f;
#pragma unroll
    for (int t = 0; t < DV / 8; ++t)
#pragma unroll
      for (int i = 0; i < 4; ++i) out[t][i] = 0.0f;
  }
  __device__ __forceinline__ void raise_maximum(const float (&score)[KEYS / 8][4]) {
    float next[2] = {top[0], top[1]};
#pragma unroll
    for (int j = 0; j < KEYS / 8; ++j)
#pragma unroll
      for (int i = 0; i < 4; ++i) next[i >> 1] = fmaxf(next[i >> 1], score[j][i]);
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      next[h] = fmaxf(next[h], __shfl_xor_sync(0xffffffffu, next[h], 1));
      next[h] = fmaxf(next[h], __shfl_xor_sync(0xffffffffu, next[h], 2));
      const float keep = exp2_approx(top[h] - next[h]);
      top[h] = next[h];
      total[h] *= keep;
#pragma unroll
      for (int t = 0; t < DV / 8; ++t) {
        out[t][2 * h] *= keep;
        out[t][2 * h + 1] *= keep;
      }
    }
  }
  __device__ __forceinline__ void absorb(float (&score)[KEYS / 8][4], const bf16* v_tile, uint32_t v_stride, uint32_t lane) {
    if (!bounded) raise_maximum(score);
    uint32_t weights[KEYS / 16][4], rests[EXTENDED ? KEYS / 16 : 1][4];
#pragma unroll
    for (int j = 0; j < KEYS / 8; ++j) {
      float e[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) e[i] = exp2_approx(score[j][i] - top[i >> 1]);
      total[0] += e[0] + e[1];
      total[1] += e[2] + e[3];
      const __nv_bfloat162 low = __floats2bfloat162_rn(e[0], e[1]), high = __floats2bfloat162_rn(e[2], e[3]);
      weights[j >> 1][(j & 1) * 2] = *reinterpret_cast<const uint32_t*>(&low);
      weights[j >> 1][(j & 1) * 2 + 1] = *reinterpret_cast<const uint32_t*>(&high);
      if (EXTENDED) {
        const __nv_bfloat162 low_rest = __floats2bfloat162_rn(e[0] - __low2float(low), e[1] - __high2float(low));
        const __nv_bfloat162 high_rest = __floats2bfloat162_rn(e[2] - __low2float(high), e[3] - __high2float(high));
        rests[EXTENDED ? j >> 1 : 0][(j & 1) * 2] = *reinterpret_cast<const uint32_t*>(&low_rest);
        rests[EXTENDED ? j >> 1 : 0][(j & 1) * 2 + 1] = *reinterpret_cast<const uint32_t*>(&high_rest);
      }
    }
#pragma unroll
    for (int s = 0; s < KEYS / 16; ++s)
#pragma unroll
      for (int t = 0; t < DV / 16; ++t) {
        uint32_t b[4];
        ldmatrix_x4_trans(b, v_tile + (16 * s + (lane & 7u) + ((lane >> 3) & 1u) * 8u) * v_stride + 16 * t + (lane >> 4) * 8u);
        mma_bf16(out[2 * t], weights[s], b[0], b[1]);
        mma_bf16(out[2 * t + 1], weights[s], b[2], b[3]);
        if (EXTENDED) {
          mma_bf16(out[2 * t], rests[EXTENDED ? s : 0], b[0], b[1]);
          mma_bf16(out[2 * t + 1], rests[EXTENDED ? s : 0], b[2], b[3]);
        }
      }
  }
};

// A raw score in units of log2 e; with a cap c, c tanh(s / c) = c - 2 c / (e^(2 s / c) + 1).
template <bool EXTENDED>
struct ScoreScale {
  float scale, cap;  // cap 0: none
  __device__ __forceinline__ explicit ScoreScale(const RowAttentionParams& p)
      : scale((EXTENDED && p.softcap > 0.0f ? p.scale / p.softcap * 2.0f : p.scale) * kLog2e), cap(p.softcap * kLog2e) {}
  __device__ __forceinline__ float operator()(float raw) const {
    const float score = raw * scale;
    return EXTENDED && cap > 0.0f ? fmaf(-2.0f * cap, __fdividef(1.0f, exp2_approx(score) + 1.0f), cap) : score;
  }
};

// 16 query rows (this warp's, at q_rows, row stride `stride`) against KEYS key rows.  DK > 0: the query
// fragments are in registers; DK == 0: they are read from shared memory for every 16 dimensions.
template <int KEYS, int DK>
__device__ __forceinline__ void scores(float (&score)[KEYS / 8][4], const uint32_t (*q_frag)[4], const bf16* q_rows,
                                       const bf16* k_tile, uint32_t stride, uint32_t steps, uint32_t lane) {
#pragma unroll
  for (int j = 0; j < KEYS / 8; ++j)
#pragma unroll
    for (int i = 0; i < 4; ++i) score[j][i] = 0.0f;
  auto step = [&](const uint32_t (&a)[4], uint32_t s) {
#pragma unroll
    for (int j = 0; j < KEYS / 16; ++j) {
      uint32_t b[4];
      ldmatrix_x4(b, k_tile + (16 * j + (lane & 7u) + (lane >> 4) * 8u) * stride + 16 * s + ((lane >> 3) & 1u) * 8u);
      mma_bf16(score[2 * j], a, b[0], b[1]);
      mma_bf16(score[2 * j + 1], a, b[2], b[3]);
    }
  };
  if (DK > 0) {
#pragma unroll
    for (int s = 0; s < DK / 16; ++s) step(q_frag[s], s);
  } else {
    for (uint32_t s = 0; s < steps; ++s) {
      uint32_t a[4];
      ldmatrix_x4(a, q_rows + ((lane & 7u) + ((lane >> 3) & 1u) * 8u) * stride + 16 * s + (lane >> 4) * 8u);
      step(a, s);
    }
  }
}

// ---- prompts -------------------------------------------------------------------------------------
constexpr uint32_t kQueryTile = 64;
// Keys per tile, and CTAs per SM to compile for (0: no bound): with smaller tiles a third CTA fits, which hides more of the
// longer way from a score to its weight.
__host__ __device__ constexpr uint32_t key_tile(int DK, bool EXTENDED) { return EXTENDED && DK == 128 ? 32u : 64u; }
constexpr int prompt_ctas(int DK, bool EXTENDED) { return DK != 128 ? 0 : EXTENDED ? 3 : 2; }

template <int DK, int DV, bool EXTENDED>
__global__ void __launch_bounds__(128, prompt_ctas(DK, EXTENDED)) attention_prompt_kernel(const bf16* query, const bf16* pool, const uint32_t* table,
                                                               const uint32_t* past_lengths, const uint32_t* sequence_rows,
                                                               bf16* out, const bf16* gate, RowAttentionParams p, uint32_t* error_word) {
  constexpr uint32_t kKeyTile = key_tile(DK, EXTENDED), kPerKey = 128u / kKeyTile;  // threads that fetch a key
  grid_chain_prologue();
  extern __shared__ __align__(16) unsigned char attention_shared[];
  const uint32_t padded = DK > 0 ? DK : round16(p.dim), k_stride = padded + 8u, v_stride = DV + 8u;
  bf16* q_tile = reinterpret_cast<bf16*>(attention_shared);
  bf16* k_tiles = q_tile + kQueryTile * k_stride;
  bf16* v_tiles = k_tiles + 2u * kKeyTile * k_stride;
  // the last query tiles see the most keys: they are scheduled first
  const uint32_t q0 = (gridDim.x - 1u - blockIdx.x) * kQueryTile, head = blockIdx.y, sequence = blockIdx.z;
  const uint32_t kv_head = head / (p.heads / p.kv_heads);
  const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31u, r = lane >> 2, c = lane & 3u;
  const uint32_t past = past_lengths[sequence];
  const KeyRows rows = key_rows(p, table, sequence_rows[sequence]);
  const uint32_t key_end = past + min(q0 + kQueryTile, p.tokens);
  // whole key tiles: those with kept keys, then from the first row's window on
  const Visible<EXTENDED> visible(p, past + q0, key_end - 1u);
  const uint32_t kept_tiles = (visible.kept + kKeyTile - 1u) / kKeyTile;
  const uint32_t skipped = max(visible.begin / kKeyTile, kept_tiles) - kept_tiles;
  const uint32_t tiles = (key_end + kKeyTile - 1u) / kKeyTile - skipped;
  auto first_key = [&](uint32_t tile) { return (tile < kept_tiles ? tile : tile + skipped) * kKeyTile; };
  const uint32_t k_chunks = padded / 8u, v_chunks = DV / 8u;

  auto fetch_tile = [&](uint32_t tile) {
    if (tile < tiles) {
      bf16* k_tile = k_tiles + (tile & 1u) * kKeyTile * k_stride;
      bf16* v_tile = v_tiles + (tile & 1u) * kKeyTile * v_stride;
      // a few threads per key row: one slot look-up, a share of the chunks each
      const uint32_t key = threadIdx.x / kPerKey, share = threadIdx.x % kPerKey, position = first_key(tile) + key;
      const bool present = position < key_end;
      const bf16* cached = pool + (size_t)(present ? rows(position, error_word) : 0u) * p.token_stride;
      const bf16* k = cached + p.key_offset + kv_head * p.dim;
      const bf16* v = cached + p.value_offset + kv_head * p.vdim;
      for (uint32_t chunk = share; chunk < k_chunks; chunk += kPerKey) {
        const bool there = present && chunk * 8u < p.dim;
        copy_async_16(k_tile + key * k_stride + chunk * 8u, there ? k + chunk * 8u : pool, there ? 16u : 0u);
      }
      for (uint32_t chunk = share; chunk < v_chunks; chunk += kPerKey) {
        const bool there = present && chunk * 8u < p.vdim;
        copy_async_16(v_tile + key * v_stride + chunk * 8u, there ? v + chunk * 8u : pool, there ? 16u : 0u);
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  fetch_tile(0);
  for (uint32_t index = threadIdx.x; index < kQueryTile * k_chunks; index += 128u) {
    const uint32_t row = index / k_chunks, chunk = index % k_chunks;
    uint4 data = make_uint4(0u, 0u, 0u, 0u);
    if (q0 + row < p.tokens && chunk * 8u < p.dim)
      data = *reinterpret_cast<const uint4*>(query + ((size_t)sequence * p.tokens + q0 + row) * p.query_stride +
                                             p.query_column + head * p.dim + chunk * 8u);
    *reinterpret_cast<uint4*>(q_tile + row * k_stride + chunk * 8u) = data;
  }
  __syncthreads();
  const bf16* q_rows = q_tile + warp * 16u * k_stride;
  uint32_t q_frag[DK > 0 ? DK / 16 : 1][4];
  if (DK > 0) {
#pragma unroll
    for (int s = 0; s < DK / 16; ++s)
      ldmatrix_x4(q_frag[s], q_rows + ((lane & 7u) + ((lane >> 3) & 1u) * 8u) * k_stride + 16 * s + (lane >> 4) * 8u);
  }
  const uint32_t row_low = q0 + warp * 16u + r;  // and row_low + 8
  const ScoreScale<EXTENDED> score_of(p);
  Softmax<kKeyTile, DV, EXTENDED> state(p);

  for (uint32_t tile = 0; tile < tiles; ++tile) {
    const uint32_t k0 = first_key(tile);
    fetch_tile(tile + 1u);  // into the other buffer, which the previous iteration's last barrier released
    asm volatile("cp.async.wait_group 1;" ::: "memory");
    __syncthreads();
    float score[kKeyTile / 8][4];
    scores<kKeyTile, DK>(score, q_frag, q_rows, k_tiles + (tile & 1u) * kKeyTile * k_stride, k_stride, padded / 16u, lane);
    const uint32_t first_row = past + q0 + warp * 16u;  // of this warp
    const bool all_visible = k0 + kKeyTile - 1u <= first_row &&
                             (!EXTENDED || !p.window || first_row + 15u - k0 < p.window || k0 + kKeyTile <= p.keep_first);
#pragma unroll
    for (int j = 0; j < (int)kKeyTile / 8; ++j)
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const uint32_t token = row_low + ((i & 2) ? 8u : 0u), key = k0 + 8u * j + 2u * c + (i & 1);
        score[j][i] = all_visible || sees<EXTENDED>(p, past + token, key) ? score_of(score[j][i]) : -INFINITY;
      }
    state.absorb(score, v_tiles + (tile & 1u) * kKeyTile * v_stride, v_stride, lane);
    __syncthreads();  // every warp is done with this buffer before the next iteration's fetch refills it
  }
  asm volatile("cp.async.wait_all;" ::: "memory");
#pragma unroll
  for (int h = 0; h < 2; ++h) {
    float total = state.total[h];
    total += __shfl_xor_sync(0xffffffffu, total, 1);
    total += __shfl_xor_sync(0xffffffffu, total, 2);
    float scale = 1.0f;
    if (p.sink) {  // bring both to the larger of the two maxima
      const float top = fmaxf(state.top[h], 0.0f);
      scale = exp2f(state.top[h] - top);
      total = total * scale + exp2f(-top);
    }
    scale /= total;
    const uint32_t token = row_low + h * 8u;
    if (token >= p.tokens) continue;
    const size_t row = (size_t)sequence * p.tokens + token;
    bf16* target = out + (row * p.heads + head) * p.vdim;
#pragma unroll
    for (int t = 0; t < DV / 8; ++t) {
      const uint32_t column = 8u * t + 2u * c;
      if (column < p.vdim)  // vdim is a multiple of eight
        *reinterpret_cast<__nv_bfloat162*>(target + column) =
            __floats2bfloat162_rn(state.out[t][2 * h] * scale * gate_of<EXTENDED>(p, gate, row, head, column),
                                  state.out[t][2 * h + 1] * scale * gate_of<EXTENDED>(p, gate, row, head, column + 1u));
    }
  }
}

// ---- decode --------------------------------------------------------------------------------------
constexpr uint32_t kWarpKeys = 16, kDecodeWarps = 4, kDecodeStages = 3, kMostSplits = 64;

// Record of one split: 16 maxima, 16 denominators, 16 x DV sums.
template <int DV>
__host__ __device__ constexpr uint32_t record_floats() { return 32u + 16u * DV; }

template <int DK, int DV, bool EXTENDED>
__global__ void __launch_bounds__(128) attention_decode_kernel(const bf16* query, const bf16* pool, const uint32_t* table,
                                                               const uint32_t* past_lengths, const uint32_t* sequence_rows,
                                                               bf16* out, const bf16* gate, uint32_t* counters, float* records,
                                                               RowAttentionParams p, uint32_t* error_word) {
  grid_chain_prologue();
  extern __shared__ __align__(16) unsigned char attention_shared[];
  const uint32_t padded = DK > 0 ? DK : round16(p.dim), k_stride = padded + 8u, v_stride = DV + 8u;
  const uint32_t stage_elements = kWarpKeys * (k_stride + v_stride);
  bf16* q_tile = reinterpret_cast<bf16*>(attention_shared);
  const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31u, r = lane >> 2, c = lane & 3u;
  bf16* ring = q_tile + 16u * k_stride + warp * kDecodeStages * stage_elements;
  const uint32_t split = blockIdx.x, kv_head = blockIdx.y, sequence = blockIdx.z;
  const uint32_t group = p.heads / p.kv_heads, query_rows = p.tokens * group;
  const uint32_t past = past_lengths[sequence];
  const Visible<EXTENDED> visible(p, past, past + p.tokens - 1u);
  const uint32_t keys = visible.count();
  const KeyRows rows = key_rows(p, table, sequence_rows[sequence]);
  // whole 64-key stretches per split
  const uint32_t stretch = (kWarpKeys * kDecodeWarps);
  const uint32_t per_split = ((keys + p.splits - 1u) / p.splits + stretch - 1u) / stretch * stretch;
  const uint32_t begin = min(split * per_split, keys), end = min(begin + per_split, keys);
  const uint32_t tiles = (end - begin + stretch - 1u) / stretch;  // of this warp
  const uint32_t k_chunks = padded / 8u, v_chunks = DV / 8u;

  auto fetch_tile = [&](uint32_t tile) {
    if (tile < tiles) {
      bf16* k_tile = ring + (tile % kDecodeStages) * stage_elements;
      bf16* v_tile = k_tile + kWarpKeys * k_stride;
      const uint32_t key = lane >> 1, half = lane & 1u, index = begin + tile * stretch + warp * kWarpKeys + key;
      const bool present = index < end;
      const bf16* cached = pool + (size_t)(present ? rows(visible.position(index), error_word) : 0u) * p.token_stride;
      const bf16* k = cached + p.key_offset + kv_head * p.dim;
      const bf16* v = cached + p.value_offset + kv_head * p.vdim;
      for (uint32_t chunk = half; chunk < k_chunks; chunk += 2u) {
        const bool there = present && chunk * 8u < p.dim;
        copy_async_16(k_tile + key * k_stride + chunk * 8u, there ? k + chunk * 8u : pool, there ? 16u : 0u);
      }
      for (uint32_t chunk = half; chunk < v_chunks; chunk += 2u) {
        const bool there = present && chunk * 8u < p.vdim;
        copy_async_16(v_tile + key * v_stride + chunk * 8u, there ? v + chunk * 8u : pool, there ? 16u : 0u);
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
#pragma unroll
  for (uint32_t s = 0; s + 1u < kDecodeStages; ++s) fetch_tile(s);
  for (uint32_t index = threadIdx.x; index < 16u * k_chunks; index += 128u) {
    const uint32_t row = index / k_chunks, chunk = index % k_chunks;
    uint4 data = make_uint4(0u, 0u, 0u, 0u);
    if (row < query_rows && chunk * 8u < p.dim)
      data = *reinterpret_cast<const uint4*>(query + ((size_t)sequence * p.tokens + row / group) * p.query_stride + p.query_column +
                                             (kv_head * group + row % group) * p.dim + chunk * 8u);
    *reinterpret_cast<uint4*>(q_tile + row * k_stride + chunk * 8u) = data;
  }
  __syncthreads();
  uint32_t q_frag[DK > 0 ? DK / 16 : 1][4];
  if (DK > 0) {
#pragma unroll
    for (int s = 0; s < DK / 16; ++s)
      ldmatrix_x4(q_frag[s], q_tile + ((lane & 7u) + ((lane >> 3) & 1u) * 8u) * k_stride + 16 * s + (lane >> 4) * 8u);
  }
  const uint32_t token_low = r / group, token_high = (r + 8u) / group;
  const ScoreScale<EXTENDED> score_of(p);
  Softmax<kWarpKeys, DV, EXTENDED> state(p);
  for (uint32_t tile = 0; tile < tiles; ++tile) {
    fetch_tile(tile + kDecodeStages - 1u);
    asm volatile("cp.async.wait_group %0;" ::"n"(kDecodeStages - 1) : "memory");
    __syncwarp();  // the other lanes' copies of this tile have landed too
    const bf16* k_tile = ring + (tile % kDecodeStages) * stage_elements;
    const uint32_t k0 = begin + tile * stretch + warp * kWarpKeys;
    float score[kWarpKeys / 8][4];
    scores<kWarpKeys, DK>(score, q_frag, q_tile, k_tile, k_stride, padded / 16u, lane);
#pragma unroll
    for (int j = 0; j < (int)kWarpKeys / 8; ++j)
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const uint32_t index = k0 + 8u * j + 2u * c + (i & 1);
        const bool seen = index < end && sees<EXTENDED>(p, past + ((i & 2) ? token_high : token_low), visible.position(index));
        score[j][i] = seen ? score_of(score[j][i]) : -INFINITY;
      }
    state.absorb(score, k_tile + kWarpKeys * k_stride, v_stride, lane);
    __syncwarp();
  }
  asm volatile("cp.async.wait_all;" ::: "memory");
#pragma unroll
  for (int h = 0; h < 2; ++h) {
    state.total[h] += __shfl_xor_sync(0xffffffffu, state.total[h], 1);
    state.total[h] += __shfl_xor_sync(0xffffffffu, state.total[h], 2);
  }
  __syncthreads();  // the rings are free: they carry the warps' results now

  constexpr uint32_t kRecord = record_floats<DV>();
  float* shared_records = reinterpret_cast<float*>(attention_shared);
  {
    float* mine = shared_records + warp * kRecord;
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      if (c == 0) {
        mine[r + 8 * h] = state.top[h];
        mine[16 + r + 8 * h] = state.total[h];
      }
#pragma unroll
      for (int t = 0; t < DV / 8; ++t)
        *reinterpret_cast<float2*>(mine + 32 + (r + 8 * h) * DV + 8 * t + 2 * c) =
            make_float2(state.out[t][2 * h], state.out[t][2 * h + 1]);
    }
  }
  __syncthreads();
  float* record = records + (((size_t)sequence * p.kv_heads + kv_head) * p.splits + split) * kRecord;
  const bool single = p.splits == 1u;
  for (uint32_t index = threadIdx.x; index < query_rows * DV; index += 128u) {
    const uint32_t row = index / DV, column = index % DV;
    float top = kLowest;
#pragma unroll
    for (uint32_t w = 0; w < kDecodeWarps; ++w) top = fmaxf(top, shared_records[w * kRecord + row]);
    float total = 0.0f, sum = 0.0f;
#pragma unroll
    for (uint32_t w = 0; w < kDecodeWarps; ++w) {
      const float weight = exp2f(shared_records[w * kRecord + row] - top);
      total += weight * shared_records[w * kRecord + 16 + row];
      sum += weight * shared_records[w * kRecord + 32 + row * DV + column];
    }
    if (single) {
      if (p.sink) {
        const float both = fmaxf(top, 0.0f), keep = exp2f(top - both);
        sum *= keep;
        total = total * keep + exp2f(-both);
      }
      const size_t token = (size_t)sequence * p.tokens + row / group;
      const uint32_t head = kv_head * group + row % group;
      if (column < p.vdim)
        out[(token * p.heads + head) * p.vdim + column] =
            __float2bfloat16_rn(sum / total * gate_of<EXTENDED>(p, gate, token, head, column));
    } else {
      record[32 + row * DV + column] = sum;
      if (column == 0) {
        record[row] = top;
        record[16 + row] = total;
      }
    }
  }
  if (single) return;

  // the last split of this (sequence, key/value head) to get here adds all of them, in split order
  __shared__ uint32_t is_last;
  __threadfence();
  __syncthreads();
  if (threadIdx.x == 0) {
    uint32_t* counter = counters + sequence * p.kv_heads + kv_head;
    const bool last = atomicAdd(counter, 1u) + 1u == p.splits;
    if (last) *counter = 0u;  // ready for the next launch
    is_last = last ? 1u : 0u;
  }
  __syncthreads();
  if (is_last == 0u) return;
  __threadfence();
  const float* first = records + ((size_t)sequence * p.kv_heads + kv_head) * p.splits * kRecord;
  const uint32_t used = (keys + per_split - 1u) / per_split;  // the others saw no key
  // weight of every split for every row, over the row's common denominator
  float* weights = shared_records;  // [query rows][used]
  for (uint32_t row = warp; row < query_rows; row += kDecodeWarps) {
    float top = p.sink ? 0.0f : kLowest;
    for (uint32_t s = lane; s < used; s += 32u) top = fmaxf(top, __ldcg(first + (size_t)s * kRecord + row));
    top = warp_max(top);
    float total = 0.0f;
    for (uint32_t s = lane; s < used; s += 32u) {
      const float weight = exp2f(__ldcg(first + (size_t)s * kRecord + row) - top);
      total += weight * __ldcg(first + (size_t)s * kRecord + 16 + row);
      weights[row * kMostSplits + s] = weight;
    }
    total = warp_sum(total) + (p.sink ? exp2f(-top) : 0.0f);
    __syncwarp();
    for (uint32_t s = lane; s < used; s += 32u) weights[row * kMostSplits + s] /= total;
  }
  __syncthreads();
  for (uint32_t index = threadIdx.x; index < query_rows * (DV / 4); index += 128u) {
    const uint32_t row = index / (DV / 4), column = index % (DV / 4) * 4u;
    const float* source = first + 32 + row * DV + column;
    float4 sum = make_float4(0.f, 0.f, 0.f, 0.f);
    uint32_t s = 0;
    for (; s + 8u <= used; s += 8u) {
      float4 part[8];
#pragma unroll
      for (int i = 0; i < 8; ++i) part[i] = __ldcg(reinterpret_cast<const float4*>(source + (size_t)(s + i) * kRecord));
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        const float weight = weights[row * kMostSplits + s + i];
        sum.x = fmaf(weight, part[i].x, sum.x);
        sum.y = fmaf(weight, part[i].y, sum.y);
        sum.z = fmaf(weight, part[i].z, sum.z);
        sum.w = fmaf(weight, part[i].w, sum.w);
      }
    }
    for (; s < used; ++s) {
      const float4 part = __ldcg(reinterpret_cast<const float4*>(source + (size_t)s * kRecord));
      const float weight = weights[row * kMostSplits + s];
      sum.x = fmaf(weight, part.x, sum.x);
      sum.y = fmaf(weight, part.y, sum.y);
      sum.z = fmaf(weight, part.z, sum.z);
      sum.w = fmaf(weight, part.w, sum.w);
    }
    if (column < p.vdim) {  // vdim is a multiple of eight
      const size_t token = (size_t)sequence * p.tokens + row / group;
      const uint32_t head = kv_head * group + row % group;
      sum.x *= gate_of<EXTENDED>(p, gate, token, head, column);
      sum.y *= gate_of<EXTENDED>(p, gate, token, head, column + 1u);
      sum.z *= gate_of<EXTENDED>(p, gate, token, head, column + 2u);
      sum.w *= gate_of<EXTENDED>(p, gate, token, head, column + 3u);
      store_four(out + (token * p.heads + head) * p.vdim + column, sum);
    }
  }
}

// ---- host ----------------------------------------------------------------------------------------
template <typename T>
int run_rows(const KernelArgs& args, const RowAttentionParams& p) {
  const size_t items = (size_t)p.sequences * p.tokens * p.heads;
  const uint32_t widest = p.dim > p.vdim ? p.dim : p.vdim;
  auto run = [&](auto kernel) {
    launch_kernel(args, kernel, dim3((uint32_t)((items + 3) / 4)), dim3(128), 0, (const T*)args.buffers[0],
                  (const T*)args.buffers[1], (const uint32_t*)args.buffers[2], (const uint32_t*)args.buffers[3],
                  (const uint32_t*)args.buffers[4], (T*)args.buffers[5], (const T*)args.buffers[7], p, context_device_error(args.ctx));
  };
  if (widest <= 64u) run(attention_rows_kernel<T, 2>);
  else if (widest <= 128u) run(attention_rows_kernel<T, 4>);
  else if (widest <= 256u) run(attention_rows_kernel<T, 8>);
  else if (widest <= 512u) run(attention_rows_kernel<T, 16>);
  else return fail(args, "head sizes above 512 are not supported");
  return check_launch(args);
}

template <int DK, int DV, bool EXTENDED>
int run_prompt(const KernelArgs& args, const RowAttentionParams& p) {
  const uint32_t padded = DK > 0 ? DK : round16(p.dim);
  constexpr uint32_t kKeyTile = key_tile(DK, EXTENDED);
  const uint32_t bytes = ((kQueryTile + 2u * kKeyTile) * (padded + 8u) + 2u * kKeyTile * (DV + 8u)) * 2u;
  auto kernel = attention_prompt_kernel<DK, DV, EXTENDED>;
  if (cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes) != cudaSuccess) {
    cudaGetLastError();
    return -1;
  }
  launch_kernel(args, kernel, dim3((p.tokens + kQueryTile - 1u) / kQueryTile, p.heads, p.sequences), dim3(128), bytes,
                (const bf16*)args.buffers[0], (const bf16*)args.buffers[1], (const uint32_t*)args.buffers[2],
                (const uint32_t*)args.buffers[3], (const uint32_t*)args.buffers[4], (bf16*)args.buffers[5],
                (const bf16*)args.buffers[7], p,
                context_device_error(args.ctx));
  return check_launch(args);
}

template <int DK, int DV, bool EXTENDED>
int run_decode(const KernelArgs& args, const RowAttentionParams& p) {
  const uint32_t padded = DK > 0 ? DK : round16(p.dim);
  uint32_t bytes = (16u * (padded + 8u) + kDecodeWarps * kDecodeStages * kWarpKeys * (padded + 8u + DV + 8u)) * 2u;
  const uint32_t merge = kDecodeWarps * record_floats<DV>() * 4u;
  if (bytes < merge) bytes = merge;
  const size_t heads = (size_t)p.sequences * p.kv_heads, counters = (heads * 4 + 255) / 256 * 256;
  LLMOPT_REQUIRE(p.splits <= kMostSplits, "at most 64 splits");
  LLMOPT_REQUIRE(p.splits == 1u || args.lengths[6] >= counters + heads * p.splits * record_floats<DV>() * 4,
                 "split scratch is too short");
  auto kernel = attention_decode_kernel<DK, DV, EXTENDED>;
  if (cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes) != cudaSuccess) {
    cudaGetLastError();
    return -1;
  }
  launch_kernel(args, kernel, dim3(p.splits, p.kv_heads, p.sequences), dim3(128), bytes, (const bf16*)args.buffers[0],
                (const bf16*)args.buffers[1], (const uint32_t*)args.buffers[2], (const uint32_t*)args.buffers[3],
                (const uint32_t*)args.buffers[4], (bf16*)args.buffers[5], (const bf16*)args.buffers[7],
                (uint32_t*)args.buffers[6],
                (float*)((uint8_t*)args.buffers[6] + counters), p, context_device_error(args.ctx));
  return check_launch(args);
}

template <int DK, int DV>
int run_tensor(const KernelArgs& args, const RowAttentionParams& p) {
  if (p.tokens * (p.heads / p.kv_heads) <= 16u)
    return p.extended() ? run_decode<DK, DV, true>(args, p) : run_decode<DK, DV, false>(args, p);
  return p.extended() ? run_prompt<DK, DV, true>(args, p) : run_prompt<DK, DV, false>(args, p);
}

int run_tensor_shapes(const KernelArgs& args, const RowAttentionParams& p) {
  if (p.dim == 128u && p.vdim == 128u) return run_tensor<128, 128>(args, p);
  if (p.dim == 64u && p.vdim == 64u) return run_tensor<64, 64>(args, p);
  if (p.vdim <= 32u) return run_tensor<0, 32>(args, p);
  if (p.vdim <= 64u) return run_tensor<0, 64>(args, p);
  if (p.vdim <= 128u) return run_tensor<0, 128>(args, p);
  return run_tensor<0, 256>(args, p);
}

// Buffers [query, pool, slot table, past, sequence rows, out, split scratch (counters zero between launches),
// gates (an absent one repeats the queries)].
template <typename T>
int launch_row_attention(const KernelArgs& args) {
  RowAttentionParams p;
  LLMOPT_REQUIRE(args.buffer_count == 8 && args.param_bytes == sizeof(p), "expects 8 buffers and 92 parameter bytes");
  memcpy(&p, args.params, sizeof(p));
  const size_t rows = (size_t)p.sequences * p.tokens, e = sizeof(T);
  LLMOPT_REQUIRE(p.heads > 0 && p.kv_heads > 0 && p.heads % p.kv_heads == 0 && p.dim > 0 && p.vdim > 0 && p.splits > 0,
                 "needs whole groups of query heads");
  LLMOPT_REQUIRE(p.key_offset + p.kv_heads * p.dim <= p.token_stride && p.value_offset + p.kv_heads * p.vdim <= p.token_stride,
                 "key or value segment lies outside the cache row");
  LLMOPT_REQUIRE(p.sequences <= 65535u && p.heads <= 65535u, "too many sequences or heads");
  LLMOPT_REQUIRE((size_t)p.query_column + p.heads * p.dim <= p.query_stride &&
                     (!p.gate_stride || (size_t)p.gate_column + p.heads * p.vdim <= p.gate_stride),
                 "query or gate columns lie outside the row");
  LLMOPT_REQUIRE(args.lengths[7] >= rows * p.gate_stride * e, "gate buffer is too short");
  LLMOPT_REQUIRE(args.lengths[0] >= rows * p.query_stride * e && args.lengths[5] >= rows * p.heads * p.vdim * e &&
                     args.lengths[1] >= (size_t)p.pool_rows * p.token_stride * e && p.pool_rows > 0 &&
                     args.lengths[2] >= (size_t)p.table_rows * p.table_stride * 4 &&
                     args.lengths[3] >= (size_t)p.sequences * 4 && args.lengths[4] >= (size_t)p.sequences * 4,
                 "buffer is too short");
  if (rows == 0) return 0;
  const bool vectors = e == 2 && p.dim % 8u == 0 && p.vdim % 8u == 0 && p.dim <= 256u && p.vdim <= 256u &&
                       p.query_stride % 8u == 0 && p.query_column % 8u == 0 && p.token_stride % 8u == 0 && p.key_offset % 8u == 0 && p.value_offset % 8u == 0 &&
                       ((uintptr_t)args.buffers[0] & 15u) == 0 && ((uintptr_t)args.buffers[1] & 15u) == 0;
  if (vectors) {
    const int status = run_tensor_shapes(args, p);
    if (status >= 0) return status;
  }
  return run_rows<T>(args, p);
}

}  // namespace

const NamedLauncher* row_attention_launchers(size_t* count) {
  static const NamedLauncher table[] = {
      {"llmopt_row_attention_bf16", launch_row_attention<bf16>},
      {"llmopt_row_attention_f32", launch_row_attention<float>},
  };
  *count = sizeof(table) / sizeof(table[0]);
  return table;
}

}  // namespace llmopt
