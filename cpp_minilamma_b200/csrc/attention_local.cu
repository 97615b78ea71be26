// Attention whose keys and values have head sizes of their own (d for queries and keys, dv for
// values), with an explicit score scale, an optional norm of the whole q and k projections, rotary
// encoding of the first `rot` dimensions of a head only, and a mask that is causal inside chunks:
// query i sees key j iff j <= i and j / chunk == i / chunk (chunk 0: every earlier key), and with a
// window w > 0 only keys j > i - w.  Chunks count from position 0 of the sequence, whatever portion of it
// a step brings.  Two further options: a query temperature (q at position p is multiplied by
// 1 + coef * ln(floor((p + 1) / every) + 1) before it is stored) and a sink in the softmax (one more term
// exp(0) in the denominator that carries no value, so a row's weights may sum to less than one).  The values
// may be the leading dv columns of the key rows (v_ld = d: a layer that caches one latent row per position and
// reads it as key and as value); otherwise they have pages of their own (v_ld = dv).
// A window may keep the sequence's first tokens (`keep_first`: key j < keep_first stays visible whatever its distance, at
// its own position), and a score may be capped smoothly (s <- cap * tanh(s / cap) after the scale).  A layer that reads
// another layer's keys and values prepares its queries only (`write_kv` 0).
//
// The projections may have biases and pass a short causal convolution over time, per channel of q, k and v, before the
// rotation (the last taps - 1 inputs of every sequence, biases included, are state; nothing comes before the first token).
//
// Kernels, for prompts and single tokens alike:
//   * prepare: one block per token.  q and k are each divided by the root mean square of their whole
//     projection (all heads at once) and multiplied by a weight, the pairs of the first `rot`
//     dimensions of every head are rotated by position * frequency (cos / sin from a table), q goes to
//     a buffer and k, v into the pages of the cache.  All arithmetic in float32.
//   * prepare behind a convolution: the same without norms; a thread owns four neighbouring channels (with their
//     partners where the rotation pairs them) and walks a run of rows, with taps and last inputs in registers; a
//     version of a channel a thread takes every other size.
//   * attend: one block per (token, kv head) and the query heads of its group.  Pages of keys and values pass
//     through shared memory; scores are float32 dot products over the head, the softmax runs online in
//     float32.  Any d and dv (16-byte copies where rows are whole 16-byte words).
#include "common.cuh"

namespace mll {

template <typename T>
struct Vec16;  // 16 bytes of T as floats
template <>
struct Vec16<float> {
  static __device__ __forceinline__ void load(const float* p, float* out) {
    const float4 v = *reinterpret_cast<const float4*>(p);
    out[0] = v.x; out[1] = v.y; out[2] = v.z; out[3] = v.w;
  }
};
template <>
struct Vec16<__nv_bfloat16> {
  static __device__ __forceinline__ void load(const __nv_bfloat16* p, float* out) {
    const uint4 v = *reinterpret_cast<const uint4*>(p);
    const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&v);
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const float2 f = __bfloat1622float2(h[i]);
      out[2 * i] = f.x;
      out[2 * i + 1] = f.y;
    }
  }
};

struct LocalPrepArgs {
  const void* qkv;        // [T, ld]: q (Hq * d), k (Hk * d), v (Hk * dv)
  const float* q_weight;  // [Hq * d] or null: no norm of the projections
  const float* k_weight;  // [Hk * d]
  const float* cos_table; // [max_pos, rot / 2] or null
  const float* sin_table;
  const int* tok_pos;
  const int* tok_seq;
  const int* seq_slot;
  const int* block_table;
  void* q_out;            // [T, Hq * d]
  void* k_cache;          // [pages, Hk, PAGE, d]
  void* v_cache;          // [pages, Hk, PAGE, dv]
  int ld, n_heads, n_kv_heads, d, dv, rot, interleaved, max_blocks;
  float eps;
  float q_temp_coef;      // query temperature: 0 and 0 for none
  int q_temp_every;
  int v_col;              // column of a row where the values begin: behind k, or k's own columns (values that are
                          // the keys as projected, before norm and rotation)
  int write_kv;           // 0: the row holds queries only; nothing goes to the cache (another layer's is read)
};

template <typename T>
__global__ void __launch_bounds__(256) local_prepare_kernel(LocalPrepArgs a) {
  __shared__ float scratch[32];
  const int t = blockIdx.x;
  const int d = a.d, nq = a.n_heads * d, nk = a.write_kv ? a.n_kv_heads * d : 0, nv = a.write_kv ? a.n_kv_heads * a.dv : 0;
  const T* row = (const T*)a.qkv + (size_t)t * a.ld;
  float fq = 1.f, fk = 1.f;
  if (a.q_weight) {
    float sq = 0.f, sk = 0.f;
    for (int i = threadIdx.x; i < nq; i += blockDim.x) {
      const float v = to_float(row[i]);
      sq += v * v;
    }
    for (int i = threadIdx.x; i < nk; i += blockDim.x) {
      const float v = to_float(row[nq + i]);
      sk += v * v;
    }
    sq = block_sum(sq, scratch);
    sk = block_sum(sk, scratch);
    fq = 1.f / sqrtf(sq / (float)nq + a.eps);
    fk = 1.f / sqrtf(sk / (float)nk + a.eps);
  }
  const int pos = a.tok_pos[t];
  if (a.q_temp_every > 0) fq *= 1.f + a.q_temp_coef * logf((float)((pos + 1) / a.q_temp_every) + 1.f);
  const int slot = a.seq_slot[a.tok_seq[t]];
  const int page = a.write_kv ? a.block_table[(size_t)slot * a.max_blocks + pos / MLL_PAGE] : 0;
  const int in_page = pos % MLL_PAGE;
  const int half = a.rot >> 1;
  const float* cs = a.cos_table ? a.cos_table + (size_t)pos * half : nullptr;
  const float* sn = a.cos_table ? a.sin_table + (size_t)pos * half : nullptr;
  for (int i = threadIdx.x; i < nq + nk; i += blockDim.x) {
    const bool is_q = i < nq;
    const int c = is_q ? i : i - nq;  // column within the q or k projection
    const int head = c / d, e = c % d;
    const float* w = is_q ? a.q_weight : a.k_weight;
    const float f = is_q ? fq : fk;
    const T* src = row + (is_q ? 0 : nq) + head * d;
    float x = to_float(src[e]) * f;
    if (w) x *= w[c];
    if (cs && e < a.rot) {
      int pair, partner;
      bool first;
      if (a.interleaved) {
        pair = e >> 1; first = !(e & 1); partner = e ^ 1;
      } else {
        first = e < half; pair = first ? e : e - half; partner = first ? e + half : e - half;
      }
      float y = to_float(src[partner]) * f;
      if (w) y *= w[head * d + partner];
      const float co = cs[pair], si = sn[pair];
      x = first ? x * co - y * si : x * co + y * si;
    }
    if (is_q)
      ((T*)a.q_out)[(size_t)t * nq + c] = from_float<T>(x);
    else
      ((T*)a.k_cache)[(((size_t)page * a.n_kv_heads + head) * MLL_PAGE + in_page) * d + e] = from_float<T>(x);
  }
  for (int i = threadIdx.x; i < nv; i += blockDim.x) {
    const int head = i / a.dv, e = i % a.dv;
    ((T*)a.v_cache)[(((size_t)page * a.n_kv_heads + head) * MLL_PAGE + in_page) * a.dv + e] = row[a.v_col + i];
  }
}

// The same for bfloat16 rows that are whole 16-byte words and rotated halves of whole words: a thread owns eight
// neighbouring dimensions.  The row waits in shared memory between the norm's sums and the rotation, which needs the
// partner half.
__global__ void __launch_bounds__(256) local_prepare_vec_kernel(LocalPrepArgs a) {
  extern __shared__ __align__(16) uint4 row_s[];
  __shared__ float scratch[32];
  const int t = blockIdx.x;
  const int dw = a.d >> 3, vw = a.dv >> 3, nq = a.n_heads * dw, nk = a.write_kv ? a.n_kv_heads * dw : 0;
  const int nv = a.write_kv ? a.n_kv_heads * vw : 0;
  const __nv_bfloat16* row = (const __nv_bfloat16*)a.qkv + (size_t)t * a.ld;
  const int pos = a.tok_pos[t];
  const int page = a.write_kv ? a.block_table[(size_t)a.seq_slot[a.tok_seq[t]] * a.max_blocks + pos / MLL_PAGE] : 0;
  const int in_page = pos % MLL_PAGE;
  float sq = 0.f, sk = 0.f;
  for (int i = threadIdx.x; i < nq + nk; i += 256) {
    const uint4 v = reinterpret_cast<const uint4*>(row)[i];
    row_s[i] = v;
    if (a.q_weight) {
      float x[8];
      Vec16<__nv_bfloat16>::load(reinterpret_cast<const __nv_bfloat16*>(&v), x);
      float s = 0.f;
#pragma unroll
      for (int k = 0; k < 8; ++k) s += x[k] * x[k];
      if (i < nq) sq += s;
      else sk += s;
    }
  }
  for (int i = threadIdx.x; i < nv; i += 256) {
    const int head = i / vw, e = i - head * vw;
    reinterpret_cast<uint4*>((__nv_bfloat16*)a.v_cache + (((size_t)page * a.n_kv_heads + head) * MLL_PAGE + in_page) * a.dv)[e] =
        reinterpret_cast<const uint4*>(row + a.v_col)[i];
  }
  float fq = 1.f, fk = 1.f;
  if (a.q_weight) {
    sq = block_sum(sq, scratch);
    sk = block_sum(sk, scratch);
    fq = 1.f / sqrtf(sq / (float)(nq * 8) + a.eps);
    fk = 1.f / sqrtf(sk / (float)(nk * 8) + a.eps);
  }
  if (a.q_temp_every > 0) fq *= 1.f + a.q_temp_coef * logf((float)((pos + 1) / a.q_temp_every) + 1.f);
  __syncthreads();
  const int hw = a.rot >> 4;  // words of a rotated half
  const float* cs = a.cos_table ? a.cos_table + (size_t)pos * (a.rot >> 1) : nullptr;
  const float* sn = a.cos_table ? a.sin_table + (size_t)pos * (a.rot >> 1) : nullptr;
  auto scaled = [&](int word, bool is_q, float* x) {  // eight normalised dimensions of the row
    Vec16<__nv_bfloat16>::load(reinterpret_cast<const __nv_bfloat16*>(row_s + word), x);
    const float f = is_q ? fq : fk;
    const float* w = a.q_weight ? (is_q ? a.q_weight + word * 8 : a.k_weight + (word - nq) * 8) : nullptr;
#pragma unroll
    for (int k = 0; k < 8; k += 4) {
      const float4 m = w ? *reinterpret_cast<const float4*>(w + k) : make_float4(1.f, 1.f, 1.f, 1.f);
      x[k] = x[k] * f * m.x; x[k + 1] = x[k + 1] * f * m.y; x[k + 2] = x[k + 2] * f * m.z; x[k + 3] = x[k + 3] * f * m.w;
    }
  };
  for (int i = threadIdx.x; i < nq + nk; i += 256) {
    const bool is_q = i < nq;
    const int c = is_q ? i : i - nq, head = c / dw, e = c - head * dw;
    float x[8];
    scaled(i, is_q, x);
    if (cs && e < 2 * hw) {
      const bool first = e < hw;
      float y[8];
      scaled(first ? i + hw : i - hw, is_q, y);
      const float* co = cs + (first ? e : e - hw) * 8;
      const float* si = sn + (first ? e : e - hw) * 8;
#pragma unroll
      for (int k = 0; k < 8; ++k) x[k] = first ? x[k] * co[k] - y[k] * si[k] : x[k] * co[k] + y[k] * si[k];
    }
    uint4 v;
    __nv_bfloat162* p = reinterpret_cast<__nv_bfloat162*>(&v);
#pragma unroll
    for (int k = 0; k < 4; ++k) p[k] = __floats2bfloat162_rn(x[2 * k], x[2 * k + 1]);
    if (is_q)
      reinterpret_cast<uint4*>((__nv_bfloat16*)a.q_out + (size_t)t * nq * 8)[c] = v;
    else
      reinterpret_cast<uint4*>((__nv_bfloat16*)a.k_cache + (((size_t)page * a.n_kv_heads + head) * MLL_PAGE + in_page) * a.d)[e] = v;
  }
}

struct ConvPrepArgs {
  const void* qkv;        // [T, ld]: q (Hq * d), k (Hk * d), v (Hk * dv): C channels
  const float* bias;      // [C] or null
  const float* conv_w;    // [C, taps], the last tap meets the current token
  const float* conv_state; // [slots, taps - 1, C]: the last inputs, biases included
  float* advance;         // conv_state to be moved on by the same kernel (every sequence brings one token), or null
  const float* cos_table; // [max_pos, rot / 2] or null
  const float* sin_table;
  const int* tok_pos;
  const int* tok_seq;
  const int* seq_slot;
  const int* seq_qstart;
  const int* block_table;
  void* q_out;            // [T, Hq * d]
  void* k_cache;          // [pages, Hk, PAGE, d]
  void* v_cache;          // [pages, Hk, PAGE, dv]
  int ld, n_heads, n_kv_heads, d, dv, rot, interleaved, max_blocks, taps;
};

// grid (tokens), 256 threads: a channel a thread; the partner of a rotated dimension is convolved again
template <typename T>
__global__ void __launch_bounds__(256) conv_prepare_kernel(ConvPrepArgs a) {
  const int t = blockIdx.x;
  const int d = a.d, nq = a.n_heads * d, nk = a.n_kv_heads * d, nv = a.n_kv_heads * a.dv, C = nq + nk + nv;
  const int seq = a.tok_seq[t], local = t - a.seq_qstart[seq], slot = a.seq_slot[seq], pos = a.tok_pos[t];
  const float* state = a.conv_state + (size_t)slot * (a.taps - 1) * C;
  const int page = a.block_table[(size_t)slot * a.max_blocks + pos / MLL_PAGE], in_page = pos % MLL_PAGE;
  const int half = a.rot >> 1;
  auto convolved = [&](int c) {
    const float b = a.bias ? a.bias[c] : 0.f;
    float y = 0.f;
    for (int back = 0; back < a.taps; ++back) {
      const float u = back <= local ? to_float(((const T*)a.qkv)[(size_t)(t - back) * a.ld + c]) + b
                                    : state[(size_t)(local - back + a.taps - 1) * C + c];
      y = fmaf(a.conv_w[(size_t)c * a.taps + (a.taps - 1 - back)], u, y);
    }
    return y;
  };
  for (int c = threadIdx.x; c < C; c += 256) {
    float x = convolved(c);
    if (c >= nq + nk) {
      const int i = c - nq - nk, head = i / a.dv, e = i % a.dv;
      ((T*)a.v_cache)[(((size_t)page * a.n_kv_heads + head) * MLL_PAGE + in_page) * a.dv + e] = from_float<T>(x);
      continue;
    }
    const int head = c / d, e = c % d;  // k heads follow the q heads
    if (e < a.rot) {
      int pair, partner;
      bool first;
      if (a.interleaved) {
        pair = e >> 1; first = !(e & 1); partner = e ^ 1;
      } else {
        first = e < half; pair = first ? e : e - half; partner = first ? e + half : e - half;
      }
      const float y = convolved(head * d + partner);
      const float co = a.cos_table[(size_t)pos * half + pair], si = a.sin_table[(size_t)pos * half + pair];
      x = first ? x * co - y * si : x * co + y * si;
    }
    if (c < nq)
      ((T*)a.q_out)[(size_t)t * nq + c] = from_float<T>(x);
    else
      ((T*)a.k_cache)[(((size_t)page * a.n_kv_heads + (head - a.n_heads)) * MLL_PAGE + in_page) * d + e] = from_float<T>(x);
  }
}

// The convolution's value y [V] at row t of channels c .. c + V - 1 in a step's first rows of a sequence (or any row: the
// inputs before the step come from the sequence's state), inputs one by one
template <typename T, int V, int TAPS>
__device__ __forceinline__ void conv_row(const ConvPrepArgs& a, int t, int local, const float* state, int C, int c,
                                         const float* w, const float* b, float* y, float* advance) {
  float past[TAPS][V];  // past[i]: the input i tokens ago
#pragma unroll
  for (int i = 0; i < TAPS; ++i) {
    if (i <= local) {
      load_floats<T, V>((const T*)a.qkv + (size_t)(t - i) * a.ld + c, past[i]);
#pragma unroll
      for (int j = 0; j < V; ++j) past[i][j] += b[j];
    } else {
      load_floats<float, V>(state + (size_t)(local - i + TAPS - 1) * C + c, past[i]);
    }
  }
#pragma unroll
  for (int j = 0; j < V; ++j) {
    y[j] = w[j * TAPS + TAPS - 1] * past[0][j];
#pragma unroll
    for (int i = 1; i < TAPS; ++i) y[j] = fmaf(w[j * TAPS + TAPS - 1 - i], past[i][j], y[j]);
  }
  if (advance) {  // one token a sequence: the state moves on by this input
#pragma unroll
    for (int i = 0; i < TAPS - 1; ++i) store_floats<float, V>(advance + (size_t)(TAPS - 2 - i) * C + c, past[i]);
  }
}

// grid (ceil(tokens / TB), ceil(units / 256)), 256 threads; a unit is a word of V channels, or the two words that the
// rotation (pairs half a rotated part apart) turns together.  A thread walks TB rows with its channels' taps in registers;
// the rows' words (and those of the TAPS - 1 rows before) are all fetched before the first is used.
template <typename T, int TAPS, int TB>
__global__ void __launch_bounds__(256) conv_prepare_walk_kernel(ConvPrepArgs a, int n_tokens) {
  constexpr int V = 4;
  __shared__ int local_s[TB], slot_s[TB], pos_s[TB], page_s[TB];
  const int t0 = blockIdx.x * TB;
  if (threadIdx.x < TB && t0 + threadIdx.x < n_tokens) {
    const int t = t0 + threadIdx.x, seq = a.tok_seq[t], slot = a.seq_slot[seq], pos = a.tok_pos[t];
    local_s[threadIdx.x] = t - a.seq_qstart[seq];
    slot_s[threadIdx.x] = slot;
    pos_s[threadIdx.x] = pos;
    page_s[threadIdx.x] = a.block_table[(size_t)slot * a.max_blocks + pos / MLL_PAGE];
  }
  __syncthreads();
  const int u = blockIdx.y * 256 + threadIdx.x;
  const int H = a.n_heads, G = a.n_kv_heads, d = a.d, dv = a.dv;
  const int hw = a.rot / (2 * V), nu = d / V - hw, vw = dv / V;
  const int nqk = (H + G) * nu;
  if (u >= nqk + G * vw) return;
  const int C = (H + G) * d + G * dv;
  const bool is_v = u >= nqk;
  int head, e, c;       // head among the q and k heads (or among the v heads), first dimension in it, column
  bool pair = false;
  if (is_v) {
    head = (u - nqk) / vw;
    e = (u - nqk - head * vw) * V;
    c = (H + G) * d + head * dv + e;
  } else {
    head = u / nu;
    const int i = u - head * nu;
    pair = i < hw;
    e = (pair ? i : i + hw) * V;
    c = head * d + e;
  }
  const int far = hw * V;  // distance to the partner
  const int cols[2] = {c, c + far};
  float w[2][V * TAPS], b[2][V];
  constexpr int ROWS = TB + TAPS - 1;
  RawWord<T, V> raw[2][TB > 1 ? ROWS : 1];
#pragma unroll
  for (int k = 0; k < 2; ++k) {
    if (k == 1 && !pair) break;
    load_floats<float, V * TAPS>(a.conv_w + (size_t)cols[k] * TAPS, w[k]);
#pragma unroll
    for (int j = 0; j < V; ++j) b[k][j] = a.bias ? a.bias[cols[k] + j] : 0.f;
    if constexpr (TB > 1) {
#pragma unroll
      for (int i = 0; i < ROWS; ++i)  // rows outside the step: any row of it, whose word is not used
        raw[k][i].fetch((const T*)a.qkv + (size_t)min(max(t0 + i - (TAPS - 1), 0), n_tokens - 1) * a.ld + cols[k]);
    }
  }
#pragma unroll
  for (int r = 0; r < TB; ++r) {
    const int t = t0 + r;
    if (t >= n_tokens) break;
    const int local = local_s[r], slot = slot_s[r], pos = pos_s[r];
    float y[2][V];
#pragma unroll
    for (int k = 0; k < 2; ++k) {
      if (k == 1 && !pair) break;
      if (TB == 1 || local < TAPS - 1) {
        const size_t own = (size_t)slot * (TAPS - 1) * C;
        conv_row<T, V, TAPS>(a, t, local, a.conv_state + own, C, cols[k], w[k], b[k], y[k], a.advance ? a.advance + own : nullptr);
      } else {
#pragma unroll
        for (int j = 0; j < V; ++j) {
          y[k][j] = 0.f;
#pragma unroll
          for (int i = 0; i < TAPS; ++i)
            y[k][j] = fmaf(w[k][j * TAPS + TAPS - 1 - i], raw[k][TB > 1 ? r + TAPS - 1 - i : 0][j] + b[k][j], y[k][j]);
        }
      }
    }
    if (pair) {
      float co[V], si[V];
      load_floats<float, V>(a.cos_table + (size_t)pos * (a.rot >> 1) + e, co);
      load_floats<float, V>(a.sin_table + (size_t)pos * (a.rot >> 1) + e, si);
#pragma unroll
      for (int j = 0; j < V; ++j) {
        const float p = y[0][j], q = y[1][j];
        y[0][j] = p * co[j] - q * si[j];
        y[1][j] = q * co[j] + p * si[j];
      }
    }
    T* dst;
    if (!is_v && head < H) {
      dst = (T*)a.q_out + (size_t)t * H * d + c;
    } else {
      const int page = page_s[r], in_page = pos % MLL_PAGE;
      dst = is_v ? (T*)a.v_cache + (((size_t)page * G + head) * MLL_PAGE + in_page) * dv + e
                 : (T*)a.k_cache + (((size_t)page * G + (head - H)) * MLL_PAGE + in_page) * d + e;
    }
    store_floats<T, V>(dst, y[0]);
    if (pair) store_floats<T, V>(dst + far, y[1]);
  }
}

static bool conv_walk_takes(int d, int dv, int rot, int interleaved, int taps, int ld) {
  return taps >= 2 && taps <= 4 && d % 4 == 0 && dv % 4 == 0 && rot % 8 == 0 && ld % 4 == 0 && (!interleaved || rot == 0);
}

template <typename T, int TAPS>
static int launch_conv_walk(const ConvPrepArgs& a, int n_tokens, cudaStream_t stream) {
  const int units = (a.n_heads + a.n_kv_heads) * (a.d / 4 - a.rot / 8) + a.n_kv_heads * (a.dv / 4);
  const int columns = (units + 255) / 256;
  // rows a thread walks: eight, as long as that leaves every multiprocessor four blocks
  if ((long long)((n_tokens + 7) / 8) * columns >= (long long)mll_sm_count() * 4)
    MLL_LAUNCH((conv_prepare_walk_kernel<T, TAPS, 8>), dim3((n_tokens + 7) / 8, columns), 256, 0, stream, a, n_tokens);
  else
    MLL_LAUNCH((conv_prepare_walk_kernel<T, TAPS, 1>), dim3(n_tokens, columns), 256, 0, stream, a, n_tokens);
  MLL_LAUNCH_CHECK();
  return 0;
}

template <typename T>
static int launch_conv_prepare(const ConvPrepArgs& a, int n_tokens, cudaStream_t stream) {
  const uintptr_t all = (uintptr_t)a.qkv | (uintptr_t)a.conv_w | (uintptr_t)a.conv_state | (uintptr_t)a.cos_table |
                        (uintptr_t)a.sin_table | (uintptr_t)a.q_out | (uintptr_t)a.k_cache | (uintptr_t)a.v_cache;
  if (conv_walk_takes(a.d, a.dv, a.rot, a.interleaved, a.taps, a.ld) && all % 16 == 0) {
    if (a.taps == 2) return launch_conv_walk<T, 2>(a, n_tokens, stream);
    if (a.taps == 3) return launch_conv_walk<T, 3>(a, n_tokens, stream);
    return launch_conv_walk<T, 4>(a, n_tokens, stream);
  }
  MLL_REQUIRE(!a.advance, "conv prepare: this size moves its state on in a kernel of its own");
  MLL_LAUNCH((conv_prepare_kernel<T>), n_tokens, 256, 0, stream, a);
  MLL_LAUNCH_CHECK();
  return 0;
}

struct LocalAttnArgs {
  const void* q;         // [T, Hq * d]
  const void* k_cache;
  const void* v_cache;
  const int* tok_pos;
  const int* tok_seq;
  const int* seq_slot;
  const int* block_table;
  void* out;             // [T, Hq * dv]
  int n_tokens, n_heads, n_kv_heads, d, dv, chunk, window, max_blocks;
  float scale;
  int sink;              // 1: the softmax's denominator has one more term exp(sink value)
  const float* sink_values;  // [Hq] the sink's score per query head (unscaled), or null: 0
  int v_ld;              // elements between value rows: dv, or d when the values are the keys' leading columns
  int keep_first;        // with a window: keys at positions below this stay visible
  float softcap;         // > 0: score <- softcap * tanh(score / softcap)
};

// grid (tokens, Hk * head chunks), 128 threads.  A block owns one token, one kv head and up to `hpb` of the
// query heads that read it; it walks the pages that hold keys first .. pos.  A page's keys and values are
// brought into shared memory by all threads (16-byte asynchronous copies where rows are whole 16-byte words,
// two pages in flight where shared memory allows), so that the loads of a page are all in flight together
// and every key and value is read once for the heads of its group.
template <typename T, int NACC>
__global__ void __launch_bounds__(128) local_attention_kernel(LocalAttnArgs a, int hpb, int stages, int vec) {
  const int d = a.d, dv = a.dv;
  const int group = a.n_heads / a.n_kv_heads;
  const int chunks = (group + hpb - 1) / hpb;
  const int t = blockIdx.x;
  const int kvh = blockIdx.y / chunks, g0 = (blockIdx.y % chunks) * hpb;
  const int ng = min(hpb, group - g0);
  const int h0 = kvh * group + g0;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int pos = a.tok_pos[t];
  int first = a.chunk > 0 ? (pos / a.chunk) * a.chunk : 0;
  if (a.window > 0) first = max(first, pos - a.window + 1);
  const int* table = a.block_table + (size_t)a.seq_slot[a.tok_seq[t]] * a.max_blocks;

  extern __shared__ __align__(16) unsigned char smem_raw[];
  constexpr int PAD = 16 / sizeof(T);
  const int d_pad = (d + 3) & ~3;
  float* q_s = reinterpret_cast<float*>(smem_raw);   // [hpb][d_pad], scaled
  float* s_s = q_s + hpb * d_pad;                     // [hpb][PAGE]
  float* m_s = s_s + hpb * MLL_PAGE;                  // [hpb] running maximum, sum, rescale factor
  float* l_s = m_s + hpb;
  float* alpha_s = l_s + hpb;
  size_t off = (size_t)((alpha_s + hpb) - q_s) * sizeof(float);
  off = (off + 15) & ~(size_t)15;
  const int k_stride = ((d + PAD - 1) / PAD) * PAD + PAD;  // elements; rows start on 16-byte boundaries
  const int v_stride = ((dv + PAD - 1) / PAD) * PAD;
  const size_t k_tile = (size_t)MLL_PAGE * k_stride, v_tile = (size_t)MLL_PAGE * v_stride;
  T* k_s = reinterpret_cast<T*>(smem_raw + off);
  T* v_s = k_s + stages * k_tile;

  for (int i = tid; i < ng * d; i += 128) {
    const int g = i / d, e = i % d;
    q_s[g * d_pad + e] = to_float(((const T*)a.q)[((size_t)t * a.n_heads + h0 + g) * d + e]) * a.scale;
  }
  for (int i = tid; i < ng; i += 128) {
    // the sink: a key with a score of its own and no value, seen before all others
    m_s[i] = a.sink ? (a.sink_values ? a.sink_values[h0 + i] : 0.f) : -INFINITY;
    l_s[i] = a.sink ? 1.f : 0.f;
  }
  float acc[NACC];
#pragma unroll
  for (int i = 0; i < NACC; ++i) acc[i] = 0.f;

  const int p_begin = first / MLL_PAGE, p_end = pos / MLL_PAGE + 1;
  // the kept first tokens that lie in front of the window: keys [0, kept), on the pages in front of p_begin and on
  // p_begin itself (whose rows between `kept` and `first` are then skipped)
  const int kept = (a.window > 0 && a.keep_first > 0) ? min(a.keep_first, first) : 0;
  const int n_kept_pages = min((kept + MLL_PAGE - 1) / MLL_PAGE, p_begin);  // walked before p_begin
  auto page_of = [&](int walk) { return walk < n_kept_pages ? walk : p_begin + (walk - n_kept_pages); };
  const int n_walk = n_kept_pages + (p_end - p_begin);
  auto load_tiles = [&](int page_index, int stage) {
    const int page = table[page_index];
    const T* kg = (const T*)a.k_cache + ((size_t)page * a.n_kv_heads + kvh) * MLL_PAGE * d;
    const T* vg = (const T*)a.v_cache + ((size_t)page * a.n_kv_heads + kvh) * MLL_PAGE * a.v_ld;
    T* kd = k_s + stage * k_tile;
    T* vd = v_s + stage * v_tile;
    // every row up to the last visible one is loaded when kept keys share the page; the scores mask the gap
    const int r_lo = page_index * MLL_PAGE < kept ? 0 : max(0, first - page_index * MLL_PAGE);
    const int r_hi = min(MLL_PAGE, pos + 1 - page_index * MLL_PAGE);
    if (vec) {
      const int kc = d / PAD, vc = dv / PAD;
      for (int c = tid; c < (r_hi - r_lo) * kc; c += 128) {
        const int r = r_lo + c / kc, cc = c % kc;
        cp_async16(kd + (size_t)r * k_stride + cc * PAD, kg + (size_t)r * d + cc * PAD);
      }
      for (int c = tid; c < (r_hi - r_lo) * vc; c += 128) {
        const int r = r_lo + c / vc, cc = c % vc;
        cp_async16(vd + (size_t)r * v_stride + cc * PAD, vg + (size_t)r * a.v_ld + cc * PAD);
      }
    } else {
      for (int c = tid; c < (r_hi - r_lo) * d; c += 128) {
        const int r = r_lo + c / d, e = c % d;
        kd[(size_t)r * k_stride + e] = kg[(size_t)r * d + e];
      }
      for (int c = tid; c < (r_hi - r_lo) * dv; c += 128) {
        const int r = r_lo + c / dv, e = c % dv;
        vd[(size_t)r * v_stride + e] = vg[(size_t)r * a.v_ld + e];
      }
    }
  };

  load_tiles(page_of(0), 0);
  cp_async_commit();
  for (int it = 0; it < n_walk; ++it) {
    const int p = page_of(it);
    const int cur = stages == 2 ? (it & 1) : 0;
    if (stages == 2 && it + 1 < n_walk) {
      load_tiles(page_of(it + 1), cur ^ 1);
      cp_async_commit();
      cp_async_wait<1>();
    } else {
      cp_async_wait<0>();
    }
    __syncthreads();
    const T* kt = k_s + cur * k_tile;
    const T* vt = v_s + cur * v_tile;
    const int jlo = p * MLL_PAGE < kept ? 0 : max(0, first - p * MLL_PAGE), jhi = min(MLL_PAGE, pos + 1 - p * MLL_PAGE);

    for (int idx = tid; idx < ng * MLL_PAGE; idx += 128) {
      const int g = idx / MLL_PAGE, j = idx % MLL_PAGE;
      float sc = -INFINITY;
      const int kpos = p * MLL_PAGE + j;
      if (j >= jlo && j < jhi && (kpos >= first || kpos < kept)) {
        const T* kr = kt + (size_t)j * k_stride;
        const float* qg = q_s + g * d_pad;
        float dot = 0.f;
        if (vec) {
          for (int e = 0; e < d; e += PAD) {
            float kv[PAD];
            Vec16<T>::load(kr + e, kv);
#pragma unroll
            for (int u = 0; u < PAD; ++u) dot = fmaf(qg[e + u], kv[u], dot);
          }
        } else {
          for (int e = 0; e < d; ++e) dot = fmaf(qg[e], to_float(kr[e]), dot);
        }
        sc = a.softcap > 0.f ? a.softcap * tanhf(dot / a.softcap) : dot;
      }
      s_s[idx] = sc;
    }
    __syncthreads();
    for (int g = warp; g < ng; g += 4) {
      const float v0 = s_s[g * MLL_PAGE + lane], v1 = s_s[g * MLL_PAGE + lane + 32];
      const float m_old = m_s[g];
      const float m_new = fmaxf(m_old, warp_max(fmaxf(v0, v1)));  // every page of the walk holds a visible key: finite
      const float alpha = expf(m_old - m_new);
      const float p0 = expf(v0 - m_new), p1 = expf(v1 - m_new);
      s_s[g * MLL_PAGE + lane] = p0;
      s_s[g * MLL_PAGE + lane + 32] = p1;
      const float psum = warp_sum(p0 + p1);
      if (lane == 0) {
        l_s[g] = l_s[g] * alpha + psum;
        m_s[g] = m_new;
        alpha_s[g] = alpha;
      }
    }
    __syncthreads();
#pragma unroll
    for (int i = 0; i < NACC; ++i) {
      const int o = tid + 128 * i;
      if (o < ng * dv) {
        const int g = o / dv, e = o % dv;
        float v = acc[i] * alpha_s[g];
        const float* pg = s_s + g * MLL_PAGE;
        for (int j = jlo; j < jhi; ++j) v = fmaf(pg[j], to_float(vt[(size_t)j * v_stride + e]), v);
        acc[i] = v;
      }
    }
    __syncthreads();
    if (stages == 1 && it + 1 < n_walk) {
      load_tiles(page_of(it + 1), 0);
      cp_async_commit();
    }
  }
#pragma unroll
  for (int i = 0; i < NACC; ++i) {
    const int o = tid + 128 * i;
    if (o < ng * dv) {
      const float l = l_s[o / dv];
      ((T*)a.out)[((size_t)t * a.n_heads + h0) * dv + o] = from_float<T>(l > 0.f ? acc[i] / l : 0.f);
    }
  }
}

template <typename T>
int launch_local_attention(const LocalAttnArgs& a, cudaStream_t stream) {
  constexpr int PAD = 16 / sizeof(T);
  const int group = a.n_heads / a.n_kv_heads;
  const int hpb = max(1, min(group, 1024 / a.dv));       // at most 8 accumulators a thread
  const int chunks = (group + hpb - 1) / hpb;
  const int vec = (a.d % PAD == 0 && a.dv % PAD == 0 && a.v_ld % PAD == 0) ? 1 : 0;
  const int k_stride = ((a.d + PAD - 1) / PAD) * PAD + PAD, v_stride = ((a.dv + PAD - 1) / PAD) * PAD;
  size_t fixed = (size_t)(hpb * ((a.d + 3) & ~3) + hpb * MLL_PAGE + 3 * hpb) * sizeof(float);
  fixed = (fixed + 15) & ~(size_t)15;
  const size_t tile = (size_t)MLL_PAGE * (k_stride + v_stride) * sizeof(T);
  const int stages = fixed + 2 * tile <= 96 * 1024 ? 2 : 1;
  const size_t smem = fixed + stages * tile;
  MLL_REQUIRE(smem <= 200 * 1024, "local attention: head sizes %d / %d need %zu bytes of shared memory", a.d, a.dv, smem);
  MLL_REQUIRE((long long)a.n_kv_heads * chunks <= 65535, "local attention: too many heads for one launch");
  const dim3 grid(a.n_tokens, a.n_kv_heads * chunks);
  const int nacc = (hpb * a.dv + 127) / 128;
#define MLL_LOCAL_LAUNCH(N)                                                                                   \
  do {                                                                                                        \
    auto kernel = local_attention_kernel<T, N>;                                                               \
    if (smem > 48 * 1024) {                                                                                   \
      cudaError_t err = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
      if (err != cudaSuccess) {                                                                               \
        mll_set_error("local attention: cannot reserve %zu bytes of shared memory: %s", smem,                 \
                      cudaGetErrorString(err));                                                               \
        return (int)err;                                                                                      \
      }                                                                                                       \
    }                                                                                                         \
    MLL_LAUNCH((kernel), grid, 128, smem, stream, a, hpb, stages, vec);                                       \
  } while (0)
  if (nacc <= 1) MLL_LOCAL_LAUNCH(1);
  else if (nacc <= 2) MLL_LOCAL_LAUNCH(2);
  else if (nacc <= 4) MLL_LOCAL_LAUNCH(4);
  else MLL_LOCAL_LAUNCH(8);
#undef MLL_LOCAL_LAUNCH
  MLL_LAUNCH_CHECK();
  return 0;
}

}  // namespace mll
// Whether mll_conv_attention_prepare can also move the convolution's state on (`advance`).
MLL_API int mll_conv_attention_advances(int d, int dv, int rot, int interleaved, int taps, int ld) {
  return mll::conv_walk_takes(d, dv, rot, interleaved, taps, ld) ? 1 : 0;
}

// qkv [n_tokens, ld] of `dtype`; see ConvPrepArgs.  advance: conv_state itself, or null.
MLL_API int mll_conv_attention_prepare(const void* qkv, const float* bias, const float* conv_w, float* conv_state, int advance,
                                       const float* cos_table, const float* sin_table, const int* tok_pos,
                                       const int* tok_seq, const int* seq_slot, const int* seq_qstart,
                                       const int* block_table, void* q_out, void* k_cache, void* v_cache, int dtype,
                                       int n_tokens, int ld, int n_heads, int n_kv_heads, int d, int dv, int rot,
                                       int interleaved, int max_blocks, int taps, cudaStream_t stream) {
  MLL_REQUIRE(n_tokens >= 0 && n_heads > 0 && n_kv_heads > 0 && d > 0 && dv > 0 && taps >= 1 && max_blocks > 0,
              "conv prepare: bad sizes");
  MLL_REQUIRE(rot >= 0 && rot <= d && rot % 2 == 0 && (rot == 0 || (cos_table && sin_table)),
              "conv prepare: %d rotated dimensions of %d, or no table", rot, d);
  MLL_REQUIRE(ld >= (n_heads + n_kv_heads) * d + n_kv_heads * dv, "conv prepare: row stride %d too short", ld);
  if (n_tokens == 0) return 0;
  mll::ConvPrepArgs a{qkv, bias, conv_w, conv_state, advance ? conv_state : nullptr, rot ? cos_table : nullptr,
                      rot ? sin_table : nullptr, tok_pos, tok_seq, seq_slot, seq_qstart, block_table, q_out, k_cache, v_cache,
                      ld, n_heads, n_kv_heads, d, dv, rot, interleaved, max_blocks, taps};
  if (dtype == MLL_F32) return mll::launch_conv_prepare<float>(a, n_tokens, stream);
  if (dtype == MLL_BF16) return mll::launch_conv_prepare<__nv_bfloat16>(a, n_tokens, stream);
  MLL_REQUIRE(false, "conv prepare: unknown dtype %d", dtype);
  return -1;
}

MLL_API int mll_local_attention_prepare(const void* qkv, const float* q_weight, const float* k_weight,
                                        const float* cos_table, const float* sin_table, const int* tok_pos,
                                        const int* tok_seq, const int* seq_slot, const int* block_table, void* q_out,
                                        void* k_cache, void* v_cache, int dtype, int n_tokens, int ld, int n_heads,
                                        int n_kv_heads, int d, int dv, int rot, int interleaved, int max_blocks,
                                        float eps, float q_temp_coef, int q_temp_every, int v_from_k, int write_kv,
                                        cudaStream_t stream) {
  MLL_REQUIRE(n_tokens >= 0 && n_heads > 0 && n_kv_heads > 0 && d > 0 && dv > 0, "local attention prepare: bad sizes");
  MLL_REQUIRE(rot >= 0 && rot <= d && rot % 2 == 0, "local attention prepare: %d rotated dimensions of %d", rot, d);
  MLL_REQUIRE((q_weight == nullptr) == (k_weight == nullptr), "local attention prepare: one norm weight without the other");
  MLL_REQUIRE(ld >= n_heads * d + (write_kv ? n_kv_heads * (v_from_k ? d : d + dv) : 0), "local attention prepare: row stride %d too short", ld);
  MLL_REQUIRE(!v_from_k || dv == d, "local attention prepare: values that are the keys need dv == d, got %d / %d", dv, d);
  MLL_REQUIRE(q_temp_every >= 0, "local attention prepare: negative temperature period");
  if (n_tokens == 0) return 0;
  mll::LocalPrepArgs a{qkv, q_weight, k_weight, rot > 0 ? cos_table : nullptr, sin_table, tok_pos, tok_seq, seq_slot,
                       block_table, q_out, k_cache, v_cache, ld, n_heads, n_kv_heads, d, dv, rot, interleaved,
                       max_blocks, eps, q_temp_coef, q_temp_every,
                       v_from_k ? n_heads * d : n_heads * d + n_kv_heads * d, write_kv ? 1 : 0};
  const auto whole = [](const void* p) { return (uintptr_t)p % 16 == 0; };
  const size_t row_bytes = (size_t)(n_heads + (write_kv ? n_kv_heads : 0)) * d * 2;
  if (dtype == MLL_BF16 && d % 8 == 0 && dv % 8 == 0 && ld % 8 == 0 && (rot == 0 || (!interleaved && rot % 16 == 0)) &&
      row_bytes <= 48 * 1024 && whole(qkv) && whole(q_out) && whole(k_cache) && whole(v_cache) && whole(q_weight) && whole(k_weight)) {
    MLL_LAUNCH((mll::local_prepare_vec_kernel), n_tokens, 256, row_bytes, stream, a);
    MLL_LAUNCH_CHECK();
    return 0;
  }
  if (dtype == MLL_F32)
    MLL_LAUNCH((mll::local_prepare_kernel<float>), n_tokens, 256, 0, stream, a);
  else if (dtype == MLL_BF16)
    MLL_LAUNCH((mll::local_prepare_kernel<__nv_bfloat16>), n_tokens, 256, 0, stream, a);
  else
    MLL_REQUIRE(false, "local attention prepare: unknown dtype %d", dtype);
  MLL_LAUNCH_CHECK();
  return 0;
}

MLL_API int mll_local_attention(const void* q, const void* k_cache, const void* v_cache, const int* tok_pos,
                                const int* tok_seq, const int* seq_slot, const int* block_table, void* out, int dtype,
                                int n_tokens, int n_heads, int n_kv_heads, int d, int dv, int chunk, int window,
                                int max_blocks, float scale, int sink, const float* sink_values, int v_in_k,
                                int keep_first, float softcap, cudaStream_t stream) {
  MLL_REQUIRE(n_tokens >= 0 && n_heads > 0 && n_kv_heads > 0 && n_heads % n_kv_heads == 0, "local attention: bad head counts");
  MLL_REQUIRE(d > 0 && d <= 1024 && dv > 0 && dv <= 1024, "local attention: head sizes %d / %d (at most 1024)", d, dv);
  MLL_REQUIRE(chunk >= 0 && window >= 0 && keep_first >= 0 && softcap >= 0.f, "local attention: negative chunk, window, kept tokens or cap");
  MLL_REQUIRE(keep_first == 0 || chunk == 0, "local attention: kept first tokens go with a window, not with chunks");
  MLL_REQUIRE(!v_in_k || dv <= d, "local attention: values of %d cannot be the leading columns of keys of %d", dv, d);
  if (n_tokens == 0) return 0;
  mll::LocalAttnArgs a{q, k_cache, v_cache, tok_pos, tok_seq, seq_slot, block_table, out, n_tokens, n_heads,
                       n_kv_heads, d, dv, chunk, window, max_blocks, scale, (sink || sink_values) ? 1 : 0, sink_values,
                       v_in_k ? d : dv, keep_first, softcap};
  if (dtype == MLL_F32) return mll::launch_local_attention<float>(a, stream);
  if (dtype == MLL_BF16) return mll::launch_local_attention<__nv_bfloat16>(a, stream);
  MLL_REQUIRE(false, "local attention: unknown dtype %d", dtype);
  return -1;
}
