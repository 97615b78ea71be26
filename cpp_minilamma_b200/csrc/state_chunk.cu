// The recurrences of recurrent.cu whose decay is one number per head (fixed, or per token), over prompts, a run of 32
// tokens at a time instead of token by token:
//
//   S_t = g_t S_(t-1) + k_t u_t^T,   o_t = S_t^T q_t,   u_t = v_t   or   u_t = beta_t (v_t - g_t S_(t-1)^T k_t)  (delta rule)
//
// Inside a run that starts from the state S, with c_i the sum of log g over its tokens up to i (g is at most 1, so every
// exponent below is at most 0):
//
//   o_i = e^(c_i) S^T q_i + sum_(j <= i) P_ij u_j,                 P_ij = e^(c_i - c_j) q_i . k_j
//   S  <- e^(c_n) S + sum_j e^(c_n - c_j) k_j u_j^T
//   and for the delta rule  u = U - W S  with  (I + A) U = diag(beta) V,  (I + A) W = diag(beta e^c) K,
//                           A_ij = beta_i e^(c_i - c_j) k_i . k_j  for j < i
//
// Kernels:
//   * state_chunk_inputs   a block per (run, head): the sums c (double), P, and for the delta rule U and W by forward
//                          substitution, a column a thread
//   * without the delta rule nothing but the sum of the states hangs from run to run: state_chunk_sums (what every run adds),
//                          state_chunk_prefix (the state in front of every run) and state_chunk_outputs
//   * state_chunk_scan     the delta rule: a block per (16 columns of the state, head, sequence) walks the runs; the columns
//                          of S in registers and in shared memory, the runs' matrices through cp.async, W and Q of the
//                          next run on their way while this one is worked on
// All products are float32 FMAs: the recurrence stays exact to float32, which bfloat16 tensor-core products would not be,
// and products cut into enough bfloat16 terms to be exact take as long on the tensor cores.
#include "common.cuh"

namespace mll {

constexpr int CH = 32;          // tokens a run
constexpr int CH_COLS = 16;     // columns of the state a block of the scan owns
constexpr int CH_FACTORS = 72;  // floats per (run, head): e^(c_i) [32], e^(c_n - c_i) [32], e^(c_n), padding
constexpr float CH_NO_DECAY_LEFT = -200.f;  // the logarithm that stands for a decay of 0: e^-200 is 0 in float32

struct ChunkArgs {
  const float* q;           // [T, G, d]
  const float* k;           // [T, G, d]
  const float* v;           // [T, H, dv]
  const float* beta;        // [T, H] (delta rule) or null
  const float* token_decay; // [T, H], or null:
  const float* head_decay;  // [H]
  float* state;             // [slots, H, d, dv]
  float* out;               // [T, H, dv]
  float* p;                 // [runs, H, 32, 32]
  float* w;                 // [runs, H, 32, d]    (delta rule)
  float* u;                 // [runs, H, 32, dv]   (delta rule)
  float* factors;           // [runs, H, CH_FACTORS]
  float* sums;              // [runs, H, d, dv]    (not the delta rule)
  const int* run_seq;       // [runs]
  const int* run_row0;      // [runs] first row among the sequence's new tokens
  const int* seq_run0;      // [sequences] the sequence's first run
  const int* seq_slot;
  const int* seq_qstart;
  const int* seq_qlen;
  int n_heads, n_kv_heads, d, dv;
};

// 16 bytes global -> shared, zeros where `valid` is false
__device__ __forceinline__ void ch_copy16(float* dst, const float* src, bool valid) {
  const unsigned s = (unsigned)__cvta_generic_to_shared(dst);
  const int bytes = valid ? 16 : 0;
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"(s), "l"(src), "r"(bytes));
}

// grid (runs, H), 128 threads.  Rows of q and k lie in shared memory as 16-byte words whose index is XORed with the row's
// low three bits: threads that read one word of eight neighbouring rows meet eight different banks.
template <int DP, bool DELTA>
__global__ void __launch_bounds__(128, 3) state_chunk_inputs_kernel(ChunkArgs a) {
  constexpr int WORDS = DP / 4, A_LD = CH + 4;
  __shared__ __align__(16) float q_s[CH * DP];
  __shared__ __align__(16) float k_s[CH * DP];
  __shared__ __align__(16) float a_s[DELTA ? CH * A_LD : 4];
  __shared__ double c_s[CH];
  __shared__ float beta_s[CH], grow_s[CH];  // beta_i, and beta_i e^(c_i)
  const int run = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, lane = tid & 31;
  const int H = a.n_heads, G = a.n_kv_heads, d = a.d, dv = a.dv, kvh = h / (H / G);
  const int seq = a.run_seq[run], row0 = a.run_row0[run];
  const int n = min(CH, a.seq_qlen[seq] - row0);
  const size_t tok0 = (size_t)a.seq_qstart[seq] + row0;
  const size_t at = (size_t)run * H + h;
  for (int i = tid; i < CH * WORDS; i += 128) {
    const int r = i / WORDS, wd = i % WORDS;
    const bool in = r < n && wd * 4 < d;
    const size_t src = in ? ((tok0 + r) * G + kvh) * d + wd * 4 : 0;
    const int dst = r * DP + ((wd ^ (r & 7)) << 2);
    ch_copy16(q_s + dst, a.q + src, in);
    ch_copy16(k_s + dst, a.k + src, in);
  }
  cp_async_commit();
  // the delta rule's first columns of values, on their way while the products run (rows past the run's end: the last row,
  // which a beta of 0 takes out again)
  float x[DELTA ? CH : 1];
  auto load_values = [&](int e) {
#pragma unroll
    for (int i = 0; i < (DELTA ? CH : 1); ++i) x[i] = a.v[((tok0 + min(i, n - 1)) * H + h) * dv + e];
  };
  if (DELTA && tid < dv) load_values(tid);
  if (tid < 32) {
    const bool in = lane < n;
    double c = 0.0;
    if (in) {
      const float g = a.token_decay ? a.token_decay[(tok0 + lane) * H + h] : a.head_decay[h];
      c = g > 0.f ? (double)logf(g) : (double)CH_NO_DECAY_LEFT;
    }
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const double before = __shfl_up_sync(0xffffffffu, c, o);
      if (lane >= o) c += before;
    }
    const double all = __shfl_sync(0xffffffffu, c, 31);  // tokens past the run's end add nothing
    c_s[lane] = c;
    const float grown = expf((float)c);
    float* f = a.factors + at * CH_FACTORS;
    f[lane] = grown;
    f[CH + lane] = in ? expf((float)(all - c)) : 0.f;
    if (lane == 0) f[2 * CH] = expf((float)all);
    if (DELTA) {
      const float b = in ? a.beta[(tok0 + lane) * H + h] : 0.f;
      beta_s[lane] = b;
      grow_s[lane] = b * grown;
    }
  }
  cp_async_wait<0>();
  __syncthreads();
  {
    // two products of 32 x 32: threads 0-63 form q k^T, threads 64-127 k k^T, rows rg + 8 i and columns cg + 8 j each
    const bool second = tid >= 64;
    const int t = tid & 63, rg = t >> 3, cg = t & 7;
    if (!second || DELTA) {
      const float* rows = second ? k_s : q_s;
      float acc[4][4];
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
#pragma unroll 4
      for (int wd = 0; wd < WORDS; ++wd) {
        float4 x[4], y[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          x[i] = *reinterpret_cast<const float4*>(rows + (rg + 8 * i) * DP + ((wd ^ rg) << 2));
          y[i] = *reinterpret_cast<const float4*>(k_s + (cg + 8 * i) * DP + ((wd ^ cg) << 2));
        }
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
          for (int j = 0; j < 4; ++j)
            acc[i][j] = fmaf(x[i].x, y[j].x, fmaf(x[i].y, y[j].y, fmaf(x[i].z, y[j].z, fmaf(x[i].w, y[j].w, acc[i][j]))));
      }
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const int r = rg + 8 * i, c = cg + 8 * j;
          const bool keep = r < n && (second ? c < r : c <= r);
          const float value = keep ? acc[i][j] * expf((float)(c_s[r] - c_s[c])) : 0.f;
          if (second) a_s[r * A_LD + c] = beta_s[r] * value;
          else a.p[(at * CH + r) * CH + c] = value;
        }
    }
  }
  if constexpr (DELTA) {
    __syncthreads();
    for (int col = tid; col < dv + d; col += 128) {
      const bool value = col < dv;
      const int e = value ? col : col - dv;
      if (value) {
        if (col != tid) load_values(e);
#pragma unroll
        for (int i = 0; i < CH; ++i) x[i] *= beta_s[i];
      } else {
#pragma unroll
        for (int i = 0; i < CH; ++i) x[i] = grow_s[i] * k_s[i * DP + (((e >> 2) ^ (i & 7)) << 2) + (e & 3)];
      }
#pragma unroll
      for (int i = 1; i < CH; ++i) {
        float s[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
        for (int m = 0; m < i; m += 4) {  // the row's entries from i on are zero, as are x's uses of them
          const float4 row = *reinterpret_cast<const float4*>(a_s + i * A_LD + m);
          s[0] = fmaf(row.x, x[m], s[0]);
          if (m + 1 < i) s[1] = fmaf(row.y, x[m + 1], s[1]);
          if (m + 2 < i) s[2] = fmaf(row.z, x[m + 2], s[2]);
          if (m + 3 < i) s[3] = fmaf(row.w, x[m + 3], s[3]);
        }
        x[i] -= (s[0] + s[1]) + (s[2] + s[3]);
      }
      float* dst = value ? a.u + at * CH * dv + e : a.w + at * CH * d + e;
      const int ld = value ? dv : d;
#pragma unroll
      for (int i = 0; i < CH; ++i) dst[(size_t)i * ld] = x[i];
    }
  }
}

// acc[i][:] += row_i[4 places] . m[4 places][4 columns]: one word (four places of the contraction) of R rows
template <int R>
__device__ __forceinline__ void ch_step(float (&acc)[R][4], const float4 (&m)[4], const float* row, int row_stride) {
#pragma unroll
  for (int i = 0; i < R; ++i) {
    const float4 x = *reinterpret_cast<const float4*>(row + i * row_stride);
    acc[i][0] = fmaf(x.x, m[0].x, fmaf(x.y, m[1].x, fmaf(x.z, m[2].x, fmaf(x.w, m[3].x, acc[i][0]))));
    acc[i][1] = fmaf(x.x, m[0].y, fmaf(x.y, m[1].y, fmaf(x.z, m[2].y, fmaf(x.w, m[3].y, acc[i][1]))));
    acc[i][2] = fmaf(x.x, m[0].z, fmaf(x.y, m[1].z, fmaf(x.z, m[2].z, fmaf(x.w, m[3].z, acc[i][2]))));
    acc[i][3] = fmaf(x.x, m[0].w, fmaf(x.y, m[1].w, fmaf(x.z, m[2].w, fmaf(x.w, m[3].w, acc[i][3]))));
  }
}

// ---- without the delta rule: nothing but the sum of the states hangs from run to run -------------------------------- //
constexpr int CH_WIDE = 64;  // columns of the state a block of the two kernels below owns

// grid (runs, H, ceil(dv / 64)), 128 threads: what a run adds to the state, sum_j e^(c_n - c_j) k_j v_j^T, to sums [runs, H,
// d, dv].  A thread owns DP / 16 rows and two groups of four columns.
template <int DP>
__global__ void __launch_bounds__(128) state_chunk_sums_kernel(ChunkArgs a) {
  constexpr int WORDS = DP / 4, TM = DP / 16, PIECE = TM < 4 ? TM : 4, PIECES = TM / PIECE;
  __shared__ __align__(16) float k_s[CH * DP];
  __shared__ __align__(16) float v_s[CH * CH_WIDE];
  __shared__ float left_s[CH];
  const int run = blockIdx.x, h = blockIdx.y, col0 = blockIdx.z * CH_WIDE, tid = threadIdx.x;
  const int H = a.n_heads, G = a.n_kv_heads, d = a.d, dv = a.dv, kvh = h / (H / G);
  const int seq = a.run_seq[run], row0 = a.run_row0[run];
  const int n = min(CH, a.seq_qlen[seq] - row0);
  const size_t tok0 = (size_t)a.seq_qstart[seq] + row0, at = (size_t)run * H + h;
#pragma unroll
  for (int i = tid; i < CH * WORDS; i += 128) {
    const int r = i / WORDS, wd = i % WORDS;
    const bool in = r < n && wd * 4 < d;
    ch_copy16(k_s + i * 4, in ? a.k + ((tok0 + r) * G + kvh) * d + wd * 4 : a.k, in);
  }
#pragma unroll
  for (int i = tid; i < CH * CH_WIDE / 4; i += 128) {
    const int r = i / (CH_WIDE / 4), wd = i % (CH_WIDE / 4);
    const bool in = r < n && col0 + wd * 4 < dv;
    ch_copy16(v_s + i * 4, in ? a.v + ((tok0 + r) * H + h) * dv + col0 + wd * 4 : a.v, in);
  }
  cp_async_commit();
  if (tid < CH) left_s[tid] = a.factors[at * CH_FACTORS + CH + tid];
  cp_async_wait<0>();
  __syncthreads();
  const int cg = tid & 7, rg = tid >> 3;
  float acc[TM][8];
#pragma unroll
  for (int i = 0; i < TM; ++i)
#pragma unroll
    for (int j = 0; j < 8; ++j) acc[i][j] = 0.f;
#pragma unroll 4
  for (int t = 0; t < CH; ++t) {
    float x[TM], y[8];
#pragma unroll
    for (int p = 0; p < PIECES; ++p) load_floats<float, PIECE>(k_s + t * DP + p * (DP / PIECES) + rg * PIECE, x + p * PIECE);
    load_floats<float, 4>(v_s + t * CH_WIDE + cg * 4, y);
    load_floats<float, 4>(v_s + t * CH_WIDE + 32 + cg * 4, y + 4);
    const float left = left_s[t];
#pragma unroll
    for (int i = 0; i < TM; ++i) x[i] *= left;
#pragma unroll
    for (int i = 0; i < TM; ++i)
#pragma unroll
      for (int j = 0; j < 8; ++j) acc[i][j] = fmaf(x[i], y[j], acc[i][j]);
  }
#pragma unroll
  for (int i = 0; i < TM; ++i) {
    const int row = (i / PIECE) * (DP / PIECES) + rg * PIECE + i % PIECE;
    if (row >= d) continue;
    float* dst = a.sums + (at * d + row) * dv + col0 + cg * 4;
    if (col0 + cg * 4 < dv) store_floats<float, 4>(dst, acc[i]);
    if (col0 + 32 + cg * 4 < dv) store_floats<float, 4>(dst + 32, acc[i] + 4);
  }
}

// grid (ceil(d dv / 1024), H, sequences), 256 threads, four neighbouring numbers of the state a thread: every run's sum
// makes room for the state in front of that run, and the sequence's state moves on by all of them.
__global__ void __launch_bounds__(256) state_chunk_prefix_kernel(ChunkArgs a) {
  const int h = blockIdx.y, seq = blockIdx.z, H = a.n_heads;
  const size_t size = (size_t)a.d * a.dv, i = ((size_t)blockIdx.x * 256 + threadIdx.x) * 4;
  if (i >= size) return;
  const int n_runs = (a.seq_qlen[seq] + CH - 1) / CH;
  float* S = a.state + ((size_t)a.seq_slot[seq] * H + h) * size + i;
  float4 s = *reinterpret_cast<const float4*>(S);
  constexpr int AHEAD = 8;  // runs whose sums are fetched together
  for (int c0 = 0; c0 < n_runs; c0 += AHEAD) {
    float4 x[AHEAD];
    float left[AHEAD];
#pragma unroll
    for (int j = 0; j < AHEAD; ++j)
      if (c0 + j < n_runs) {
        const size_t at = (size_t)(a.seq_run0[seq] + c0 + j) * H + h;
        x[j] = *reinterpret_cast<const float4*>(a.sums + at * size + i);
        left[j] = a.factors[at * CH_FACTORS + 2 * CH];
      }
#pragma unroll
    for (int j = 0; j < AHEAD; ++j)
      if (c0 + j < n_runs) {
        const size_t at = (size_t)(a.seq_run0[seq] + c0 + j) * H + h;
        *reinterpret_cast<float4*>(a.sums + at * size + i) = s;
        s.x = fmaf(left[j], s.x, x[j].x); s.y = fmaf(left[j], s.y, x[j].y);
        s.z = fmaf(left[j], s.z, x[j].z); s.w = fmaf(left[j], s.w, x[j].w);
      }
  }
  *reinterpret_cast<float4*>(S) = s;
}

template <int DP>
struct ChunkOutputsSmem {  // offsets in floats; the warps' partial sums lie over the states once they are used
  static constexpr int Q = 0, P = Q + CH * DP, V = P + CH * CH, S = V + CH * CH_WIDE;
  static constexpr int SUMS = 4 * CH * CH_WIDE, FLOATS = S + (DP * CH_WIDE > SUMS ? DP * CH_WIDE : SUMS);
  static constexpr size_t BYTES = (size_t)FLOATS * sizeof(float);
};

// grid (runs, H, ceil(dv / 64)), 128 threads: o_i = e^(c_i) S^T q_i + sum_j P_ij v_j of a run, S the state in front of it.
// A warp takes every fourth word of either contraction, a thread rows lane / 8 + 4 i (i < 8) and two groups of four columns.
template <int DP>
__global__ void __launch_bounds__(128) state_chunk_outputs_kernel(ChunkArgs a) {
  using L = ChunkOutputsSmem<DP>;
  constexpr int WORDS = DP / 4, WIDE_WORDS = CH_WIDE / 4;
  extern __shared__ __align__(16) float sm[];
  const int run = blockIdx.x, h = blockIdx.y, col0 = blockIdx.z * CH_WIDE;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, cg = lane & 7, rg = lane >> 3;
  const int H = a.n_heads, G = a.n_kv_heads, d = a.d, dv = a.dv, kvh = h / (H / G);
  const int seq = a.run_seq[run], row0 = a.run_row0[run];
  const int n = min(CH, a.seq_qlen[seq] - row0);
  const size_t tok0 = (size_t)a.seq_qstart[seq] + row0, at = (size_t)run * H + h;
#pragma unroll
  for (int i = tid; i < CH * WORDS; i += 128) {
    const int r = i / WORDS, wd = i % WORDS;
    const bool in = r < n && wd * 4 < d;
    ch_copy16(sm + L::Q + i * 4, in ? a.q + ((tok0 + r) * G + kvh) * d + wd * 4 : a.q, in);
  }
#pragma unroll
  for (int i = tid; i < DP * WIDE_WORDS; i += 128) {
    const int r = i / WIDE_WORDS, wd = i % WIDE_WORDS;
    const bool in = r < d && col0 + wd * 4 < dv;
    ch_copy16(sm + L::S + i * 4, in ? a.sums + (at * d + r) * dv + col0 + wd * 4 : a.sums, in);
  }
#pragma unroll
  for (int i = tid; i < CH * CH / 4; i += 128) ch_copy16(sm + L::P + i * 4, a.p + at * CH * CH + i * 4, true);
#pragma unroll
  for (int i = tid; i < CH * WIDE_WORDS; i += 128) {
    const int r = i / WIDE_WORDS, wd = i % WIDE_WORDS;
    const bool in = r < n && col0 + wd * 4 < dv;
    ch_copy16(sm + L::V + i * 4, in ? a.v + ((tok0 + r) * H + h) * dv + col0 + wd * 4 : a.v, in);
  }
  cp_async_commit();
  float grown[8];
#pragma unroll
  for (int i = 0; i < 8; ++i) grown[i] = a.factors[at * CH_FACTORS + rg + 4 * i];
  cp_async_wait<0>();
  __syncthreads();
  float lo[8][4], hi[8][4];  // columns cg 4 .. + 3 and 32 further
#pragma unroll
  for (int i = 0; i < 8; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) lo[i][j] = hi[i][j] = 0.f;
  auto word = [&](const float* rows, int row_stride, const float* m_s, int wd) {
    float4 m[4];
#pragma unroll
    for (int e = 0; e < 4; ++e) m[e] = *reinterpret_cast<const float4*>(m_s + (4 * wd + e) * CH_WIDE + cg * 4);
    ch_step<8>(lo, m, rows + rg * row_stride + wd * 4, 4 * row_stride);
#pragma unroll
    for (int e = 0; e < 4; ++e) m[e] = *reinterpret_cast<const float4*>(m_s + (4 * wd + e) * CH_WIDE + 32 + cg * 4);
    ch_step<8>(hi, m, rows + rg * row_stride + wd * 4, 4 * row_stride);
  };
#pragma unroll 2
  for (int wd = warp; wd < WORDS; wd += 4) word(sm + L::Q, DP, sm + L::S, wd);
#pragma unroll
  for (int i = 0; i < 8; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      lo[i][j] *= grown[i];
      hi[i][j] *= grown[i];
    }
#pragma unroll
  for (int wd = warp; wd < CH / 4; wd += 4) word(sm + L::P, CH, sm + L::V, wd);
  __syncthreads();
  float* part = sm + L::S + warp * CH * CH_WIDE;
#pragma unroll
  for (int i = 0; i < 8; ++i) {
    store_floats<float, 4>(part + (rg + 4 * i) * CH_WIDE + cg * 4, lo[i]);
    store_floats<float, 4>(part + (rg + 4 * i) * CH_WIDE + 32 + cg * 4, hi[i]);
  }
  __syncthreads();
#pragma unroll
  for (int i = tid; i < CH * WIDE_WORDS; i += 128) {
    const int r = i / WIDE_WORDS, wd = i % WIDE_WORDS;
    if (r >= n || col0 + wd * 4 >= dv) continue;
    float x[4], y[4];
    load_floats<float, 4>(sm + L::S + i * 4, x);
#pragma unroll
    for (int w = 1; w < 4; ++w) {
      load_floats<float, 4>(sm + L::S + w * CH * CH_WIDE + i * 4, y);
#pragma unroll
      for (int j = 0; j < 4; ++j) x[j] += y[j];
    }
    store_floats<float, 4>(a.out + ((tok0 + r) * H + h) * dv + col0 + wd * 4, x);
  }
}

// ---- with the delta rule -------------------------------------------------------------------------------------------- //
template <int DP>
struct ChunkScanSmem {  // offsets in floats
  static constexpr int ROWS = CH * DP, COL_LD = CH_COLS + 4;
  static constexpr int Q = 0, W = Q + 2 * ROWS, K = W + 2 * ROWS, P = K + ROWS, U = P + CH * CH;
  static constexpr int F = U + CH * COL_LD, S = F + CH_FACTORS, X = S + DP * COL_LD, Y = X + CH * COL_LD;
  static constexpr int FLOATS = Y + CH * COL_LD;
  static constexpr size_t BYTES = (size_t)FLOATS * sizeof(float);
};

// The four lanes kg = 0 .. 3 of a tile hold partial sums of its four rows: afterwards lane kg holds the full sums of row
// number 2 (kg & 1) + (kg >> 1).
__device__ __forceinline__ float4 ch_reduce(const float (&acc)[4][4], int kg) {
  float half[2][4];
  const bool odd = kg & 1;
#pragma unroll
  for (int i = 0; i < 2; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const float give = odd ? acc[i][j] : acc[i + 2][j], keep = odd ? acc[i + 2][j] : acc[i][j];
      half[i][j] = keep + __shfl_xor_sync(0xffffffffu, give, 1);
    }
  const bool upper = kg & 2;
  float out[4];
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    const float give = upper ? half[0][j] : half[1][j], keep = upper ? half[1][j] : half[0][j];
    out[j] = keep + __shfl_xor_sync(0xffffffffu, give, 2);
  }
  return make_float4(out[0], out[1], out[2], out[3]);
}

// Where columns 4 cg .. + 3 of row `row` lie in a tile of 16 columns (rows of COL_LD floats): the column group is XORed with
// a bit of the row's word, so that the eight lanes of a quarter warp (four words kg, two column groups) meet 32 banks.
template <int LD>
__device__ __forceinline__ int ch_place(int row, int cg) { return row * LD + ((cg ^ (((row >> 3) & 1) << 1)) << 2); }

// grid (ceil(dv / 16), H, sequences), 128 threads.  For products with S a thread owns rows rg + 8 i (i < 4) of the run,
// four columns and a quarter of the contraction (every fourth 16-byte word).
template <int DP>
__global__ void __launch_bounds__(128, 2) state_chunk_scan_kernel(ChunkArgs a) {
  using L = ChunkScanSmem<DP>;
  constexpr int WORDS = DP / 4, LD = L::COL_LD, RS = DP / 32;
  extern __shared__ __align__(16) float sm[];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int kg = lane & 3, cg = (lane >> 2) & 3, rg = 2 * warp + (lane >> 4);
  const int row_of_lane = rg + 8 * (2 * (kg & 1) + (kg >> 1));  // the row whose sums this lane ends up with
  const int col0 = blockIdx.x * CH_COLS, h = blockIdx.y, seq = blockIdx.z;
  const int H = a.n_heads, G = a.n_kv_heads, d = a.d, dv = a.dv, kvh = h / (H / G);
  const int len = a.seq_qlen[seq], n_runs = (len + CH - 1) / CH;
  const int run0 = a.seq_run0[seq];
  const size_t tok_base = (size_t)a.seq_qstart[seq];

  // A thread copies one word of every (128 / WORDS)-th row: its place in the first of them, in each matrix
  constexpr int STEP = 128 / WORDS;
  const int load_row = tid / WORDS, load_word = (tid % WORDS) * 4;
  const bool load_col = load_word < d;
  const size_t qk_ld = (size_t)G * d;
  const float* q_at = a.q + (tok_base + load_row) * qk_ld + (size_t)kvh * d + load_word;
  const float* k_at = a.k + (tok_base + load_row) * qk_ld + (size_t)kvh * d + load_word;
  const float* w_at = a.w + (((size_t)run0 * H + h) * CH + load_row) * d + load_word;
  const float* p_at = a.p + ((size_t)run0 * H + h) * CH * CH + tid * 4;
  const float* u_at = a.u + (((size_t)run0 * H + h) * CH + (tid >> 2)) * dv + col0 + (tid & 3) * 4;
  const float* f_at = a.factors + ((size_t)run0 * H + h) * CH_FACTORS + tid * 4;
  auto load_products = [&](int c) {  // Q and W of run c, which follow those of run c - 1
    float* q_s = sm + L::Q + (c & 1) * L::ROWS + tid * 4;
    float* w_s = sm + L::W + (c & 1) * L::ROWS + tid * 4;
    const int rows = load_col ? len - c * CH - load_row : 0;
#pragma unroll 2
    for (int j = 0; j < CH / STEP; ++j) {
      const bool in = j * STEP < rows;
      ch_copy16(q_s + j * 512, in ? q_at + j * STEP * qk_ld : a.q, in);
      ch_copy16(w_s + j * 512, load_col ? w_at + (size_t)j * STEP * d : a.w, load_col);
    }
    q_at += CH * qk_ld;
    w_at += (size_t)H * CH * d;
  };
  auto load_writes = [&](int c) {  // K, P, U and the factors of run c, likewise
    float* k_s = sm + L::K + tid * 4;
    const int rows = load_col ? len - c * CH - load_row : 0;
#pragma unroll 2
    for (int j = 0; j < CH / STEP; ++j) {
      const bool in = j * STEP < rows;
      ch_copy16(k_s + j * 512, in ? k_at + j * STEP * qk_ld : a.k, in);
    }
    ch_copy16(sm + L::P + tid * 4, p_at, true);
    ch_copy16(sm + L::P + tid * 4 + 512, p_at + 512, true);
    const bool in = col0 + (tid & 3) * 4 < dv;
    ch_copy16(sm + L::U + (tid >> 2) * LD + (tid & 3) * 4, in ? u_at : a.u, in);
    if (tid < CH_FACTORS / 4) ch_copy16(sm + L::F + tid * 4, f_at, true);
    k_at += CH * qk_ld;
    p_at += (size_t)H * CH * CH;
    u_at += (size_t)H * CH * dv;
    f_at += (size_t)H * CH_FACTORS;
  };

  // this thread's piece of the state: rows dg RS .. + RS - 1, columns 4 sc .. 4 sc + 3
  const int sc = tid & 3, dg = tid >> 2;
  float s[RS][4];
  float* S = a.state + ((size_t)a.seq_slot[seq] * H + h) * d * dv;
  const bool s_col = col0 + sc * 4 < dv;
#pragma unroll
  for (int i = 0; i < RS; ++i) {
    const int row = dg * RS + i;
    float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
    if (row < d && s_col) x = *reinterpret_cast<const float4*>(S + (size_t)row * dv + col0 + sc * 4);
    s[i][0] = x.x; s[i][1] = x.y; s[i][2] = x.z; s[i][3] = x.w;
    *reinterpret_cast<float4*>(sm + L::S + ch_place<LD>(row, sc)) = x;
  }
  load_products(0);
  cp_async_commit();
  load_writes(0);
  cp_async_commit();
  for (int c = 0; c < n_runs; ++c) {
    if (c + 1 < n_runs) load_products(c + 1);
    cp_async_commit();
    cp_async_wait<2>();  // this run's Q and W; its K, P, U and the next run's Q and W may still be on their way
    __syncthreads();
    const float* q_s = sm + L::Q + (c & 1) * L::ROWS + rg * DP;
    const float* w_s = sm + L::W + (c & 1) * L::ROWS + rg * DP;
    float acc[4][4], corr[4][4];
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) acc[i][j] = corr[i][j] = 0.f;
    // rolled loops: the whole of a run's work unrolled is more than the instruction caches hold
#pragma unroll 2
    for (int step = 0; step < WORDS / 4; ++step) {
      const int wd = kg + 4 * step;
      float4 m[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) m[e] = *reinterpret_cast<const float4*>(sm + L::S + ch_place<LD>(4 * wd + e, cg));
      ch_step<4>(acc, m, q_s + wd * 4, 8 * DP);
      ch_step<4>(corr, m, w_s + wd * 4, 8 * DP);
    }
    cp_async_wait<1>();
    __syncthreads();  // K, P, U and the factors are here
    const float* f = sm + L::F;
    {
      float4 x = *reinterpret_cast<const float4*>(sm + L::U + row_of_lane * LD + cg * 4);
      const float4 y = ch_reduce(corr, kg);
      x.x -= y.x; x.y -= y.y; x.z -= y.z; x.w -= y.w;
      const float left = f[CH + row_of_lane];
      *reinterpret_cast<float4*>(sm + L::X + ch_place<LD>(row_of_lane, cg)) = x;
      *reinterpret_cast<float4*>(sm + L::Y + row_of_lane * LD + cg * 4) = make_float4(left * x.x, left * x.y, left * x.z, left * x.w);
    }
    __syncthreads();
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const float grown = f[rg + 8 * i];
#pragma unroll
      for (int j = 0; j < 4; ++j) acc[i][j] *= grown;
    }
#pragma unroll 1
    for (int step = 0; step < CH / 16; ++step) {
      const int wd = kg + 4 * step;
      float4 m[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) m[e] = *reinterpret_cast<const float4*>(sm + L::X + ch_place<LD>(4 * wd + e, cg));
      ch_step<4>(acc, m, sm + L::P + rg * CH + wd * 4, 8 * CH);
    }
    {
      const float4 o = ch_reduce(acc, kg);
      const int t = c * CH + row_of_lane;
      if (t < len && col0 + cg * 4 < dv)
        *reinterpret_cast<float4*>(a.out + ((tok_base + t) * H + h) * dv + col0 + cg * 4) = o;
    }
    const float left = f[2 * CH];
#pragma unroll
    for (int i = 0; i < RS; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) s[i][j] *= left;
#pragma unroll 8
    for (int t = 0; t < CH; ++t) {
      float kr[RS];
      load_floats<float, RS>(sm + L::K + t * DP + dg * RS, kr);
      const float4 y = *reinterpret_cast<const float4*>(sm + L::Y + t * LD + sc * 4);
#pragma unroll
      for (int i = 0; i < RS; ++i) {
        s[i][0] = fmaf(kr[i], y.x, s[i][0]); s[i][1] = fmaf(kr[i], y.y, s[i][1]);
        s[i][2] = fmaf(kr[i], y.z, s[i][2]); s[i][3] = fmaf(kr[i], y.w, s[i][3]);
      }
    }
#pragma unroll
    for (int i = 0; i < RS; ++i)  // nobody reads S between the barrier behind the products with it and the next run's
      *reinterpret_cast<float4*>(sm + L::S + ch_place<LD>(dg * RS + i, sc)) = make_float4(s[i][0], s[i][1], s[i][2], s[i][3]);
    __syncthreads();
    if (c + 1 < n_runs) load_writes(c + 1);
    cp_async_commit();
  }
  if (s_col) {
#pragma unroll
    for (int i = 0; i < RS; ++i) {
      const int row = dg * RS + i;
      if (row < d) *reinterpret_cast<float4*>(S + (size_t)row * dv + col0 + sc * 4) = make_float4(s[i][0], s[i][1], s[i][2], s[i][3]);
    }
  }
}

template <typename Kernel>
static int reserve(Kernel kernel, size_t smem) {
  const cudaError_t err = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  if (err == cudaSuccess) return 0;
  mll_set_error("state chunks: cannot reserve %zu bytes of shared memory: %s", smem, cudaGetErrorString(err));
  return (int)err;
}

template <int DP>
static int launch_chunks(const ChunkArgs& a, int n_runs, int n_seqs, cudaStream_t stream) {
  if (a.beta) {
    MLL_LAUNCH((state_chunk_inputs_kernel<DP, true>), dim3(n_runs, a.n_heads), 128, 0, stream, a);
    MLL_LAUNCH_CHECK();
    constexpr size_t smem = ChunkScanSmem<DP>::BYTES;
    if (const int err = reserve(state_chunk_scan_kernel<DP>, smem)) return err;
    MLL_LAUNCH((state_chunk_scan_kernel<DP>), dim3((a.dv + CH_COLS - 1) / CH_COLS, a.n_heads, n_seqs), 128, smem, stream, a);
    MLL_LAUNCH_CHECK();
    return 0;
  }
  const dim3 tiles(n_runs, a.n_heads, (a.dv + CH_WIDE - 1) / CH_WIDE);
  MLL_LAUNCH((state_chunk_inputs_kernel<DP, false>), dim3(n_runs, a.n_heads), 128, 0, stream, a);
  MLL_LAUNCH_CHECK();
  MLL_LAUNCH((state_chunk_sums_kernel<DP>), tiles, 128, 0, stream, a);
  MLL_LAUNCH_CHECK();
  const unsigned words = (unsigned)(((long long)a.d * a.dv + 1023) / 1024);
  MLL_LAUNCH((state_chunk_prefix_kernel), dim3(words, a.n_heads, n_seqs), 256, 0, stream, a);
  MLL_LAUNCH_CHECK();
  constexpr size_t smem = ChunkOutputsSmem<DP>::BYTES;
  if (const int err = reserve(state_chunk_outputs_kernel<DP>, smem)) return err;
  MLL_LAUNCH((state_chunk_outputs_kernel<DP>), tiles, 128, smem, stream, a);
  MLL_LAUNCH_CHECK();
  return 0;
}

}  // namespace mll

// Tokens a run of mll_state_chunks.
MLL_API int mll_state_chunk_tokens() { return mll::CH; }

MLL_API int mll_state_chunks_supported(int d, int dv) { return d > 0 && d <= 128 && d % 4 == 0 && dv > 0 && dv % 4 == 0; }

// Floats of scratch memory for `n_runs` runs.
MLL_API long long mll_state_chunks_scratch(int n_runs, int n_heads, int d, int dv, int delta) {
  return (long long)n_runs * n_heads * (mll::CH * mll::CH + mll::CH_FACTORS + (delta ? mll::CH * (d + dv) : d * dv));
}

// As mll_state_scan modes 0, 3 (token_decay given) and 4 (beta too), a run of tokens at a time.  run_seq, run_row0
// [n_runs]: every sequence's runs one after another, each of up to 32 tokens; seq_run0 [n_seqs]: its first run.
MLL_API int mll_state_chunks(const float* q, const float* k, const float* v, const float* beta, const float* token_decay,
                             const float* head_decay, float* state, float* out, float* scratch, const int* run_seq,
                             const int* run_row0, const int* seq_run0, const int* seq_slot, const int* seq_qstart,
                             const int* seq_qlen, int n_runs, int n_seqs, int n_heads, int n_kv_heads, int d, int dv,
                             cudaStream_t stream) {
  MLL_REQUIRE(n_runs >= 0 && n_seqs >= 0 && n_heads > 0 && n_kv_heads > 0 && n_heads % n_kv_heads == 0, "state chunks: bad head counts");
  MLL_REQUIRE(mll_state_chunks_supported(d, dv), "state chunks: head sizes %d / %d", d, dv);
  MLL_REQUIRE(n_heads <= 65535 && n_seqs <= 65535, "state chunks: too many heads or sequences for one launch");
  MLL_REQUIRE((token_decay == nullptr) != (head_decay == nullptr) && (!beta || token_decay), "state chunks: the decay's inputs do not fit");
  MLL_REQUIRE(((uintptr_t)q | (uintptr_t)k | (uintptr_t)v | (uintptr_t)state | (uintptr_t)out | (uintptr_t)scratch) % 16 == 0,
              "state chunks: operands must be 16-byte aligned");
  if (n_seqs == 0 || n_runs == 0) return 0;
  const size_t pairs = (size_t)n_runs * n_heads;
  float* p = scratch;
  float* factors = p + pairs * mll::CH * mll::CH;
  float* u = factors + pairs * mll::CH_FACTORS;
  float* w = u + pairs * mll::CH * dv;  // without the delta rule the runs' sums stand in the place of u and w
  mll::ChunkArgs a{q, k, v, beta, token_decay, head_decay, state, out, p, beta ? w : nullptr, beta ? u : nullptr, factors, beta ? nullptr : u,
                   run_seq, run_row0, seq_run0, seq_slot, seq_qstart, seq_qlen, n_heads, n_kv_heads, d, dv};
  if (d <= 32) return mll::launch_chunks<32>(a, n_runs, n_seqs, stream);
  if (d <= 64) return mll::launch_chunks<64>(a, n_runs, n_seqs, stream);
  return mll::launch_chunks<128>(a, n_runs, n_seqs, stream);
}
