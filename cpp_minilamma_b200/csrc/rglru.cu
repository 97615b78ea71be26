// A gated linear recurrent unit behind a short convolution:
//
//   u_t = conv(x_t + b_x) + b_c         causal, `taps` inputs per channel, nothing before a sequence's first token
//   r_t = sigmoid(A u_t + a),  i_t = sigmoid(I u_t + c)       A, I block-diagonal: n square blocks of `bs` channels
//   decay_t = exp(-rate * r_t * softplus(lam))      rate * softplus(lam) is a number per channel, formed once
//   S_t = decay_t S_(t-1) + sqrt(1 - decay_t^2) i_t u_t       one number per channel, float32, zero at the start
//   out_t = S_t * gelu(y_t + b_y)       (the tanh form)
//
// x and y are columns of one projection row.  u, the gates, the decays and the state are float32.
//
// Kernels (each for prompts and single tokens alike; a step's tokens of one sequence are consecutive rows):
//   * lru_gates       decay and write (sqrt(1 - decay^2) i u) of every token and channel.  A block owns a tile of tokens
//                     and channels of one diagonal block; it forms u for the tile's tokens and the whole diagonal
//                     block in shared memory and multiplies.  Two versions: float32 FMAs (any block size, either dtype),
//                     and mma.sync for bfloat16 matrices: u is cut into three bfloat16 terms that add up to all 24 bits
//                     of its float32 value, so the products are those of the float32 u, accumulated in float32.
//                     In steps of single tokens the same blocks also advance the state and write the output.
//   * lru_scan        the recurrence over a prompt's tokens: a warp per run of tokens, a lane per channel.  Every run is
//                     summarised (product of decays, state from zero), the runs' carries are chained through shared
//                     memory, and a second pass over the run applies the carry, multiplies by gelu(y) and writes.
#include "attention_decode.cuh"
#include "common.cuh"

namespace mll {

// 1 / (1 + e^-z); FAST: the hardware's exponential and reciprocal (a few units in the last place of a float32)
template <bool FAST>
__device__ __forceinline__ float lru_sigmoid(float z) {
  return FAST ? __fdividef(1.f, 1.f + __expf(-z)) : 1.f / (1.f + expf(-z));
}
template <bool FAST>
__device__ __forceinline__ float lru_sqrt(float x) {
  if (!FAST) return sqrtf(x);
  float r;
  asm("sqrt.approx.f32 %0, %1;" : "=f"(r) : "f"(x));
  return r;
}
// 1 - e^-x for x >= 0, given e = e^-x: near 0 by the first terms of its Taylor series (the next one is below 1e-9 of the
// result), else by the difference, which loses less than two bits there
__device__ __forceinline__ float lru_one_minus(float x, float e) {
  float p = fmaf(x, -1.f / 7.f, 1.f);
  p = fmaf(x * p, -1.f / 6.f, 1.f);
  p = fmaf(x * p, -1.f / 5.f, 1.f);
  p = fmaf(x * p, -1.f / 4.f, 1.f);
  p = fmaf(x * p, -1.f / 3.f, 1.f);
  p = fmaf(x * p, -1.f / 2.f, 1.f);
  return x < 0.25f ? x * p : 1.f - e;
}
__device__ __forceinline__ float lru_gelu(float z) {
  return 0.5f * z * (1.f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
}

struct LruArgs {
  const void* proj;         // [T, ld]: y in columns y_col .. + width, x in columns x_col .. + width
  const float* x_bias;      // [width]
  const float* y_bias;      // [width]
  const float* conv_w;      // [width, taps]
  const float* conv_b;      // [width]
  const float* conv_state;  // [slots, taps - 1, width]: the last inputs of every sequence, without x_bias
  const void* gate_w;       // mma: bfloat16 [n, 2, bs(out), bs(in)]; FMA: float32 [n, bs(in), 2 bs(out)]
  const float* gate_b;      // [2, width]: r's, then i's
  const float* rates;       // [width]: rate * softplus(lam)
  float* state;             // [slots, width]
  float* decay;             // [T, width]
  float* write;             // [T, width]
  void* out;                // [T, width] in the run's dtype
  const int* tok_pos;
  const int* tok_seq;
  const int* seq_slot;
  const int* seq_qstart;
  const int* seq_qlen;
  int n_tokens, ld, x_col, y_col, width, blocks, taps, single;
};

// u of token t, channel c (see above): inputs of this step come from the projection, earlier ones from the state.
template <typename T>
__device__ __forceinline__ float lru_conv(const LruArgs& a, int t, int c, int pos, int local, const float* state) {
  float u = a.conv_b[c];
  const float xb = a.x_bias[c];
  for (int back = 0; back < a.taps; ++back) {  // the input `back` tokens ago meets tap taps - 1 - back
    if (pos - back < 0) break;                  // before the sequence: nothing, not even the bias
    const float x = back <= local ? to_float(((const T*)a.proj)[(size_t)(t - back) * a.ld + a.x_col + c])
                                  : state[(size_t)(local - back + a.taps - 1) * a.width + c];
    u = fmaf(a.conv_w[(size_t)c * a.taps + (a.taps - 1 - back)], x + xb, u);
  }
  return u;
}

// What one channel brings to every token: the gates' biases, its rate, y's bias.
struct __align__(16) LruChannel {
  float br, bi, rate, yb;
};
__device__ __forceinline__ LruChannel lru_channel(const LruArgs& a, int c) {
  return {a.gate_b[c], a.gate_b[a.width + c], a.rates[c], a.y_bias[c]};
}

// From the two gates' pre-activations to the recurrence's inputs (decay, write).
template <bool FAST>
__device__ __forceinline__ float2 lru_inputs(const LruChannel& ch, float zr, float zi, float u) {
  const float r = lru_sigmoid<FAST>(zr + ch.br), i = lru_sigmoid<FAST>(zi + ch.bi);
  const float x = ch.rate * r;
  const float decay = expf(-x);
  return make_float2(decay, lru_sqrt<FAST>(lru_one_minus(2.f * x, decay * decay)) * i * u);
}

// A step of one token: the state advances, the output is written.
template <typename T>
__device__ __forceinline__ void lru_advance(const LruArgs& a, const LruChannel& ch, int t, int slot, int c, float2 in) {
  float* S = a.state + (size_t)slot * a.width + c;
  const float y = to_float(((const T*)a.proj)[(size_t)t * a.ld + a.y_col + c]) + ch.yb;
  const float s = fmaf(in.x, *S, in.y);
  *S = s;
  ((T*)a.out)[(size_t)t * a.width + c] = from_float<T>(s * lru_gelu(y));
}

// grid (ceil(tokens / 16), n * ceil(bs / 64)), 256 threads: a thread owns one channel and four tokens.
template <typename T>
__global__ void __launch_bounds__(256) lru_gates_kernel(LruArgs a) {
  extern __shared__ float u_s[];  // [16][bs]
  const int bs = a.width / a.blocks, tiles = (bs + 63) / 64;
  const int block = blockIdx.y / tiles, col = (blockIdx.y % tiles) * 64 + (threadIdx.x & 63);
  const int t0 = blockIdx.x * 16, n = min(16, a.n_tokens - t0);
  for (int i = threadIdx.x; i < n * bs; i += 256) {
    const int t = t0 + i / bs, seq = a.tok_seq[t];
    u_s[i] = lru_conv<T>(a, t, block * bs + i % bs, a.tok_pos[t], t - a.seq_qstart[seq],
                         a.conv_state + (size_t)a.seq_slot[seq] * (a.taps - 1) * a.width);
  }
  __syncthreads();
  if (col >= bs) return;
  const float* w = (const float*)a.gate_w + (size_t)block * bs * 2 * bs;
  const int q0 = (threadIdx.x >> 6) * 4;
  float r[4] = {0.f, 0.f, 0.f, 0.f}, z[4] = {0.f, 0.f, 0.f, 0.f};
  for (int k = 0; k < bs; ++k) {
    const float wr = w[(size_t)k * 2 * bs + col], wi = w[(size_t)k * 2 * bs + bs + col];
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const float u = q0 + i < n ? u_s[(q0 + i) * bs + k] : 0.f;
      r[i] = fmaf(wr, u, r[i]);
      z[i] = fmaf(wi, u, z[i]);
    }
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
    if (q0 + i < n) {
      const int t = t0 + q0 + i, c = block * bs + col;
      const LruChannel ch = lru_channel(a, c);
      const float2 in = lru_inputs<false>(ch, r[i], z[i], u_s[(q0 + i) * bs + col]);
      if (a.single) {
        lru_advance<T>(a, ch, t, a.seq_slot[a.tok_seq[t]], c, in);
      } else {
        a.decay[(size_t)t * a.width + c] = in.x;
        a.write[(size_t)t * a.width + c] = in.y;
      }
    }
}

// grid (ceil(tokens / M), n * column parts), 256 threads; M = 16 WM MT tokens.  A block forms u for its tokens and one
// whole diagonal block in shared memory - three bfloat16 planes [3][M][row] (high, middle, low term) - and walks `passes`
// runs of 64 channels of it.  Warps: WM along the tokens, 8 / WM along the channels; a warp owns MT x 16 tokens and NT x 8
// channels of both gates, so that a thread ends with r and i of the same (token, channel) pairs.
// The k-order inside a product is free as long as both operands agree: a thread's 16 bytes (eight neighbouring inputs)
// serve two k-steps.
template <int WM, int MT, int NT>
__global__ void __launch_bounds__(256) lru_gates_mma_kernel(LruArgs a, int row, int passes) {
  extern __shared__ __align__(16) __nv_bfloat16 planes[];
  constexpr int M = 16 * WM * MT;
  static_assert(8 / WM * NT * 8 == 64, "a pass covers 64 channels");
  __shared__ int pos_s[M], back_s[M];           // a token's position; how many of its inputs lie in this step
  __shared__ int slot_s[M];                     // its sequence's slot
  const int bs = a.width / a.blocks, tiles = (bs + 63) / 64, parts = (tiles + passes - 1) / passes;
  const int block = blockIdx.y / parts, tile0 = (blockIdx.y % parts) * passes, tile1 = min(tiles, tile0 + passes);
  const int t0 = blockIdx.x * M, n = min(M, a.n_tokens - t0);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, q = lane & 3;
  const int k_pad = (bs + 31) & ~31;
  LruChannel* channel_s = reinterpret_cast<LruChannel*>(planes + (size_t)3 * M * row);  // of the block's channels
  for (int i = threadIdx.x; i < min(bs, tile1 * 64) - tile0 * 64; i += 256) channel_s[i] = lru_channel(a, block * bs + tile0 * 64 + i);
  if (threadIdx.x < M && threadIdx.x < n) {
    const int t = t0 + threadIdx.x, seq = a.tok_seq[t];
    pos_s[threadIdx.x] = a.tok_pos[t];
    back_s[threadIdx.x] = t - a.seq_qstart[seq];
    slot_s[threadIdx.x] = a.seq_slot[seq];
  }
  __syncthreads();
  // u: a thread owns a pair of channels and every (256 / pairs)-th token
  const __nv_bfloat16* proj = (const __nv_bfloat16*)a.proj;
  const int pairs = k_pad / 2;
  for (int p = threadIdx.x % min(pairs, 256); p < pairs; p += 256) {
    const int k = 2 * p, c = block * bs + k;
    const bool real = k < bs;  // bs is even: both channels or none
    const float2 xb = real ? make_float2(a.x_bias[c], a.x_bias[c + 1]) : make_float2(0.f, 0.f);
    const float2 cb = real ? make_float2(a.conv_b[c], a.conv_b[c + 1]) : make_float2(0.f, 0.f);
    const float* w = a.conv_w + (size_t)c * a.taps + a.taps - 1;
    float2 w4[4];  // the taps of the last four inputs stay in registers
#pragma unroll
    for (int i = 0; i < 4; ++i) w4[i] = real && i < a.taps ? make_float2(w[-i], w[a.taps - i]) : make_float2(0.f, 0.f);
    const int step = pairs >= 256 ? 1 : 256 / pairs;
    if (pairs < 256 && threadIdx.x >= step * pairs) break;
#pragma unroll 4
    for (int m = pairs >= 256 ? 0 : threadIdx.x / pairs; m < M; m += step) {
      float2 u = make_float2(0.f, 0.f);
      if (real && m < n) {
        u = cb;
        const int local = back_s[m], reach = min(a.taps - 1, pos_s[m]);  // nothing before the sequence, not even the bias
        const __nv_bfloat16* x0 = proj + (size_t)(t0 + m) * a.ld + a.x_col + c;
        const float* s0 = a.conv_state + ((size_t)slot_s[m] * (a.taps - 1) + local + a.taps - 1) * a.width + c;
        auto input = [&](int back) {
          if (back <= local)
            return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(x0 - (size_t)back * a.ld));
          return make_float2(s0[-(ptrdiff_t)back * a.width], s0[1 - (ptrdiff_t)back * a.width]);
        };
        float2 x[4];
#pragma unroll
        for (int back = 0; back < 4; ++back)
          if (back <= reach) x[back] = input(back);
#pragma unroll
        for (int back = 0; back < 4; ++back)
          if (back <= reach) {
            u.x = fmaf(w4[back].x, x[back].x + xb.x, u.x);
            u.y = fmaf(w4[back].y, x[back].y + xb.y, u.y);
          }
        for (int back = 4; back <= reach; ++back) {
          const float2 v = input(back);
          u.x = fmaf(w[-back], v.x + xb.x, u.x);
          u.y = fmaf(w[a.taps - back], v.y + xb.y, u.y);
        }
      }
      const __nv_bfloat162 hi = __floats2bfloat162_rn(u.x, u.y);
      const float2 h = __bfloat1622float2(hi);
      const float2 rest = make_float2(u.x - h.x, u.y - h.y);  // exact
      const __nv_bfloat162 mid = __floats2bfloat162_rn(rest.x, rest.y);
      const float2 f = __bfloat1622float2(mid);
      *reinterpret_cast<__nv_bfloat162*>(planes + (size_t)m * row + k) = hi;
      *reinterpret_cast<__nv_bfloat162*>(planes + (size_t)(M + m) * row + k) = mid;
      *reinterpret_cast<__nv_bfloat162*>(planes + (size_t)(2 * M + m) * row + k) = __floats2bfloat162_rn(rest.x - f.x, rest.y - f.y);
    }
  }
  __syncthreads();
  const int m0 = (warp % WM) * MT * 16, n0 = (warp / WM) * NT * 8;
  const __nv_bfloat16* w = (const __nv_bfloat16*)a.gate_w + (size_t)block * 2 * bs * bs;
  const uint4 zero = make_uint4(0, 0, 0, 0);
  for (int tile = tile0; tile < tile1; ++tile) {
    const int c0 = tile * 64 + n0;
    if (c0 >= bs) break;
    float acc[2][NT][MT][4];
#pragma unroll
    for (int e = 0; e < 2; ++e)
#pragma unroll
      for (int j = 0; j < NT; ++j)
#pragma unroll
        for (int m = 0; m < MT; ++m)
#pragma unroll
          for (int i = 0; i < 4; ++i) acc[e][j][m][i] = 0.f;
    const uint4* rows[2][NT];  // this lane's rows of the two matrices
    bool have[NT];
#pragma unroll
    for (int j = 0; j < NT; ++j) {
      const int col = min(c0 + 8 * j + g, bs - 1);
      have[j] = c0 + 8 * j + g < bs;
      rows[0][j] = reinterpret_cast<const uint4*>(w + (size_t)col * bs) + q;
      rows[1][j] = reinterpret_cast<const uint4*>(w + (size_t)(bs + col) * bs) + q;
    }
    uint4 next[2][NT];  // the matrices' words of the step ahead
    auto fetch = [&](int k) {
      const bool in = k + 8 * q < bs;  // bs is a multiple of 8: eight inputs are inside or outside together
#pragma unroll
      for (int e = 0; e < 2; ++e)
#pragma unroll
        for (int j = 0; j < NT; ++j) next[e][j] = in && have[j] ? rows[e][j][k >> 3] : zero;
    };
    fetch(0);
#pragma unroll 2
    for (int k = 0; k < k_pad; k += 32) {
      uint4 b[2][NT];
#pragma unroll
      for (int e = 0; e < 2; ++e)
#pragma unroll
        for (int j = 0; j < NT; ++j) b[e][j] = next[e][j];
      if (k + 32 < k_pad) fetch(k + 32);
#pragma unroll
      for (int p = 0; p < 3; ++p)
#pragma unroll
        for (int m = 0; m < MT; ++m) {
          const __nv_bfloat16* src = planes + (size_t)(p * M + m0 + m * 16 + g) * row + k + 8 * q;
          const uint4 lo = *reinterpret_cast<const uint4*>(src);
          const uint4 up = *reinterpret_cast<const uint4*>(src + 8 * row);
          const unsigned a0[4] = {lo.x, up.x, lo.y, up.y}, a1[4] = {lo.z, up.z, lo.w, up.w};
#pragma unroll
          for (int e = 0; e < 2; ++e)
#pragma unroll
            for (int j = 0; j < NT; ++j) {
              mma_16816(acc[e][j][m], a0, b[e][j].x, b[e][j].y);
              mma_16816(acc[e][j][m], a1, b[e][j].z, b[e][j].w);
            }
        }
    }
#pragma unroll
    for (int j = 0; j < NT; ++j) {
      const int c = c0 + 8 * j + 2 * q, full = block * bs + c;  // a pair of channels: bs is even, both or none
      if (c >= bs) continue;
      const LruChannel ch0 = channel_s[c - tile0 * 64], ch1 = channel_s[c - tile0 * 64 + 1];
#pragma unroll
      for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          const int tok = m0 + m * 16 + g + 8 * half, t = t0 + tok;
          if (tok >= n) continue;
          const unsigned* src = reinterpret_cast<const unsigned*>(planes + (size_t)tok * row + c);
          const float2 h = unpack_bf162(src[0]), mid = unpack_bf162(src[(size_t)M * row / 2]), lo = unpack_bf162(src[(size_t)M * row]);
          const float2 in0 = lru_inputs<true>(ch0, acc[0][j][m][2 * half], acc[1][j][m][2 * half], (h.x + mid.x) + lo.x);
          const float2 in1 = lru_inputs<true>(ch1, acc[0][j][m][2 * half + 1], acc[1][j][m][2 * half + 1], (h.y + mid.y) + lo.y);
          if (a.single) {
            lru_advance<__nv_bfloat16>(a, ch0, t, slot_s[tok], full, in0);
            lru_advance<__nv_bfloat16>(a, ch1, t, slot_s[tok], full + 1, in1);
          } else {
            const size_t at = (size_t)t * a.width + full;
            *reinterpret_cast<float2*>(a.decay + at) = make_float2(in0.x, in1.x);
            *reinterpret_cast<float2*>(a.write + at) = make_float2(in0.y, in1.y);
          }
        }
    }
  }
}

// grid (ceil(width / 32), sequences), (32, runs) threads: lane = channel, warp = run of tokens.
template <typename T>
__global__ void __launch_bounds__(1024) lru_scan_kernel(LruArgs a) {
  __shared__ float prod_s[32][33], end_s[32][33];
  const int lane = threadIdx.x, run = threadIdx.y, runs = blockDim.y;
  const int seq = blockIdx.y, c = blockIdx.x * 32 + lane;
  const int row0 = a.seq_qstart[seq], n = a.seq_qlen[seq];
  const int per = (n + runs - 1) / runs;
  const int lo = row0 + min(n, run * per), hi = row0 + min(n, (run + 1) * per);
  const bool live = c < a.width;
  const float* dec = a.decay + c;
  const float* wri = a.write + c;
  float* S = a.state + (size_t)a.seq_slot[seq] * a.width + c;
  float carry = live ? *S : 0.f;
  if (runs > 1) {
    float prod = 1.f, s = 0.f;
    if (live) {
      int t = lo;
      for (; t + 8 <= hi; t += 8) {
        float d[8], w[8];
#pragma unroll
        for (int i = 0; i < 8; ++i) {
          d[i] = dec[(size_t)(t + i) * a.width];
          w[i] = wri[(size_t)(t + i) * a.width];
        }
#pragma unroll
        for (int i = 0; i < 8; ++i) {
          s = fmaf(d[i], s, w[i]);
          prod *= d[i];
        }
      }
      for (; t < hi; ++t) {
        const float d = dec[(size_t)t * a.width];
        s = fmaf(d, s, wri[(size_t)t * a.width]);
        prod *= d;
      }
    }
    prod_s[run][lane] = prod;
    end_s[run][lane] = s;
    __syncthreads();  // every run has read the old state too: the last one may write it below
    for (int e = 0; e < run; ++e) carry = fmaf(prod_s[e][lane], carry, end_s[e][lane]);
  }
  if (!live) return;
  const float yb = a.y_bias[c];
  const T* y = (const T*)a.proj + a.y_col + c;
  T* out = (T*)a.out + c;
  int t = lo;
  for (; t + 8 <= hi; t += 8) {
    float d[8], w[8], v[8];
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      d[i] = dec[(size_t)(t + i) * a.width];
      w[i] = wri[(size_t)(t + i) * a.width];
      v[i] = to_float(y[(size_t)(t + i) * a.ld]);
    }
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      carry = fmaf(d[i], carry, w[i]);
      out[(size_t)(t + i) * a.width] = from_float<T>(carry * lru_gelu(v[i] + yb));
    }
  }
  for (; t < hi; ++t) {
    carry = fmaf(dec[(size_t)t * a.width], carry, wri[(size_t)t * a.width]);
    out[(size_t)t * a.width] = from_float<T>(carry * lru_gelu(to_float(y[(size_t)t * a.ld]) + yb));
  }
  if (hi == row0 + n && lo < hi) *S = carry;  // exactly one run ends with the sequence's last token
}

// Bytes of shared memory and elements between rows of a plane: 16-byte words of neighbouring rows in different banks.
inline int lru_plane_row(int bs) { return ((bs + 31) / 32) * 32 + (((bs + 31) / 32) % 2 ? 0 : 32); }

template <int WM, int MT, int NT>
int launch_lru_gates_mma(const LruArgs& a, cudaStream_t stream) {
  constexpr int M = 16 * WM * MT;
  const int bs = a.width / a.blocks, row = lru_plane_row(bs), tiles = (bs + 63) / 64;
  // a block that walks more channels forms u once for all of them; enough blocks for the device come first
  const int n_tiles = (a.n_tokens + M - 1) / M;
  int passes = tiles;
  while (passes > 1 && (long long)n_tiles * a.blocks * ((tiles + passes - 1) / passes) < mll_sm_count()) passes = (passes + 1) / 2;
  const size_t smem = (size_t)3 * M * row * 2 + (size_t)passes * 64 * sizeof(LruChannel);
  auto kernel = lru_gates_mma_kernel<WM, MT, NT>;
  if (smem > 48 * 1024) {
    cudaError_t err = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (err != cudaSuccess) {
      mll_set_error("linear recurrent unit: cannot reserve %zu bytes of shared memory: %s", smem, cudaGetErrorString(err));
      return (int)err;
    }
  }
  const dim3 grid(n_tiles, a.blocks * ((tiles + passes - 1) / passes));
  MLL_LAUNCH((kernel), grid, 256, smem, stream, a, row, passes);
  MLL_LAUNCH_CHECK();
  return 0;
}

template <typename T>
int launch_lru_gates(const LruArgs& a, cudaStream_t stream) {
  const int bs = a.width / a.blocks;
  const size_t smem = (size_t)16 * bs * sizeof(float);
  auto kernel = lru_gates_kernel<T>;
  if (smem > 48 * 1024) {
    cudaError_t err = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (err != cudaSuccess) {
      mll_set_error("linear recurrent unit: cannot reserve %zu bytes of shared memory: %s", smem, cudaGetErrorString(err));
      return (int)err;
    }
  }
  const dim3 grid((a.n_tokens + 15) / 16, a.blocks * ((bs + 63) / 64));
  MLL_LAUNCH((kernel), grid, 256, smem, stream, a);
  MLL_LAUNCH_CHECK();
  return 0;
}

}  // namespace mll

// Whether the tensor-core version takes diagonal blocks of this size (bfloat16 matrices).
MLL_API int mll_lru_mma_supported(int dtype, int bs) {
  return dtype == MLL_BF16 && bs % 8 == 0 && bs >= 8 && (size_t)3 * 16 * mll::lru_plane_row(bs) * 2 <= 160 * 1024;  // and the channels' numbers beside them
}

// `mma`: gate_w is bfloat16 [n, 2, bs, bs] (rows are outputs), else float32 [n, bs(in), 2 bs(out)].
// `single`: every sequence brings one token; the state advances and `out` is written here (decay, write may be null).
MLL_API int mll_lru_gates(const void* proj, const float* x_bias, const float* y_bias, const float* conv_w,
                          const float* conv_b, const float* conv_state, const void* gate_w, const float* gate_b,
                          const float* rates, float* state, float* decay, float* write, void* out, const int* tok_pos,
                          const int* tok_seq, const int* seq_slot, const int* seq_qstart, int dtype, int n_tokens, int ld,
                          int x_col, int y_col, int width, int blocks, int taps, int mma, int single,
                          cudaStream_t stream) {
  MLL_REQUIRE(n_tokens >= 0 && width > 0 && blocks > 0 && width % blocks == 0 && taps > 0, "linear recurrent unit: bad sizes");
  MLL_REQUIRE(x_col >= 0 && y_col >= 0 && x_col + width <= ld && y_col + width <= ld,
              "linear recurrent unit: columns outside rows of %d", ld);
  MLL_REQUIRE(single ? (state && out) : (decay && write), "linear recurrent unit: an output is missing");
  const int bs = width / blocks;
  MLL_REQUIRE((size_t)16 * bs * 4 <= 200 * 1024, "linear recurrent unit: blocks of %d exceed the 3200 the kernel takes", bs);
  MLL_REQUIRE((long long)blocks * ((bs + 63) / 64) <= 65535, "linear recurrent unit: too many blocks for one launch");
  if (n_tokens == 0) return 0;
  mll::LruArgs a{proj, x_bias, y_bias, conv_w, conv_b, conv_state, gate_w, gate_b, rates, state, decay, write, out, tok_pos,
                 tok_seq, seq_slot, seq_qstart, nullptr, n_tokens, ld, x_col, y_col, width, blocks, taps, single};
  if (mma) {
    MLL_REQUIRE(ld % 2 == 0 && x_col % 2 == 0 && (uintptr_t)proj % 4 == 0, "linear recurrent unit: projection rows must be pairs");
    MLL_REQUIRE(mll_lru_mma_supported(dtype, bs), "linear recurrent unit: blocks of %d on tensor cores", bs);
    const size_t per16 = (size_t)3 * 16 * mll::lru_plane_row(bs) * 2;
    // a tall tile reads the matrices less often, a low one gives more blocks
    if (n_tokens > 256 && 4 * per16 <= 190 * 1024) return mll::launch_lru_gates_mma<2, 2, 2>(a, stream);
    return mll::launch_lru_gates_mma<1, 1, 1>(a, stream);
  }
  if (dtype == MLL_F32) return mll::launch_lru_gates<float>(a, stream);
  if (dtype == MLL_BF16) return mll::launch_lru_gates<__nv_bfloat16>(a, stream);
  MLL_REQUIRE(false, "linear recurrent unit: unknown dtype %d", dtype);
  return -1;
}

// `longest`: the most tokens any sequence of the step brings (how many warps share a sequence follows from it).
MLL_API int mll_lru_scan(const float* decay, const float* write, const void* proj, const float* y_bias, float* state,
                         void* out, const int* seq_slot, const int* seq_qstart, const int* seq_qlen, int dtype, int n_seqs,
                         int ld, int y_col, int width, int longest, cudaStream_t stream) {
  MLL_REQUIRE(n_seqs >= 0 && n_seqs <= 65535 && width > 0 && longest >= 0 && y_col >= 0 && y_col + width <= ld,
              "linear recurrent scan: bad sizes");
  if (n_seqs == 0 || longest == 0) return 0;
  mll::LruArgs a{};
  a.decay = const_cast<float*>(decay); a.write = const_cast<float*>(write);
  a.proj = proj; a.y_bias = y_bias; a.state = state; a.out = out;
  a.seq_slot = seq_slot; a.seq_qstart = seq_qstart; a.seq_qlen = seq_qlen;
  a.ld = ld; a.y_col = y_col; a.width = width;
  const int runs = min(32, max(1, (longest + 15) / 16));
  const dim3 grid((width + 31) / 32, n_seqs), block(32, runs);
  if (dtype == MLL_F32)
    MLL_LAUNCH((mll::lru_scan_kernel<float>), grid, block, 0, stream, a);
  else if (dtype == MLL_BF16)
    MLL_LAUNCH((mll::lru_scan_kernel<__nv_bfloat16>), grid, block, 0, stream, a);
  else
    MLL_REQUIRE(false, "linear recurrent scan: unknown dtype %d", dtype);
  MLL_LAUNCH_CHECK();
  return 0;
}
