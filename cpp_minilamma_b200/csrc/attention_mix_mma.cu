// Attention with mixed scores and sigmoid weights (attention_mix.cu) in bfloat16 on tensor cores, for prompt tiles and
// for single tokens.
//
// A key's weight in head h needs the scores of all H heads at that key, so a block owns R query rows of one sequence with
// all their heads and walks the window in runs of N keys.  Per run:
//   1. S = q k^T by mma.sync: the 16 rows of a tile are R query rows of 16 / R heads of one key head's group; scores go to
//      shared memory as float32.
//   2. z = M S + b on the FMA pipe (two float32 FMAs an instruction), sigmoid, mask; weights go to shared memory as
//      bfloat16.  A thread holds a few positions of a few output heads, so M is read as broadcasts.
//   3. O += P V by mma.sync: a warp keeps up to TPW units of 16 rows x 64 value columns in registers for the whole walk.
// Nothing is normalised, so there is no running maximum and no rescaling, and context splits simply add up.
// K and V of a run have one buffer each: the next run's keys load while 2 and 3 work, its values while 1 and 2 do.
// Where the H x R rows' outputs exceed what one block's registers hold, grid y splits the output heads and every block
// recomputes the scores.
#include "attention_decode.cuh"
#include "attention_mix.cuh"

namespace mll {

struct MixMmaArgs {
  const __nv_bfloat16* q;
  const __nv_bfloat16* k_cache;
  const __nv_bfloat16* v_cache;
  const int* seq_slot;
  const int* seq_ctx;
  const int* seq_qstart;
  const int* seq_qlen;
  const int* tile_seq;    // prompt tiles of 64 rows; null: single tokens, grid x runs over the sequences
  const int* tile_row0;
  const int* block_table;
  const float* mix;       // [H, H] or null
  const float* bias;      // [H] or null
  __nv_bfloat16* out;
  float* part;            // [sequences, n_splits, H, dv] sums of the context's runs (n_splits > 1)
  int n_heads, n_kv_heads, d, dv, window, max_blocks, n_splits;
  float scale;
};

constexpr int MIX_WARPS = 8;

// Shared memory of a block, in bytes from its start.  Rows of q and P are compact: row h * R + r.
struct MixMmaLayout {
  int qs, vs, hp;                 // elements between rows of q / k and of v; heads rounded up to a multiple of 8
  int k, v, s, p, m, b, total;    // q starts at 0
};
__host__ __device__ inline MixMmaLayout mix_mma_layout(int H, int G, int d, int dv, int R, int N) {
  MixMmaLayout l;
  l.qs = ((d + 15) & ~15) + 8;
  l.vs = ((dv + 15) & ~15) + 8;
  l.hp = (H + 7) & ~7;
  int at = H * R * l.qs * 2;
  l.k = at; at += G * N * l.qs * 2;
  l.v = at; at += G * N * l.vs * 2;
  l.s = at; at += H * R * (N + 8) * 4;
  l.p = at; at += H * R * (N + 8) * 2;
  at = (at + 15) & ~15;
  l.m = at; at += H * l.hp * 4;
  l.b = at; at += l.hp * 4;
  l.total = at;
  return l;
}

typedef unsigned long long mix_f32x2;
__device__ __forceinline__ mix_f32x2 mix_pack2(float lo, float hi) {
  mix_f32x2 r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(lo), "f"(hi));
  return r;
}
__device__ __forceinline__ void mix_unpack2(mix_f32x2 v, float& lo, float& hi) {
  asm("mov.b64 {%0, %1}, %2;" : "=f"(lo), "=f"(hi) : "l"(v));
}
__device__ __forceinline__ mix_f32x2 mix_fma2(mix_f32x2 a, mix_f32x2 b, mix_f32x2 c) {
  mix_f32x2 r;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
  return r;
}
// large |z|: e^-z overflows to infinity (weight 0) or falls to 0 (weight 1)
__device__ __forceinline__ float mix_sigmoid(float z) { return __fdividef(1.f, 1.f + __expf(-z)); }

template <int R, int N, int TPW>
__global__ void __launch_bounds__(MIX_WARPS * 32, TPW <= 2 ? 2 : 1) mixed_attention_mma_kernel(MixMmaArgs a) {
  extern __shared__ __align__(16) unsigned char smem_raw[];
  constexpr int THREADS = MIX_WARPS * 32;
  constexpr int HPT = 16 / R;         // heads in the 16 rows of a tile
  constexpr int QP = R == 1 ? 1 : 2;  // tiles of one key head that share the key fragments in step 1
  constexpr int SS = N + 8;           // elements between rows of S and of P
  const int H = a.n_heads, G = a.n_kv_heads, group = H / G, d = a.d, dv = a.dv;
  const MixMmaLayout L = mix_mma_layout(H, G, d, dv, R, N);
  __nv_bfloat16* q_s = reinterpret_cast<__nv_bfloat16*>(smem_raw);
  __nv_bfloat16* k_s = reinterpret_cast<__nv_bfloat16*>(smem_raw + L.k);
  __nv_bfloat16* v_s = reinterpret_cast<__nv_bfloat16*>(smem_raw + L.v);
  float* s_s = reinterpret_cast<float*>(smem_raw + L.s);
  __nv_bfloat16* p_s = reinterpret_cast<__nv_bfloat16*>(smem_raw + L.p);
  float* m_s = reinterpret_cast<float*>(smem_raw + L.m);  // [H in][hp out], times scale
  float* b_s = reinterpret_cast<float*>(smem_raw + L.b);

  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int g = lane >> 2, t = lane & 3;
  const bool single = a.tile_seq == nullptr;
  constexpr int SUB = 64 / R;  // tiles of R rows in a listed tile of 64
  const int seq = single ? blockIdx.x : a.tile_seq[blockIdx.x / SUB];
  const int row0 = single ? 0 : a.tile_row0[blockIdx.x / SUB] + (int)(blockIdx.x % SUB) * R;
  const int ctx = a.seq_ctx[seq], qlen = single ? 1 : a.seq_qlen[seq];
  const int rows = min(R, qlen - row0);
  if (rows <= 0) return;
  const int pos0 = ctx - qlen + row0, last = pos0 + rows - 1;
  const int first = a.window > 0 ? max(0, pos0 - a.window + 1) : 0;
  const size_t tok0 = (size_t)a.seq_qstart[seq] + row0;
  const int* table = a.block_table + (size_t)a.seq_slot[seq] * a.max_blocks;
  int run = first / N, run_end = last / N + 1;
  if (a.n_splits > 1) {
    const int per = (run_end - run + a.n_splits - 1) / a.n_splits;
    run += (int)blockIdx.z * per;
    run_end = min(run_end, run + per);
  }

  // the units (16 rows x 64 value columns) of this block and warp; neighbours share a key head where they can
  const int tpg = (group + HPT - 1) / HPT;            // tiles of a key head
  const int cps = (L.vs - 8 + 63) / 64;               // column parts of a value head
  const int n_units = G * cps * tpg;
  const int unit0 = (int)blockIdx.y * MIX_WARPS * TPW;
  const int unit1 = min(n_units, unit0 + MIX_WARPS * TPW);
  const int kv_lo = unit0 / (cps * tpg), kv_hi = (unit1 - 1) / (cps * tpg);

  const int kw = (L.qs - 8) >> 3, vw = (L.vs - 8) >> 3;  // 16-byte words of a padded row
  auto load_run = [&](const __nv_bfloat16* cache, __nv_bfloat16* dst, int size, int stride, int words, int which) {
    const int page = table[which * N / MLL_PAGE];
    const int in_page = which * N % MLL_PAGE, valid = ctx - which * N;  // rows past the cached length hold no data
    for (int i = tid; i < N * words; i += THREADS) {
      const int r = i / words, c = (i - r * words) * 8;
      const bool in = c < size && r < valid;
      const __nv_bfloat16* src = cache + ((size_t)page * G * MLL_PAGE + in_page + r) * size + (in ? c : 0);
      for (int h = 0; h < G; ++h)
        cp_async16_zfill(dst + (size_t)(h * N + r) * stride + c, src + (size_t)h * MLL_PAGE * size, in);
    }
  };
  for (int i = tid; i < H * R * kw; i += THREADS) {
    const int row = i / kw, c = (i - row * kw) * 8, h = row / R, r = row % R;
    const bool in = c < d && r < rows;
    cp_async16_zfill(q_s + (size_t)row * L.qs + c, a.q + ((tok0 + (in ? r : 0)) * H + h) * d + (in ? c : 0), in);
  }
  if (run < run_end) load_run(a.k_cache, k_s, d, L.qs, kw, run);
  cp_async_commit();
  if (run < run_end) load_run(a.v_cache, v_s, dv, L.vs, vw, run);
  cp_async_commit();
  for (int i = tid; i < H * L.hp; i += THREADS) {
    const int in = i / L.hp, to = i % L.hp;
    m_s[i] = to < H ? (a.mix ? a.mix[(size_t)to * H + in] : (to == in ? 1.f : 0.f)) * a.scale : 0.f;
  }
  for (int i = tid; i < L.hp; i += THREADS) b_s[i] = (i < H && a.bias) ? a.bias[i] : 0.f;

  float o[TPW][8][4];
#pragma unroll
  for (int j = 0; j < TPW; ++j)
#pragma unroll
    for (int n = 0; n < 8; ++n)
#pragma unroll
      for (int i = 0; i < 4; ++i) o[j][n][i] = 0.f;

  // step 1's units: QP tiles of one key head against N keys (or, where that leaves warps idle, half of them)
  const int pairs = (tpg + QP - 1) / QP;
  const int halves = (N == 32 && G * pairs * 2 <= MIX_WARPS) ? 2 : 1;
  // row of q / P that the tile's row rr stands for (rows past the group repeat its last head and are not stored)
  auto compact = [&](int kv, int tile, int rr) { return (kv * group + min(tile * HPT + rr / R, group - 1)) * R + rr % R; };

  cp_async_wait<1>();
  __syncthreads();
  for (; run < run_end; ++run) {
    for (int u = warp; u < G * pairs * halves; u += MIX_WARPS) {
      const int half = u % halves, pair = (u / halves) % pairs, kv = u / (halves * pairs);
      const int np0 = half * (N / 16) / halves, np1 = (half + 1) * (N / 16) / halves;
      float acc[QP][N / 8][4];
#pragma unroll
      for (int m = 0; m < QP; ++m)
#pragma unroll
        for (int n = 0; n < N / 8; ++n)
#pragma unroll
          for (int i = 0; i < 4; ++i) acc[m][n][i] = 0.f;
      const __nv_bfloat16* qa[QP];
#pragma unroll
      for (int m = 0; m < QP; ++m)
        qa[m] = q_s + (size_t)compact(kv, min(pair * QP + m, tpg - 1), (lane & 7) + (((lane >> 3) & 1) << 3)) * L.qs + ((lane >> 4) << 3);
      const __nv_bfloat16* kb = k_s + (size_t)(kv * N + (lane & 7) + ((lane >> 4) << 3)) * L.qs + (((lane >> 3) & 1) << 3);
#pragma unroll 4
      for (int e = 0; e < L.qs - 8; e += 16) {
        unsigned qf[QP][4];
#pragma unroll
        for (int m = 0; m < QP; ++m) ldmatrix_x4(qf[m], qa[m] + e);
#pragma unroll
        for (int np = 0; np < N / 16; ++np) {
          if (np < np0 || np >= np1) continue;
          unsigned kf[4];
          ldmatrix_x4(kf, kb + (size_t)np * 16 * L.qs + e);
#pragma unroll
          for (int m = 0; m < QP; ++m) {
            mma_16816(acc[m][2 * np], qf[m], kf[0], kf[1]);
            mma_16816(acc[m][2 * np + 1], qf[m], kf[2], kf[3]);
          }
        }
      }
#pragma unroll
      for (int m = 0; m < QP; ++m) {
        const int tile = pair * QP + m;
        if (tile >= tpg) continue;
#pragma unroll
        for (int half8 = 0; half8 < 2; ++half8) {
          const int rr = g + 8 * half8;
          if (tile * HPT + rr / R >= group) continue;
          float* dst = s_s + (size_t)compact(kv, tile, rr) * SS + 2 * t;
#pragma unroll
          for (int n = 0; n < N / 8; ++n)
            if (n >= 2 * np0 && n < 2 * np1)
              *reinterpret_cast<float2*>(dst + n * 8) = make_float2(acc[m][n][2 * half8], acc[m][n][2 * half8 + 1]);
        }
      }
    }
    __syncthreads();  // scores are there, this run's keys are done with
    if (run + 1 < run_end) load_run(a.k_cache, k_s, d, L.qs, kw, run + 1);
    cp_async_commit();

    // step 2: PK positions (neighbouring keys of one row) x HC output heads a thread
    constexpr int PK = R == 1 ? 1 : 4, HC = R == 1 ? 4 : 8;
    const int h_begin = kv_lo * group / HC, h_end = ((kv_hi + 1) * group + HC - 1) / HC;
    constexpr int POS = R * N / PK;
    for (int item = tid; item < POS * (h_end - h_begin); item += THREADS) {
      const int at = item % POS, hc = (h_begin + item / POS) * HC;
      const int r = at / (N / PK), key = (at % (N / PK)) * PK;
      mix_f32x2 z[PK][HC / 2];
#pragma unroll
      for (int c = 0; c < HC / 2; ++c) {
        const mix_f32x2 b = mix_pack2(b_s[hc + 2 * c], b_s[hc + 2 * c + 1]);
#pragma unroll
        for (int k = 0; k < PK; ++k) z[k][c] = b;
      }
      const float* s = s_s + (size_t)r * SS + key;
      const float* m = m_s + hc;
#pragma unroll 4
      for (int in = 0; in < H; ++in) {
        float sv[PK];
        if (PK == 4) {
          const float4 v = *reinterpret_cast<const float4*>(s + (size_t)in * R * SS);
          sv[0] = v.x; sv[1 % PK] = v.y; sv[2 % PK] = v.z; sv[3 % PK] = v.w;
        } else {
          sv[0] = s[(size_t)in * R * SS];
        }
        mix_f32x2 mv[HC / 2];
#pragma unroll
        for (int c = 0; c < HC / 4; ++c) {
          const ulonglong2 v = *reinterpret_cast<const ulonglong2*>(m + in * L.hp + 4 * c);
          mv[2 * c] = v.x;
          mv[2 * c + 1] = v.y;
        }
#pragma unroll
        for (int k = 0; k < PK; ++k) {
          const mix_f32x2 sd = mix_pack2(sv[k], sv[k]);
#pragma unroll
          for (int c = 0; c < HC / 2; ++c) z[k][c] = mix_fma2(sd, mv[c], z[k][c]);
        }
      }
      const int qpos = pos0 + r, kpos = run * N + key;
      bool ok[PK];
#pragma unroll
      for (int k = 0; k < PK; ++k)
        ok[k] = r < rows && kpos + k <= qpos && (a.window <= 0 || kpos + k > qpos - a.window);
#pragma unroll
      for (int c = 0; c < HC / 2; ++c) {
        float w[2][PK];
#pragma unroll
        for (int k = 0; k < PK; ++k) {
          float lo, hi;
          mix_unpack2(z[k][c], lo, hi);
          w[0][k] = ok[k] ? mix_sigmoid(lo) : 0.f;
          w[1][k] = ok[k] ? mix_sigmoid(hi) : 0.f;
        }
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int h = hc + 2 * c + e;
          if (h >= H) continue;
          __nv_bfloat16* dst = p_s + (size_t)(h * R + r) * SS + key;
          if (PK == 4) {
            uint2 v;
            v.x = pack_bf162(w[e][0], w[e][1 % PK]);
            v.y = pack_bf162(w[e][2 % PK], w[e][3 % PK]);
            *reinterpret_cast<uint2*>(dst) = v;
          } else {
            *dst = __float2bfloat16_rn(w[e][0]);
          }
        }
      }
    }
    cp_async_wait<1>();  // this run's values (the next run's keys may still be on their way)
    __syncthreads();

    // step 3
#pragma unroll
    for (int ks = 0; ks < N / 16; ++ks) {
      unsigned pf[TPW][4];
#pragma unroll
      for (int j = 0; j < TPW; ++j) {
        const int u = min(unit0 + warp * TPW + j, n_units - 1);
        const int kv = u / (cps * tpg), tile = u % tpg;
        ldmatrix_x4(pf[j], p_s + (size_t)compact(kv, tile, (lane & 7) + (((lane >> 3) & 1) << 3)) * SS + ks * 16 + ((lane >> 4) << 3));
      }
#pragma unroll
      for (int np = 0; np < 4; ++np) {
        unsigned vf[4];
        int held = -1;
#pragma unroll
        for (int j = 0; j < TPW; ++j) {
          const int u = unit0 + warp * TPW + j;
          if (u >= unit1) continue;
          const int kc = u / tpg, kv = kc / cps, col = (kc % cps) * 64 + np * 16;
          if (col >= L.vs - 8) continue;
          if (kc != held) {
            ldmatrix_x4_trans(vf, v_s + (size_t)(kv * N + ks * 16 + (lane & 7) + (((lane >> 3) & 1) << 3)) * L.vs + col + ((lane >> 4) << 3));
            held = kc;
          }
          mma_16816(o[j][2 * np], pf[j], vf[0], vf[1]);
          mma_16816(o[j][2 * np + 1], pf[j], vf[2], vf[3]);
        }
      }
    }
    cp_async_wait<0>();  // the next run's keys
    __syncthreads();     // this run's values, weights and scores are done with
    if (run + 1 < run_end) load_run(a.v_cache, v_s, dv, L.vs, vw, run + 1);
    cp_async_commit();
  }
  cp_async_wait<0>();

#pragma unroll
  for (int j = 0; j < TPW; ++j) {
    const int u = unit0 + warp * TPW + j;
    if (u >= unit1) continue;
    const int kc = u / tpg, kv = kc / cps, tile = u % tpg;
#pragma unroll
    for (int half8 = 0; half8 < 2; ++half8) {
      const int rr = g + 8 * half8, r = rr % R;
      if (tile * HPT + rr / R >= group || r >= rows) continue;
      const int h = kv * group + tile * HPT + rr / R;
#pragma unroll
      for (int n = 0; n < 8; ++n) {
        const int col = (kc % cps) * 64 + n * 8 + 2 * t;
        if (col >= dv) continue;  // dv is even: a pair is inside or outside as a whole
        if (a.n_splits > 1)
          *reinterpret_cast<float2*>(a.part + (((size_t)seq * a.n_splits + blockIdx.z) * H + h) * dv + col) =
              make_float2(o[j][n][2 * half8], o[j][n][2 * half8 + 1]);
        else
          *reinterpret_cast<__nv_bfloat162*>(a.out + ((tok0 + r) * H + h) * dv + col) =
              __floats2bfloat162_rn(o[j][n][2 * half8], o[j][n][2 * half8 + 1]);
      }
    }
  }
}

// out[sequence's token] = the sum of its context splits, in split order; a thread owns a pair of columns
__global__ void __launch_bounds__(256) mixed_attention_sum_kernel(const float* __restrict__ part, const int* __restrict__ seq_qstart,
                                                                  __nv_bfloat16* __restrict__ out, int n_seqs, int n_splits, int width) {
  const long long at = (long long)blockIdx.x * 256 + threadIdx.x;
  if (at >= (long long)n_seqs * (width / 2)) return;
  const int seq = (int)(at / (width / 2)), c = (int)(at % (width / 2)) * 2;
  const float* p = part + (size_t)seq * n_splits * width + c;
  float2 sum = make_float2(0.f, 0.f);
#pragma unroll 4
  for (int s = 0; s < n_splits; ++s) {
    const float2 v = *reinterpret_cast<const float2*>(p + (size_t)s * width);
    sum.x += v.x;
    sum.y += v.y;
  }
  *reinterpret_cast<__nv_bfloat162*>(out + (size_t)seq_qstart[seq] * width + c) = __floats2bfloat162_rn(sum.x, sum.y);
}

constexpr int MIX_SMEM_MAX = 227 * 1024;

inline int mix_units(int H, int G, int dv, int R) {
  const int group = H / G, tpg = (group + 16 / R - 1) / (16 / R);
  return G * tpg * ((((dv + 15) & ~15) + 63) / 64);
}

// Rows and keys per run of a launch: R * 256 + N, or 0 where shared memory holds no combination.
inline int mix_mma_shape(int single, int H, int G, int d, int dv) {
  auto fits = [&](int R, int N, int limit) { return mix_mma_layout(H, G, d, dv, R, N).total <= limit; };
  if (single) {
    if (fits(1, 32, MIX_SMEM_MAX / 2 - 1024)) return 256 + 32;  // two blocks a multiprocessor
    return fits(1, 16, MIX_SMEM_MAX) ? 256 + 16 : 0;
  }
  if (mix_units(H, G, dv, 16) <= 4 * MIX_WARPS) {
    if (fits(16, 32, MIX_SMEM_MAX)) return 16 * 256 + 32;
    if (fits(16, 16, MIX_SMEM_MAX)) return 16 * 256 + 16;
  }
  for (int R = 8; R <= 16; R += 8)
    for (int N = 32; N >= 16; N -= 16)
      if (fits(R, N, MIX_SMEM_MAX)) return R * 256 + N;
  return 0;
}

template <int R, int N, int TPW>
int launch_mixed_mma(const MixMmaArgs& a, int n_blocks, cudaStream_t stream) {
  const int smem = mix_mma_layout(a.n_heads, a.n_kv_heads, a.d, a.dv, R, N).total;
  auto kernel = mixed_attention_mma_kernel<R, N, TPW>;
  cudaError_t err = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
  if (err != cudaSuccess) {
    mll_set_error("mixed attention (mma): cannot reserve %d bytes of shared memory: %s", smem, cudaGetErrorString(err));
    return (int)err;
  }
  const int units = mix_units(a.n_heads, a.n_kv_heads, a.dv, R);
  const dim3 grid(n_blocks, (units + MIX_WARPS * TPW - 1) / (MIX_WARPS * TPW), a.n_splits);
  MLL_LAUNCH((kernel), grid, MIX_WARPS * 32, smem, stream, a);
  MLL_LAUNCH_CHECK();
  return 0;
}

}  // namespace mll

MLL_API int mll_mixed_attention_mma_supported(int dtype, int single, int n_heads, int n_kv_heads, int d, int dv) {
  return dtype == MLL_BF16 && d % 8 == 0 && d >= 8 && d <= 256 && dv % 8 == 0 && dv >= 8 && dv <= 256 && n_kv_heads > 0 &&
         n_heads % n_kv_heads == 0 && mll::mix_mma_shape(single, n_heads, n_kv_heads, d, dv) != 0;
}

// tile_seq / tile_row0: tiles of up to 64 query rows as (sequence, first row among the sequence's new tokens), n_tiles of
// them; null: every sequence brings one token and n_tiles is the number of sequences.  n_splits > 1 (single tokens only)
// cuts every context into that many runs and needs scratch: n_tiles * n_splits * H * dv floats.
MLL_API int mll_mixed_attention_mma(const void* q, const void* k_cache, const void* v_cache, const int* seq_slot,
                                    const int* seq_ctx, const int* seq_qstart, const int* seq_qlen, const int* tile_seq,
                                    const int* tile_row0, const int* block_table, const float* mix, const float* bias,
                                    void* out, float* scratch, int n_tiles, int n_heads, int n_kv_heads, int d, int dv,
                                    int window, int max_blocks, int n_splits, float scale, cudaStream_t stream) {
  const int single = tile_seq == nullptr;
  MLL_REQUIRE(mll_mixed_attention_mma_supported(MLL_BF16, single, n_heads, n_kv_heads, d, dv),
              "mixed attention (mma): %d heads of %d / %d over %d", n_heads, d, dv, n_kv_heads);
  MLL_REQUIRE(n_tiles >= 0 && window >= 0 && (single || tile_row0), "mixed attention (mma): bad tile list or window");
  MLL_REQUIRE(n_splits >= 1 && n_splits <= 64 && (n_splits == 1 || (single && scratch)),
              "mixed attention (mma): %d context splits need single tokens and scratch memory", n_splits);
  if (n_tiles == 0) return 0;
  mll::MixMmaArgs a{(const __nv_bfloat16*)q, (const __nv_bfloat16*)k_cache, (const __nv_bfloat16*)v_cache, seq_slot, seq_ctx,
                    seq_qstart, seq_qlen, tile_seq, tile_row0, block_table, mix, bias, (__nv_bfloat16*)out, scratch,
                    n_heads, n_kv_heads, d, dv, window, max_blocks, n_splits, scale};
  const int shape = mll::mix_mma_shape(single, n_heads, n_kv_heads, d, dv), R = shape / 256, N = shape % 256;
  const int units = mll::mix_units(n_heads, n_kv_heads, dv, R);
  int code;
  if (R == 1) {
    if (units <= mll::MIX_WARPS)
      code = N == 32 ? mll::launch_mixed_mma<1, 32, 1>(a, n_tiles, stream) : mll::launch_mixed_mma<1, 16, 1>(a, n_tiles, stream);
    else
      code = N == 32 ? mll::launch_mixed_mma<1, 32, 2>(a, n_tiles, stream) : mll::launch_mixed_mma<1, 16, 2>(a, n_tiles, stream);
  } else if (R == 8) {
    code = N == 32 ? mll::launch_mixed_mma<8, 32, 4>(a, n_tiles * 8, stream) : mll::launch_mixed_mma<8, 16, 4>(a, n_tiles * 8, stream);
  } else if (units <= 2 * mll::MIX_WARPS) {
    code = N == 32 ? mll::launch_mixed_mma<16, 32, 2>(a, n_tiles * 4, stream) : mll::launch_mixed_mma<16, 16, 2>(a, n_tiles * 4, stream);
  } else {
    code = N == 32 ? mll::launch_mixed_mma<16, 32, 4>(a, n_tiles * 4, stream) : mll::launch_mixed_mma<16, 16, 4>(a, n_tiles * 4, stream);
  }
  if (code != 0 || n_splits == 1) return code;
  const long long items = (long long)n_tiles * (n_heads * dv / 2);
  MLL_LAUNCH((mll::mixed_attention_sum_kernel), (unsigned)((items + 255) / 256), 256, 0, stream, scratch, seq_qstart,
             (__nv_bfloat16*)out, n_tiles, n_splits, n_heads * dv);
  MLL_LAUNCH_CHECK();
  return 0;
}
