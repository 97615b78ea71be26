// Attention with mixed scores and sigmoid weights (attention_mix.cu) in bfloat16 on tensor cores, for prompt tiles and
// for single tokens.
//
// A key's weight in head h needs the scores of all H heads at that key, so a block owns R query rows of one sequence with
// all their heads and walks the window in runs of N keys.  Per run:
//   1. S = q k^T by mma.sync: the 16 rows of a tile are R query rows of 16 / R heads of one key head's group; scores go to
//      shared memory - for prompts as three bfloat16 planes that add up to all 24 bits of the float32 score.
//   2. z = M S + b, sigmoid, mask; weights go to shared memory as bfloat16.  For prompts the mixing is three more mma.sync
//      products (the planes are exact: a float32 product of float32 scores), or six where M has values that are no
//      bfloat16 numbers and is cut into planes as well; for single tokens it is float32 FMAs, two an instruction.
//   3. O += P V by mma.sync: a warp keeps TP x 16 rows x CP x 64 value columns in registers for the whole walk.
// Nothing is normalised, so there is no running maximum and no rescaling, and context splits simply add up.
// K and V of a run have one buffer each.  Single tokens: the next run's keys load while 2 and 3 work, its values while 1
// and 2 do.  Prompts: step 3 of a run shares an interval between barriers with step 1 of the next one (two streams of
// independent products a warp), and the copies into both buffers pass while 2 works.
// A prompt's tile may be cut along its keys too: the blocks of a thread-block cluster walk a share of the runs each and add
// their sums up through distributed shared memory, every block the columns it writes.
// Where the H x R rows' outputs exceed what one block's registers hold, grid y splits the output heads and every block
// recomputes the scores.
#include "attention_decode.cuh"
#include "attention_mix.cuh"

#include <cooperative_groups.h>

#include <type_traits>

namespace mll {

namespace cg = cooperative_groups;

struct MixMmaArgs {
  const __nv_bfloat16* q;
  const __nv_bfloat16* k_cache;
  const __nv_bfloat16* v_cache;
  const int* seq_slot;
  const int* seq_ctx;
  const int* seq_qstart;
  const int* seq_qlen;
  const int* tile_seq;    // prompt tiles of 128 rows, walked from the back; null: single tokens, grid x runs over the sequences
  const int* tile_row0;
  const int* block_table;
  const float* mix;       // [H, H] or null
  const float* bias;      // [H] or null
  __nv_bfloat16* out;
  float* part;            // single tokens: [sequences, n_splits, H, dv] sums of the context's runs (n_splits > 1)
  int n_heads, n_kv_heads, d, dv, window, max_blocks;
  int mix_planes;         // prompts: 1 where every entry of mix is a bfloat16 number, else 3
  int n_splits;           // blocks (grid z) that share a tile's runs; for prompts they are one cluster
  float scale;
};


// Shared memory of a block, in bytes from its start.  Rows of q are compact: row h * R + r.  Scores and weights of head h
// and row r begin at element h * ps + r * (N + 8): rows of 16-byte words of which neighbours - in a head, or of heads -
// lie in different banks.
struct MixMmaLayout {
  int qs, vs, ps, hp;             // elements between rows of q / k, of v, between heads of S / P; heads rounded up to 16
  int k, v, s, p, m, b, total;    // q starts at 0
};
__host__ __device__ inline MixMmaLayout mix_mma_layout(int H, int G, int d, int dv, int R, int N) {
  MixMmaLayout l;
  l.qs = ((d + 15) & ~15) + 8;
  l.vs = ((dv + 15) & ~15) + 8;
  l.ps = R * (N + 8) + (R > 1 ? 8 : 0);
  l.hp = (H + 15) & ~15;
  int at = H * R * l.qs * 2;
  l.k = at; at += G * N * l.qs * 2;
  l.v = at; at += G * N * l.vs * 2;
  l.s = at; at += R > 1 ? 3 * l.hp * l.ps * 2 : H * l.ps * 4;
  l.p = at; at += l.hp * l.ps * 2;
  at = (at + 15) & ~15;
  l.m = at; at += R > 1 ? 3 * l.hp * (l.hp + 8) * 2 : H * l.hp * 4;
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
// sigmoid(z) from y = -z log2 e: 1 / (1 + 2^y); large |z|: 2^y overflows to infinity (weight 0) or falls to 0 (weight 1)
__device__ __forceinline__ float mix_sigmoid(float y) {
  float e, r;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(e) : "f"(y));
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(1.f + e));
  return r;
}
constexpr float MIX_LOG2E = 1.4426950408889634f;

// Shared memory by 32-bit address: the walk's inner loops add small offsets to a few bases.
__device__ __forceinline__ void mix_ldsm(unsigned (&r)[4], unsigned at) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(at));
}
__device__ __forceinline__ void mix_ldsm_trans(unsigned (&r)[4], unsigned at) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];\n"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(at));
}
// as mma_16816, free to move between the fragment loads around it
__device__ __forceinline__ void mix_mma(float (&c)[4], const unsigned (&a)[4], unsigned b0, unsigned b1) {
  asm("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void mix_sts(unsigned at, unsigned v) {
  asm volatile("st.shared.b32 [%0], %1;\n" ::"r"(at), "r"(v) : "memory");
}
__device__ __forceinline__ void mix_sts2(unsigned at, float x, float y) {
  asm volatile("st.shared.v2.f32 [%0], {%1, %2};\n" ::"r"(at), "f"(x), "f"(y) : "memory");
}
__device__ __forceinline__ void mix_copy16(unsigned at, const void* src, bool valid) {
  const int bytes = valid ? 16 : 0;  // fewer source bytes than 16: the rest is written as zero
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"(at), "l"(src), "r"(bytes) : "memory");
}

// DIM: the head size of keys and values where it is known at compile time (strides and word counts are then constants), or 0.
// W warps a block; with 8 of them two blocks share a multiprocessor.  CUT: the mixing matrix comes in three terms.
template <int R, int N, int W, int TP, int CP, int DIM, bool CUT>
__global__ void __launch_bounds__(W * 32, W == 8 ? 2 : 1)
mixed_attention_mma_kernel(MixMmaArgs a) {
  extern __shared__ __align__(16) unsigned char smem_raw[];
  constexpr int WARPS = W, THREADS = W * 32;
  constexpr int HPT = 16 / R;         // heads in the 16 rows of a tile
  constexpr int QP = W == 8 ? 1 : 2;  // tiles of one key head that share the key fragments in step 1
  constexpr int SS = N + 8;           // elements between rows of S and of P
  constexpr bool MERGED = R > 1;      // step 3 of a run beside step 1 of the next
  const int H = a.n_heads, G = a.n_kv_heads, group = H / G, d = DIM ? DIM : a.d, dv = DIM ? DIM : a.dv;
  const MixMmaLayout L = mix_mma_layout(H, G, d, dv, R, N);
  __nv_bfloat16* q_s = reinterpret_cast<__nv_bfloat16*>(smem_raw);
  float* s_s = reinterpret_cast<float*>(smem_raw + L.s);
  __nv_bfloat16* p_s = reinterpret_cast<__nv_bfloat16*>(smem_raw + L.p);
  __nv_bfloat16* planes = reinterpret_cast<__nv_bfloat16*>(smem_raw + L.s);  // R > 1: three of them, hp * ps elements each
  float* m_s = reinterpret_cast<float*>(smem_raw + L.m);                     // R == 1: [H in][hp out], times -scale log2 e
  __nv_bfloat16* mb_s = reinterpret_cast<__nv_bfloat16*>(smem_raw + L.m);    // R > 1: planes of [hp out][hp in + 8]
  float* b_s = reinterpret_cast<float*>(smem_raw + L.b);                     // times -log2 e

  const int tid = threadIdx.x, lane = tid & 31;
  const int warp = __shfl_sync(0xffffffffu, tid >> 5, 0);  // the same register value in all lanes: branches on it are uniform
  const int g = lane >> 2, t = lane & 3;
  const bool single = a.tile_seq == nullptr;
  constexpr int SUB = 128 / R;  // tiles of R rows in a listed tile of 128
  const int work = gridDim.x - 1 - blockIdx.x;  // from the back: the tiles with the most keys in front of them start first
  const int seq = single ? blockIdx.x : a.tile_seq[work / SUB];
  const int row0 = single ? 0 : a.tile_row0[work / SUB] + work % SUB * R;
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

  // the units of step 3 (TP tiles of 16 rows of one key head x CP x 64 value columns): one a warp
  const int tpg = (group + HPT - 1) / HPT, tgs = (tpg + TP - 1) / TP;                  // tiles of a key head, groups of them
  const int cgs = (L.vs - 8 + CP * 64 - 1) / (CP * 64);                                // column groups of a value head
  const int unit0 = (int)blockIdx.y * WARPS, unit1 = min(G * cgs * tgs, unit0 + WARPS);
  const int kv_lo = unit0 / (cgs * tgs), kv_hi = (unit1 - 1) / (cgs * tgs);

  const int kw = (L.qs - 8) >> 3, vw = (L.vs - 8) >> 3;  // 16-byte words of a padded row
  // a thread's words of a run: the first (row, word) and the way to the next one
  const int k_r = tid / kw, k_c = tid % kw * 8, v_r = tid / vw, v_c = tid % vw * 8;
  const unsigned base = (unsigned)__cvta_generic_to_shared(smem_raw);
  auto load_run = [&](const __nv_bfloat16* cache, unsigned dst, int size, int stride, int words, int r, int c, int which, int page) {
    const int valid = ctx - which * N;  // rows past the cached length hold no data
    const __nv_bfloat16* from = cache + (size_t)(page * G * MLL_PAGE + which * N % MLL_PAGE) * size;
    const int head = MLL_PAGE * size, head_to = N * stride * 2;
    auto column = [&](int row, int col) {  // the same word of every head
      const bool in = col < size && row < valid;
      const __nv_bfloat16* src = from + (in ? row * size + col : 0);
      unsigned to = dst + (row * stride + col) * 2;
      int h = 0;
      for (; h + 4 <= G; h += 4) {
#pragma unroll
        for (int i = 0; i < 4; ++i) mix_copy16(to + i * head_to, src + (size_t)i * head, in);
        src += (size_t)4 * head;
        to += 4 * head_to;
      }
      for (; h < G; ++h, src += head, to += head_to) mix_copy16(to, src, in);
    };
    if (r < N) column(r, c);
    if (N * words > THREADS)
      for (int i = tid + THREADS; i < N * words; i += THREADS) column(i / words, i % words * 8);
  };
  auto load_keys = [&](int which, int page) { load_run(a.k_cache, base + L.k, d, L.qs, kw, k_r, k_c, which, page); };
  auto load_values = [&](int which, int page) { load_run(a.v_cache, base + L.v, dv, L.vs, vw, v_r, v_c, which, page); };
  int page = run < run_end ? table[run * N / MLL_PAGE] : 0;  // of the run whose loads come next
  for (int i = tid; i < H * R * kw; i += THREADS) {
    const int row = i / kw, c = (i - row * kw) * 8, h = row / R, r = row % R;
    const bool in = c < d && r < rows;
    cp_async16_zfill(q_s + (size_t)row * L.qs + c, a.q + ((tok0 + (in ? r : 0)) * H + h) * d + (in ? c : 0), in);
  }
  if (run < run_end) load_keys(run, page);
  cp_async_commit();
  if (!MERGED && run < run_end) load_values(run, page);
  cp_async_commit();
  auto mix_at = [&](int to, int in) { return to >= H || in >= H ? 0.f : a.mix ? a.mix[(size_t)to * H + in] : (to == in ? 1.f : 0.f); };
  if (R == 1) {
    for (int i = tid; i < H * L.hp; i += THREADS) m_s[i] = mix_at(i % L.hp, i / L.hp) * (-MIX_LOG2E * a.scale);
  } else {
    for (int i = tid; i < L.hp * L.hp; i += THREADS) {
      float rest = mix_at(i / L.hp, i % L.hp);
      for (int p = 0; p < (CUT ? 3 : 1); ++p) {
        const __nv_bfloat16 term = __float2bfloat16_rn(rest);
        mb_s[(p * L.hp + i / L.hp) * (L.hp + 8) + i % L.hp] = term;
        rest -= __bfloat162float(term);  // exact
      }
    }
    // heads that do not exist enter the products with a factor of 0: their scores must be numbers
    for (int i = tid; i < 3 * (L.hp - H) * L.ps; i += THREADS)
      planes[(size_t)(i / ((L.hp - H) * L.ps)) * L.hp * L.ps + (size_t)H * L.ps + i % ((L.hp - H) * L.ps)] = __float2bfloat16_rn(0.f);
  }
  for (int i = tid; i < L.hp; i += THREADS) b_s[i] = (i < H && a.bias) ? -MIX_LOG2E * a.bias[i] : 0.f;

  float o[TP][CP][8][4];
#pragma unroll
  for (int i = 0; i < TP * CP * 32; ++i) (&o[0][0][0][0])[i] = 0.f;

  // the head that the tile's row rr stands for (rows past the group repeat its last head and are not stored)
  auto head_of = [&](int kv, int tile, int rr) { return kv * group + min(tile * HPT + rr / R, group - 1); };
  const int ld_row = (lane & 7) + (((lane >> 3) & 1) << 3), ld_col = (lane >> 4) << 3;  // ldmatrix: this lane's row and column

  // step 3's unit of this warp: where the lane reads its rows of P and the values, how many of its columns exist (0: no unit)
  const int unit = min(unit0 + warp, unit1 - 1), my_kv = unit / (cgs * tgs), my_col = unit / tgs % cgs * CP * 64, my_tile = unit % tgs * TP;
  const int my_cols = unit0 + warp < unit1 ? min(CP * 64, L.vs - 8 - my_col) : 0;
  const unsigned p_at = base + L.p + (head_of(my_kv, my_tile, ld_row) * L.ps + ld_row % R * SS + ld_col) * 2;
  // the second tile's rows: HPT heads on, or the first tile's again where there is none (or where it is not whole)
  const int p_step = my_tile + 1 < tpg ? HPT * L.ps * 2 : 0;
  const unsigned v_at = base + L.v + ((my_kv * N + ld_row) * L.vs + my_col + ld_col) * 2;

  // step 1's units: QP tiles of one key head against 16 keys.  Where the lane reads q and k and where its scores
  // go; the second tile and the rows 8 further down lie at fixed distances
  const int pairs = (tpg + QP - 1) / QP;
  const int qk_units = G * pairs * (N / 16), plane = L.hp * L.ps * 2;
  unsigned q_at = 0, k_at = 0;
  int q_step = 0, s_at = 0, rows_in = 0;  // rows_in: bit 2 m + i set where row i of tile m is a row of the group
  constexpr int SB = R == 1 ? 4 : 2;  // bytes of a score in S (R == 1), of one of its terms
  auto set_qk = [&](int u) {
    const int strip = u % (N / 16), pair = (u / (N / 16)) % pairs, kv = u / (N / 16 * pairs);
    k_at = base + L.k + ((kv * N + strip * 16 + (lane & 7) + ((lane >> 4) << 3)) * L.qs + (((lane >> 3) & 1) << 3)) * 2;
    const int tile = pair * QP;
    q_at = base + ((head_of(kv, tile, ld_row) * R + ld_row % R) * L.qs + ld_col) * 2;
    q_step = tile + 1 < tpg ? HPT * R * L.qs * 2 : 0;
    s_at = base + L.s + ((kv * group + tile * HPT + g / R) * L.ps + g % R * SS + strip * 16 + 2 * t) * SB;
    rows_in = 0;
#pragma unroll
    for (int m = 0; m < QP; ++m)
#pragma unroll
      for (int i = 0; i < 2; ++i) rows_in |= (tile + m) * HPT + (g + 8 * i) / R < group ? 1 << (2 * m + i) : 0;
  };
  set_qk(min(warp, qk_units - 1));
  // step 3 of a run; `all`: every column of the unit exists
  auto weigh_values = [&](auto all) {
#pragma unroll
    for (int ks = 0; ks < N / 16; ++ks) {
      unsigned pf[TP][4], vf[2][4];
#pragma unroll
      for (int i = 0; i < TP; ++i) mix_ldsm(pf[i], p_at + i * p_step + ks * 32);
      const unsigned v = v_at + ks * 32 * L.vs;
      mix_ldsm_trans(vf[0], v);
#pragma unroll
      for (int np = 0; np < CP * 4; ++np)
        if (decltype(all)::value || np * 16 < my_cols) {
          if (np + 1 < CP * 4 && (decltype(all)::value || np * 16 + 16 < my_cols)) mix_ldsm_trans(vf[(np + 1) & 1], v + np * 32 + 32);
#pragma unroll
          for (int i = 0; i < TP; ++i) {
            mix_mma(o[i][np / 4][np % 4 * 2], pf[i], vf[np & 1][0], vf[np & 1][1]);
            mix_mma(o[i][np / 4][np % 4 * 2 + 1], pf[i], vf[np & 1][2], vf[np & 1][3]);
          }
        }
    }
  };
  const float neg_scale = -MIX_LOG2E * a.scale;

  auto step3 = [&] {
    if (my_cols == CP * 64)
      weigh_values(std::true_type{});
    else if (my_cols > 0)
      weigh_values(std::false_type{});
  };
  cp_async_wait<1>();
  __syncthreads();
  const bool any_runs = run < run_end;
  for (const int run0 = run; run < run_end; ++run) {
    const int page_now = page;
    if (run + 1 < run_end) page = table[(run + 1) * N / MLL_PAGE];
    for (int u = warp; u < qk_units; u += WARPS) {
      if (qk_units > WARPS) set_qk(u);  // else the warp keeps the one it has
      float acc[QP][2][4];
#pragma unroll
      for (int m = 0; m < QP; ++m)
#pragma unroll
        for (int n = 0; n < 2; ++n)
#pragma unroll
          for (int i = 0; i < 4; ++i) acc[m][n][i] = 0.f;
      unsigned qf[2][QP][4], kf[2][4];  // this step's fragments and the next one's
      auto fetch = [&](int to, int e) {
        mix_ldsm(kf[to], k_at + e);
#pragma unroll
        for (int m = 0; m < QP; ++m) mix_ldsm(qf[to][m], q_at + m * q_step + e);
      };
      auto multiply = [&](int from) {
#pragma unroll
        for (int m = 0; m < QP; ++m) {
          mix_mma(acc[m][0], qf[from][m], kf[from][0], kf[from][1]);
          mix_mma(acc[m][1], qf[from][m], kf[from][2], kf[from][3]);
        }
      };
      const int e_end = (L.qs - 8) * 2;
      fetch(0, 0);
#pragma unroll 4
      for (int e = 0; e < e_end; e += 64) {
        if (e + 32 < e_end) fetch(1, e + 32);
        multiply(0);
        if (e + 32 < e_end) {
          if (e + 64 < e_end) fetch(0, e + 64);
          multiply(1);
        }
      }
#pragma unroll
      for (int m = 0; m < QP; ++m)
#pragma unroll
        for (int half8 = 0; half8 < 2; ++half8) {
          if (!(rows_in >> (2 * m + half8) & 1)) continue;
          const unsigned to = s_at + (m * HPT * L.ps + half8 * (8 / R * L.ps + 8 % R * SS)) * SB;
#pragma unroll
          for (int n = 0; n < 2; ++n) {
            const float x = acc[m][n][2 * half8], y = acc[m][n][2 * half8 + 1];
            if (R == 1) {
              mix_sts2(to + n * 8 * SB, x, y);
            } else {
              const unsigned hi = pack_bf162(x, y);
              const float2 h = unpack_bf162(hi);
              const float rx = x - h.x, ry = y - h.y;  // exact
              const unsigned mid = pack_bf162(rx, ry);
              const float2 f = unpack_bf162(mid);
              mix_sts(to + n * 8 * SB, hi);
              mix_sts(to + n * 8 * SB + plane, mid);
              mix_sts(to + n * 8 * SB + 2 * plane, pack_bf162(rx - f.x, ry - f.y));
            }
          }
        }
    }
    if (MERGED && run > run0) step3();  // of the run before
    __syncthreads();  // scores are there, this run's keys (and, merged, the values and weights of the run before) are done with
    if (run + 1 < run_end) load_keys(run + 1, page);
    if (MERGED) load_values(run, page_now);
    cp_async_commit();

    // step 2
    if constexpr (R == 1) {
      // one key x four output heads a thread
      const int h_begin = kv_lo * group / 4, h_end = ((kv_hi + 1) * group + 3) / 4;
      for (int item = tid; item < N * (h_end - h_begin); item += THREADS) {
        const int key = item % N, hc = (h_begin + item / N) * 4;
        mix_f32x2 z[2] = {mix_pack2(b_s[hc], b_s[hc + 1]), mix_pack2(b_s[hc + 2], b_s[hc + 3])};
        const float* s = s_s + key;
        const float* m = m_s + hc;
#pragma unroll 8
        for (int in = 0; in < H; ++in) {
          const float sv = s[in * SS];
          const ulonglong2 mv = *reinterpret_cast<const ulonglong2*>(m + in * L.hp);
          const mix_f32x2 sd = mix_pack2(sv, sv);
          z[0] = mix_fma2(sd, mv.x, z[0]);
          z[1] = mix_fma2(sd, mv.y, z[1]);
        }
        const int kpos = run * N + key;
        const bool ok = kpos <= pos0 && (a.window <= 0 || kpos > pos0 - a.window);
#pragma unroll
        for (int c = 0; c < 2; ++c) {
          float lo, hi;
          mix_unpack2(z[c], lo, hi);
          p_s[(hc + 2 * c) * L.ps + key] = __float2bfloat16_rn(ok ? mix_sigmoid(lo) : 0.f);
          p_s[(hc + 2 * c + 1) * L.ps + key] = __float2bfloat16_rn(ok ? mix_sigmoid(hi) : 0.f);
        }
      }
    } else {
      // a warp owns one row's keys x 16 output heads
      const int mt0 = kv_lo * group / 16, mts = ((kv_hi + 1) * group + 15) / 16 - mt0;
      const bool edge = rows < R || run * N + N - 1 > pos0 || (a.window > 0 && run * N <= last - a.window);
      for (int item = warp; item < R * mts; item += WARPS) {
        const int r = item % R, h = (mt0 + item / R) * 16;
        float z[N / 8][4];
#pragma unroll
        for (int n = 0; n < N / 8; ++n)
#pragma unroll
          for (int i = 0; i < 4; ++i) z[n][i] = 0.f;
        unsigned m = base + L.m + ((h + ld_row) * (L.hp + 8) + ld_col) * 2;
        unsigned s = base + L.s + (ld_row * L.ps + r * SS + ld_col) * 2;
        for (int kt = 0; kt < L.hp; kt += 16, m += 32, s += L.ps * 32) {
          unsigned mf[4], sf[3][N / 16][4];
          mix_ldsm(mf, m);
#pragma unroll
          for (int p = 0; p < 3; ++p)
#pragma unroll
            for (int n = 0; n < N / 16; ++n) mix_ldsm_trans(sf[p][n], s + p * plane + n * 32);
          if (CUT) {  // the smaller terms of M with the terms of S that still count, smallest first
#pragma unroll
            for (int k = 2; k >= 1; --k) {
              unsigned mk[4];
              mix_ldsm(mk, m + k * L.hp * (L.hp + 8) * 2);
#pragma unroll
              for (int p = 2 - k; p >= 0; --p)
#pragma unroll
                for (int n = 0; n < N / 16; ++n) {
                  mix_mma(z[2 * n], mk, sf[p][n][0], sf[p][n][1]);
                  mix_mma(z[2 * n + 1], mk, sf[p][n][2], sf[p][n][3]);
                }
            }
          }
#pragma unroll
          for (int p = 2; p >= 0; --p)
#pragma unroll
            for (int n = 0; n < N / 16; ++n) {
              mix_mma(z[2 * n], mf, sf[p][n][0], sf[p][n][1]);
              mix_mma(z[2 * n + 1], mf, sf[p][n][2], sf[p][n][3]);
            }
        }
        const float b0 = b_s[h + g], b1 = b_s[h + g + 8];
        const unsigned to = base + L.p + ((h + g) * L.ps + r * SS + 2 * t) * 2, to8 = to + 16 * L.ps;
#pragma unroll
        for (int n = 0; n < N / 8; ++n) {
          z[n][0] = mix_sigmoid(fmaf(z[n][0], neg_scale, b0));
          z[n][1] = mix_sigmoid(fmaf(z[n][1], neg_scale, b0));
          z[n][2] = mix_sigmoid(fmaf(z[n][2], neg_scale, b1));
          z[n][3] = mix_sigmoid(fmaf(z[n][3], neg_scale, b1));
        }
        if (edge) {  // the run meets the diagonal, the window's far edge or a row that does not exist
          const int qpos = pos0 + r, kpos = run * N + 2 * t;
          const int lo = a.window > 0 ? qpos - a.window + 1 : 0, hi = r < rows ? qpos : -1;
#pragma unroll
          for (int n = 0; n < N / 8; ++n)
#pragma unroll
            for (int i = 0; i < 4; ++i) {
              const int k = kpos + 8 * n + (i & 1);
              if (k < lo || k > hi) z[n][i] = 0.f;
            }
        }
#pragma unroll
        for (int n = 0; n < N / 8; ++n) {
          mix_sts(to + 16 * n, pack_bf162(z[n][0], z[n][1]));
          mix_sts(to8 + 16 * n, pack_bf162(z[n][2], z[n][3]));
        }
      }
    }
    if (MERGED) {
      cp_async_wait<0>();  // the next run's keys, this run's values
      __syncthreads();
      continue;
    }
    cp_async_wait<1>();  // this run's values (the next run's keys may still be on their way)
    __syncthreads();
    step3();
    cp_async_wait<0>();  // the next run's keys
    __syncthreads();     // this run's values, weights and scores are done with
    if (run + 1 < run_end) load_values(run + 1, page);
    cp_async_commit();
  }
  if (MERGED && any_runs) step3();  // of the last run
  cp_async_wait<0>();

  if constexpr (R > 1) {
    if (a.n_splits > 1) {  // the same in all blocks of the cluster: each gets here, with or without runs of its own
      cg::cluster_group cluster = cg::this_cluster();
      float2* mine = reinterpret_cast<float2*>(smem_raw);  // [TP * CP * 16][THREADS], over what the walk no longer needs
      __syncthreads();
#pragma unroll
      for (int i = 0; i < TP * CP * 8; ++i)
#pragma unroll
        for (int half8 = 0; half8 < 2; ++half8) {
          const float* f = &o[0][0][0][0] + i * 4 + 2 * half8;
          mine[(i * 2 + half8) * THREADS + tid] = make_float2(f[0], f[1]);
        }
      cluster.sync();
      const int rank = (int)cluster.block_rank(), share = 8 / a.n_splits;  // n_splits divides 8
#pragma unroll
      for (int i = 0; i < TP; ++i)
#pragma unroll
        for (int half8 = 0; half8 < 2; ++half8) {
          const int rr = g + 8 * half8, r = rr % R, tile = my_tile + i;
          if (tile * HPT + rr / R >= group || r >= rows) continue;
          const int h = my_kv * group + tile * HPT + rr / R;
          for (int c = 0; c < CP; ++c)
            for (int n = rank * share; n < (rank + 1) * share; ++n) {
              const int col = c * 64 + n * 8 + 2 * t;
              if (col >= my_cols || my_col + col >= dv) continue;
              const float2* at = mine + (((i * CP + c) * 8 + n) * 2 + half8) * THREADS + tid;
              float2 sum = make_float2(0.f, 0.f);
              for (int sp = 0; sp < a.n_splits; ++sp) {  // in the order of the runs
                const float2 v = *cluster.map_shared_rank(at, sp);
                sum.x += v.x;
                sum.y += v.y;
              }
              *reinterpret_cast<__nv_bfloat162*>(a.out + ((tok0 + r) * H + h) * dv + my_col + col) = __floats2bfloat162_rn(sum.x, sum.y);
            }
        }
      cluster.sync();  // nobody leaves while another block may still read its shared memory
      return;
    }
  }
#pragma unroll
  for (int i = 0; i < TP; ++i)
#pragma unroll
    for (int half8 = 0; half8 < 2; ++half8) {
      const int rr = g + 8 * half8, r = rr % R, tile = my_tile + i;
      if (tile * HPT + rr / R >= group || r >= rows) continue;
      const int h = my_kv * group + tile * HPT + rr / R;
#pragma unroll
      for (int c = 0; c < CP; ++c)
#pragma unroll
        for (int n = 0; n < 8; ++n) {
          const int col = c * 64 + n * 8 + 2 * t;
          if (col >= my_cols || my_col + col >= dv) continue;  // dv is even: a pair is inside or outside as a whole
          const float x = o[i][c][n][2 * half8], y = o[i][c][n][2 * half8 + 1];
          if (a.n_splits > 1)
            *reinterpret_cast<float2*>(a.part + (((size_t)seq * a.n_splits + blockIdx.z) * H + h) * dv + my_col + col) = make_float2(x, y);
          else
            *reinterpret_cast<__nv_bfloat162*>(a.out + ((tok0 + r) * H + h) * dv + my_col + col) = __floats2bfloat162_rn(x, y);
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

inline int mix_units(int H, int G, int dv, int R, int TP, int CP) {
  const int group = H / G, tpg = (group + 16 / R - 1) / (16 / R);
  return G * ((tpg + TP - 1) / TP) * ((((dv + 15) & ~15) + CP * 64 - 1) / (CP * 64));
}

// How a launch cuts its work: rows, keys per run and warps of a block (rows 0: shared memory holds no cut).
struct MixShape {
  int R, N, W;
};
inline MixShape mix_mma_shape(int single, int H, int G, int d, int dv) {
  auto fits = [&](int R, int N, int limit) { return mix_mma_layout(H, G, d, dv, R, N).total <= limit; };
  const int half = MIX_SMEM_MAX / 2 - 1024;  // two blocks a multiprocessor
  if (single) {
    if (fits(1, 32, half)) return {1, 32, 8};
    return {fits(1, 16, MIX_SMEM_MAX) ? 1 : 0, 16, 8};
  }
  if (mix_units(H, G, dv, 16, 2, 1) <= 16) {
    if (fits(16, 32, MIX_SMEM_MAX)) return {16, 32, 16};
    if (fits(16, 16, MIX_SMEM_MAX)) return {16, 16, 16};
  }
  for (int R = 8; R <= 16; R += 8)
    for (int N = 32; N >= 16; N -= 16)
      if (fits(R, N, MIX_SMEM_MAX)) return {R, N, 16};
  return {0, 0, 0};
}

template <int R, int N, int W, int TP, int CP, int DIM, bool CUT>
int launch_mixed_mma_cut(const MixMmaArgs& a, int n_blocks, cudaStream_t stream) {
  const int exchange = R > 1 && a.n_splits > 1 ? TP * CP * 16 * W * 32 * (int)sizeof(float2) : 0;
  const int smem = max(mix_mma_layout(a.n_heads, a.n_kv_heads, a.d, a.dv, R, N).total, exchange);
  auto kernel = mixed_attention_mma_kernel<R, N, W, TP, CP, DIM, CUT>;
  cudaError_t err = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
  if (err != cudaSuccess) {
    mll_set_error("mixed attention (mma): cannot reserve %d bytes of shared memory: %s", smem, cudaGetErrorString(err));
    return (int)err;
  }
  const int units = mix_units(a.n_heads, a.n_kv_heads, a.dv, R, TP, CP);
  cudaLaunchConfig_t config = {};
  config.gridDim = dim3(n_blocks, (units + W - 1) / W, a.n_splits);
  config.blockDim = dim3(W * 32);
  config.dynamicSmemBytes = smem;
  config.stream = stream;
  cudaLaunchAttribute attr[1];
  if (R > 1 && a.n_splits > 1) {
    attr[0].id = cudaLaunchAttributeClusterDimension;
    attr[0].val.clusterDim.x = 1;
    attr[0].val.clusterDim.y = 1;
    attr[0].val.clusterDim.z = a.n_splits;
    config.attrs = attr;
    config.numAttrs = 1;
  }
  mll_launch_status = cudaLaunchKernelEx(&config, kernel, a);
  MLL_LAUNCH_CHECK();
  return 0;
}

template <int R, int N, int W, int TP, int CP, int DIM>
int launch_mixed_mma_dim(const MixMmaArgs& a, int n_blocks, cudaStream_t stream) {
  if constexpr (R > 1) {
    if (a.mix_planes > 1) return launch_mixed_mma_cut<R, N, W, TP, CP, DIM, true>(a, n_blocks, stream);
  }
  return launch_mixed_mma_cut<R, N, W, TP, CP, DIM, false>(a, n_blocks, stream);
}

template <int R, int N, int W, int TP, int CP>
int launch_mixed_mma(const MixMmaArgs& a, int n_blocks, cudaStream_t stream) {
  return a.d == 128 && a.dv == 128 ? launch_mixed_mma_dim<R, N, W, TP, CP, 128>(a, n_blocks, stream)
                                   : launch_mixed_mma_dim<R, N, W, TP, CP, 0>(a, n_blocks, stream);
}

}  // namespace mll

MLL_API int mll_mixed_attention_mma_supported(int dtype, int single, int n_heads, int n_kv_heads, int d, int dv) {
  return dtype == MLL_BF16 && d % 8 == 0 && d >= 8 && d <= 256 && dv % 8 == 0 && dv >= 8 && dv <= 256 && n_kv_heads > 0 &&
         n_heads % n_kv_heads == 0 && mll::mix_mma_shape(single, n_heads, n_kv_heads, d, dv).R != 0;
}

// mix: float32; mix_planes: for prompts, 1 says that every entry is a bfloat16 number, 3 that it may be any float32.
// tile_seq / tile_row0: tiles of up to 128 query rows as (sequence, first row among the sequence's new tokens), n_tiles of
// them; null: every sequence brings one token and n_tiles is the number of sequences.  n_splits > 1 blocks share every
// tile's keys: the blocks of a cluster for prompts (2, 4 or 8), else blocks that need scratch, n_tiles * n_splits * H * dv
// floats.
MLL_API int mll_mixed_attention_mma(const void* q, const void* k_cache, const void* v_cache, const int* seq_slot,
                                    const int* seq_ctx, const int* seq_qstart, const int* seq_qlen, const int* tile_seq,
                                    const int* tile_row0, const int* block_table, const float* mix, const float* bias,
                                    void* out, float* scratch, int n_tiles, int n_heads, int n_kv_heads, int d, int dv,
                                    int window, int max_blocks, int mix_planes, int n_splits, float scale, cudaStream_t stream) {
  const int single = tile_seq == nullptr;
  MLL_REQUIRE(mll_mixed_attention_mma_supported(MLL_BF16, single, n_heads, n_kv_heads, d, dv),
              "mixed attention (mma): %d heads of %d / %d over %d", n_heads, d, dv, n_kv_heads);
  MLL_REQUIRE(n_tiles >= 0 && window >= 0 && (single || tile_row0), "mixed attention (mma): bad tile list or window");
  MLL_REQUIRE(n_splits >= 1 && n_splits <= 64 && (n_splits == 1 || (single ? scratch != nullptr : 8 % n_splits == 0)),
              "mixed attention (mma): %d context splits (single tokens: scratch memory; prompts: 1, 2, 4 or 8)", n_splits);
  MLL_REQUIRE(mix_planes == 1 || mix_planes == 3, "mixed attention (mma): a matrix of 1 or 3 planes, not %d", mix_planes);
  if (n_tiles == 0) return 0;
  mll::MixMmaArgs a{(const __nv_bfloat16*)q, (const __nv_bfloat16*)k_cache, (const __nv_bfloat16*)v_cache, seq_slot, seq_ctx,
                    seq_qstart, seq_qlen, tile_seq, tile_row0, block_table, mix, bias, (__nv_bfloat16*)out, scratch,
                    n_heads, n_kv_heads, d, dv, window, max_blocks, mix_planes, n_splits, scale};
  const mll::MixShape shape = mll::mix_mma_shape(single, n_heads, n_kv_heads, d, dv);
  const bool wide = shape.N == 32;
  int code;
  if (shape.R == 1) {
    if (mll::mix_units(n_heads, n_kv_heads, dv, 1, 1, 1) <= 8)
      code = wide ? mll::launch_mixed_mma<1, 32, 8, 1, 1>(a, n_tiles, stream) : mll::launch_mixed_mma<1, 16, 8, 1, 1>(a, n_tiles, stream);
    else
      code = wide ? mll::launch_mixed_mma<1, 32, 8, 1, 2>(a, n_tiles, stream) : mll::launch_mixed_mma<1, 16, 8, 1, 2>(a, n_tiles, stream);
  } else if (shape.R == 8) {
    code = wide ? mll::launch_mixed_mma<8, 32, 16, 2, 1>(a, n_tiles * 16, stream) : mll::launch_mixed_mma<8, 16, 16, 2, 1>(a, n_tiles * 16, stream);
  } else {
    code = wide ? mll::launch_mixed_mma<16, 32, 16, 2, 1>(a, n_tiles * 8, stream) : mll::launch_mixed_mma<16, 16, 16, 2, 1>(a, n_tiles * 8, stream);
  }
  if (code != 0 || n_splits == 1 || !single) return code;
  const long long items = (long long)n_tiles * (n_heads * dv / 2);
  MLL_LAUNCH((mll::mixed_attention_sum_kernel), (unsigned)((items + 255) / 256), 256, 0, stream, scratch, seq_qstart,
             (__nv_bfloat16*)out, n_tiles, n_splits, n_heads * dv);
  MLL_LAUNCH_CHECK();
  return 0;
}

// Blocks along the rows that a prompt tile of 128 rows becomes (what a choice of n_splits goes by), or 0.
MLL_API int mll_mixed_attention_mma_blocks(int n_heads, int n_kv_heads, int d, int dv) {
  const mll::MixShape shape = mll::mix_mma_shape(0, n_heads, n_kv_heads, d, dv);
  if (shape.R == 0) return 0;
  return 128 / shape.R * ((mll::mix_units(n_heads, n_kv_heads, dv, shape.R, 2, 1) + shape.W - 1) / shape.W);
}
