// Windowed attention whose heads look at each other's scores and whose weights are no softmax:
//
//   s_g(i, j) = scale * q_g(i) . k_(g / group)(j)               H query heads of d over Hk key heads
//   z_h(i, j) = sum_g M[h, g] s_g(i, j) + b_h                   one matrix over the heads (null: z = s + b)
//   out_h(i)  = sum_j sigmoid(z_h(i, j)) v_(h / group)(j)       j <= i, and j > i - window where window > 0
//
// The weights of a row are not normalised over its keys, so there is no running maximum, and sums over runs of keys
// simply add up.  Scores, mixing, weights and sums are float32.
//
// This file is the general kernel: every dtype, head count and head size, prompts and single tokens alike.  One block
// owns a token and up to `hpb` output heads; it needs the scores of all H heads at every key, so it walks the window in
// runs of 32 keys: the scores of the run (a key head's rows at a time pass through shared memory), the mixed weights,
// then the weighted values.
#include "attention_mix.cuh"

namespace mll {

constexpr int MIX_KEYS = 32;
constexpr int MIX_THREADS = 256;

template <typename T, int NACC>
__global__ void __launch_bounds__(MIX_THREADS) mixed_attention_kernel(MixAttnArgs a, int hpb) {
  extern __shared__ __align__(16) unsigned char smem_raw[];
  const int H = a.n_heads, G = a.n_kv_heads, d = a.d, dv = a.dv, group = H / G;
  const int t = blockIdx.x, h0 = blockIdx.y * hpb, nh = min(hpb, H - h0);
  const int tid = threadIdx.x;
  const int pos = a.tok_pos[t];
  const int first = a.window > 0 ? max(0, pos - a.window + 1) : 0;
  const int* table = a.block_table + (size_t)a.seq_slot[a.tok_seq[t]] * a.max_blocks;

  float* q_s = reinterpret_cast<float*>(smem_raw);      // [H][d], scaled
  float* s_s = q_s + (size_t)H * d;                      // [H][MIX_KEYS]
  float* p_s = s_s + (size_t)H * MIX_KEYS;               // [hpb][MIX_KEYS]
  T* tile = reinterpret_cast<T*>(p_s + (size_t)hpb * MIX_KEYS);  // [MIX_KEYS][max(d, dv) + 1]
  const int stride = max(d, dv) + 1;

  for (int i = tid; i < H * d; i += MIX_THREADS) q_s[i] = to_float(((const T*)a.q)[(size_t)t * H * d + i]) * a.scale;
  float acc[NACC];
#pragma unroll
  for (int i = 0; i < NACC; ++i) acc[i] = 0.f;
  const int kv_lo = h0 / group, kv_hi = (h0 + nh - 1) / group;

  for (int base = first / MIX_KEYS * MIX_KEYS; base <= pos; base += MIX_KEYS) {
    // a run of 32 keys lies inside one page of 64
    const size_t page = (size_t)table[base / MLL_PAGE];
    const int in_page = base % MLL_PAGE;
    const int lo = max(0, first - base), hi = min(MIX_KEYS, pos + 1 - base);  // visible rows of the run
    for (int g = 0; g < G; ++g) {
      const T* src = (const T*)a.k_cache + ((page * G + g) * MLL_PAGE + in_page) * d;
      __syncthreads();
      for (int i = tid; i < (hi - lo) * d; i += MIX_THREADS) {
        const int r = lo + i / d, e = i % d;
        tile[r * stride + e] = src[(size_t)r * d + e];
      }
      __syncthreads();
      for (int i = tid; i < group * MIX_KEYS; i += MIX_THREADS) {
        const int h = g * group + i / MIX_KEYS, j = i % MIX_KEYS;
        float dot = 0.f;
        if (j >= lo && j < hi) {
          const float* q = q_s + (size_t)h * d;
          const T* k = tile + j * stride;
          for (int e = 0; e < d; ++e) dot = fmaf(q[e], to_float(k[e]), dot);
        }
        s_s[h * MIX_KEYS + j] = dot;
      }
    }
    __syncthreads();
    for (int i = tid; i < nh * MIX_KEYS; i += MIX_THREADS) {
      const int h = i / MIX_KEYS, j = i % MIX_KEYS;
      float z;
      if (a.mix) {
        z = 0.f;
        const float* row = a.mix + (size_t)(h0 + h) * H;
        for (int g = 0; g < H; ++g) z = fmaf(__ldg(row + g), s_s[g * MIX_KEYS + j], z);
      } else {
        z = s_s[(h0 + h) * MIX_KEYS + j];
      }
      z += a.bias ? a.bias[h0 + h] : 0.f;
      p_s[h * MIX_KEYS + j] = (j >= lo && j < hi) ? 1.f / (1.f + expf(-z)) : 0.f;
    }
    for (int g = kv_lo; g <= kv_hi; ++g) {
      const T* src = (const T*)a.v_cache + ((page * G + g) * MLL_PAGE + in_page) * dv;
      __syncthreads();
      for (int i = tid; i < (hi - lo) * dv; i += MIX_THREADS) {
        const int r = lo + i / dv, e = i % dv;
        tile[r * stride + e] = src[(size_t)r * dv + e];
      }
      __syncthreads();
#pragma unroll
      for (int i = 0; i < NACC; ++i) {
        const int o = tid + MIX_THREADS * i;
        if (o < nh * dv && (h0 + o / dv) / group == g) {
          const float* p = p_s + (o / dv) * MIX_KEYS;
          const T* v = tile + o % dv;
          float sum = acc[i];
          for (int j = lo; j < hi; ++j) sum = fmaf(p[j], to_float(v[j * stride]), sum);
          acc[i] = sum;
        }
      }
    }
  }
#pragma unroll
  for (int i = 0; i < NACC; ++i) {
    const int o = tid + MIX_THREADS * i;
    if (o < nh * dv) ((T*)a.out)[((size_t)t * H + h0) * dv + o] = from_float<T>(acc[i]);
  }
}

template <typename T>
int launch_mixed_attention(const MixAttnArgs& a, cudaStream_t stream) {
  const int hpb = max(1, min(a.n_heads, MIX_THREADS * 8 / a.dv));  // at most 8 accumulators a thread
  const int chunks = (a.n_heads + hpb - 1) / hpb;
  const size_t smem = ((size_t)a.n_heads * a.d + (size_t)(a.n_heads + hpb) * MIX_KEYS) * sizeof(float) +
                      (size_t)MIX_KEYS * (max(a.d, a.dv) + 1) * sizeof(T);
  MLL_REQUIRE(smem <= 200 * 1024, "mixed attention: %d heads of %d / %d need %zu bytes of shared memory", a.n_heads, a.d,
              a.dv, smem);
  const dim3 grid(a.n_tokens, chunks);
  const int nacc = (hpb * a.dv + MIX_THREADS - 1) / MIX_THREADS;
#define MLL_MIX_LAUNCH(N)                                                                                     \
  do {                                                                                                        \
    auto kernel = mixed_attention_kernel<T, N>;                                                               \
    if (smem > 48 * 1024) {                                                                                   \
      cudaError_t err = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
      if (err != cudaSuccess) {                                                                               \
        mll_set_error("mixed attention: cannot reserve %zu bytes of shared memory: %s", smem,                 \
                      cudaGetErrorString(err));                                                               \
        return (int)err;                                                                                      \
      }                                                                                                       \
    }                                                                                                         \
    MLL_LAUNCH((kernel), grid, MIX_THREADS, smem, stream, a, hpb);                                            \
  } while (0)
  if (nacc <= 1) MLL_MIX_LAUNCH(1);
  else if (nacc <= 2) MLL_MIX_LAUNCH(2);
  else if (nacc <= 4) MLL_MIX_LAUNCH(4);
  else MLL_MIX_LAUNCH(8);
#undef MLL_MIX_LAUNCH
  MLL_LAUNCH_CHECK();
  return 0;
}

}  // namespace mll

MLL_API int mll_mixed_attention(const void* q, const void* k_cache, const void* v_cache, const int* tok_pos,
                                const int* tok_seq, const int* seq_slot, const int* block_table, const float* mix,
                                const float* bias, void* out, int dtype, int n_tokens, int n_heads, int n_kv_heads, int d,
                                int dv, int window, int max_blocks, float scale, cudaStream_t stream) {
  MLL_REQUIRE(n_tokens >= 0 && n_heads > 0 && n_kv_heads > 0 && n_heads % n_kv_heads == 0, "mixed attention: bad head counts");
  MLL_REQUIRE(d > 0 && d <= 2048 && dv > 0 && dv <= 2048 && window >= 0, "mixed attention: head sizes %d / %d, window %d", d,
              dv, window);
  if (n_tokens == 0) return 0;
  mll::MixAttnArgs a{};
  a.q = q; a.k_cache = k_cache; a.v_cache = v_cache;
  a.tok_pos = tok_pos; a.tok_seq = tok_seq; a.seq_slot = seq_slot; a.block_table = block_table;
  a.mix = mix; a.bias = bias; a.out = out;
  a.n_tokens = n_tokens; a.n_heads = n_heads; a.n_kv_heads = n_kv_heads; a.d = d; a.dv = dv;
  a.window = window; a.max_blocks = max_blocks; a.scale = scale;
  if (dtype == MLL_F32) return mll::launch_mixed_attention<float>(a, stream);
  if (dtype == MLL_BF16) return mll::launch_mixed_attention<__nv_bfloat16>(a, stream);
  MLL_REQUIRE(false, "mixed attention: unknown dtype %d", dtype);
  return -1;
}
