// Embedding gather, dtype casts and the gated activations (SwiGLU and its relatives).
//
// Replaces the reference's EmbeddingKernel, SiluKernel and ElementWiseMulKernel
// (src/cuda_ops.cu:165-192) with batched kernels; SiLU and the product are one pass.
#include <stdarg.h>
#include <stdio.h>

#include "common.cuh"

static thread_local char g_error[512] = "";

void mll_set_error(const char* fmt, ...) {
  va_list args;
  va_start(args, fmt);
  vsnprintf(g_error, sizeof(g_error), fmt, args);
  va_end(args);
}

MLL_API const char* mll_last_error() { return g_error; }

thread_local cudaError_t mll_launch_status = cudaSuccess;

// Identifies the build; the Python side checks it after loading the library.
MLL_API int mll_abi_version() { return 35; }

// Cache positions per page, for the Python side to check against its own constant.
MLL_API int mll_page() { return MLL_PAGE; }

int mll_sm_count() {
  constexpr int kMaxDevices = 64;
  static int known[kMaxDevices] = {0};
  int device = 0, count = 0;
  if (cudaGetDevice(&device) != cudaSuccess || device < 0 || device >= kMaxDevices) {
    cudaGetLastError();
    device = 0;
  }
  if (known[device] == 0) {
    if (cudaDeviceGetAttribute(&count, cudaDevAttrMultiProcessorCount, device) != cudaSuccess || count < 1) {
      cudaGetLastError();
      count = 148;  // a B200, the device this library is written for
    }
    known[device] = count;
  }
  return known[device];
}

MLL_API int mll_multiprocessor_count() { return mll_sm_count(); }

namespace mll {

// x[t, :] = scale * float(table[token[t], :]); the residual stream is float32.
template <typename TableT>
__global__ void embedding_kernel(const int* __restrict__ tokens, const TableT* __restrict__ table,
                                 float* __restrict__ x, int width, float scale) {
  const int t = blockIdx.x;
  const TableT* row = table + (size_t)tokens[t] * width;
  float* out = x + (size_t)t * width;
  for (int i = threadIdx.x; i < width; i += blockDim.x) out[i] = to_float(row[i]) * scale;
}

// the same for a bfloat16 table whose rows are multiples of 8 elements: 16-byte loads, one per thread and pass
__global__ void embedding_bf16_vec8_kernel(const int* __restrict__ tokens, const __nv_bfloat16* __restrict__ table,
                                           float* __restrict__ x, int width, float scale) {
  const int t = blockIdx.x;
  const uint4* row = reinterpret_cast<const uint4*>(table + (size_t)tokens[t] * width);
  float4* out = reinterpret_cast<float4*>(x + (size_t)t * width);
  for (int i = threadIdx.x; i < (width >> 3); i += blockDim.x) {
    const uint4 raw = row[i];
    const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&raw);
    const float2 a = __bfloat1622float2(h[0]), b = __bfloat1622float2(h[1]);
    const float2 c = __bfloat1622float2(h[2]), d = __bfloat1622float2(h[3]);
    out[2 * i] = make_float4(a.x * scale, a.y * scale, b.x * scale, b.y * scale);
    out[2 * i + 1] = make_float4(c.x * scale, c.y * scale, d.x * scale, d.y * scale);
  }
}

// x[t, :] = scale * table[token[t], :] + pairs[row(t), :], row(t) a hash of the token before and the token itself:
// (mul_prev * previous + mul_cur * token) mod buckets, and row `buckets` (the table's last) for a sequence's first
// token.  The token before the first one of a step is the sequence's state (prev_token[slot]); the block of that
// first token also leaves the step's last token of its sequence there for the next step.
struct PairEmbedArgs {
  const int* tokens;
  const int* tok_pos;
  const int* tok_seq;
  const int* seq_slot;
  const int* seq_qstart;
  const int* seq_qlen;
  int* prev_token;   // [slots]
  float* x;          // [T, width]
  int width, buckets;
  long long mul_prev, mul_cur;
  float scale;
};

template <typename TableT>
__global__ void __launch_bounds__(128) embedding_pair_kernel(PairEmbedArgs a, const TableT* __restrict__ table,
                                                             const TableT* __restrict__ pairs) {
  __shared__ int pair_row;
  const int t = blockIdx.x;
  const int token = a.tokens[t];
  if (threadIdx.x == 0) {
    const int seq = a.tok_seq[t];
    const int first = a.seq_qstart[seq];
    int row = a.buckets;
    if (a.tok_pos[t] > 0) {
      const int before = t == first ? a.prev_token[a.seq_slot[seq]] : a.tokens[t - 1];
      long long v = (a.mul_prev * before + a.mul_cur * token) % a.buckets;
      row = (int)(v < 0 ? v + a.buckets : v);
    }
    if (t == first) a.prev_token[a.seq_slot[seq]] = a.tokens[first + a.seq_qlen[seq] - 1];  // read above, by this thread
    pair_row = row;
  }
  __syncthreads();
  const TableT* row = table + (size_t)token * a.width;
  float* out = a.x + (size_t)t * a.width;
  if (!pairs) {  // no pair table: the scaled row alone
    for (int i = threadIdx.x; i < a.width; i += blockDim.x) out[i] = a.scale * to_float(row[i]);
    return;
  }
  const TableT* prow = pairs + (size_t)pair_row * a.width;
  for (int i = threadIdx.x; i < a.width; i += blockDim.x) out[i] = fmaf(a.scale, to_float(row[i]), to_float(prow[i]));
}

template <typename In, typename Out>
__global__ void cast_kernel(const In* __restrict__ in, Out* __restrict__ out, size_t n) {
  size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
  const size_t stride = (size_t)gridDim.x * blockDim.x;
  for (; i < n; i += stride) out[i] = from_float<Out>(to_float(in[i]));
}

// out[t, i] = act(gate) * up, act silu or gelu in its tanh form (GATE_ACT_*).  `gu` rows hold gate and up either as two halves
// ([gate(0..I) | up(0..I)], block == 0) or interleaved in blocks of `block` columns
// ([gate(0..b) | up(0..b) | gate(b..2b) | ...]); I is a multiple of `block` then.
// `bias` (float32 [2 I], in the order of a row of gu, or null) is added to gate and up first.
template <typename T>
__global__ void swiglu_kernel(const T* __restrict__ gu, T* __restrict__ out, int tokens,
                              int inter, int block, const float* __restrict__ bias, int act) {
  const size_t total = (size_t)tokens * inter;
  size_t idx = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
  const size_t stride = (size_t)gridDim.x * blockDim.x;
  for (; idx < total; idx += stride) {
    const int t = (int)(idx / inter), i = (int)(idx % inter);
    const T* row = gu + (size_t)t * 2 * inter;
    float g, u;
    const int gc = block == 0 ? i : (i / block) * 2 * block + i % block;
    const int uc = block == 0 ? inter + i : gc + block;
    g = to_float(row[gc]);
    u = to_float(row[uc]);
    if (bias) {
      g += bias[gc];
      u += bias[uc];
    }
    out[idx] = from_float<T>(gate_act_mul<false>(act, g, u));
  }
}

// The same over groups of 8 consecutive outputs (inter % 8 == 0, block 0 or 8): 16- or
// 32-byte loads of a gate group and its up group, one vector store.
template <typename T>
struct Pack8;
template <>
struct Pack8<__nv_bfloat16> {
  static __device__ __forceinline__ void load(const __nv_bfloat16* p, float* v) {
    const uint4 raw = *reinterpret_cast<const uint4*>(p);
    const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const float2 f = __bfloat1622float2(h[i]);
      v[2 * i] = f.x;
      v[2 * i + 1] = f.y;
    }
  }
  static __device__ __forceinline__ void store(__nv_bfloat16* p, const float* v) {
    uint4 raw;
    __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&raw);
#pragma unroll
    for (int i = 0; i < 4; ++i) h[i] = __floats2bfloat162_rn(v[2 * i], v[2 * i + 1]);
    *reinterpret_cast<uint4*>(p) = raw;
  }
};
template <>
struct Pack8<float> {
  static __device__ __forceinline__ void load(const float* p, float* v) {
    const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
    v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
  }
  static __device__ __forceinline__ void store(float* p, const float* v) {
    *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
    *reinterpret_cast<float4*>(p + 4) = make_float4(v[4], v[5], v[6], v[7]);
  }
};

// The float32 path keeps the accurate exponential and division; a bfloat16 result
// is rounded to 8 bits anyway, so it takes the fast ones (a prefill step spends a tenth of its
// non-GEMM time here, and the accurate forms make the kernel compute-bound).
template <typename T>
__global__ void swiglu_vec8_kernel(const T* __restrict__ gu, T* __restrict__ out, int tokens, int inter, int block,
                                   const float* __restrict__ bias, int act) {
  const int groups = inter >> 3;
  const size_t total = (size_t)tokens * groups;
  size_t idx = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
  const size_t stride = (size_t)gridDim.x * blockDim.x;
  for (; idx < total; idx += stride) {
    const int t = (int)(idx / groups), b = (int)(idx % groups);
    const T* row = gu + (size_t)t * 2 * inter;
    const T* gp = block ? row + (size_t)b * 16 : row + (size_t)b * 8;
    const T* up = block ? gp + 8 : row + inter + (size_t)b * 8;
    float g[8], u[8], r[8];
    Pack8<T>::load(gp, g);
    Pack8<T>::load(up, u);
    if (bias) {  // groups of 8 floats start on 32-byte boundaries of the bias (the launch checks its base)
      float gb[8], ub[8];
      Pack8<float>::load(bias + (gp - row), gb);
      Pack8<float>::load(bias + (up - row), ub);
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        g[i] += gb[i];
        u[i] += ub[i];
      }
    }
#pragma unroll
    for (int i = 0; i < 8; ++i) r[i] = gate_act_mul<sizeof(T) == 2>(act, g[i], u[i]);
    Pack8<T>::store(out + (size_t)t * inter + (size_t)b * 8, r);
  }
}

__global__ void scale_kernel(float* __restrict__ x, size_t n, float factor) {
  size_t idx = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
  const size_t stride = (size_t)gridDim.x * blockDim.x;
  for (; idx < n; idx += stride) x[idx] *= factor;
}

// x = cap * tanh(factor * x / cap)
__global__ void softcap_kernel(float* __restrict__ x, size_t n, float factor, float cap) {
  const size_t at = ((size_t)blockIdx.x * blockDim.x + threadIdx.x) * 4, stride = (size_t)gridDim.x * blockDim.x * 4;
  const float inv = 1.f / cap;
  for (size_t i = at; i < n; i += stride) {
    if (i + 4 <= n) {  // the launch checks that x starts on a 16-byte boundary
      float4 v = *reinterpret_cast<float4*>(x + i);
      v.x = cap * tanhf(factor * v.x * inv); v.y = cap * tanhf(factor * v.y * inv);
      v.z = cap * tanhf(factor * v.z * inv); v.w = cap * tanhf(factor * v.w * inv);
      *reinterpret_cast<float4*>(x + i) = v;
    } else {
      for (size_t j = i; j < n; ++j) x[j] = cap * tanhf(factor * x[j] * inv);
    }
  }
}

// x[t, i] += bias[i] (bias float32, sum in float32)
template <typename T>
__global__ void add_bias_kernel(T* __restrict__ x, const float* __restrict__ bias, size_t total, int width) {
  size_t idx = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
  const size_t stride = (size_t)gridDim.x * blockDim.x;
  for (; idx < total; idx += stride) x[idx] = from_float<T>(to_float(x[idx]) + bias[idx % width]);
}

// The same in bfloat16, eight neighbouring columns a thread (width a multiple of 8).
__global__ void __launch_bounds__(256) add_bias_vec8_kernel(__nv_bfloat16* __restrict__ x, const float* __restrict__ bias,
                                                            size_t words, int row_words) {
  for (size_t i = (size_t)blockIdx.x * 256 + threadIdx.x; i < words; i += (size_t)gridDim.x * 256) {
    float v[8], b[8];
    Pack8<__nv_bfloat16>::load(x + i * 8, v);
    Pack8<float>::load(bias + (i % row_words) * 8, b);
#pragma unroll
    for (int k = 0; k < 8; ++k) v[k] += b[k];
    Pack8<__nv_bfloat16>::store(x + i * 8, v);
  }
}

// As swiglu_vec8_kernel (bfloat16, gate and up interleaved in blocks of 8), for rows of gate/up that still lack their
// RMS norm's factor (the product ran on x * w_norm): both are multiplied by the row's factor first.  One row per
// blockIdx.y; warp 0 computes the factor from the row's partial sums of squares.
__global__ void swiglu_rows_kernel(const __nv_bfloat16* __restrict__ gu, __nv_bfloat16* __restrict__ out, int inter,
                                   int block, RowNormIn in, int width, int act) {
  __shared__ float factor;
  const int m = blockIdx.y;
  if (threadIdx.x < 32) {
    const float f = row_norm_factor<32>(in.sumsq + (size_t)m * in.stride, in.partials, width, in.eps, threadIdx.x,
                                        0xffffffffu);
    if (threadIdx.x == 0) factor = f;
  }
  __syncthreads();
  const float f = factor;
  const int groups = inter >> 3;
  const int b = blockIdx.x * blockDim.x + threadIdx.x;
  if (b >= groups) return;
  const __nv_bfloat16* row = gu + (size_t)m * 2 * inter;
  const __nv_bfloat16* gp = block ? row + (size_t)b * 16 : row + (size_t)b * 8;
  const __nv_bfloat16* up = block ? gp + 8 : row + inter + (size_t)b * 8;
  float g[8], u[8], r[8];
  Pack8<__nv_bfloat16>::load(gp, g);
  Pack8<__nv_bfloat16>::load(up, u);
#pragma unroll
  for (int i = 0; i < 8; ++i) r[i] = gate_act_mul<true>(act, g[i] * f, u[i] * f);
  Pack8<__nv_bfloat16>::store(out + (size_t)m * inter + (size_t)b * 8, r);
}

// table[staged[r][0]][:] = staged[r][1 : 1 + width] for r < n_rows: rows of a block table that changed on
// the host, brought over inside the step's index buffer.
__global__ void scatter_rows_kernel(int* __restrict__ table, const int* __restrict__ staged, int width, int table_rows) {
  const int* row = staged + (size_t)blockIdx.x * (width + 1);
  const int target = row[0];
  if (target < 0 || target >= table_rows) return;
  for (int i = threadIdx.x; i < width; i += blockDim.x) table[(size_t)target * width + i] = row[1 + i];
}

// dst[i] = src[index[i]] for i < n; an index outside [0, n_src) gives 0.
__global__ void gather_int32_kernel(int* __restrict__ dst, const int* __restrict__ src, const int* __restrict__ index, int n,
                                    int n_src) {
  const int i = blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= n) return;
  const int at = index[i];
  dst[i] = at >= 0 && at < n_src ? src[at] : 0;
}

// out[t, 0:D] = x[t] + delta[t] (delta optional), out[t, D:2D] = x0[t]: the float32 residual stream (with the
// output of the last part still to be added) beside an earlier state of it, as one row for the product that
// mixes the two.  The sum is float32; T is the product's input type.
template <typename T>
__global__ void stream_concat_kernel(const float* __restrict__ x, const T* __restrict__ delta,
                                     const float* __restrict__ x0, T* __restrict__ out, size_t total, int width) {
  for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (size_t)gridDim.x * blockDim.x) {
    const size_t t = i / (2 * width);
    const int c = (int)(i % (2 * width));
    float v;
    if (c < width) {
      v = x[t * width + c];
      if (delta) v += to_float(delta[t * width + c]);
    } else {
      v = x0[t * width + c - width];
    }
    out[i] = from_float<T>(v);
  }
}

// out[t, h * dv + i] = in[t * in_t + h * in_h + i] * sigmoid(gate[t * gate_ld + (per_head ? h : h * dv + i)]):
// the output gate of an attention layer, one number per head or one per element, read from the projection's
// own row; the input may lie head-major (a batched product's result).  out may be in itself when the layouts agree.
template <typename T>
__global__ void heads_gate_kernel(const T* __restrict__ in, const T* __restrict__ gate, T* __restrict__ out,
                                  size_t total, int n_heads, int dv, long long in_t, long long in_h, int gate_ld,
                                  int per_head) {
  for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (size_t)gridDim.x * blockDim.x) {
    const size_t t = i / ((size_t)n_heads * dv);
    const int c = (int)(i % ((size_t)n_heads * dv));
    const int h = c / dv, e = c % dv;
    const float g = to_float(gate[t * gate_ld + (per_head ? h : c)]);
    const float v = to_float(in[t * in_t + (size_t)h * in_h + e]);
    out[i] = from_float<T>(v / (1.f + expf(-g)));
  }
}

// The same in bfloat16 with one gate per head, eight neighbouring values a thread (dv and the strides multiples of 8).
__global__ void __launch_bounds__(256) heads_gate_vec_kernel(const __nv_bfloat16* in, const __nv_bfloat16* gate, __nv_bfloat16* out,
                                                             size_t words, int n_heads, int dv, long long in_t, long long in_h,
                                                             int gate_ld) {
  const int per_head = dv / 8, per_token = n_heads * per_head;
  for (size_t i = (size_t)blockIdx.x * 256 + threadIdx.x; i < words; i += (size_t)gridDim.x * 256) {
    const size_t t = i / per_token;
    const int w = (int)(i - t * per_token), h = w / per_head;
    uint4 v = *reinterpret_cast<const uint4*>(in + t * in_t + (size_t)h * in_h + (w - h * per_head) * 8);
    const float f = 1.f / (1.f + expf(-__bfloat162float(gate[t * gate_ld + h])));
    __nv_bfloat162* p = reinterpret_cast<__nv_bfloat162*>(&v);
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      const float2 x = __bfloat1622float2(p[k]);
      p[k] = __floats2bfloat162_rn(x.x * f, x.y * f);
    }
    *reinterpret_cast<uint4*>(out + i * 8) = v;
  }
}

// out = act(in), elementwise, evaluated in float32.  kind 0: gelu in its erf form, 0.5 z (1 + erf(z / sqrt 2));
// 1: gelu in its tanh form, 0.5 z (1 + tanh(sqrt(2 / pi) (z + 0.044715 z^3))).
template <typename T>
__global__ void activation_kernel(const T* __restrict__ in, T* __restrict__ out, size_t total, int kind) {
  for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (size_t)gridDim.x * blockDim.x) {
    const float z = to_float(in[i]);
    const float v = kind == 0 ? 0.5f * z * (1.f + erff(z * 0.70710678118654752f))
                              : 0.5f * z * (1.f + tanhf(0.79788456080286536f * (z + 0.044715f * z * z * z)));
    out[i] = from_float<T>(v);
  }
}

}  // namespace mll

// in, out: [n] of `dtype` (out may be in); kind: see activation_kernel.
MLL_API int mll_activation(const void* in, void* out, int dtype, long long n, int kind, cudaStream_t stream) {
  MLL_REQUIRE(n >= 0 && (kind == 0 || kind == 1), "activation: bad size %lld or kind %d", n, kind);
  if (n == 0) return 0;
  long long blocks = (n + 255) / 256;
  if (blocks > mll_sm_count() * 16) blocks = mll_sm_count() * 16;
  if (dtype == MLL_F32)
    MLL_LAUNCH((mll::activation_kernel<float>), (int)blocks, 256, 0, stream, (const float*)in, (float*)out, (size_t)n, kind);
  else if (dtype == MLL_BF16)
    MLL_LAUNCH((mll::activation_kernel<__nv_bfloat16>), (int)blocks, 256, 0, stream, (const __nv_bfloat16*)in,
               (__nv_bfloat16*)out, (size_t)n, kind);
  else
    MLL_REQUIRE(false, "activation: unknown dtype %d", dtype);
  MLL_LAUNCH_CHECK();
  return 0;
}

// dst: int32 [n]; src: int32 [n_src]; index: int32 [n].  dst and src must not overlap.
MLL_API int mll_gather_int32(int* dst, const int* src, const int* index, int n, int n_src, cudaStream_t stream) {
  MLL_REQUIRE(n >= 0 && n_src > 0, "gather_int32: bad sizes n=%d n_src=%d", n, n_src);
  if (n == 0) return 0;
  MLL_LAUNCH((mll::gather_int32_kernel), (n + 127) / 128, 128, 0, stream, dst, src, index, n, n_src);
  MLL_LAUNCH_CHECK();
  return 0;
}

// table: int32 [table_rows, width]; staged: int32 [n_rows, 1 + width], column 0 the row of `table` to replace.
MLL_API int mll_scatter_rows(int* table, const int* staged, int n_rows, int width, int table_rows, cudaStream_t stream) {
  MLL_REQUIRE(n_rows >= 0 && width > 0 && table_rows > 0, "scatter_rows: bad sizes rows=%d width=%d", n_rows, width);
  if (n_rows == 0) return 0;
  MLL_LAUNCH((mll::scatter_rows_kernel), n_rows, width >= 128 ? 128 : 32, 0, stream, table, staged, width, table_rows);
  MLL_LAUNCH_CHECK();
  return 0;
}

// x[i] *= factor (float32, in place)
MLL_API int mll_scale(float* x, long long n, float factor, cudaStream_t stream) {
  MLL_REQUIRE(n >= 0, "scale: bad size %lld", n);
  if (n == 0) return 0;
  long long blocks = (n + 255) / 256;
  if (blocks > mll_sm_count() * 16) blocks = mll_sm_count() * 16;
  MLL_LAUNCH((mll::scale_kernel), (int)blocks, 256, 0, stream, x, (size_t)n, factor);
  MLL_LAUNCH_CHECK();
  return 0;
}

// x[i] = cap * tanh(factor * x[i] / cap) (float32, in place)
MLL_API int mll_softcap(float* x, long long n, float factor, float cap, cudaStream_t stream) {
  MLL_REQUIRE(n >= 0 && cap > 0.f, "softcap: bad size %lld or cap", n);
  MLL_REQUIRE((uintptr_t)x % 16 == 0, "softcap: the tensor must be 16-byte aligned");
  if (n == 0) return 0;
  long long blocks = (n + 1023) / 1024;
  if (blocks > mll_sm_count() * 16) blocks = mll_sm_count() * 16;
  MLL_LAUNCH((mll::softcap_kernel), (int)blocks, 256, 0, stream, x, (size_t)n, factor, cap);
  MLL_LAUNCH_CHECK();
  return 0;
}

MLL_API int mll_add_bias(void* x, const float* bias, int dtype, int n_rows, int width, cudaStream_t stream) {
  MLL_REQUIRE(n_rows >= 0 && width > 0, "add_bias: bad sizes rows=%d width=%d", n_rows, width);
  if (n_rows == 0) return 0;
  const size_t total = (size_t)n_rows * width;
  if (dtype == MLL_BF16 && width % 8 == 0 && (uintptr_t)x % 16 == 0 && (uintptr_t)bias % 16 == 0) {
    const long long want = (long long)((total / 8 + 255) / 256), most = (long long)mll_sm_count() * 16;
    MLL_LAUNCH((mll::add_bias_vec8_kernel), (int)(want < most ? want : most), 256, 0, stream, (__nv_bfloat16*)x, bias,
               total / 8, width / 8);
    MLL_LAUNCH_CHECK();
    return 0;
  }
  long long blocks = (long long)((total + 255) / 256);
  if (blocks > mll_sm_count() * 16) blocks = mll_sm_count() * 16;
  if (dtype == MLL_F32)
    MLL_LAUNCH((mll::add_bias_kernel<float>), (int)blocks, 256, 0, stream, (float*)x, bias, total, width);
  else if (dtype == MLL_BF16)
    MLL_LAUNCH((mll::add_bias_kernel<__nv_bfloat16>), (int)blocks, 256, 0, stream, (__nv_bfloat16*)x, bias, total, width);
  else
    MLL_REQUIRE(false, "add_bias: unknown dtype %d", dtype);
  MLL_LAUNCH_CHECK();
  return 0;
}

MLL_API int mll_embedding(const int* tokens, const void* table, int table_dtype, float* x,
                          int n_tokens, int width, float scale, cudaStream_t stream) {
  MLL_REQUIRE(n_tokens >= 0 && width > 0, "embedding: bad sizes tokens=%d width=%d", n_tokens, width);
  if (n_tokens == 0) return 0;
  const int threads = width >= 1024 ? 256 : 128;
  if (table_dtype == MLL_F32)
    MLL_LAUNCH((mll::embedding_kernel<float>), n_tokens, threads, 0, stream, tokens, (const float*)table, x, width, scale);
  else if (table_dtype == MLL_BF16 && width % 8 == 0 && ((uintptr_t)table % 16 == 0) && ((uintptr_t)x % 16 == 0))
    MLL_LAUNCH((mll::embedding_bf16_vec8_kernel), n_tokens, width >= 2048 ? 256 : 64, 0, stream, tokens,
               (const __nv_bfloat16*)table, x, width, scale);
  else if (table_dtype == MLL_BF16)
    MLL_LAUNCH((mll::embedding_kernel<__nv_bfloat16>), n_tokens, threads, 0, stream, tokens, (const __nv_bfloat16*)table, x, width, scale);
  else
    MLL_REQUIRE(false, "embedding: unknown table dtype %d", table_dtype);
  MLL_LAUNCH_CHECK();
  return 0;
}

// tokens, tok_pos, tok_seq: int32 [n_tokens]; seq_slot, seq_qstart, seq_qlen: int32 per sequence; prev_token: int32
// [slots]; table [vocab, width] and pairs [buckets + 1, width] of `table_dtype`; x: float32 [n_tokens, width].
MLL_API int mll_embedding_pair(const int* tokens, const int* tok_pos, const int* tok_seq, const int* seq_slot,
                               const int* seq_qstart, const int* seq_qlen, int* prev_token, const void* table,
                               const void* pairs, int table_dtype, float* x, int n_tokens, int width, int buckets,
                               long long mul_prev, long long mul_cur, float scale, cudaStream_t stream) {
  MLL_REQUIRE(n_tokens >= 0 && width > 0 && buckets > 0, "pair embedding: bad sizes tokens=%d width=%d buckets=%d",
              n_tokens, width, buckets);
  if (n_tokens == 0) return 0;
  mll::PairEmbedArgs a{tokens, tok_pos, tok_seq, seq_slot, seq_qstart, seq_qlen, prev_token, x, width, buckets,
                       mul_prev, mul_cur, scale};
  if (table_dtype == MLL_F32)
    MLL_LAUNCH((mll::embedding_pair_kernel<float>), n_tokens, 128, 0, stream, a, (const float*)table, (const float*)pairs);
  else if (table_dtype == MLL_BF16)
    MLL_LAUNCH((mll::embedding_pair_kernel<__nv_bfloat16>), n_tokens, 128, 0, stream, a, (const __nv_bfloat16*)table,
               (const __nv_bfloat16*)pairs);
  else
    MLL_REQUIRE(false, "pair embedding: unknown table dtype %d", table_dtype);
  MLL_LAUNCH_CHECK();
  return 0;
}

MLL_API int mll_cast(const void* in, int in_dtype, void* out, int out_dtype, long long n,
                     cudaStream_t stream) {
  MLL_REQUIRE(n >= 0, "cast: negative size");
  if (n == 0) return 0;
  const int threads = 256;
  long long blocks = (n + threads - 1) / threads;
  if (blocks > mll_sm_count() * 16) blocks = mll_sm_count() * 16;
  if (in_dtype == MLL_F32 && out_dtype == MLL_BF16)
    MLL_LAUNCH((mll::cast_kernel<float, __nv_bfloat16>), (int)blocks, threads, 0, stream, (const float*)in, (__nv_bfloat16*)out, (size_t)n);
  else if (in_dtype == MLL_BF16 && out_dtype == MLL_F32)
    MLL_LAUNCH((mll::cast_kernel<__nv_bfloat16, float>), (int)blocks, threads, 0, stream, (const __nv_bfloat16*)in, (float*)out, (size_t)n);
  else
    MLL_REQUIRE(false, "cast: unsupported dtype pair %d -> %d", in_dtype, out_dtype);
  MLL_LAUNCH_CHECK();
  return 0;
}

// bfloat16 gu [n_tokens, 2 inter] (halves: block 0; blocks of 8: block 8) computed from rows that lack their RMS
// norm's factor 1 / sqrt(sum_p sumsq[m][p] / width + eps): out = act(gate f) * (up f).
MLL_API int mll_swiglu_rows(const void* gu, void* out, int n_tokens, int inter, int block, const float* sumsq, int partials,
                            int stride, float eps, int width, int act, cudaStream_t stream) {
  MLL_REQUIRE(act == mll::GATE_ACT_SILU || act == mll::GATE_ACT_GELU_TANH, "swiglu_rows: unknown activation %d", act);
  MLL_REQUIRE(n_tokens >= 0 && n_tokens <= 65535 && inter > 0 && inter % 8 == 0 && (block == 0 || block == 8),
              "swiglu_rows: bad sizes tokens=%d inter=%d block=%d", n_tokens, inter, block);
  MLL_REQUIRE(sumsq && partials >= 1 && stride >= partials && eps >= 0.f && width > 0,
              "swiglu_rows: partial sums: %d of stride %d", partials, stride);
  MLL_REQUIRE(((uintptr_t)gu % 16 == 0) && ((uintptr_t)out % 16 == 0), "swiglu_rows: operands must be 16-byte aligned");
  if (n_tokens == 0) return 0;
  const int groups = inter / 8;
  MLL_LAUNCH((mll::swiglu_rows_kernel), dim3((groups + 255) / 256, n_tokens), 256, 0, stream, (const __nv_bfloat16*)gu,
             (__nv_bfloat16*)out, inter, block, mll::RowNormIn{sumsq, partials, stride, eps}, width, act);
  MLL_LAUNCH_CHECK();
  return 0;
}

MLL_API int mll_swiglu(const void* gu, void* out, int dtype, int n_tokens, int inter, int block, const float* bias,
                       int act, cudaStream_t stream) {
  MLL_REQUIRE(act == mll::GATE_ACT_SILU || act == mll::GATE_ACT_GELU_TANH, "swiglu: unknown activation %d", act);
  MLL_REQUIRE(n_tokens >= 0 && inter > 0, "swiglu: bad sizes tokens=%d inter=%d", n_tokens, inter);
  MLL_REQUIRE(block >= 0 && (block == 0 || inter % block == 0),
              "swiglu: intermediate size %d is not a multiple of the interleave block %d", inter, block);
  if (n_tokens == 0) return 0;
  const int threads = 256;
  const bool vec = inter % 8 == 0 && (block == 0 || block == 8) && ((uintptr_t)gu % 16 == 0) &&
                   ((uintptr_t)out % 16 == 0) && ((uintptr_t)bias % 16 == 0);
  if (vec) {
    long long groups = ((long long)n_tokens * (inter / 8) + threads - 1) / threads;
    if (groups > mll_sm_count() * 32) groups = mll_sm_count() * 32;
    if (dtype == MLL_F32)
      MLL_LAUNCH((mll::swiglu_vec8_kernel<float>), (int)groups, threads, 0, stream, (const float*)gu, (float*)out, n_tokens,
                                                                       inter, block, bias, act);
    else if (dtype == MLL_BF16)
      MLL_LAUNCH((mll::swiglu_vec8_kernel<__nv_bfloat16>), (int)groups, threads, 0, stream, (const __nv_bfloat16*)gu, (__nv_bfloat16*)out, n_tokens, inter, block, bias, act);
    else
      MLL_REQUIRE(false, "swiglu: unknown dtype %d", dtype);
    MLL_LAUNCH_CHECK();
    return 0;
  }
  long long blocks = ((long long)n_tokens * inter + threads - 1) / threads;
  if (blocks > mll_sm_count() * 32) blocks = mll_sm_count() * 32;
  if (dtype == MLL_F32)
    MLL_LAUNCH((mll::swiglu_kernel<float>), (int)blocks, threads, 0, stream, (const float*)gu, (float*)out, n_tokens, inter, block, bias, act);
  else if (dtype == MLL_BF16)
    MLL_LAUNCH((mll::swiglu_kernel<__nv_bfloat16>), (int)blocks, threads, 0, stream, (const __nv_bfloat16*)gu, (__nv_bfloat16*)out, n_tokens, inter, block, bias, act);
  else
    MLL_REQUIRE(false, "swiglu: unknown dtype %d", dtype);
  MLL_LAUNCH_CHECK();
  return 0;
}

// x, x0: float32 [n_tokens, width]; delta: optional [n_tokens, width] of `dtype`; out: [n_tokens, 2 width] of `dtype`.
MLL_API int mll_stream_concat(const float* x, const void* delta, const float* x0, void* out, int dtype, int n_tokens,
                              int width, cudaStream_t stream) {
  MLL_REQUIRE(n_tokens >= 0 && width > 0, "stream_concat: bad sizes tokens=%d width=%d", n_tokens, width);
  if (n_tokens == 0) return 0;
  const size_t total = (size_t)n_tokens * 2 * width;
  long long blocks = (long long)((total + 255) / 256);
  if (blocks > mll_sm_count() * 16) blocks = mll_sm_count() * 16;
  if (dtype == MLL_F32)
    MLL_LAUNCH((mll::stream_concat_kernel<float>), (int)blocks, 256, 0, stream, x, (const float*)delta, x0, (float*)out,
               total, width);
  else if (dtype == MLL_BF16)
    MLL_LAUNCH((mll::stream_concat_kernel<__nv_bfloat16>), (int)blocks, 256, 0, stream, x, (const __nv_bfloat16*)delta,
               x0, (__nv_bfloat16*)out, total, width);
  else
    MLL_REQUIRE(false, "stream_concat: unknown dtype %d", dtype);
  MLL_LAUNCH_CHECK();
  return 0;
}

// in: element (t, h, i) at t * in_t + h * in_h + i; gate: [n_tokens, gate_ld] (already offset to the gate's first
// column); out: [n_tokens, n_heads * dv]; all of `dtype`.
MLL_API int mll_heads_gate(const void* in, const void* gate, void* out, int dtype, int n_tokens, int n_heads, int dv,
                           long long in_t, long long in_h, int gate_ld, int per_head, cudaStream_t stream) {
  MLL_REQUIRE(n_tokens >= 0 && n_heads > 0 && dv > 0 && gate_ld > 0, "heads_gate: bad sizes");
  if (n_tokens == 0) return 0;
  const size_t total = (size_t)n_tokens * n_heads * dv;
  if (dtype == MLL_BF16 && per_head && dv % 8 == 0 && in_t % 8 == 0 && in_h % 8 == 0 && (uintptr_t)in % 16 == 0 && (uintptr_t)out % 16 == 0) {
    const long long want = (long long)((total / 8 + 255) / 256), most = (long long)mll_sm_count() * 8;
    MLL_LAUNCH((mll::heads_gate_vec_kernel), (int)(want < most ? want : most), 256, 0, stream, (const __nv_bfloat16*)in,
               (const __nv_bfloat16*)gate, (__nv_bfloat16*)out, total / 8, n_heads, dv, in_t, in_h, gate_ld);
    MLL_LAUNCH_CHECK();
    return 0;
  }
  long long blocks = (long long)((total + 255) / 256);
  if (blocks > mll_sm_count() * 16) blocks = mll_sm_count() * 16;
  if (dtype == MLL_F32)
    MLL_LAUNCH((mll::heads_gate_kernel<float>), (int)blocks, 256, 0, stream, (const float*)in, (const float*)gate,
               (float*)out, total, n_heads, dv, in_t, in_h, gate_ld, per_head);
  else if (dtype == MLL_BF16)
    MLL_LAUNCH((mll::heads_gate_kernel<__nv_bfloat16>), (int)blocks, 256, 0, stream, (const __nv_bfloat16*)in,
               (const __nv_bfloat16*)gate, (__nv_bfloat16*)out, total, n_heads, dv, in_t, in_h, gate_ld, per_head);
  else
    MLL_REQUIRE(false, "heads_gate: unknown dtype %d", dtype);
  MLL_LAUNCH_CHECK();
  return 0;
}
