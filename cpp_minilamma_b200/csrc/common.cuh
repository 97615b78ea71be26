// Shared device helpers of the kernel library (sm_100a).
//
// Every exported entry point is `extern "C"`, takes raw device pointers, sizes and
// a stream, validates its arguments on the host and returns 0 on success.  A refused
// argument returns a negative code and leaves a message for mll_last_error(); a CUDA
// launch error returns the positive cudaError_t.  Nothing here allocates memory or
// synchronises.
#pragma once

#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#define MLL_API extern "C" __attribute__((visibility("default")))

// dtype codes shared with the Python binding
enum : int { MLL_F32 = 0, MLL_BF16 = 1 };

// number of cache positions in one page
#define MLL_PAGE 64

void mll_set_error(const char* fmt, ...);

#define MLL_REQUIRE(cond, ...)        \
  do {                                \
    if (!(cond)) {                    \
      mll_set_error(__VA_ARGS__);     \
      return -1;                      \
    }                                 \
  } while (0)

// Launches `kernel` on `stream`; the outcome is picked up by MLL_LAUNCH_CHECK.
#define MLL_LAUNCH(kernel, grid, block, smem, stream, ...) \
  mll_launch_status = mll::launch_kernel(kernel, dim3(grid), dim3(block), (size_t)(smem), stream, ##__VA_ARGS__)

#define MLL_LAUNCH_CHECK()                          \
  do {                                              \
    cudaError_t err__ = mll_launch_status;          \
    mll_launch_status = cudaSuccess;                \
    if (err__ == cudaSuccess) err__ = cudaGetLastError(); \
    if (err__ != cudaSuccess) {                     \
      mll_set_error("%s:%d launch failed: %s", __FILE__, __LINE__, cudaGetErrorString(err__)); \
      return (int)err__;                            \
    }                                               \
  } while (0)

extern thread_local cudaError_t mll_launch_status;

// Multiprocessors of the current device (asked once per device; the kernels size their grids by it).
int mll_sm_count();

namespace mll {

template <typename... KernelArgs, typename... Args>
inline cudaError_t launch_kernel(void (*kernel)(KernelArgs...), dim3 grid, dim3 block, size_t smem,
                                 cudaStream_t stream, Args... args) {
  cudaLaunchConfig_t config = {};
  config.gridDim = grid;
  config.blockDim = block;
  config.dynamicSmemBytes = smem;
  config.stream = stream;
  return cudaLaunchKernelEx(&config, kernel, static_cast<KernelArgs>(args)...);
}

__device__ __forceinline__ float to_float(float v) { return v; }
__device__ __forceinline__ float to_float(__nv_bfloat16 v) { return __bfloat162float(v); }

template <typename T>
__device__ __forceinline__ T from_float(float v);
template <>
__device__ __forceinline__ float from_float<float>(float v) { return v; }
template <>
__device__ __forceinline__ __nv_bfloat16 from_float<__nv_bfloat16>(float v) {
  return __float2bfloat16_rn(v);
}

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}

__device__ __forceinline__ float warp_max(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, o));
  return v;
}

// Block-wide sum with a fixed reduction tree (same result on every run).
// `scratch` holds at least 32 floats; every thread gets the total.
__device__ __forceinline__ float block_sum(float v, float* scratch) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int nwarps = (blockDim.x + 31) >> 5;
  v = warp_sum(v);
  __syncthreads();
  if (lane == 0) scratch[warp] = v;
  __syncthreads();
  float total = (lane < nwarps) ? scratch[lane] : 0.f;
  total = warp_sum(total);
  return total;
}

__device__ __forceinline__ float block_max(float v, float* scratch) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int nwarps = (blockDim.x + 31) >> 5;
  v = warp_max(v);
  __syncthreads();
  if (lane == 0) scratch[warp] = v;
  __syncthreads();
  float total = (lane < nwarps) ? scratch[lane] : -INFINITY;
  total = warp_max(total);
  return total;
}

// First key that the one query token of a decode step may see, `ctx` being the sequence's length with that token.
// window > 0: the last `window` positions.  window < 0 names a chunk of -window positions instead: the keys of
// the query's own chunk, chunks counted from position 0 (the query sits at ctx - 1).
__device__ __forceinline__ int decode_first_key(int ctx, int window) {
  if (window > 0) return max(0, ctx - window);
  if (window < 0) return ((ctx - 1) / -window) * -window;
  return 0;
}

// V neighbouring values (V * sizeof(T) a power of two; p aligned to as many bytes, 16 at most) as floats
template <typename T, int V>
__device__ __forceinline__ void load_floats(const T* p, float* out) {
  if constexpr (sizeof(T) == 4) {
    if constexpr (V % 4 == 0) {
#pragma unroll
      for (int i = 0; i < V; i += 4) {
        const float4 v = *reinterpret_cast<const float4*>((const float*)p + i);
        out[i] = v.x; out[i + 1] = v.y; out[i + 2] = v.z; out[i + 3] = v.w;
      }
    } else {
#pragma unroll
      for (int i = 0; i < V; ++i) out[i] = to_float(p[i]);
    }
  } else if constexpr (V == 1) {
    out[0] = to_float(p[0]);
  } else {
    unsigned raw[(V + 1) / 2];
    if constexpr (V == 8) {
      const uint4 v = *reinterpret_cast<const uint4*>(p);
      raw[0] = v.x; raw[1] = v.y; raw[2] = v.z; raw[3] = v.w;
    } else if constexpr (V == 4) {
      const uint2 v = *reinterpret_cast<const uint2*>(p);
      raw[0] = v.x; raw[1] = v.y;
    } else {
      raw[0] = *reinterpret_cast<const unsigned*>(p);
    }
#pragma unroll
    for (int i = 0; i < V / 2; ++i) {
      const float2 f = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw[i]));
      out[2 * i] = f.x;
      out[2 * i + 1] = f.y;
    }
  }
}
template <typename T, int V>
__device__ __forceinline__ void store_floats(T* p, const float* v) {
  if constexpr (sizeof(T) == 4) {
    if constexpr (V % 4 == 0) {
#pragma unroll
      for (int i = 0; i < V; i += 4) *reinterpret_cast<float4*>((float*)p + i) = make_float4(v[i], v[i + 1], v[i + 2], v[i + 3]);
    } else {
#pragma unroll
      for (int i = 0; i < V; ++i) p[i] = from_float<T>(v[i]);
    }
  } else if constexpr (V == 1) {
    p[0] = from_float<T>(v[0]);
  } else {
    unsigned raw[(V + 1) / 2];
#pragma unroll
    for (int i = 0; i < V / 2; ++i) {
      const __nv_bfloat162 h = __floats2bfloat162_rn(v[2 * i], v[2 * i + 1]);
      raw[i] = *reinterpret_cast<const unsigned*>(&h);
    }
    if constexpr (V == 8) *reinterpret_cast<uint4*>(p) = make_uint4(raw[0], raw[1], raw[2], raw[3]);
    else if constexpr (V == 4) *reinterpret_cast<uint2*>(p) = make_uint2(raw[0], raw[1]);
    else *reinterpret_cast<unsigned*>(p) = raw[0];
  }
}

// V neighbouring values as they lie in memory, fetched through the read-only path (nothing writes them while the kernel
// runs): a run of such words can be on its way before the first is used, whatever the kernel stores in between
template <typename T, int V>
struct RawWord {
  static constexpr int REGS = V * (int)sizeof(T) / 4;
  unsigned r[REGS];
  __device__ __forceinline__ void fetch(const T* p) {
    if constexpr (REGS % 4 == 0) {
#pragma unroll
      for (int i = 0; i < REGS; i += 4) {
        const uint4 v = __ldg(reinterpret_cast<const uint4*>(p) + i / 4);
        r[i] = v.x; r[i + 1] = v.y; r[i + 2] = v.z; r[i + 3] = v.w;
      }
    } else if constexpr (REGS == 2) {
      const uint2 v = __ldg(reinterpret_cast<const uint2*>(p));
      r[0] = v.x; r[1] = v.y;
    } else {
      r[0] = __ldg(reinterpret_cast<const unsigned*>(p));
    }
  }
  __device__ __forceinline__ float operator[](int i) const {
    if constexpr (sizeof(T) == 4) return __uint_as_float(r[i]);
    else return __uint_as_float(i & 1 ? r[i >> 1] & 0xffff0000u : r[i >> 1] << 16);  // bfloat16 is float32's upper half
  }
};

// 16-byte asynchronous copy global -> shared (both 16-byte aligned)
__device__ __forceinline__ void cp_async16(void* smem, const void* gmem) {
  unsigned s = (unsigned)__cvta_generic_to_shared(smem);
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"(s), "l"(gmem));
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;\n" ::); }
template <int N>
__device__ __forceinline__ void cp_async_wait() {
  asm volatile("cp.async.wait_group %0;\n" ::"n"(N));
}

// Activations of a gated feed-forward's gate (GATE_ACT_*), exact and as one multiplication and one division:
// silu(z) = z / (1 + e^-z); gelu in its tanh form, 0.5 z (1 + tanh y) with y = sqrt(2 / pi) (z + 0.044715 z^3), is
// z / (1 + e^-2y), since (1 + tanh y) / 2 is the logistic function of 2y.  FAST: hardware exponential and division, for
// results that are rounded to bfloat16.
enum : int { GATE_ACT_SILU = 0, GATE_ACT_GELU_TANH = 1 };

template <bool FAST>
__device__ __forceinline__ float gate_act_mul(int kind, float g, float u) {
  const float y = kind == GATE_ACT_GELU_TANH ? 1.5957691216057308f * fmaf(0.044715f * g * g, g, g) : g;
  return FAST ? __fdividef(g, 1.f + __expf(-y)) * u : g / (1.f + expf(-y)) * u;
}

// Rows whose RMS norm is still to be applied.  The kernel that added to the residual stream wrote, for
// every row m, `partials` sums of squares over column tiles at sumsq[m * stride + p] and the row itself
// multiplied by the norm's weight; a product over such rows multiplies its result by
// 1 / sqrt(sum_p sumsq[m][p] / width + eps), which is what the norm would have put into the row.
struct RowNormIn {
  const float* sumsq;  // null: the rows are taken as they are
  int partials, stride;
  float eps;
};

// That factor for one row, computed by LANES consecutive lanes of a warp (LANES 16 or 32; `sub` is the
// lane's index among them, `mask` names them) in a fixed order; every one of them gets the result.
template <int LANES>
__device__ __forceinline__ float row_norm_factor(const float* row_partials, int partials, int width, float eps,
                                                 int sub, unsigned mask) {
  float s = 0.f;
  for (int p0 = sub; p0 < partials; p0 += 8 * LANES) {
    float v[8];  // eight loads in flight: the sum below must not wait for one load after the other
#pragma unroll
    for (int i = 0; i < 8; ++i) v[i] = p0 + i * LANES < partials ? row_partials[p0 + i * LANES] : 0.f;
#pragma unroll
    for (int i = 0; i < 8; ++i) s += v[i];
  }
#pragma unroll
  for (int o = LANES / 2; o > 0; o >>= 1) s += __shfl_xor_sync(mask, s, o);
  return 1.f / sqrtf(s / (float)width + eps);
}

// The same for two rows at once (the second only if `second`): their loads are in flight together, so that
// a warp with two rows to do pays one memory latency, and each sum is formed as above.
__device__ __forceinline__ void row_norm_factors2(const float* row_a, const float* row_b, bool second, int partials,
                                                  int width, float eps, int lane, float& fa, float& fb) {
  float sa = 0.f, sb = 0.f;
  for (int p0 = lane; p0 < partials; p0 += 8 * 32) {
    float va[8], vb[8];
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      const bool in = p0 + i * 32 < partials;
      va[i] = in ? row_a[p0 + i * 32] : 0.f;
      vb[i] = in && second ? row_b[p0 + i * 32] : 0.f;
    }
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      sa += va[i];
      sb += vb[i];
    }
  }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    sa += __shfl_xor_sync(0xffffffffu, sa, o);
    sb += __shfl_xor_sync(0xffffffffu, sb, o);
  }
  fa = 1.f / sqrtf(sa / (float)width + eps);
  fb = 1.f / sqrtf(sb / (float)width + eps);
}

}  // namespace mll
