// Arguments shared by the kernels of attention with mixed scores and sigmoid weights (attention_mix.cu: every size and
// dtype; attention_mix_mma.cuh: bfloat16 on tensor cores).
#pragma once

#include "common.cuh"

namespace mll {

struct MixAttnArgs {
  const void* q;           // [T, H * d]
  const void* k_cache;     // [pages, Hk, PAGE, d]
  const void* v_cache;     // [pages, Hk, PAGE, dv]
  const int* tok_pos;
  const int* tok_seq;
  const int* seq_slot;
  const int* block_table;
  const float* mix;        // [H, H] row h: how the heads' scores enter head h; or null
  const float* bias;       // [H] or null
  void* out;               // [T, H * dv]
  int n_tokens, n_heads, n_kv_heads, d, dv, window, max_blocks;
  float scale;
};

}  // namespace mll
