"""Attention whose heads look at each other's scores and whose weights are sigmoids, not a softmax.

    q = W_q h, k = W_k h, v = W_v h                       H heads of d, G heads of d, G heads of dv
    q <- q / rms(q) * w_q,  k <- k / rms(k) * w_k         over the whole projection, all heads at once (optional)
    rotate the first `rotary_dims` dimensions of every q and k head by position * f_i
    s_g(i, j) = scale * q_g(i) . k_(g G / H)(j)           for j <= i, and j > i - window where window > 0
    z_h = sum_g M[h, g] s_g + b_h                         M mixes the heads' scores (optional), b a number per head (optional)
    out = W_o concat_heads(sum_j sigmoid(z_h(i, j)) v(j)) not normalised over the keys

Since nothing is normalised, the sums over any runs of keys simply add up: no maximum is carried along, and a context
can be cut between blocks at will.  Preparation (norm, rotation, cache write) is the chunked attention's; so is the
cache, with a window that hands pages back.
"""
from __future__ import annotations

from typing import List, Optional

import torch

from ..csrc import kernels as K
from .base import BuildContext, CacheNeed, KVNeed, Mixer, WeightSpec, register_part
from .chunked_attention import prompt_tiles
from .linear import Linear
from .rope import shared_position_encoding


class MixedHeadsAttention(Mixer):
    """params:
      n_heads, n_kv_heads, head_dim, v_head_dim     sizes
      scale                                         factor on q . k
      window                                        0 = every earlier key
      position, rotary_dims                         PartSpec of a rotary encoding over `rotary_dims` dimensions, or None
      qk_norm                                       None or {"q": tensor name, "k": tensor name, "eps": float}
      out_name                                      workspace name of the result (default "o")
      names                                         {"q","k","v","o"} and optionally "mix" ([n_heads, n_heads]) and "bias"
                                                    ([n_heads]): tensor names
    """

    capturable = True
    workspace = "attention"

    def __init__(self, params, ctx: BuildContext):
        super().__init__(params, ctx)
        self.n_heads = int(params["n_heads"])
        self.n_kv_heads = int(params["n_kv_heads"])
        self.d = int(params["head_dim"])
        self.dv = int(params.get("v_head_dim") or self.d)
        self.scale = float(params["scale"])
        self.window = int(params.get("window") or 0)
        self.names = dict(params["names"])
        self.qk_norm = dict(params["qk_norm"]) if params.get("qk_norm") else None
        self.out_name = params.get("out_name") or "o"
        self.rot = int(params.get("rotary_dims") or 0) if params.get("position") else 0
        if self.n_heads % self.n_kv_heads:
            raise ValueError(f"mixed attention: {self.n_heads} heads are not a multiple of {self.n_kv_heads} kv heads")
        if self.rot % 2 or self.rot > self.d:
            raise ValueError(f"mixed attention: {self.rot} rotated dimensions of a head of {self.d}")
        self.position = shared_position_encoding(params["position"], ctx) if self.rot else None
        self.qkv: Optional[Linear] = None
        self.o: Optional[Linear] = None
        self.q_weight = self.k_weight = self.mix = self.bias = None
        self.mix_narrow = True  # the mixing matrix holds bfloat16 numbers: fewer products in the prompt kernel

    def weight_specs(self) -> List[WeightSpec]:
        D, H, G = self.ctx.hidden_size, self.n_heads, self.n_kv_heads
        specs = [WeightSpec(self.names["q"], (H * self.d, D)), WeightSpec(self.names["k"], (G * self.d, D)),
                 WeightSpec(self.names["v"], (G * self.dv, D)), WeightSpec(self.names["o"], (D, H * self.dv))]
        if "mix" in self.names:
            specs.append(WeightSpec(self.names["mix"], (H, H)))
        if "bias" in self.names:
            specs.append(WeightSpec(self.names["bias"], (H,), kind="vector"))
        if self.qk_norm:
            specs.append(WeightSpec(self.qk_norm["q"], (H * self.d,), kind="vector", init="norm"))
            specs.append(WeightSpec(self.qk_norm["k"], (G * self.d,), kind="vector", init="norm"))
        return specs

    def bind(self, store) -> None:
        mats = [store.take(self.names[p]) for p in ("q", "k", "v")]
        if len({m.dtype for m in mats}) > 1:
            mats = [m.float() for m in mats]
        fused = torch.cat(mats, dim=0)
        spare = -fused.shape[0] % 8  # rows of zeros up to a multiple of 8: the product's rows stay 16-byte aligned
        if spare:
            fused = torch.cat([fused, torch.zeros((spare, fused.shape[1]), dtype=fused.dtype, device=fused.device)], dim=0)
        self.qkv = Linear(fused, self.names["q"] + "+k+v")
        del mats, fused
        self.o = Linear(store.take(self.names["o"]), self.names["o"])
        if "mix" in self.names:
            self.mix = store.take(self.names["mix"]).float()  # a score is float32: so is what mixes it
            self.mix_narrow = bool((self.mix.to(torch.bfloat16).float() == self.mix).all())
        if "bias" in self.names:
            self.bias = store.take(self.names["bias"])
        if self.qk_norm:
            self.q_weight = store.take(self.qk_norm["q"])
            self.k_weight = store.take(self.qk_norm["k"])

    def parameter_bytes(self) -> int:
        return self.qkv.parameter_bytes() + self.o.parameter_bytes()

    def cache_need(self) -> CacheNeed:
        return CacheNeed(kv=KVNeed(self.n_kv_heads, self.d, self.window, self.dv if self.dv != self.d else 0))

    def forward(self, step, h, cache):
        T = h.shape[0]
        act = self.ctx.act_dtype
        if cache.k is None:
            raise RuntimeError("mixed attention: the cache view has no key/value storage")
        qkv = self.qkv.forward(step, h, "qkv")
        cos, sin = self.position.tables() if self.position is not None else (None, None)
        q = step.ws.buffer("q", (T, self.n_heads * self.d), act)
        K.local_attention_prepare(qkv, self.q_weight, self.k_weight, cos, sin, step.tok_pos, step.tok_seq, step.seq_slot,
                                  cache.block_table, q, cache.k, cache.v, self.n_heads, self.n_kv_heads, self.d, self.dv,
                                  self.rot, bool(self.position.interleaved) if self.position is not None else False,
                                  float(self.qk_norm["eps"]) if self.qk_norm else 0.0)
        out = step.ws.buffer("attn", (T, self.n_heads * self.dv), act)
        self._attend(step, q, cache, out)
        return self.o.forward(step, out, self.out_name)

    def step_metadata_key(self):
        # the tile list of prompt steps on tensor cores, shared with the other attention layers
        return ("chunked_attention.tiles", K.PREFILL_TILE) if self.ctx.act_dtype == torch.bfloat16 else None

    def prepare_step(self, shape):
        return prompt_tiles(shape)

    def _attend(self, step, q, cache, out) -> None:
        sizes = (self.n_heads, self.n_kv_heads, self.d, self.dv)
        tiles = step.meta.get(self.step_metadata_key()) if not step.all_decode else None
        if (step.all_decode or tiles) and K.mixed_attention_mma_supported(self.ctx.act_dtype, step.all_decode, *sizes):
            seqs = (q, cache.k, cache.v, step.seq_slot, step.seq_ctx, step.seq_qstart, step.seq_qlen)
            if tiles:
                splits = K.mixed_attention_tile_splits(tiles["wide_seq"].shape[0], *sizes, self.ctx.multiprocessors)
                K.mixed_attention_tiles(*seqs, tiles["wide_seq"], tiles["wide_row0"], cache.block_table, self.mix, self.bias,
                                        out, *sizes, self.window, self.scale, n_splits=splits, narrow_mix=self.mix_narrow)
                return
            splits = K.mixed_attention_single_splits(step.n_seqs, self.ctx.multiprocessors)
            scratch = step.ws.buffer("attn.parts", (K.mixed_attention_single_scratch(step.n_seqs, self.n_heads, self.dv, splits),),
                                     torch.float32) if splits > 1 else None
            K.mixed_attention_single(*seqs, cache.block_table, self.mix, self.bias, out, step.n_seqs, *sizes, self.window,
                                     self.scale, n_splits=splits, scratch=scratch)
            return
        K.mixed_attention(q, cache.k, cache.v, step.tok_pos, step.tok_seq, step.seq_slot, cache.block_table, self.mix,
                          self.bias, out, self.n_heads, self.n_kv_heads, self.d, self.dv, self.window, self.scale)


register_part("mixer", "mixed_heads_attention", MixedHeadsAttention)
