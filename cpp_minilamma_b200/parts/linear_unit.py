"""A gated linear recurrent unit behind a short convolution: a state of one number per channel.

    y = gelu(W_y h + b_y),  u = conv(W_x h + b_x) + b_c       gelu in its tanh form; a causal convolution per channel over
                                                              the last `conv` tokens, nothing before the first one
    r = sigmoid(A u + a),  i = sigmoid(I u + c)               A, I block-diagonal: `blocks` equal square blocks
    decay = exp(-rate * r * softplus(lam))
    S_t = decay * S_(t-1) + sqrt(1 - decay^2) * i * u         from S = 0
    out = W_o (S * y)

Per sequence the cache keeps S and the last conv - 1 inputs of the convolution (as projected, without b_x).  What
enters the recurrence is float32: u, both gates with their products, decays, the state.
"""
from __future__ import annotations

from typing import List, Optional

import torch

from ..csrc import kernels as K
from .base import BuildContext, CacheNeed, Mixer, StateNeed, WeightSpec, register_part
from .linear import Linear


class LinearRecurrentUnit(Mixer):
    """params: width (channels), blocks (of the gates' matrices), conv (taps), rate (the factor in the decay's exponent),
    out_name (workspace name of the result, default "o"), names: tensor names for "y", "y_bias", "x", "x_bias", "conv",
    "conv_bias", "ra", "ra_bias", "ri", "ri_bias", "lam", "o"."""

    capturable = True
    workspace = "lru"

    def __init__(self, params, ctx: BuildContext):
        super().__init__(params, ctx)
        self.width = int(params["width"])
        self.blocks = int(params["blocks"])
        self.taps = int(params["conv"])
        self.rate = float(params["rate"])
        self.names = dict(params["names"])
        self.out_name = params.get("out_name") or "o"
        if self.blocks < 1 or self.width % self.blocks:
            raise ValueError(f"linear recurrent unit: {self.width} channels in {self.blocks} equal blocks")
        if self.taps < 1:
            raise ValueError("linear recurrent unit: the convolution needs at least one tap")
        self.proj: Optional[Linear] = None
        self.o: Optional[Linear] = None

    def weight_specs(self) -> List[WeightSpec]:
        D, W, n, bs = self.ctx.hidden_size, self.width, self.names, self.width // self.blocks
        vector = lambda name, *shape: WeightSpec(n[name], shape, kind="vector")
        return [WeightSpec(n["y"], (W, D)), vector("y_bias", W), WeightSpec(n["x"], (W, D)), vector("x_bias", W),
                vector("conv", W, self.taps), vector("conv_bias", W),
                WeightSpec(n["ra"], (self.blocks, bs, bs)), vector("ra_bias", self.blocks, bs),
                WeightSpec(n["ri"], (self.blocks, bs, bs)), vector("ri_bias", self.blocks, bs),
                vector("lam", W), WeightSpec(n["o"], (D, W))]

    def bind(self, store) -> None:
        n, W, bs = self.names, self.width, self.width // self.blocks
        mats = [store.take(n["y"]), store.take(n["x"])]
        if len({m.dtype for m in mats}) > 1:
            mats = [m.float() for m in mats]
        fused = torch.cat(mats, dim=0)
        spare = -fused.shape[0] % 8  # rows of zeros up to a multiple of 8: the product's rows stay 16-byte aligned
        if spare:
            fused = torch.cat([fused, torch.zeros((spare, fused.shape[1]), dtype=fused.dtype, device=fused.device)], dim=0)
        self.proj = Linear(fused, n["y"] + "+x")
        del mats, fused
        self.y_bias, self.x_bias, self.conv_b = (store.take(n[p]) for p in ("y_bias", "x_bias", "conv_bias"))
        # the decay's exponent per channel, once: softplus(lam) = max(lam, 0) + log(1 + exp(-|lam|)) in double, then float32
        lam = store.take(n["lam"]).double()
        self.rates = (self.rate * (lam.clamp_min(0) + torch.log1p(torch.exp(-lam.abs())))).float().contiguous()
        self.conv_w = store.take(n["conv"]).contiguous()
        self.gate_b = torch.stack([store.take(n["ra_bias"]).reshape(W), store.take(n["ri_bias"]).reshape(W)]).contiguous()
        ra, ri = store.take(n["ra"]), store.take(n["ri"])
        if (ra.dtype == ri.dtype == torch.bfloat16 and self.ctx.device.type == "cuda"
                and K.lru_mma_supported(self.ctx.act_dtype, bs)):
            self.gate_w = torch.stack([ra, ri], dim=1).contiguous()  # [blocks, 2, out, in]
        else:
            self.gate_w = torch.cat([ra.float(), ri.float()], dim=1).transpose(1, 2).contiguous()  # [blocks, in, 2 out]
        self.o = Linear(store.take(n["o"]), n["o"])

    def parameter_bytes(self) -> int:
        return self.proj.parameter_bytes() + self.o.parameter_bytes() + self.gate_w.numel() * self.gate_w.element_size()

    def cache_need(self) -> CacheNeed:
        return CacheNeed(state=StateNeed((("S", (self.width,)), ("conv", (self.taps - 1, self.width)))))

    def forward(self, step, h, cache):
        T, W, ws = h.shape[0], self.width, step.ws
        proj = self.proj.forward(step, h, "lru.proj")
        out = ws.buffer("lru.out", (T, W), self.ctx.act_dtype)
        gates = (proj, W, 0, self.x_bias, self.y_bias, self.conv_w, self.conv_b, cache.state["conv"], self.gate_w,
                 self.gate_b, self.rates, cache.state["S"], step.tok_pos, step.tok_seq, step.seq_slot, step.seq_qstart,
                 self.blocks)
        if step.all_decode:
            K.lru_gates(*gates, out=out)  # one token each: the state advances in the same kernel
        else:
            decay = ws.buffer("lru.decay", (T, W), torch.float32)
            write = ws.buffer("lru.write", (T, W), torch.float32)
            K.lru_gates(*gates, decay=decay, write=write)
        if self.taps > 1:
            K.conv_state_update(proj, cache.state["conv"], step.seq_slot, step.seq_qstart, step.seq_qlen, step.n_seqs, W,
                                self.taps, first_column=W)
        if not step.all_decode:
            K.lru_scan(decay, write, proj, 0, self.y_bias, cache.state["S"], out, step.seq_slot, step.seq_qstart,
                       step.seq_qlen, step.n_seqs, max(step.shape.lens))
        return self.o.forward(step, out, self.out_name)


register_part("mixer", "linear_recurrent_unit", LinearRecurrentUnit)
