"""Mixers that keep a matrix per sequence and head instead of keys and values.

All run   S_t = diag(g_t) S_(t-1) + k_t u_t^T,   o_t = S_t^T q_t   (S is [d, dv], float32, zero at the start of a
sequence, carried from step to step in the cache's per-slot state), so the read-out sees the current token's
write, and normalise o by its root mean square (per head, or a row at once) before a gate and the output projection.

`retention`          one fixed decay per head, u = v; q and k carry rotary positions, k / sqrt(d);
                     out = W_o (o / rms(o) * silu(W_g h))
`gated_delta_rule`   a decay per head and key channel, g = exp(-exp(A) softplus(W_a2 W_a1 h + b)), and the delta
                     rule u = beta (v - S^T k) with beta = sigmoid(W_b h); q, k, v pass a short causal
                     convolution over time and silu, q and k are scaled to unit length per head, q / sqrt(d);
                     the last taps - 1 convolution inputs of a sequence are state too;
                     out = W_o (o / rms(o) * w * sigmoid(W_g2 W_g1 h))

`delta_rule_head_decay`  the delta rule with one decay per head, g = exp(-exp(A) softplus(W_a h + b)), and an output
                     gate of full rank: out = W_o (o / rms(o) * w * silu(W_g h)); everything else as above

`lightning_attention`  one fixed decay per head, u = v, silu on q, k and v; the row of all heads' o is normalised at once:
                     out = W_o (o / rms(o) * w * sigmoid(W_g h))

`gated_linear_attention`  a decay per head and key channel, g = sigmoid(W_a2 W_a1 h + b)^(1 / tau), u = v, q / sqrt(d);
                     out = W_o (o / rms(o) * w * silu(W_g h))

`state_space`        (the state-space duality form) one projection W_in h = [z | x | B | C | dt]; x, B and C pass a short
                     causal convolution with a bias and silu; dt = softplus(dt + bias) per head; one decay per token
                     and head, g = exp(-exp(A_h) dt); k = B and q = C are shared by the heads of a group, u = dt x;
                     o + D_h x, times silu(z), normalised in a few equal parts of the row, times a weight, then W_o;
                     the last taps - 1 convolution inputs of a sequence are state too

Where the decay is one number per head - fixed or per token - prompts take the recurrence a run of tokens at a time
(`_recur`); decays per key channel and single tokens take it token by token.

What enters the recurrence is float32 (decays, step sizes, gates, unit vectors, the state); the projections are
products in the run's dtype.  Sizes, decays, tap counts and eps are parameters.
"""
from __future__ import annotations

import math
from typing import List, Optional

import torch

from ..csrc import kernels as K
from .base import BuildContext, CacheNeed, Mixer, StateNeed, WeightSpec, register_part, row_count
from .linear import Linear
from .rope import shared_position_encoding


def _pad_rows(matrix: torch.Tensor, multiple: int = 8) -> torch.Tensor:
    """Zero rows up to a multiple of 8: the product's row stride then keeps 16-byte alignment."""
    spare = -matrix.shape[0] % multiple
    if not spare:
        return matrix
    return torch.cat([matrix, torch.zeros((spare, matrix.shape[1]), dtype=matrix.dtype, device=matrix.device)], dim=0)


RUNS = ("state_mixers.runs",)  # key of the step's lists of runs, shared by all layers
CHUNK_FROM = 8                 # tokens a sequence (on average) from which a step takes its recurrences a run at a time


def _run_lists(shape):
    """The index arrays of a prompt step's recurrences taken a run of tokens at a time: (sequence, first row among its new
    tokens) of every run, and every sequence's first run.  Steps of single tokens need no list."""
    if shape.all_decode:
        return {}
    lists = {"run_seq": [], "run_row0": [], "seq_run0": []}
    for i, n in enumerate(shape.lens):
        lists["seq_run0"].append(len(lists["run_seq"]))
        for row0 in range(0, n, K.STATE_RUN):
            lists["run_seq"].append(i)
            lists["run_row0"].append(row0)
    return lists


def _recur(step, q, k, v, state, o, H: int, G: int, d: int, dv: int, head_decay=None, token_decay=None, beta=None,
           runs: bool = True) -> None:
    """The recurrence with one decay per head over the step's tokens: a run of tokens at a time in prompt steps, token by
    token otherwise (and where `runs` is off: a decay outside [0, 1] has no logarithm to work with)."""
    lists = step.meta.get(RUNS) if runs and not step.all_decode else None
    if lists and step.n_tokens >= CHUNK_FROM * step.n_seqs and K.state_chunks_supported(d, dv):
        scratch = step.ws.buffer("state.runs", (K.state_chunks_scratch(lists["run_seq"].shape[0], H, d, dv, beta is not None),),
                                 torch.float32)
        K.state_chunks(q, k, v, state, o, scratch, lists["run_seq"], lists["run_row0"], lists["seq_run0"], step.seq_slot,
                       step.seq_qstart, step.seq_qlen, step.n_seqs, H, G, d, dv, head_decay=head_decay,
                       token_decay=token_decay, beta=beta)
        return
    K.state_scan(q, k, v, None, beta, head_decay, state, o, step.seq_slot, step.seq_qstart, step.seq_qlen, step.n_seqs, H, G,
                 d, dv, token_decay=token_decay)


class _RecursInRuns(Mixer):
    """A state mixer whose prompt steps want the lists of runs."""

    def step_metadata_key(self):
        return RUNS

    def prepare_step(self, shape):
        return _run_lists(shape)


def _same_dtype(mats):
    return [m.float() for m in mats] if len({m.dtype for m in mats}) > 1 else list(mats)


class Retention(_RecursInRuns):
    """params: n_heads, head_dim, v_head_dim, decay (one per head), eps (of the head norm),
    position (PartSpec of a rotary encoding over `rotary_dims` dimensions, or None), rotary_dims,
    names {"q","k","v","g","o"}: tensor names."""

    capturable = True
    workspace = "mix"

    def __init__(self, params, ctx: BuildContext):
        super().__init__(params, ctx)
        self.n_heads = int(params["n_heads"])
        self.d = int(params["head_dim"])
        self.dv = int(params["v_head_dim"])
        self.decay = [float(x) for x in params["decay"]]
        self.eps = float(params["eps"])
        self.names = dict(params["names"])
        self.rot = int(params.get("rotary_dims") or 0) if params.get("position") else 0
        if len(self.decay) != self.n_heads:
            raise ValueError(f"retention: {len(self.decay)} decays for {self.n_heads} heads")
        if self.rot % 2 or self.rot > self.d:
            raise ValueError(f"retention: {self.rot} rotated dimensions of a head of {self.d}")
        self.position = shared_position_encoding(params["position"], ctx) if self.rot else None
        self.decay_t = torch.tensor(self.decay, dtype=torch.float32, device=ctx.device)
        self.in_runs = all(0.0 <= x <= 1.0 for x in self.decay)
        self.proj: Optional[Linear] = None
        self.o: Optional[Linear] = None

    def weight_specs(self) -> List[WeightSpec]:
        D, H = self.ctx.hidden_size, self.n_heads
        return [WeightSpec(self.names["q"], (H * self.d, D)), WeightSpec(self.names["k"], (H * self.d, D)),
                WeightSpec(self.names["v"], (H * self.dv, D)), WeightSpec(self.names["g"], (H * self.dv, D)),
                WeightSpec(self.names["o"], (D, H * self.dv))]

    def bind(self, store) -> None:
        mats = _same_dtype([store.take(self.names[p]) for p in ("q", "k", "v", "g")])
        self.proj = Linear(_pad_rows(torch.cat(mats, dim=0)), self.names["q"] + "+k+v+g")
        del mats
        self.o = Linear(store.take(self.names["o"]), self.names["o"])

    def parameter_bytes(self) -> int:
        return self.proj.parameter_bytes() + self.o.parameter_bytes()

    def cache_need(self) -> CacheNeed:
        return CacheNeed(state=StateNeed((("S", (self.n_heads, self.d, self.dv)),)))

    def forward(self, step, h, cache):
        T, H, d, dv = h.shape[0], self.n_heads, self.d, self.dv
        ws = step.ws
        proj = self.proj.forward(step, h, "mix.proj")
        q = ws.buffer("mix.q", (T, H * d), torch.float32)
        k = ws.buffer("mix.k", (T, H * d), torch.float32)
        v = ws.buffer("mix.v", (T, H * dv), torch.float32)
        cos, sin = self.position.tables() if self.position is not None else (None, None)
        K.retention_prepare(proj, cos, sin, step.tok_pos, q, k, v, H, d, dv, self.rot,
                            bool(self.position.interleaved) if self.position is not None else False,
                            1.0 / math.sqrt(d))
        o = ws.buffer("mix.o", (T, H * dv), torch.float32)
        _recur(step, q, k, v, cache.state["S"], o, H, H, d, dv, head_decay=self.decay_t, runs=self.in_runs)
        gated = ws.buffer("mix.gated", (T, H * dv), self.ctx.act_dtype)
        K.head_norm_gate(o, None, proj, gated, H, dv, self.eps, K.GATE_SILU, gate_col=H * (2 * d + dv))
        return self.o.forward(step, gated, "o")


class GatedDeltaRule(Mixer):
    """params: n_heads, n_kv_heads (q and k heads; value head h reads q/k head h // (n_heads / n_kv_heads)),
    head_dim, v_head_dim, conv (taps), eps (of the head norm), unit_eps (inside the root of the unit length),
    names: tensor names for "q","k","v" (their convolution taps are "<name>.conv"), "b", "a1", "a2", "dt_bias",
    "A_log", "g1", "g2", "norm", "o"; decay_rank, gate_rank: inner sizes of the two low-rank pairs (-1: as stored)."""

    capturable = True
    workspace = "mix"

    def __init__(self, params, ctx: BuildContext):
        super().__init__(params, ctx)
        self.n_heads = int(params["n_heads"])
        self.n_kv_heads = int(params["n_kv_heads"])
        self.d = int(params["head_dim"])
        self.dv = int(params["v_head_dim"])
        self.taps = int(params["conv"])
        self.eps = float(params["eps"])
        self.unit_eps = float(params.get("unit_eps", 1e-6))
        self.decay_rank = int(params.get("decay_rank") or -1)  # -1: whatever the tensors have
        self.gate_rank = int(params.get("gate_rank") or -1)
        self.names = dict(params["names"])
        if self.n_heads % self.n_kv_heads:
            raise ValueError(f"delta rule: {self.n_heads} heads are not a multiple of {self.n_kv_heads} q/k heads")
        if self.taps < 1:
            raise ValueError("delta rule: the convolution needs at least one tap")
        self.channels = 2 * self.n_kv_heads * self.d + self.n_heads * self.dv
        self.proj: Optional[Linear] = None      # q, k, v, b
        self.low: Optional[Linear] = None       # a1, g1
        self.high: Optional[Linear] = None      # a2 and g2 side by side on the low ranks
        self.o: Optional[Linear] = None

    def weight_specs(self) -> List[WeightSpec]:
        D, H, G, d, dv, n = self.ctx.hidden_size, self.n_heads, self.n_kv_heads, self.d, self.dv, self.names
        return [WeightSpec(n["q"], (G * d, D)), WeightSpec(n["q"] + ".conv", (G * d, self.taps), kind="vector"),
                WeightSpec(n["k"], (G * d, D)), WeightSpec(n["k"] + ".conv", (G * d, self.taps), kind="vector"),
                WeightSpec(n["v"], (H * dv, D)), WeightSpec(n["v"] + ".conv", (H * dv, self.taps), kind="vector"),
                WeightSpec(n["b"], (H, D)), WeightSpec(n["A_log"], (H,), kind="vector"),
                WeightSpec(n["norm"], (dv,), kind="vector", init="norm"),
                WeightSpec(n["a1"], (self.decay_rank, D)), WeightSpec(n["a2"], (H * d, self.decay_rank)),
                WeightSpec(n["dt_bias"], (H * d,), kind="vector"),
                WeightSpec(n["g1"], (self.gate_rank, D)), WeightSpec(n["g2"], (H * dv, self.gate_rank)),
                WeightSpec(n["o"], (D, H * dv))]

    def bind(self, store) -> None:
        n = self.names
        mats = _same_dtype([store.take(n[p]) for p in ("q", "k", "v", "b")])
        self.proj = Linear(_pad_rows(torch.cat(mats, dim=0)), n["q"] + "+k+v+b")
        low = _same_dtype([store.take(n["a1"]), store.take(n["g1"])])
        self.low = Linear(_pad_rows(torch.cat(low, dim=0)), n["a1"] + "+g1")
        # the second level of both low-rank pairs as one product: [[a2, 0], [0, g2]] over the columns (a1 | g1 | padding)
        a2, g2 = _same_dtype([store.take(n["a2"]), store.take(n["g2"])])
        ra, rg, width = low[0].shape[0], low[1].shape[0], self.low.out_features
        if a2.shape[1] != ra or g2.shape[1] != rg:
            raise ValueError(f"delta rule: {n['a2']} / {n['g2']} read {a2.shape[1]} / {g2.shape[1]} inputs, "
                             f"{n['a1']} / {n['g1']} give {ra} / {rg}")
        high = torch.zeros((a2.shape[0] + g2.shape[0], width), dtype=a2.dtype, device=a2.device)
        high[:a2.shape[0], :ra] = a2
        high[a2.shape[0]:, ra:ra + rg] = g2
        self.high = Linear(_pad_rows(high), n["a2"] + "+g2")
        del mats, low, a2, g2, high
        self.conv_w = torch.cat([store.take(n[p] + ".conv") for p in ("q", "k", "v")], dim=0).contiguous()
        self.a_log = store.take(n["A_log"])
        self.dt_bias = store.take(n["dt_bias"])
        self.norm_w = store.take(n["norm"])
        self.o = Linear(store.take(n["o"]), n["o"])

    def parameter_bytes(self) -> int:
        return sum(l.parameter_bytes() for l in (self.proj, self.low, self.high, self.o))

    def cache_need(self) -> CacheNeed:
        return CacheNeed(state=StateNeed((("S", (self.n_heads, self.d, self.dv)),
                                          ("conv", (self.taps - 1, self.channels)))))

    def forward(self, step, h, cache):
        T, H, G, d, dv = h.shape[0], self.n_heads, self.n_kv_heads, self.d, self.dv
        ws = step.ws
        proj = self.proj.forward(step, h, "mix.proj")
        low = self.low.forward(step, h, "mix.low")
        high = self.high.forward(step, low, "mix.high", out_dtype=torch.float32)  # [T, H d (decay) + H dv (gate) + padding]
        q = ws.buffer("mix.q", (T, G * d), torch.float32)
        k = ws.buffer("mix.k", (T, G * d), torch.float32)
        v = ws.buffer("mix.v", (T, H * dv), torch.float32)
        g = ws.buffer("mix.g", (T, H * d), torch.float32)
        beta = ws.buffer("mix.beta", (T, H), torch.float32)
        K.delta_prepare(proj, high, self.conv_w, cache.state["conv"], self.a_log, self.dt_bias, step.tok_seq,
                        step.seq_slot, step.seq_qstart, q, k, v, g, beta, H, G, d, dv, self.taps, self.unit_eps)
        K.conv_state_update(proj, cache.state["conv"], step.seq_slot, step.seq_qstart, step.seq_qlen, step.n_seqs,
                            self.channels, self.taps)
        o = ws.buffer("mix.o", (T, H * dv), torch.float32)
        K.state_scan(q, k, v, g, beta, None, cache.state["S"], o, step.seq_slot, step.seq_qstart, step.seq_qlen,
                     step.n_seqs, H, G, d, dv)
        gated = ws.buffer("mix.gated", (T, H * dv), self.ctx.act_dtype)
        K.head_norm_gate(o, self.norm_w, high, gated, H, dv, self.eps, K.GATE_SIGMOID, gate_col=H * d)
        return self.o.forward(step, gated, "o")


class HeadDecayDeltaRule(_RecursInRuns):
    """params: n_heads, n_kv_heads (q and k heads; value head h reads q/k head h // (n_heads / n_kv_heads)), head_dim,
    v_head_dim, conv (taps), eps (of the head norm), unit_eps (inside the root of the unit length), out_name (workspace name
    of the result, default "o"), names: tensor names for "q", "k", "v" (their convolution taps are "<name>.conv"), "b", "a",
    "dt_bias", "A_log", "g", "norm", "o"."""

    capturable = True
    workspace = "mix"
    takes_prenormed = True
    adds_residual = True

    def __init__(self, params, ctx: BuildContext):
        super().__init__(params, ctx)
        self.n_heads = int(params["n_heads"])
        self.n_kv_heads = int(params["n_kv_heads"])
        self.d = int(params["head_dim"])
        self.dv = int(params["v_head_dim"])
        self.taps = int(params["conv"])
        self.eps = float(params["eps"])
        self.unit_eps = float(params.get("unit_eps", 1e-6))
        self.names = dict(params["names"])
        self.out_name = params.get("out_name") or "o"
        if self.n_heads % self.n_kv_heads:
            raise ValueError(f"delta rule: {self.n_heads} heads are not a multiple of {self.n_kv_heads} q/k heads")
        if self.taps < 1:
            raise ValueError("delta rule: the convolution needs at least one tap")
        self.channels = 2 * self.n_kv_heads * self.d + self.n_heads * self.dv
        # a row of the one product: q, k, v | beta, decay | the gate, from a multiple of eight columns on
        self.gate_col = self.channels + 2 * self.n_heads
        self.gate_col += -self.gate_col % 8
        self.proj: Optional[Linear] = None
        self.o: Optional[Linear] = None
        self.advances: Optional[bool] = None  # the preparation kernel moves the convolution's state on itself

    def weight_specs(self) -> List[WeightSpec]:
        D, H, G, d, dv, n = self.ctx.hidden_size, self.n_heads, self.n_kv_heads, self.d, self.dv, self.names
        return [WeightSpec(n["q"], (G * d, D)), WeightSpec(n["q"] + ".conv", (G * d, self.taps), kind="vector"),
                WeightSpec(n["k"], (G * d, D)), WeightSpec(n["k"] + ".conv", (G * d, self.taps), kind="vector"),
                WeightSpec(n["v"], (H * dv, D)), WeightSpec(n["v"] + ".conv", (H * dv, self.taps), kind="vector"),
                WeightSpec(n["b"], (H, D)), WeightSpec(n["A_log"], (H,), kind="vector"),
                WeightSpec(n["norm"], (dv,), kind="vector", init="norm"), WeightSpec(n["a"], (H, D)),
                WeightSpec(n["dt_bias"], (H,), kind="vector"), WeightSpec(n["g"], (H * dv, D)),
                WeightSpec(n["o"], (D, H * dv))]

    def bind(self, store) -> None:
        n = self.names
        mats = _same_dtype([store.take(n[p]) for p in ("q", "k", "v", "b", "a", "g")])
        front = _pad_rows(torch.cat(mats[:5], dim=0))
        self.proj = Linear(_pad_rows(torch.cat([front, mats[5]], dim=0)), n["q"] + "+k+v+b+a+g")
        del mats, front
        self.conv_w = torch.cat([store.take(n[p] + ".conv") for p in ("q", "k", "v")], dim=0).contiguous()
        self.a_log = store.take(n["A_log"])
        self.dt_bias = store.take(n["dt_bias"])
        self.norm_w = store.take(n["norm"])
        self.o = Linear(store.take(n["o"]), n["o"])

    def parameter_bytes(self) -> int:
        return self.proj.parameter_bytes() + self.o.parameter_bytes()

    def cache_need(self) -> CacheNeed:
        return CacheNeed(state=StateNeed((("S", (self.n_heads, self.d, self.dv)),
                                          ("conv", (self.taps - 1, self.channels)))))

    def forward(self, step, h, cache, into=None):
        T, H, G, d, dv = row_count(h), self.n_heads, self.n_kv_heads, self.d, self.dv
        ws = step.ws
        proj = self.proj.forward(step, h, "mix.proj")
        q = ws.buffer("mix.q", (T, G * d), torch.float32)
        k = ws.buffer("mix.k", (T, G * d), torch.float32)
        v = ws.buffer("mix.v", (T, H * dv), torch.float32)
        decay = ws.buffer("mix.decay", (T, H), torch.float32)
        beta = ws.buffer("mix.beta", (T, H), torch.float32)
        if self.advances is None:
            self.advances = K.delta_prepare_advances(H, G, d, dv, self.taps, proj.shape[1])
        advance = self.advances and step.all_decode
        K.delta_prepare(proj, None, self.conv_w, cache.state["conv"], self.a_log, self.dt_bias, step.tok_seq,
                        step.seq_slot, step.seq_qstart, q, k, v, decay, beta, H, G, d, dv, self.taps, self.unit_eps,
                        advance=advance)
        if self.taps > 1 and not advance:
            K.conv_state_update(proj, cache.state["conv"], step.seq_slot, step.seq_qstart, step.seq_qlen, step.n_seqs,
                                self.channels, self.taps)
        o = ws.buffer("mix.o", (T, H * dv), torch.float32)
        _recur(step, q, k, v, cache.state["S"], o, H, G, d, dv, token_decay=decay, beta=beta)
        gated = ws.buffer("mix.gated", (T, H * dv), self.ctx.act_dtype)
        K.head_norm_gate(o, self.norm_w, proj, gated, H, dv, self.eps, K.GATE_SILU, gate_col=self.gate_col)
        return self.o.forward(step, gated, self.out_name, into=into)


class LightningAttention(_RecursInRuns):
    """params: n_heads, head_dim, v_head_dim, decay (one per head), eps (of the norm over the row of all heads), out_name
    (workspace name of the result, default "o"), names: tensor names for "q", "k", "v", "g", "norm", "o"."""

    capturable = True
    workspace = "lightning"
    takes_prenormed = True

    def __init__(self, params, ctx: BuildContext):
        super().__init__(params, ctx)
        self.n_heads = int(params["n_heads"])
        self.d = int(params["head_dim"])
        self.dv = int(params["v_head_dim"])
        self.decay = [float(x) for x in params["decay"]]
        self.eps = float(params["eps"])
        self.names = dict(params["names"])
        self.out_name = params.get("out_name") or "o"
        if len(self.decay) != self.n_heads:
            raise ValueError(f"lightning attention: {len(self.decay)} decays for {self.n_heads} heads")
        self.decay_t = torch.tensor(self.decay, dtype=torch.float32, device=ctx.device)
        self.in_runs = all(0.0 <= x <= 1.0 for x in self.decay)
        self.proj: Optional[Linear] = None
        self.o: Optional[Linear] = None

    def weight_specs(self) -> List[WeightSpec]:
        D, H, d, dv, n = self.ctx.hidden_size, self.n_heads, self.d, self.dv, self.names
        return [WeightSpec(n["q"], (H * d, D)), WeightSpec(n["k"], (H * d, D)), WeightSpec(n["v"], (H * dv, D)),
                WeightSpec(n["g"], (H * dv, D)), WeightSpec(n["norm"], (H * dv,), kind="vector", init="norm"),
                WeightSpec(n["o"], (D, H * dv))]

    def bind(self, store) -> None:
        mats = _same_dtype([store.take(self.names[p]) for p in ("q", "k", "v", "g")])
        self.proj = Linear(_pad_rows(torch.cat(mats, dim=0)), self.names["q"] + "+k+v+g")
        del mats
        self.norm_w = store.take(self.names["norm"])
        self.o = Linear(store.take(self.names["o"]), self.names["o"])

    def parameter_bytes(self) -> int:
        return self.proj.parameter_bytes() + self.o.parameter_bytes()

    def cache_need(self) -> CacheNeed:
        return CacheNeed(state=StateNeed((("S", (self.n_heads, self.d, self.dv)),)))

    def forward(self, step, h, cache):
        T, H, d, dv = row_count(h), self.n_heads, self.d, self.dv
        ws = step.ws
        proj = self.proj.forward(step, h, "lightning.proj")
        q = ws.buffer("lightning.q", (T, H * d), torch.float32)
        k = ws.buffer("lightning.k", (T, H * d), torch.float32)
        v = ws.buffer("lightning.v", (T, H * dv), torch.float32)
        K.retention_prepare(proj, None, None, step.tok_pos, q, k, v, H, d, dv, 0, False, 1.0, silu=True)
        o = ws.buffer("lightning.o", (T, H * dv), torch.float32)
        _recur(step, q, k, v, cache.state["S"], o, H, H, d, dv, head_decay=self.decay_t, runs=self.in_runs)
        gated = ws.buffer("lightning.gated", (T, H * dv), self.ctx.act_dtype)
        K.row_norm_gate(o, self.norm_w, proj, gated, self.eps, K.GATE_SIGMOID, gate_col=H * (2 * d + dv))
        return self.o.forward(step, gated, self.out_name)


class GatedLinearAttention(Mixer):
    """params: n_heads, head_dim, v_head_dim, tau (the decay is sigmoid(z)^(1 / tau)), eps (of the head norm),
    decay_rank (inner size of the low-rank pair, -1: as stored), out_name (workspace name of the result, default "o"),
    names: tensor names for "q", "k", "v", "g", "a1", "a2", "a2_bias", "norm", "o"."""

    capturable = True
    workspace = "gla"

    def __init__(self, params, ctx: BuildContext):
        super().__init__(params, ctx)
        self.n_heads = int(params["n_heads"])
        self.d = int(params["head_dim"])
        self.dv = int(params["v_head_dim"])
        self.tau = float(params["tau"])
        self.eps = float(params["eps"])
        self.decay_rank = int(params.get("decay_rank") or -1)
        self.names = dict(params["names"])
        self.out_name = params.get("out_name") or "o"
        if self.tau <= 0:
            raise ValueError(f"gated linear attention: tau {self.tau} must be positive")
        self.proj: Optional[Linear] = None   # q, k, v, g
        self.low: Optional[Linear] = None    # a1
        self.high: Optional[Linear] = None   # a2 over the columns of a1
        self.o: Optional[Linear] = None

    def weight_specs(self) -> List[WeightSpec]:
        D, H, d, dv, n = self.ctx.hidden_size, self.n_heads, self.d, self.dv, self.names
        return [WeightSpec(n["q"], (H * d, D)), WeightSpec(n["k"], (H * d, D)), WeightSpec(n["v"], (H * dv, D)),
                WeightSpec(n["g"], (H * dv, D)), WeightSpec(n["a1"], (self.decay_rank, D)),
                WeightSpec(n["a2"], (H * d, self.decay_rank)), WeightSpec(n["a2_bias"], (H * d,), kind="vector"),
                WeightSpec(n["norm"], (dv,), kind="vector", init="norm"), WeightSpec(n["o"], (D, H * dv))]

    def bind(self, store) -> None:
        n = self.names
        a1 = store.take(n["a1"])
        a2 = store.take(n["a2"])
        if a2.shape[1] != a1.shape[0]:
            raise ValueError(f"gated linear attention: {n['a2']} reads {a2.shape[1]} inputs, {n['a1']} gives {a1.shape[0]}")
        mats = _same_dtype([store.take(n[p]) for p in ("q", "k", "v", "g")])
        self.proj = Linear(_pad_rows(torch.cat(mats, dim=0)), n["q"] + "+k+v+g")
        a1, a2 = _same_dtype([a1, a2])
        self.low = Linear(_pad_rows(a1), n["a1"])
        # the second level over the first level's columns (and its padding)
        high = torch.zeros((a2.shape[0], self.low.out_features), dtype=a2.dtype, device=a2.device)
        high[:, :a2.shape[1]] = a2
        self.high = Linear(_pad_rows(high), n["a2"])
        del mats, a1, a2, high
        self.bias = store.take(n["a2_bias"])
        self.norm_w = store.take(n["norm"])
        self.o = Linear(store.take(n["o"]), n["o"])

    def parameter_bytes(self) -> int:
        return sum(l.parameter_bytes() for l in (self.proj, self.low, self.high, self.o))

    def cache_need(self) -> CacheNeed:
        return CacheNeed(state=StateNeed((("S", (self.n_heads, self.d, self.dv)),)))

    def forward(self, step, h, cache):
        T, H, d, dv = h.shape[0], self.n_heads, self.d, self.dv
        ws = step.ws
        proj = self.proj.forward(step, h, "gla.proj")
        low = self.low.forward(step, h, "gla.low")
        rate = self.high.forward(step, low, "gla.rate", out_dtype=torch.float32)  # [T, H d (+ padding)]
        q = ws.buffer("gla.q", (T, H * d), torch.float32)
        k = ws.buffer("gla.k", (T, H * d), torch.float32)
        v = ws.buffer("gla.v", (T, H * dv), torch.float32)
        g = ws.buffer("gla.g", (T, H * d), torch.float32)
        K.channel_decay_prepare(proj, rate, self.bias, q, k, v, g, H, d, dv, 1.0 / math.sqrt(d), self.tau)
        o = ws.buffer("gla.o", (T, H * dv), torch.float32)
        K.state_scan(q, k, v, g, None, None, cache.state["S"], o, step.seq_slot, step.seq_qstart, step.seq_qlen,
                     step.n_seqs, H, H, d, dv)
        gated = ws.buffer("gla.gated", (T, H * dv), self.ctx.act_dtype)
        K.head_norm_gate(o, self.norm_w, proj, gated, H, dv, self.eps, K.GATE_SILU, gate_col=H * (2 * d + dv))
        return self.o.forward(step, gated, self.out_name)


class StateSpace(_RecursInRuns):
    """params: n_heads, n_groups (heads of one group share B and C), v_head_dim (columns of x per head), state (rows of
    the state per head: the size of B and C), conv (taps), norm_groups (equal parts of the row that are normalised
    each by itself), eps (of that norm), out_name (workspace name of the result, default "o"),
    names: tensor names for "in", "conv", "conv_bias", "dt_bias", "A_log", "D", "norm", "o"."""

    capturable = True
    workspace = "ssd"

    def __init__(self, params, ctx: BuildContext):
        super().__init__(params, ctx)
        self.n_heads = int(params["n_heads"])
        self.n_groups = int(params["n_groups"])
        self.dv = int(params["v_head_dim"])
        self.d = int(params["state"])
        self.taps = int(params["conv"])
        self.parts = int(params.get("norm_groups") or 1)
        self.eps = float(params["eps"])
        self.names = dict(params["names"])
        self.out_name = params.get("out_name") or "o"
        if self.n_groups < 1 or self.n_heads % self.n_groups:
            raise ValueError(f"state space: {self.n_heads} heads are not a multiple of {self.n_groups} groups")
        if self.taps < 1:
            raise ValueError("state space: the convolution needs at least one tap")
        self.inner = self.n_heads * self.dv
        if self.parts < 1 or self.inner % self.parts:
            raise ValueError(f"state space: {self.inner} columns cannot be normalised in {self.parts} equal parts")
        self.channels = self.inner + 2 * self.n_groups * self.d        # what passes the convolution: x, B, C
        self.rows = 2 * self.inner + 2 * self.n_groups * self.d + self.n_heads
        self.proj: Optional[Linear] = None
        self.o: Optional[Linear] = None

    def weight_specs(self) -> List[WeightSpec]:
        D, H, n = self.ctx.hidden_size, self.n_heads, self.names
        return [WeightSpec(n["in"], (self.rows, D)),
                WeightSpec(n["conv"], (self.channels, self.taps), kind="vector"),
                WeightSpec(n["conv_bias"], (self.channels,), kind="vector"),
                WeightSpec(n["dt_bias"], (H,), kind="vector"), WeightSpec(n["A_log"], (H,), kind="vector"),
                WeightSpec(n["D"], (H,), kind="vector", init="norm"),
                WeightSpec(n["norm"], (self.inner,), kind="vector", init="norm"),
                WeightSpec(n["o"], (D, self.inner))]

    def bind(self, store) -> None:
        n = self.names
        self.proj = Linear(_pad_rows(store.take(n["in"])), n["in"])
        self.conv_w = store.take(n["conv"]).contiguous()
        self.conv_b = store.take(n["conv_bias"])
        self.dt_bias = store.take(n["dt_bias"])
        self.a_log = store.take(n["A_log"])
        self.skip = store.take(n["D"])
        self.norm_w = store.take(n["norm"])
        self.o = Linear(store.take(n["o"]), n["o"])

    def parameter_bytes(self) -> int:
        return self.proj.parameter_bytes() + self.o.parameter_bytes()

    def cache_need(self) -> CacheNeed:
        return CacheNeed(state=StateNeed((("S", (self.n_heads, self.d, self.dv)),
                                          ("conv", (self.taps - 1, self.channels)))))

    def forward(self, step, h, cache):
        T, H, G, d, dv = h.shape[0], self.n_heads, self.n_groups, self.d, self.dv
        ws = step.ws
        proj = self.proj.forward(step, h, "ssd.proj")
        q = ws.buffer("ssd.q", (T, G * d), torch.float32)
        k = ws.buffer("ssd.k", (T, G * d), torch.float32)
        u = ws.buffer("ssd.u", (T, self.inner), torch.float32)
        xs = ws.buffer("ssd.x", (T, self.inner), torch.float32)
        decay = ws.buffer("ssd.decay", (T, H), torch.float32)
        K.ssd_prepare(proj, self.conv_w, self.conv_b, cache.state["conv"], self.a_log, self.dt_bias, step.tok_seq,
                      step.seq_slot, step.seq_qstart, q, k, u, xs, decay, H, G, d, dv, self.taps)
        K.conv_state_update(proj, cache.state["conv"], step.seq_slot, step.seq_qstart, step.seq_qlen, step.n_seqs,
                            self.channels, self.taps, first_column=self.inner)
        o = ws.buffer("ssd.o", (T, self.inner), torch.float32)
        _recur(step, q, k, u, cache.state["S"], o, H, G, d, dv, token_decay=decay)
        gated = ws.buffer("ssd.gated", (T, self.inner), self.ctx.act_dtype)
        K.gated_group_norm(o, xs, self.skip, proj, self.norm_w, gated, dv, self.parts, self.eps)
        return self.o.forward(step, gated, self.out_name)


register_part("mixer", "state_space", StateSpace)
register_part("mixer", "delta_rule_head_decay", HeadDecayDeltaRule)
register_part("mixer", "lightning_attention", LightningAttention)
register_part("mixer", "gated_linear_attention", GatedLinearAttention)
register_part("mixer", "retention", Retention)
register_part("mixer", "gated_delta_rule", GatedDeltaRule)
