"""The Mefolorn decoder as data: `MefolornConfig` -> `ModelSpec`.

A scaled token embedding; layers whose mixer and feed-forward read two norms of the same stream, norms that squash every
column through a tanh instead of computing a mean or a variance; two kinds of mixer - attention over a shared low-rank
latent without positions, with queries from a latent of their own, a sliding window, a learned sink per head and a gate
per head; and, side by side, windowed attention whose heads' scores are mixed and weighted by a sigmoid, beside a gated
linear recurrent unit - and a dense gated feed-forward; a final norm and a head that is the embedding table.  This file
is the only one that knows Mefolorn's tensor names: `embed`, `l<i>.norm1`, `l<i>.norm2` (with `.alpha`, `.b`),
`l<i>.mix.*`, `l<i>.mix.{left, right}.*`, `l<i>.mlp.{gate, up, down}`, `final.norm`.
"""
from __future__ import annotations

from ..config.base import register_architecture
from ..config.mefolorn import MefolornConfig, MefolornLayer
from ..parts.base import LayerSpec, ModelSpec, PartSpec, ScheduleEntry


def _mixer(layer: MefolornLayer, prefix: str, eps: float) -> PartSpec:
    pre = prefix + "mix."
    if layer.type == "latent_attention":
        names = {p: pre + p for p in ("uq", "dkv", "uk", "uv", "g", "o")}
        names.update(dq=pre + "dq", dq_norm=pre + "dq.norm", dkv_norm=pre + "dkv.norm")
        return PartSpec("latent_attention", {
            "n_heads": layer.heads, "head_dim": layer.dim, "rot_dim": 0, "v_head_dim": layer.vdim,
            "kv_rank": layer.kv_rank, "q_rank": layer.q_rank, "scale": layer.scale, "position": None, "eps": eps,
            "gate": "head", "window": layer.window, "sink": pre + "sink", "names": names})
    left, right = layer.left, layer.right
    lp, rp = pre + "left.", pre + "right."
    position = None
    if left.rot_dims:
        position = PartSpec("rotary", {"head_dim": left.rot_dims, "theta": left.rot_base, "scaling": None,
                                       "interleaved": False})
    attention = PartSpec("mixed_heads_attention", {
        "n_heads": left.heads, "n_kv_heads": left.kv_heads, "head_dim": left.dim, "v_head_dim": left.vdim,
        "scale": left.scale, "window": left.window, "position": position, "rotary_dims": left.rot_dims,
        "qk_norm": {"q": lp + "q.norm", "k": lp + "k.norm", "eps": eps}, "out_name": "o.left",
        "names": {**{p: lp + p for p in ("q", "k", "v", "o")}, "mix": lp + "talk", "bias": lp + "pb"}})
    names = {p: rp + p for p in ("y", "x", "conv", "ra", "ri", "lam", "o")}
    names.update({p + "_bias": rp + p + ".b" for p in ("y", "x", "conv", "ra", "ri")})
    unit = PartSpec("linear_recurrent_unit", {
        "width": right.width, "blocks": right.blocks, "conv": right.conv, "rate": 8.0, "out_name": "o.right",
        "names": names})
    return PartSpec("side_by_side", {"left": attention, "right": unit, "scale_left": layer.left_scale,
                                     "scale_right": layer.right_scale})


def build_mefolorn_spec(config: MefolornConfig) -> ModelSpec:
    def norm(name, optional=False):
        return PartSpec("dynamic_tanh", {"width": config.width, "name": name, "alpha": name + ".alpha",
                                         "bias": name + ".b", "optional": optional})

    layers = []
    for i, layer in enumerate(config.layers):
        prefix = f"l{i}."
        feed = PartSpec("none")
        if layer.ff:
            feed = PartSpec("swiglu", {"intermediate": layer.ff, "bare_names": True,
                                       "names": {p: f"{prefix}mlp.{p}" for p in ("gate", "up", "down")}})
        layers.append(LayerSpec(block=PartSpec("parallel_two_norms"), mixer=_mixer(layer, prefix, config.eps),
                                feed_forward=feed,
                                norms={"mixer": norm(prefix + "norm1"),
                                       # nothing reads the second norm of a layer without a feed-forward
                                       "feed_forward": norm(prefix + "norm2", optional=not layer.ff)}))
    return ModelSpec(
        hidden_size=config.width, vocab_size=config.vocab, max_positions=config.max_positions,
        embedding=PartSpec("token_embedding", {"vocab": config.vocab, "name": "embed", "scale": config.embed_scale}),
        layers=layers, schedule=[ScheduleEntry(i) for i in range(len(layers))], final_norm=norm("final.norm"),
        lm_head=PartSpec("linear_head", {"vocab": config.vocab, "name": "head", "tied_to": "embed"}))


register_architecture("Mefolorn", MefolornConfig, build_mefolorn_spec)
