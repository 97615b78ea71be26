"""The Gopitar decoder as data: `GopitarConfig` -> `ModelSpec`.

A scaled token embedding; pre-norm layers with two kinds of mixer - side by side, attention under a sliding window whose
queries, keys and values pass a short convolution over time, with biases and a gate per head, beside lightning attention (a
matrix state per head with one fixed decay); and the gated delta rule with one decay per token and head - and a dense
feed-forward gated by gelu; a stretch of layers that may run several times over, with the embedding's output added to the
stream in front of every repeat; a final norm and an untied head whose logits are capped smoothly.  This file is the only
one that knows Gopitar's tensor names: `embed`, `l<i>.norm1`, `l<i>.norm2`, `l<i>.mix.*`, `l<i>.mix.{left, right}.*`,
`l<i>.mlp.{gate, up, down}`, `final.norm`, `head`.
"""
from __future__ import annotations

from ..config.base import register_architecture
from ..config.gopitar import GopitarConfig, GopitarLayer
from ..parts.base import LayerSpec, ModelSpec, PartSpec, ScheduleEntry


def _mixer(layer: GopitarLayer, prefix: str, eps: float) -> PartSpec:
    pre = prefix + "mix."
    if layer.type == "delta":
        return PartSpec("delta_rule_head_decay", {
            "n_heads": layer.heads, "n_kv_heads": layer.kv_heads, "head_dim": layer.dim, "v_head_dim": layer.vdim,
            "conv": layer.conv, "eps": eps, "unit_eps": 1e-6,
            "names": {p: pre + p for p in ("q", "k", "v", "b", "a", "dt_bias", "A_log", "g", "norm", "o")}})
    left, right = layer.left, layer.right
    lp, rp = pre + "left.", pre + "right."
    position, rot_dims = None, 0
    if left.rot is not None and left.rot.dims:
        rot_dims = left.rot.dims
        position = PartSpec("rotary", {"head_dim": rot_dims, "theta": left.rot.base, "scaling": None, "interleaved": False})
    attention = PartSpec("chunked_attention", {
        "n_heads": left.heads, "n_kv_heads": left.kv_heads, "head_dim": left.dim, "v_head_dim": left.vdim,
        "scale": left.scale, "chunk": 0, "window": left.window, "position": position, "rotary_dims": rot_dims,
        "qk_norm": None, "gate": "head", "conv": left.conv, "bias": True, "out_name": "o.left",
        "names": {p: lp + p for p in ("q", "k", "v", "g", "o")}})
    lightning = PartSpec("lightning_attention", {
        "n_heads": right.heads, "head_dim": right.dim, "v_head_dim": right.vdim, "decay": list(right.decay), "eps": eps,
        "out_name": "o.right", "names": {p: rp + p for p in ("q", "k", "v", "g", "norm", "o")}})
    return PartSpec("side_by_side", {"left": attention, "right": lightning, "scale_left": layer.left_scale,
                                     "scale_right": layer.right_scale})


def build_gopitar_spec(config: GopitarConfig) -> ModelSpec:
    def norm(name, optional=False):
        return PartSpec("rms_norm", {"width": config.width, "eps": config.eps, "name": name, "optional": optional})

    layers = []
    for i, layer in enumerate(config.layers):
        prefix = f"l{i}."
        feed = PartSpec("none")
        if layer.ff:
            feed = PartSpec("swiglu", {"intermediate": layer.ff, "bare_names": True, "activation": "gelu_tanh",
                                       "names": {p: f"{prefix}mlp.{p}" for p in ("gate", "up", "down")}})
        layers.append(LayerSpec(block=PartSpec("pre_norm"), mixer=_mixer(layer, prefix, config.eps), feed_forward=feed,
                                norms={"input": norm(prefix + "norm1"),
                                       # nothing reads the second norm of a layer without a feed-forward
                                       "post_mixer": norm(prefix + "norm2", optional=not layer.ff)}))
    schedule = [ScheduleEntry(i, enter=(0, turn) if turn else None) for i, turn in config.schedule()]
    again = any(entry.enter is not None for entry in schedule)
    return ModelSpec(
        hidden_size=config.width, vocab_size=config.vocab, max_positions=config.max_positions,
        embedding=PartSpec("token_embedding", {"vocab": config.vocab, "name": "embed", "scale": config.embed_scale}),
        layers=layers, schedule=schedule, final_norm=norm("final.norm"),
        lm_head=PartSpec("linear_head", {"vocab": config.vocab, "name": "head", "tied_to": None,
                                         "softcap": config.logit_softcap}),
        stream_ops=[PartSpec("embedding_again")] if again else [])


register_architecture("Gopitar", GopitarConfig, build_gopitar_spec)
