"""`MefolornConfig`: the configuration of the Mefolorn decoder, typed and checked.

A Mefolorn folder's config.json names the design in "architecture" and gives every size and constant:

    vocab, width, norm.eps, embedding.scale
    layers[i].type     "latent_attention" | "parallel"
    layers[i].mixer    latent_attention:  heads, dim, vdim, q_rank, kv_rank, scale, mask {size}
                       parallel:          left {heads, kv_heads, dim, vdim, scale, mask {size}, rot {base, dims}},
                                          right {width, blocks, conv}, left_scale, right_scale
    layers[i].mlp      {"kind": "dense", "ff": n}, or null for a layer without a feed-forward

Nothing here knows tensor names or kernels; `models/mefolorn.py` turns the typed configuration into parts.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Dict, List, Optional

from .base import ConfigError, ModelConfig, take_float, take_int
from .kupirax import _object

MIXER_TYPES = ("latent_attention", "parallel")


def _window(raw: Dict[str, Any], what: str) -> int:
    """mask.size; 0 without a mask (every earlier key is seen)."""
    if raw.get("mask") is None:
        return 0
    return take_int(_object(raw["mask"], what + ".mask"), "size", minimum=1)


@dataclass
class MixedHeadsSide:
    """The left side of a `parallel` mixer: attention with mixed scores and sigmoid weights."""

    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: int = 0
    rot_base: float = 10000.0
    rot_dims: int = 0

    @classmethod
    def from_dict(cls, raw: Any, what: str) -> "MixedHeadsSide":
        raw = _object(raw, what)
        heads = take_int(raw, "heads", minimum=1)
        side = cls(heads=heads, kv_heads=take_int(raw, "kv_heads", default=heads, minimum=1),
                   dim=take_int(raw, "dim", minimum=1), vdim=take_int(raw, "vdim", minimum=1),
                   scale=take_float(raw, "scale"), window=_window(raw, what))
        if raw.get("rot") is not None:
            rot = _object(raw["rot"], what + ".rot")
            side.rot_dims = take_int(rot, "dims", minimum=0)
            if side.rot_dims:
                side.rot_base = take_float(rot, "base")
        if side.heads % side.kv_heads:
            raise ConfigError(f"config.json: {what}: {side.heads} heads are not a multiple of {side.kv_heads} kv_heads")
        if side.rot_dims % 2 or side.rot_dims > side.dim or side.rot_base <= 0:
            raise ConfigError(f"config.json: {what}: rot needs a positive base and an even number of at most {side.dim} dims")
        return side

    def to_dict(self) -> Dict[str, Any]:
        return {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "scale": self.scale,
                "mask": {"size": self.window} if self.window else None,
                "rot": {"base": self.rot_base, "dims": self.rot_dims} if self.rot_dims else None}


@dataclass
class LinearUnitSide:
    """The right side of a `parallel` mixer: a gated linear recurrent unit behind a short convolution."""

    width: int
    blocks: int
    conv: int

    @classmethod
    def from_dict(cls, raw: Any, what: str) -> "LinearUnitSide":
        raw = _object(raw, what)
        side = cls(width=take_int(raw, "width", minimum=1), blocks=take_int(raw, "blocks", minimum=1),
                   conv=take_int(raw, "conv", minimum=1))
        if side.width % side.blocks:
            raise ConfigError(f"config.json: {what}: {side.width} columns in {side.blocks} equal blocks")
        return side

    def to_dict(self) -> Dict[str, Any]:
        return {"width": self.width, "blocks": self.blocks, "conv": self.conv}


@dataclass
class MefolornLayer:
    type: str
    # latent_attention
    heads: int = 0
    dim: int = 0
    vdim: int = 0
    q_rank: int = 0
    kv_rank: int = 0
    scale: float = 0.0
    window: int = 0
    # parallel
    left: Optional[MixedHeadsSide] = None
    right: Optional[LinearUnitSide] = None
    left_scale: float = 1.0
    right_scale: float = 1.0
    ff: int = 0  # 0: no feed-forward

    @classmethod
    def from_dict(cls, raw: Any, index: int) -> "MefolornLayer":
        what = f"layers[{index}]"
        raw = _object(raw, what)
        kind = raw.get("type")
        if kind not in MIXER_TYPES:
            raise ConfigError(f"config.json: {what}.type {kind!r} is not one of {', '.join(MIXER_TYPES)}")
        m = _object(raw.get("mixer"), what + ".mixer")
        layer = cls(type=kind)
        if kind == "latent_attention":
            for key in ("heads", "dim", "vdim", "q_rank", "kv_rank"):
                setattr(layer, key, take_int(m, key, minimum=1))
            layer.scale = take_float(m, "scale")
            layer.window = _window(m, what + ".mixer")
        else:
            layer.left = MixedHeadsSide.from_dict(m.get("left"), what + ".mixer.left")
            layer.right = LinearUnitSide.from_dict(m.get("right"), what + ".mixer.right")
            layer.left_scale = take_float(m, "left_scale", default=1.0)
            layer.right_scale = take_float(m, "right_scale", default=1.0)
        if raw.get("mlp") is not None:
            mlp = _object(raw["mlp"], what + ".mlp")
            if mlp.get("kind") != "dense":
                raise ConfigError(f"config.json: {what}.mlp.kind {mlp.get('kind')!r} is not supported (known: dense)")
            layer.ff = take_int(mlp, "ff", minimum=1)
        return layer

    def to_dict(self) -> Dict[str, Any]:
        if self.type == "latent_attention":
            mixer: Dict[str, Any] = {"heads": self.heads, "dim": self.dim, "vdim": self.vdim, "q_rank": self.q_rank,
                                     "kv_rank": self.kv_rank, "scale": self.scale,
                                     "mask": {"size": self.window} if self.window else None}
        else:
            mixer = {"left": self.left.to_dict(), "right": self.right.to_dict(), "left_scale": self.left_scale,
                     "right_scale": self.right_scale}
        return {"type": self.type, "mixer": mixer, "mlp": {"kind": "dense", "ff": self.ff} if self.ff else None}


@dataclass
class MefolornConfig(ModelConfig):
    vocab: int = 0
    width: int = 0
    eps: float = 1e-5
    embed_scale: float = 1.0
    layers: List[MefolornLayer] = field(default_factory=list)
    max_positions: int = 1 << 20   # not part of the design: the most positions a sequence may have
    torch_dtype: str = "bfloat16"  # storage of a folder written from this configuration

    @classmethod
    def from_dict(cls, raw: Dict[str, Any]) -> "MefolornConfig":
        layers = raw.get("layers")
        if not isinstance(layers, list) or not layers:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        config = cls(vocab=take_int(raw, "vocab", minimum=1), width=take_int(raw, "width", minimum=1),
                     eps=take_float(_object(raw.get("norm"), "'norm'"), "eps"),
                     layers=[MefolornLayer.from_dict(l, i) for i, l in enumerate(layers)])
        config.embed_scale = take_float(_object(raw.get("embedding") or {}, "'embedding'"), "scale", default=1.0)
        config.max_positions = take_int(raw, "max_positions", default=cls.max_positions, minimum=1)
        config.torch_dtype = raw.get("torch_dtype", "bfloat16")
        return config

    def validate(self) -> None:
        if self.eps < 0:
            raise ConfigError("config.json: norm.eps must not be negative")

    @property
    def vocab_size(self) -> int:
        return self.vocab

    def to_dict(self) -> Dict[str, Any]:
        return {"architecture": self.architecture or "Mefolorn", "vocab": self.vocab, "width": self.width,
                "norm": {"eps": self.eps}, "embedding": {"scale": self.embed_scale},
                "layers": [l.to_dict() for l in self.layers],
                "max_positions": self.max_positions, "torch_dtype": self.torch_dtype}
