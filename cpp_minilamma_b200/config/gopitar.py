"""`GopitarConfig`: the configuration of the Gopitar decoder, typed and checked.

A Gopitar folder's config.json names the design in "architecture" and gives every size and constant:

    vocab, width, norm.eps, embedding.scale, logit_softcap
    layers[i].type     "parallel" | "delta"
    layers[i].mixer    parallel:  left {heads, kv_heads, dim, vdim, conv, scale, mask {size}, rot {base, dims}},
                                  right {heads, dim, vdim, decay [one per head]}, left_scale, right_scale
                       delta:     heads, kv_heads, dim, vdim, conv
    layers[i].mlp      {"kind": "dense", "ff": n}, or null for a layer without a feed-forward
    loop               {"start", "stop", "times"}: layers start .. stop - 1 run `times` times in a row, or null

Nothing here knows tensor names or kernels; `models/gopitar.py` turns the typed configuration into parts.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Dict, List, Optional, Tuple

from .base import ConfigError, ModelConfig, take_float, take_int
from .kupirax import Rotation, _object
from .mefolorn import _window

MIXER_TYPES = ("parallel", "delta")


@dataclass
class WindowSide:
    """The left side of a `parallel` mixer: windowed attention behind a short convolution."""

    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int
    scale: float
    window: int = 0
    rot: Optional[Rotation] = None

    @classmethod
    def from_dict(cls, raw: Any, what: str) -> "WindowSide":
        raw = _object(raw, what)
        heads, dim = take_int(raw, "heads", minimum=1), take_int(raw, "dim", minimum=1)
        side = cls(heads=heads, kv_heads=take_int(raw, "kv_heads", default=heads, minimum=1), dim=dim,
                   vdim=take_int(raw, "vdim", default=dim, minimum=1), conv=take_int(raw, "conv", minimum=1),
                   scale=take_float(raw, "scale"), window=_window(raw, what), rot=Rotation.from_dict(raw.get("rot"), what + ".rot"))
        if side.heads % side.kv_heads:
            raise ConfigError(f"config.json: {what}: {side.heads} heads are not a multiple of {side.kv_heads} kv_heads")
        if side.rot is not None and (side.rot.dims > side.dim or side.rot.scaling):
            raise ConfigError(f"config.json: {what}.rot rotates at most {side.dim} dims and knows no scaling")
        return side

    def to_dict(self) -> Dict[str, Any]:
        return {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "conv": self.conv,
                "scale": self.scale, "mask": {"size": self.window} if self.window else None,
                "rot": self.rot.to_dict() if self.rot is not None else None}


@dataclass
class LightningSide:
    """The right side of a `parallel` mixer: lightning attention, one fixed decay per head."""

    heads: int
    dim: int
    vdim: int
    decay: List[float] = field(default_factory=list)

    @classmethod
    def from_dict(cls, raw: Any, what: str) -> "LightningSide":
        raw = _object(raw, what)
        heads, dim = take_int(raw, "heads", minimum=1), take_int(raw, "dim", minimum=1)
        decay = raw.get("decay")
        if not isinstance(decay, list) or len(decay) != heads or \
                any(isinstance(x, bool) or not isinstance(x, (int, float)) for x in decay):
            raise ConfigError(f"config.json: {what}.decay must list one number per head")
        return cls(heads=heads, dim=dim, vdim=take_int(raw, "vdim", default=dim, minimum=1), decay=[float(x) for x in decay])

    def to_dict(self) -> Dict[str, Any]:
        return {"heads": self.heads, "dim": self.dim, "vdim": self.vdim, "decay": list(self.decay)}


@dataclass
class GopitarLayer:
    type: str
    # delta
    heads: int = 0
    kv_heads: int = 0
    dim: int = 0
    vdim: int = 0
    conv: int = 0
    # parallel
    left: Optional[WindowSide] = None
    right: Optional[LightningSide] = None
    left_scale: float = 1.0
    right_scale: float = 1.0
    ff: int = 0  # 0: no feed-forward

    @classmethod
    def from_dict(cls, raw: Any, index: int) -> "GopitarLayer":
        what = f"layers[{index}]"
        raw = _object(raw, what)
        kind = raw.get("type")
        if kind not in MIXER_TYPES:
            raise ConfigError(f"config.json: {what}.type {kind!r} is not one of {', '.join(MIXER_TYPES)}")
        m = _object(raw.get("mixer"), what + ".mixer")
        layer = cls(type=kind)
        if kind == "delta":
            layer.heads, layer.dim = take_int(m, "heads", minimum=1), take_int(m, "dim", minimum=1)
            layer.kv_heads = take_int(m, "kv_heads", default=layer.heads, minimum=1)
            layer.vdim = take_int(m, "vdim", default=layer.dim, minimum=1)
            layer.conv = take_int(m, "conv", minimum=1)
            if layer.heads % layer.kv_heads:
                raise ConfigError(f"config.json: {what}: {layer.heads} heads are not a multiple of {layer.kv_heads} kv_heads")
        else:
            layer.left = WindowSide.from_dict(m.get("left"), what + ".mixer.left")
            layer.right = LightningSide.from_dict(m.get("right"), what + ".mixer.right")
            layer.left_scale = take_float(m, "left_scale", default=1.0)
            layer.right_scale = take_float(m, "right_scale", default=1.0)
        if raw.get("mlp") is not None:
            mlp = _object(raw["mlp"], what + ".mlp")
            if mlp.get("kind") != "dense":
                raise ConfigError(f"config.json: {what}.mlp.kind {mlp.get('kind')!r} is not supported (known: dense)")
            layer.ff = take_int(mlp, "ff", minimum=1)
        return layer

    def to_dict(self) -> Dict[str, Any]:
        if self.type == "delta":
            mixer: Dict[str, Any] = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim,
                                     "conv": self.conv}
        else:
            mixer = {"left": self.left.to_dict(), "right": self.right.to_dict(), "left_scale": self.left_scale,
                     "right_scale": self.right_scale}
        return {"type": self.type, "mixer": mixer, "mlp": {"kind": "dense", "ff": self.ff} if self.ff else None}


@dataclass
class GopitarConfig(ModelConfig):
    vocab: int = 0
    width: int = 0
    eps: float = 1e-5
    embed_scale: float = 1.0
    logit_softcap: float = 0.0     # 0: the logits are not capped
    layers: List[GopitarLayer] = field(default_factory=list)
    loop_start: int = 0
    loop_stop: int = 0
    loop_times: int = 1
    max_positions: int = 1 << 20   # not part of the design: the most positions a sequence may have
    torch_dtype: str = "bfloat16"  # storage of a folder written from this configuration

    @classmethod
    def from_dict(cls, raw: Dict[str, Any]) -> "GopitarConfig":
        layers = raw.get("layers")
        if not isinstance(layers, list) or not layers:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        config = cls(vocab=take_int(raw, "vocab", minimum=1), width=take_int(raw, "width", minimum=1),
                     eps=take_float(_object(raw.get("norm"), "'norm'"), "eps"),
                     layers=[GopitarLayer.from_dict(l, i) for i, l in enumerate(layers)])
        config.embed_scale = take_float(_object(raw.get("embedding") or {}, "'embedding'"), "scale", default=1.0)
        config.logit_softcap = take_float(raw, "logit_softcap", default=0.0)
        if raw.get("loop") is not None:
            loop = _object(raw["loop"], "'loop'")
            config.loop_start = take_int(loop, "start", minimum=0)
            config.loop_stop = take_int(loop, "stop", minimum=0)
            config.loop_times = take_int(loop, "times", minimum=1)
        config.max_positions = take_int(raw, "max_positions", default=cls.max_positions, minimum=1)
        config.torch_dtype = raw.get("torch_dtype", "bfloat16")
        return config

    def validate(self) -> None:
        if self.eps < 0:
            raise ConfigError("config.json: norm.eps must not be negative")
        if self.logit_softcap < 0:
            raise ConfigError("config.json: logit_softcap must not be negative")
        if not 0 <= self.loop_start <= self.loop_stop <= len(self.layers):
            raise ConfigError(f"config.json: loop [{self.loop_start}, {self.loop_stop}) does not lie inside the "
                              f"{len(self.layers)} layers")

    @property
    def vocab_size(self) -> int:
        return self.vocab

    def schedule(self) -> List[Tuple[int, int]]:
        """(layer, n) in the order they run; n > 0 in front of the first layer of the n-th repeat of the loop, else 0."""
        runs = [(i, 0) for i in range(self.loop_start)]
        for turn in range(self.loop_times):
            runs += [(i, turn if i == self.loop_start else 0) for i in range(self.loop_start, self.loop_stop)]
        return runs + [(i, 0) for i in range(self.loop_stop, len(self.layers))]

    def to_dict(self) -> Dict[str, Any]:
        out: Dict[str, Any] = {"architecture": self.architecture or "Gopitar", "vocab": self.vocab, "width": self.width,
                               "norm": {"eps": self.eps}, "embedding": {"scale": self.embed_scale},
                               "layers": [l.to_dict() for l in self.layers], "max_positions": self.max_positions,
                               "torch_dtype": self.torch_dtype}
        if self.logit_softcap:
            out["logit_softcap"] = self.logit_softcap
        if self.loop_stop > self.loop_start:
            out["loop"] = {"start": self.loop_start, "stop": self.loop_stop, "times": self.loop_times}
        return out
