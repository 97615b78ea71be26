"""Small Gopitar configurations and weights for the tests, made here from NumPy random numbers and written with this
file's own safetensors writer (bfloat16 storage), so that nothing of the product takes part in what the oracle reads.
Sizes are unlike each other on purpose: head counts and groups of 1, 2, 3, 5 and all, key and value sizes that differ
both ways, rotated parts that are a whole head, a part of it or nothing, windows of one token, shorter and longer than a
page and none at all, convolutions of one to five taps, decays from quick forgetting to almost none, layers without a
feed-forward, loops over the first, the middle or all layers (and none), mixer weights of 0 on one side (so that the other
side stands alone) or 1, an embedding scale of 1, caps that bend the logits strongly or hardly at all."""
import json
import struct

import numpy as np


def left(heads=4, kv_heads=2, dim=16, vdim=24, conv=3, scale=0.3, size=40, rot=8, base=100.0):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv, "scale": scale}
    if size:
        m["mask"] = {"size": size}
    if rot is not None:
        m["rot"] = {"base": base, "dims": rot}
    return m


def right(heads=2, dim=12, vdim=20, decay=(0.7, 0.995)):
    return {"heads": heads, "dim": dim, "vdim": vdim, "decay": list(decay)}


def pair(l, r, scales=(0.9, 1.3)):
    return "parallel", {"left": l, "right": r, "left_scale": scales[0], "right_scale": scales[1]}


def delta(heads=4, kv_heads=2, dim=12, vdim=20, conv=4):
    return "delta", {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}


def layer(mixer, ff=0):
    return {"type": mixer[0], "mixer": mixer[1], "mlp": {"kind": "dense", "ff": ff} if ff else None}


def config(layers, width=48, vocab=97, eps=1e-5, embed_scale=3.0, cap=20.0, loop=None):
    out = {"architecture": "Gopitar", "vocab": vocab, "width": width, "norm": {"eps": eps},
           "embedding": {"scale": embed_scale}, "logit_softcap": cap, "layers": layers}
    if loop:
        out["loop"] = dict(zip(("start", "stop", "times"), loop))
    return out


CONFIGS = {
    # each mixer alone, without a feed-forward
    "span": lambda: config([layer(pair(left(heads=6, kv_heads=2), right(), (1.3, 0.0)))], width=40),
    "glow": lambda: config([layer(pair(left(heads=1, kv_heads=1), right(3, 16, 8, (0.3, 0.9, 0.999)), (0.0, 1.2)))], width=40),
    "delta": lambda: config([layer(delta(heads=6, kv_heads=3))], width=40),
    # everything, every layer with sizes of its own, a loop over the middle
    "mixed": lambda: config([
        layer(pair(left(heads=6, kv_heads=3, dim=8, vdim=12, conv=4, scale=0.5, size=33, rot=4, base=50.0),
                   right(3, 20, 12, (0.2, 0.97, 0.9995)), (1.4, 0.6)), 40),
        layer(delta(heads=2, kv_heads=1, dim=24, vdim=8, conv=2), 24),
        layer(pair(left(heads=5, kv_heads=1, dim=12, vdim=4, conv=5, scale=0.4, size=130, rot=12, base=1000.0),
                   right(1, 8, 32, (0.99,)), (0.7, 1.2))),
        layer(delta(heads=5, kv_heads=5, dim=8, vdim=28, conv=5)),
        layer(pair(left(heads=3, kv_heads=3, dim=10, vdim=10, conv=2, scale=0.3, size=64, rot=None), right(), (0.5, 0.5)), 36)],
        width=56, vocab=131, eps=1e-6, embed_scale=7.0, cap=9.0, loop=(1, 4, 3)),
    # sizes of one: one head, one dimension, a window of one token, one tap, every factor 1; no window; a loop of one pass
    "ones": lambda: config([
        layer(pair(left(heads=1, kv_heads=1, dim=2, vdim=1, conv=1, scale=1.0, size=1, rot=2, base=3.0), right(1, 1, 1, (1.0,)), (1.0, 1.0)), 1),
        layer(delta(heads=1, kv_heads=1, dim=1, vdim=1, conv=1), 8),
        layer(pair(left(heads=2, kv_heads=1, dim=8, vdim=8, conv=1, size=0, rot=0), right(2, 4, 4, (0.5, 0.0)), (1.0, 1.0)), 16)],
        width=36, vocab=61, embed_scale=1.0, cap=50.0, loop=(0, 3, 1)),
    # a loop over all layers whose last has no feed-forward: two pending outputs and the embedding meet in one norm
    "loop": lambda: config([layer(delta(heads=2, kv_heads=2), 32), layer(pair(left(), right()))], width=44, loop=(0, 2, 4)),
    # windows just shorter than, as long as and just longer than a page, and of several pages
    "windows": lambda: config([
        layer(pair(left(heads=2, kv_heads=1, dim=8, vdim=8, size=63, rot=8), right(1, 8, 8, (0.95,)))),
        layer(pair(left(heads=2, kv_heads=1, dim=8, vdim=16, size=64, rot=8), right(1, 8, 8, (0.95,)))),
        layer(pair(left(heads=2, kv_heads=2, dim=16, vdim=8, size=65, rot=4), right(1, 8, 8, (0.95,))), 12),
        layer(pair(left(heads=3, kv_heads=3, dim=8, vdim=8, size=128), right(1, 8, 8, (0.95,))))], width=32, vocab=50),
    # sizes at which the bfloat16 run takes its tensor-core kernels, values wider and narrower than keys
    "tensor": lambda: config([
        layer(pair(left(heads=8, kv_heads=2, dim=64, vdim=128, conv=3, scale=0.12, size=90, rot=32, base=10000.0),
                   right(2, 64, 64, (0.7, 0.998))), 128),
        layer(delta(heads=4, kv_heads=2, dim=64, vdim=64, conv=4), 96),
        layer(pair(left(heads=4, kv_heads=4, dim=128, vdim=64, conv=4, scale=0.1, size=70, rot=128, base=100.0),
                   right(3, 32, 128, (0.9, 0.98, 0.9999))), 64),
        layer(pair(left(heads=6, kv_heads=2, dim=64, vdim=64, conv=2, scale=0.12, size=150, rot=64, base=100.0),
                   right(2, 128, 32, (0.8, 0.99))), 64),
        layer(delta(heads=3, kv_heads=1, dim=128, vdim=128, conv=3), 72)],
        width=128, vocab=89, embed_scale=5.0, loop=(1, 3, 2)),
    # nothing divisible by four: a width of 50, heads of 6 and 10, the kernels' scalar paths
    "odd": lambda: config([
        layer(pair(left(heads=3, kv_heads=1, dim=6, vdim=10, conv=3, size=13, rot=2, base=7.0), right(3, 5, 7, (0.4, 0.8, 0.99)), (1.2, 0.9)), 14),
        layer(delta(heads=3, kv_heads=3, dim=7, vdim=9, conv=3), 30)],
        width=50, vocab=53, cap=4.0),
}


def tensor_shapes(cfg):
    D = cfg["width"]
    shapes = {"embed": (cfg["vocab"], D), "final.norm": (D,), "head": (cfg["vocab"], D)}
    for i, lay in enumerate(cfg["layers"]):
        p, m = f"l{i}.", lay["mixer"]
        shapes[p + "norm1"] = (D,)
        if lay["type"] == "delta":
            H, G, d, dv, taps = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"]
            q = p + "mix."
            for name, rows in (("q", G * d), ("k", G * d), ("v", H * dv)):
                shapes.update({q + name: (rows, D), q + name + ".conv": (rows, taps)})
            shapes.update({q + "b": (H, D), q + "a": (H, D), q + "A_log": (H,), q + "dt_bias": (H,), q + "norm": (dv,),
                           q + "g": (H * dv, D), q + "o": (D, H * dv)})
        else:
            l, r = m["left"], m["right"]
            H, G, d, dv, taps = l["heads"], l["kv_heads"], l["dim"], l["vdim"], l["conv"]
            q = p + "mix.left."
            for name, rows in (("q", H * d), ("k", G * d), ("v", G * dv)):
                shapes.update({q + name: (rows, D), q + name + ".b": (rows,), q + name + ".conv": (rows, taps)})
            shapes.update({q + "g": (H, D), q + "o": (D, H * dv), q + "o.b": (D,)})
            H, d, dv = r["heads"], r["dim"], r["vdim"]
            q = p + "mix.right."
            shapes.update({q + "q": (H * d, D), q + "k": (H * d, D), q + "v": (H * dv, D), q + "g": (H * dv, D),
                           q + "norm": (H * dv,), q + "o": (D, H * dv)})
        if lay["mlp"]:
            ff = lay["mlp"]["ff"]
            shapes.update({p + "norm2": (D,), p + "mlp.gate": (ff, D), p + "mlp.up": (ff, D), p + "mlp.down": (D, ff)})
    return shapes


def to_bf16_bits(a):
    bits = np.ascontiguousarray(a, dtype=np.float32).view(np.uint32).astype(np.uint64)
    return (((bits + 0x7FFF + ((bits >> 16) & 1)) >> 16) & 0xFFFF).astype(np.uint16)


def make_weights(cfg, seed):
    """name -> float32 array holding bfloat16 values.  Scales are chosen so that every mechanism matters: scores large
    enough that single keys win, biases and every tap of a convolution as large as what they join, decays between quick
    forgetting and hardly any, betas and gates neither open nor shut, outputs as large as the stream they join."""
    rng = np.random.RandomState(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        leaf = name.split(".", 1)[-1]
        fan_in = shape[-1]
        if leaf in ("norm1", "norm2") or leaf.endswith("norm"):
            a = 1.0 + 0.3 * rng.randn(*shape)
        elif leaf.endswith("A_log"):
            a = np.log(0.05 + 1.5 * rng.rand(*shape))
        elif leaf.endswith("dt_bias"):
            a = -2.0 + rng.randn(*shape)
        elif leaf.endswith(".conv"):
            a = 0.8 * rng.randn(*shape)
        elif leaf.endswith(".b") and len(shape) == 1:
            a = 0.5 * rng.randn(*shape)
        elif name == "embed":
            a = rng.randn(*shape) / cfg["embedding"]["scale"] ** 0.5
        elif name == "head":
            a = 3.0 * rng.randn(*shape) / np.sqrt(fan_in)
        elif leaf.endswith("left.q"):
            a = 2.5 * rng.randn(*shape) / np.sqrt(fan_in)
        elif leaf.endswith((".o", ".down")):
            a = 0.7 * rng.randn(*shape) / np.sqrt(fan_in)
        else:
            a = 1.2 * rng.randn(*shape) / np.sqrt(fan_in)
        bits = to_bf16_bits(a)
        out[name] = (bits.astype(np.uint32) << 16).view(np.float32).reshape(shape)
    return out


def write_folder(cfg, weights, folder):
    folder.mkdir(parents=True, exist_ok=True)
    (folder / "config.json").write_text(json.dumps(cfg, indent=1))
    header, blobs, at = {}, [], 0
    for name, a in weights.items():
        raw = to_bf16_bits(a).astype("<u2").tobytes()
        header[name] = {"dtype": "BF16", "shape": list(a.shape), "data_offsets": [at, at + len(raw)]}
        blobs.append(raw)
        at += len(raw)
    text = json.dumps(header).encode()
    text += b" " * (-len(text) % 8)
    with open(folder / "model.safetensors", "wb") as fh:
        fh.write(struct.pack("<Q", len(text)))
        fh.write(text)
        for raw in blobs:
            fh.write(raw)
    return str(folder)


def make_folder(name, folder, seed=0):
    cfg = CONFIGS[name]() if isinstance(name, str) else name
    weights = make_weights(cfg, seed)
    return write_folder(cfg, weights, folder), cfg, {k: v.astype(np.float64) for k, v in weights.items()}


def tokens(cfg, length, seed):
    return [int(t) for t in np.random.RandomState(seed).randint(0, cfg["vocab"], size=length)]


def random_config(seed):
    """A configuration drawn from a fixed seed: two to five layers of either kind in any order, sizes from lists that
    hold tensor-core sizes and others, any loop."""
    import random
    rng = random.Random(seed)
    layers = []
    for _ in range(rng.randint(2, 5)):
        if rng.random() < 0.45:
            G = rng.choice([1, 2, 3, 4])
            mixer = delta(heads=G * rng.choice([1, 1, 2, 3]), kv_heads=G, dim=rng.choice([8, 16, 24, 32, 64, 96, 128]),
                          vdim=rng.choice([8, 16, 40, 64, 128]), conv=rng.choice([1, 2, 3, 4, 6]))
        else:
            G, d, R = rng.choice([1, 2, 3, 4]), rng.choice([8, 16, 32, 48, 64, 64, 128]), rng.choice([1, 2, 3, 4])
            mixer = pair(left(heads=G * rng.choice([1, 2, 3, 4]), kv_heads=G, dim=d, vdim=rng.choice([d, 16, 40, 64, 128]),
                              conv=rng.choice([1, 2, 3, 4, 5]), scale=rng.choice([0.1, 0.15, 0.25]),
                              size=rng.choice([1, 17, 40, 64, 65, 100, 130, 200]), rot=rng.choice([d, d // 2, 8, 4]),
                              base=rng.choice([100.0, 10000.0])),
                         right(R, rng.choice([8, 16, 32, 64, 128]), rng.choice([8, 24, 32, 64, 128]),
                               [rng.choice([0.3, 0.6, 0.95, 0.99, 0.999, 1.0]) for _ in range(R)]),
                         (rng.choice([0.4, 0.8]), rng.choice([0.5, 1.0, 1.6])))
        layers.append(layer(mixer, rng.choice([0, 64, 96, 200])))
    start = rng.randint(0, len(layers) - 1)
    loop = rng.choice([None, (start, rng.randint(start, len(layers)), rng.choice([1, 2, 3]))])
    return config(layers, width=rng.choice([64, 72, 96, 128, 192, 256]), vocab=rng.choice([211, 384, 1000]),
                  eps=rng.choice([1e-5, 1e-6]), embed_scale=rng.choice([1.0, 3.0, 8.0]), cap=rng.choice([10.0, 30.0]), loop=loop)
