"""Small Mefolorn configurations and weights for the tests, made here from NumPy random numbers and written with this
file's own safetensors writer (bfloat16 storage), so that nothing of the product takes part in what the oracle reads.
Sizes are unlike each other on purpose: head counts and groups of 1, 2, 3, 5 and all, key and value sizes that differ,
rotated parts that are a whole head, a part of it or nothing, windows of one token, shorter and longer than a page and
none at all, latent ranks that are no multiples of eight, recurrent widths in one block, several, or a block per channel,
convolutions of one to five taps, layers without a feed-forward, mixer weights of 0 on one side (so that the other side
stands alone) or 1, an embedding scale of 1."""
import json
import struct

import numpy as np


def latent(heads=3, dim=8, vdim=12, q_rank=10, rank=20, scale=0.4, size=40):
    m = {"heads": heads, "dim": dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": rank, "scale": scale}
    if size:
        m["mask"] = {"size": size}
    return "latent_attention", m


def left(heads=4, kv_heads=2, dim=16, vdim=16, scale=0.3, size=40, rot=16, base=100.0):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if size:
        m["mask"] = {"size": size}
    if rot is not None:
        m["rot"] = {"base": base, "dims": rot}
    return m


def right(width=24, blocks=2, conv=4):
    return {"width": width, "blocks": blocks, "conv": conv}


def pair(l, r, scales=(1.0, 1.0)):
    return "parallel", {"left": l, "right": r, "left_scale": scales[0], "right_scale": scales[1]}


def layer(mixer, ff=0):
    return {"type": mixer[0], "mixer": mixer[1], "mlp": {"kind": "dense", "ff": ff} if ff else None}


def config(layers, width=48, vocab=97, eps=1e-5, embed_scale=3.0):
    return {"architecture": "Mefolorn", "vocab": vocab, "width": width, "norm": {"eps": eps},
            "embedding": {"scale": embed_scale}, "layers": layers}


CONFIGS = {
    # each mixer alone, without a feed-forward
    "latent": lambda: config([layer(latent())], width=40),
    "talk": lambda: config([layer(pair(left(heads=6, kv_heads=2, rot=8), right(), (1.3, 0.0)))], width=40),
    "drift": lambda: config([layer(pair(left(heads=1, kv_heads=1), right(width=40, blocks=5), (0.0, 0.8)))], width=40),
    # everything, every layer with sizes of its own
    "mixed": lambda: config([
        layer(pair(left(heads=6, kv_heads=3, dim=8, vdim=12, scale=0.5, size=33, rot=4, base=50.0), right(36, 3, 3), (1.4, 0.6)), 40),
        layer(latent(heads=2, dim=16, vdim=8, q_rank=7, rank=12, scale=0.3, size=70), 24),
        layer(pair(left(heads=5, kv_heads=1, dim=12, vdim=4, scale=0.4, size=130, rot=12, base=1000.0), right(28, 1, 5), (0.7, 1.2))),
        layer(latent(heads=4, dim=4, vdim=20, q_rank=30, rank=9, scale=0.6, size=5)),
        layer(pair(left(heads=3, kv_heads=3, dim=10, vdim=10, scale=0.3, size=64, rot=None), right(20, 4, 2), (0.5, 0.5)), 36)],
        width=56, vocab=131, eps=1e-6, embed_scale=7.0),
    # sizes of one: one head, a rank of one, a window of one token, one tap, a block per channel, every factor 1; no window
    "ones": lambda: config([
        layer(latent(heads=1, dim=1, vdim=1, q_rank=1, rank=1, scale=1.0, size=1), 8),
        layer(pair(left(heads=1, kv_heads=1, dim=2, vdim=1, scale=1.0, size=1, rot=2, base=3.0), right(6, 6, 1)), 1),
        layer(pair(left(heads=2, kv_heads=1, dim=8, vdim=8, size=0, rot=0), right(1, 1, 4)), 16),
        layer(latent(heads=2, dim=8, vdim=8, q_rank=16, rank=24, size=0))],
        width=36, vocab=61, embed_scale=1.0),
    # windows just shorter than, as long as and just longer than a page, and of several pages
    "windows": lambda: config([
        layer(latent(heads=2, dim=8, vdim=8, q_rank=8, rank=16, size=63)),
        layer(pair(left(heads=2, kv_heads=1, dim=8, vdim=8, size=64, rot=8), right(8, 2, 2))),
        layer(pair(left(heads=2, kv_heads=2, dim=8, vdim=8, size=65, rot=4), right(8, 1, 3)), 12),
        layer(latent(heads=3, dim=8, vdim=8, q_rank=8, rank=16, size=128))], width=32, vocab=50),
    # sizes at which the bfloat16 run takes its tensor-core kernels
    "tensor": lambda: config([
        layer(latent(heads=8, dim=32, vdim=32, q_rank=48, rank=64, scale=0.2, size=90), 128),
        layer(pair(left(heads=8, kv_heads=2, dim=64, vdim=64, scale=0.1, size=70, rot=64, base=10000.0), right(96, 3, 4), (0.5, 0.7)), 96),
        layer(pair(left(heads=6, kv_heads=2, dim=32, vdim=128, scale=0.2, size=150, rot=16, base=100.0), right(128, 1, 4), (0.6, 0.4)), 64),
        layer(latent(heads=5, dim=64, vdim=24, q_rank=32, rank=136, scale=0.15, size=33))],
        width=128, vocab=89, embed_scale=5.0),
    # many heads: tiles of eight rows, and more outputs than one block's registers hold
    "heads": lambda: config([
        layer(pair(left(heads=24, kv_heads=3, dim=16, vdim=72, scale=0.3, size=50, rot=16), right(64, 2, 4), (0.3, 1.0)), 64),
        layer(pair(left(heads=40, kv_heads=5, dim=8, vdim=16, scale=0.4, size=30, rot=8), right(32, 4, 3), (0.4, 1.0)))],
        width=96, vocab=71),
    # nothing divisible by four: a width of 50, heads of 6 and 10, the kernels' scalar paths
    "odd": lambda: config([
        layer(pair(left(heads=3, kv_heads=1, dim=6, vdim=10, size=13, rot=2, base=7.0), right(30, 3, 3), (1.2, 0.9)), 14),
        layer(latent(heads=5, dim=6, vdim=10, q_rank=11, rank=7, size=21), 30)],
        width=50, vocab=53),
}


def tensor_shapes(cfg):
    D = cfg["width"]
    shapes = {"embed": (cfg["vocab"], D)}

    def norm(name):
        shapes.update({name: (D,), name + ".b": (D,), name + ".alpha": ()})

    norm("final.norm")
    for i, lay in enumerate(cfg["layers"]):
        p, m = f"l{i}.", lay["mixer"]
        norm(p + "norm1")
        if lay["type"] == "latent_attention":
            H, d, dv, qr, rank = m["heads"], m["dim"], m["vdim"], m["q_rank"], m["kv_rank"]
            shapes.update({p + "mix.dq": (qr, D), p + "mix.dq.norm": (qr,), p + "mix.uq": (H * d, qr),
                           p + "mix.dkv": (rank, D), p + "mix.dkv.norm": (rank,), p + "mix.uk": (H * d, rank),
                           p + "mix.uv": (H * dv, rank), p + "mix.sink": (H,), p + "mix.g": (H, D), p + "mix.o": (D, H * dv)})
        else:
            l, r = m["left"], m["right"]
            H, G, d, dv = l["heads"], l["kv_heads"], l["dim"], l["vdim"]
            q = p + "mix.left."
            shapes.update({q + "q": (H * d, D), q + "k": (G * d, D), q + "v": (G * dv, D), q + "q.norm": (H * d,),
                           q + "k.norm": (G * d,), q + "talk": (H, H), q + "pb": (H,), q + "o": (D, H * dv)})
            w, n = r["width"], r["blocks"]
            q = p + "mix.right."
            shapes.update({q + "y": (w, D), q + "y.b": (w,), q + "x": (w, D), q + "x.b": (w,), q + "conv": (w, r["conv"]),
                           q + "conv.b": (w,), q + "ra": (n, w // n, w // n), q + "ra.b": (n, w // n),
                           q + "ri": (n, w // n, w // n), q + "ri.b": (n, w // n), q + "lam": (w,), q + "o": (D, w)})
        if lay["mlp"]:
            ff = lay["mlp"]["ff"]
            norm(p + "norm2")
            shapes.update({p + "mlp.gate": (ff, D), p + "mlp.up": (ff, D), p + "mlp.down": (D, ff)})
    return shapes


def to_bf16_bits(a):
    bits = np.ascontiguousarray(a, dtype=np.float32).view(np.uint32).astype(np.uint64)
    return (((bits + 0x7FFF + ((bits >> 16) & 1)) >> 16) & 0xFFFF).astype(np.uint16)


def make_weights(cfg, seed):
    """name -> float32 array holding bfloat16 values.  Scales are chosen so that every mechanism matters: alphas that
    neither leave the norms linear nor saturate them, scores large enough that single keys win, sinks from far below to
    above them, mixing matrices whose off-diagonal part is as large as the diagonal, decays between quick forgetting and
    hardly any, gates neither open nor shut, biases that are no rounding noise."""
    rng = np.random.RandomState(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        leaf = name.split(".", 1)[-1]
        fan_in = shape[-1] if shape else 1
        if leaf.endswith("alpha"):
            a = np.asarray(0.3 + 0.5 * rng.rand())
        elif leaf in ("norm1", "norm2", "norm") or leaf.endswith(("dq.norm", "dkv.norm", "q.norm", "k.norm")):
            a = 1.0 + 0.3 * rng.randn(*shape)
        elif leaf.endswith("sink"):
            a = 2.5 * rng.randn(*shape)
        elif leaf.endswith("talk"):
            a = 0.7 * np.eye(shape[0]) + 0.8 * rng.randn(*shape) / np.sqrt(shape[0])
        elif leaf.endswith(".pb"):
            a = -1.5 + rng.randn(*shape)
        elif leaf.endswith(".lam"):
            a = -3.0 + 2.0 * rng.randn(*shape)
        elif leaf.endswith(".conv"):
            a = 0.6 * rng.randn(*shape)
        elif leaf.endswith(".b"):
            a = 0.4 * rng.randn(*shape)
        elif leaf.endswith(".uq"):
            a = 2.5 * rng.randn(*shape) / np.sqrt(fan_in)
        elif name == "embed":
            a = rng.randn(*shape) / cfg["embedding"]["scale"] ** 0.5
        elif leaf.endswith("left.o"):  # the weights of a row add up to as many as there are keys
            window = (cfg["layers"][int(name[1:name.index(".")])]["mixer"]["left"].get("mask") or {}).get("size", 100)
            a = 2.0 * rng.randn(*shape) / np.sqrt(fan_in) / np.sqrt(window)
        elif leaf.endswith((".o", ".down")):
            a = 0.7 * rng.randn(*shape) / np.sqrt(fan_in)
        else:
            a = 1.5 * rng.randn(*shape) / np.sqrt(fan_in)
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
    hold tensor-core sizes and others."""
    import random
    rng = random.Random(seed)
    layers = []
    for _ in range(rng.randint(2, 5)):
        size = rng.choice([1, 17, 40, 64, 65, 100, 130, 200])
        if rng.random() < 0.5:
            mixer = latent(heads=rng.choice([1, 2, 3, 4, 8]), dim=rng.choice([16, 24, 32, 64]), vdim=rng.choice([16, 24, 40, 64]),
                           q_rank=rng.choice([16, 24, 50, 96]), rank=rng.choice([16, 32, 44, 64, 128]),
                           scale=rng.choice([0.1, 0.2, 0.3]), size=size)
        else:
            G, d = rng.choice([1, 2, 3, 4]), rng.choice([8, 16, 24, 32, 48, 64, 96])
            n = rng.choice([1, 2, 4])
            mixer = pair(left(heads=G * rng.choice([1, 2, 3, 4, 8]), kv_heads=G, dim=d, vdim=rng.choice([d, d, 16, 40, 72]),
                              scale=rng.choice([0.1, 0.15, 0.25]), size=size, rot=rng.choice([d, d, d // 2, 0]),
                              base=rng.choice([100.0, 10000.0])),
                         right(width=n * rng.choice([8, 16, 20, 40, 72]), blocks=n, conv=rng.choice([1, 2, 4, 6])),
                         (rng.choice([0.4, 0.7]), rng.choice([0.5, 1.0, 1.6])))
        layers.append(layer(mixer, rng.choice([0, 64, 96, 200])))
    return config(layers, width=rng.choice([64, 72, 96, 128, 192, 256]), vocab=rng.choice([211, 384, 1000]),
                  eps=rng.choice([1e-5, 1e-6]), embed_scale=rng.choice([1.0, 3.0, 8.0]))
