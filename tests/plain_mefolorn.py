"""Plain, slow Mefolorn decoder used as the oracle of the tests.

Whole sequences, NumPy float64, one function per mechanism, dense score matrices, the recurrence walked token by
token.  Nothing here is imported by the product and nothing of the product is imported here.

The design in this file's own notation (D model width, T tokens, p positions from 0):

  x_0       = c_e E[token]
  layer     : x <- x + mixer(squash_1(x)) + ff(squash_2(x))         both read the same x
  squash    = tanh(alpha x) w + b                                   alpha one number per norm, w and b per column
  logits    = E squash_final(x)                                     the embedding table again, without c_e

  latent    q_h = (W_uq rms(W_dq h) w_q)_h, c = rms(W_dkv h) w_c, k_h = W_uk,h c, v_h = W_uv,h c; no positions;
            s = scale q.k over the last `size` tokens; weights exp(s_j) / (exp(sink_h) + sum_j exp(s_j)); head h's
            output times sigmoid(W_g h)_h; W_o
  side by side: c_l mix_l(h) + c_r mix_r(h), the two that follow
  talk      grouped-query heads; q and k divided by the root mean square of their whole projections, times weights,
            then rotated (pairs (i, i + r/2) of the first r dimensions by p base^(-2i/r)); s_g = scale q_g.k;
            s'_h = sum_g M[h, g] s_g; weights sigmoid(s'_h + b_h) over the last `size` tokens, not normalised; W_o
  drift     y = gelu(W_y h + b_y), u = conv(W_x h + b_x) + b_c over the last `taps` tokens; in every one of n equal parts
            r = sigmoid(A u + a), i = sigmoid(I u + c); decay exp(-8 r softplus(lam));
            S_p = decay S_(p-1) + sqrt(1 - decay^2) i u; W_o (S y)
  ff        W_down(silu(W_gate h) W_up h)
"""
from __future__ import annotations

import json
import struct
from pathlib import Path

import numpy as np


# --------------------------------------------------------------------------- #
# model folder                                                                #
# --------------------------------------------------------------------------- #
def read_folder(path):
    """(config dict, {name: float64 array}) of a folder with config.json and model.safetensors."""
    path = Path(path)
    config = json.loads((path / "config.json").read_text())
    blob = (path / "model.safetensors").read_bytes()
    (n,) = struct.unpack("<Q", blob[:8])
    header = json.loads(blob[8:8 + n].decode("utf-8"))
    tensors = {}
    for name, info in header.items():
        if name == "__metadata__":
            continue
        lo, hi = info["data_offsets"]
        raw = blob[8 + n + lo:8 + n + hi]
        if info["dtype"] == "BF16":
            a = (np.frombuffer(raw, dtype="<u2").astype(np.uint32) << 16).view(np.float32)
        elif info["dtype"] == "F32":
            a = np.frombuffer(raw, dtype="<f4")
        elif info["dtype"] == "I32":
            a = np.frombuffer(raw, dtype="<i4")
        else:
            raise ValueError(f"dtype {info['dtype']} of {name}")
        tensors[name] = a.reshape(tuple(info["shape"])).astype(np.float64)
    return config, tensors


# --------------------------------------------------------------------------- #
# small functions                                                             #
# --------------------------------------------------------------------------- #
def rms(x, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def squash(x, W, name):
    return np.tanh(W[name + ".alpha"] * x) * W[name] + W[name + ".b"]


def sigmoid(z):
    return 0.5 * (1.0 + np.tanh(0.5 * z))


def silu(z):
    return z * sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (z + 0.044715 * z ** 3)))


def softplus(z):
    return np.logaddexp(0.0, z)


def visible(T, size):
    """[T, T]: query i sees key j; size 0 means every earlier key."""
    i, j = np.arange(T)[:, None], np.arange(T)[None, :]
    return (j <= i) & ((i - j < size) if size else True)


def mask_size(m):
    return (m.get("mask") or {}).get("size", 0)


# --------------------------------------------------------------------------- #
# rotation                                                                    #
# --------------------------------------------------------------------------- #
def rotate_halves(x, positions, rot):
    """x [T, heads, d]: among the first r dimensions, (i, i + r/2) turn by positions * base^(-2i/r); the rest pass."""
    r = rot["dims"] if rot else 0
    if not r:
        return x
    f = rot["base"] ** (-2.0 * np.arange(r // 2, dtype=np.float64) / r)
    angle = positions[:, None, None] * f
    c, s = np.cos(angle), np.sin(angle)
    u, v = x[..., :r // 2], x[..., r // 2:r]
    out = x.copy()
    out[..., :r // 2] = u * c - v * s
    out[..., r // 2:r] = v * c + u * s
    return out


# --------------------------------------------------------------------------- #
# mixers                                                                      #
# --------------------------------------------------------------------------- #
def latent(h, W, pre, m, eps):
    T = h.shape[0]
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    cq = rms(h @ W[pre + "dq"].T, eps) * W[pre + "dq.norm"]
    q = (cq @ W[pre + "uq"].T).reshape(T, H, d)
    c = rms(h @ W[pre + "dkv"].T, eps) * W[pre + "dkv.norm"]
    k = (c @ W[pre + "uk"].T).reshape(T, H, d)
    v = (c @ W[pre + "uv"].T).reshape(T, H, dv)
    gate = sigmoid(h @ W[pre + "g"].T)
    see = visible(T, mask_size(m))
    out = np.zeros((T, H, dv))
    for head in range(H):
        s = np.where(see, (q[:, head] @ k[:, head].T) * m["scale"], -np.inf)
        sink = W[pre + "sink"][head]
        top = np.maximum(s.max(axis=1, keepdims=True), sink)
        e = np.exp(s - top)
        p = e / (np.exp(sink - top) + e.sum(axis=1, keepdims=True))
        out[:, head] = (p @ v[:, head]) * gate[:, head:head + 1]
    return out.reshape(T, H * dv) @ W[pre + "o"].T


def talk(h, W, pre, m, eps):
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    pos = np.arange(T, dtype=np.float64)
    q = (rms(h @ W[pre + "q"].T, eps) * W[pre + "q.norm"]).reshape(T, H, d)
    k = (rms(h @ W[pre + "k"].T, eps) * W[pre + "k.norm"]).reshape(T, G, d)
    v = (h @ W[pre + "v"].T).reshape(T, G, dv)
    q, k = rotate_halves(q, pos, m.get("rot")), rotate_halves(k, pos, m.get("rot"))
    s = np.stack([q[:, g] @ k[:, g // (H // G)].T * m["scale"] for g in range(H)])  # [H, T, T]
    s = np.einsum("hg,gij->hij", W[pre + "talk"], s)
    p = np.where(visible(T, mask_size(m)), sigmoid(s + W[pre + "pb"][:, None, None]), 0.0)
    out = np.stack([p[g] @ v[:, g // (H // G)] for g in range(H)], axis=1)
    return out.reshape(T, H * dv) @ W[pre + "o"].T


def short_convolution(z, w, b):
    """y[t, c] = b[c] + sum_i w[c, taps - 1 - i] z[t - i, c], nothing before the first token."""
    y = np.broadcast_to(b, z.shape).copy()
    taps = w.shape[1]
    for back in range(min(taps, z.shape[0])):
        y[back:] += w[:, taps - 1 - back] * z[:z.shape[0] - back]
    return y


def block_products(u, A, a):
    """[T, n, k] = A[n] u_n + a[n] for the n equal parts of u's columns."""
    n, k, _ = A.shape
    return np.einsum("noi,tni->tno", A, u.reshape(u.shape[0], n, k)) + a


def drift_inputs(h, W, pre, m):
    """(decay, write, y), each [T, width]."""
    T, width = h.shape[0], m["width"]
    y = gelu_tanh(h @ W[pre + "y"].T + W[pre + "y.b"])
    u = short_convolution(h @ W[pre + "x"].T + W[pre + "x.b"], W[pre + "conv"], W[pre + "conv.b"])
    r = sigmoid(block_products(u, W[pre + "ra"], W[pre + "ra.b"])).reshape(T, width)
    i = sigmoid(block_products(u, W[pre + "ri"], W[pre + "ri.b"])).reshape(T, width)
    decay = np.exp(-8.0 * r * softplus(W[pre + "lam"]))
    return decay, np.sqrt(1.0 - decay * decay) * i * u, y


def drift(h, W, pre, m):
    decay, write, y = drift_inputs(h, W, pre, m)
    S = np.zeros(m["width"])
    out = np.zeros_like(write)
    for t in range(h.shape[0]):
        S = decay[t] * S + write[t]
        out[t] = S * y[t]
    return out @ W[pre + "o"].T


def mixer(h, W, pre, layer, eps):
    m = layer["mixer"]
    if layer["type"] == "latent_attention":
        return latent(h, W, pre, m, eps)
    if layer["type"] != "parallel":
        raise ValueError(f"layer type {layer['type']}")
    return m["left_scale"] * talk(h, W, pre + "left.", m["left"], eps) + \
        m["right_scale"] * drift(h, W, pre + "right.", m["right"])


def feed_forward(h, W, pre):
    return (silu(h @ W[pre + "gate"].T) * (h @ W[pre + "up"].T)) @ W[pre + "down"].T


# --------------------------------------------------------------------------- #
# the model                                                                   #
# --------------------------------------------------------------------------- #
def forward(config, W, tokens, with_layers=False):
    """logits [T, vocab] of a whole sequence; with_layers: also the stream after every layer."""
    eps = config["norm"]["eps"]
    x = W["embed"][np.asarray(tokens)] * config["embedding"]["scale"]
    after = []
    for index, layer in enumerate(config["layers"]):
        pre = f"l{index}."
        add = mixer(squash(x, W, pre + "norm1"), W, pre + "mix.", layer, eps)
        if layer.get("mlp"):
            add = add + feed_forward(squash(x, W, pre + "norm2"), W, pre + "mlp.")
        x = x + add
        after.append(x)
    logits = squash(x, W, "final.norm") @ W["embed"].T
    return (logits, np.stack(after)) if with_layers else logits
