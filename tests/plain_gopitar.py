"""Plain, slow Gopitar decoder used as the oracle of the tests.

Whole sequences, NumPy float64, one function per mechanism, dense score matrices, recurrences walked token by token.
Nothing here is imported by the product and nothing of the product is imported here.

The design in this file's own notation (D model width, T tokens, p positions from 0, unit(x) = x / sqrt(mean(x^2) + eps)):

  x_0      = c_e E[token]
  layer    : r = x + mixer(w_1 unit(x)),  x' = r + ff(w_2 unit(r))       a layer without a feed-forward ends at r
  order    : layers [a, b) run n times in a row, in front of every run but the first x <- x + x_0
  logits   = c tanh(W_head(w_f unit(x)) / c)

  side by side: c_l span(h) + c_r glow(h), the two that follow
  span     q, k, v = conv(W h + b) each, over the last `taps` tokens (nothing, not even b, before the first);
           q and k rotated (pairs (i, i + r/2) of the first r dimensions by p base^(-2i/r)); softmax(scale q.k) over the
           last `size` tokens; head h's output times sigmoid(W_g h)_h; W_o + b_o
  glow     q, k, v = silu(W h); S_p = a_h S_(p-1) + k v^T from 0; o = S^T q; the row of all heads' o: unit times w, times
           sigmoid(W_g h); W_o
  delta    q, k, v = silu(conv(W h)); q and k to unit length per head, q / sqrt(d); beta = sigmoid(W_b h),
           g = exp(-exp(A) softplus(W_a h + t)); S <- g S; u = beta (v - S^T k); S <- S + k u^T; o = S^T q;
           per head unit(o) times w, times silu(W_g h); W_o
  ff       W_down(gelu(W_gate h) W_up h), gelu in its tanh form
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
def short_convolution(z, w):
    """y[t, c] = sum_i w[c, taps - 1 - i] z[t - i, c], nothing before the first token."""
    y = np.zeros_like(z)
    taps = w.shape[1]
    for back in range(min(taps, z.shape[0])):
        y[back:] += w[:, taps - 1 - back] * z[:z.shape[0] - back]
    return y


def span_inputs(h, W, pre, m):
    """q [T, H, d], k [T, G, d], v [T, G, dv] as the scores and the sums read them."""
    T = h.shape[0]
    pos = np.arange(T, dtype=np.float64)
    q, k, v = (short_convolution(h @ W[pre + p].T + W[pre + p + ".b"], W[pre + p + ".conv"]) for p in "qkv")
    q, k = q.reshape(T, m["heads"], m["dim"]), k.reshape(T, m["kv_heads"], m["dim"])
    return (rotate_halves(q, pos, m.get("rot")), rotate_halves(k, pos, m.get("rot")),
            v.reshape(T, m["kv_heads"], m["vdim"]))


def span(h, W, pre, m):
    T, H, dv = h.shape[0], m["heads"], m["vdim"]
    q, k, v = span_inputs(h, W, pre, m)
    gate = sigmoid(h @ W[pre + "g"].T)
    see = visible(T, mask_size(m))
    out = np.zeros((T, H, dv))
    for head in range(H):
        at = head // (H // m["kv_heads"])
        s = np.where(see, (q[:, head] @ k[:, at].T) * m["scale"], -np.inf)
        e = np.exp(s - s.max(axis=1, keepdims=True))
        out[:, head] = (e @ v[:, at]) / e.sum(axis=1, keepdims=True) * gate[:, head:head + 1]
    return out.reshape(T, H * dv) @ W[pre + "o"].T + W[pre + "o.b"]


def glow(h, W, pre, m, eps):
    T, H, d, dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = silu(h @ W[pre + "q"].T).reshape(T, H, d)
    k = silu(h @ W[pre + "k"].T).reshape(T, H, d)
    v = silu(h @ W[pre + "v"].T).reshape(T, H, dv)
    decay = np.asarray(m["decay"], dtype=np.float64)[:, None, None]
    S = np.zeros((H, d, dv))
    o = np.zeros((T, H, dv))
    for t in range(T):
        S = decay * S + k[t][:, :, None] * v[t][:, None, :]
        o[t] = np.einsum("hkv,hk->hv", S, q[t])
    row = rms(o.reshape(T, H * dv), eps) * W[pre + "norm"]
    return (row * sigmoid(h @ W[pre + "g"].T)) @ W[pre + "o"].T


def delta_inputs(h, W, pre, m):
    """(q, k per value head [T, H, d], v [T, H, dv], g [T, H], beta [T, H])."""
    T, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (silu(short_convolution(h @ W[pre + p].T, W[pre + p + ".conv"])) for p in "qkv")
    q, k = q.reshape(T, G, d), k.reshape(T, G, d)
    length = lambda x: np.sqrt(np.sum(x * x, axis=-1, keepdims=True) + 1e-6)
    q, k = q / length(q) / np.sqrt(d), k / length(k)
    g = np.exp(-np.exp(W[pre + "A_log"]) * softplus(h @ W[pre + "a"].T + W[pre + "dt_bias"]))
    share = np.arange(H) // (H // G)
    return q[:, share], k[:, share], v.reshape(T, H, dv), g, sigmoid(h @ W[pre + "b"].T)


def delta(h, W, pre, m, eps):
    T, H, d, dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q, k, v, g, beta = delta_inputs(h, W, pre, m)
    S = np.zeros((H, d, dv))
    o = np.zeros((T, H, dv))
    for t in range(T):
        S = g[t][:, None, None] * S
        u = beta[t][:, None] * (v[t] - np.einsum("hkv,hk->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        o[t] = np.einsum("hkv,hk->hv", S, q[t])
    o = rms(o, eps) * W[pre + "norm"] * silu(h @ W[pre + "g"].T).reshape(T, H, dv)
    return o.reshape(T, H * dv) @ W[pre + "o"].T


def mixer(h, W, pre, layer, eps):
    m = layer["mixer"]
    if layer["type"] == "delta":
        return delta(h, W, pre, m, eps)
    if layer["type"] != "parallel":
        raise ValueError(f"layer type {layer['type']}")
    return m["left_scale"] * span(h, W, pre + "left.", m["left"]) + \
        m["right_scale"] * glow(h, W, pre + "right.", m["right"], eps)


def feed_forward(h, W, pre):
    return (gelu_tanh(h @ W[pre + "gate"].T) * (h @ W[pre + "up"].T)) @ W[pre + "down"].T


# --------------------------------------------------------------------------- #
# the model                                                                   #
# --------------------------------------------------------------------------- #
def order(config):
    """[(layer, whether the embedding's output joins the stream in front of it)] as they run."""
    n = len(config["layers"])
    loop = config.get("loop") or {"start": 0, "stop": 0, "times": 1}
    a, b = loop["start"], loop["stop"]
    runs = [(i, False) for i in range(a)]
    for again in range(loop["times"]):
        runs += [(i, again > 0 and i == a) for i in range(a, b)]
    return runs + [(i, False) for i in range(b, n)]


def forward(config, W, tokens, with_layers=False):
    """logits [T, vocab] of a whole sequence; with_layers: also the stream after every layer run."""
    eps = config["norm"]["eps"]
    x0 = W["embed"][np.asarray(tokens)] * config["embedding"]["scale"]
    x, after = x0, []
    for index, again in order(config):
        layer, pre = config["layers"][index], f"l{index}."
        if again:
            x = x + x0
        x = x + mixer(rms(x, eps) * W[pre + "norm1"], W, pre + "mix.", layer, eps)
        if layer.get("mlp"):
            x = x + feed_forward(rms(x, eps) * W[pre + "norm2"], W, pre + "mlp.")
        after.append(x)
    cap = config["logit_softcap"]
    logits = cap * np.tanh((rms(x, eps) * W["final.norm"]) @ W["head"].T / cap)
    return (logits, np.stack(after)) if with_layers else logits
