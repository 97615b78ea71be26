"""The Mefolorn oracle against the same mechanisms written the other way round, and the configuration, tensor list and
cache needs of the product - all without a GPU."""
import json

import numpy as np
import pytest
import torch

import plain_mefolorn as pm
import tiny_mefolorn as tm
from cpp_minilamma_b200.config.base import ConfigError, config_from_dict
from cpp_minilamma_b200.config.mefolorn import MefolornConfig
from cpp_minilamma_b200.engine.model import Model
from cpp_minilamma_b200.models.mefolorn import build_mefolorn_spec


def logistic(z):
    return 1.0 / (1.0 + np.exp(-z))


def test_norm_has_no_statistics():
    """Every column by itself: one column's value does not depend on the others', and nothing is divided by a size."""
    W = {"n": np.array([2.0, -1.0, 0.5]), "n.b": np.array([0.1, 0.2, -0.3]), "n.alpha": np.asarray(0.7)}
    x = np.array([[0.5, -3.0, 40.0], [0.5, 9.0, -2.0]])
    got = pm.squash(x, W, "n")
    assert got[0, 0] == got[1, 0] == 2.0 * np.tanh(0.35) + 0.1
    assert np.isclose(got[0, 1], np.tanh(2.1) + 0.2) and np.isclose(got[0, 2], 0.5 - 0.3)


def test_latent_attention_query_by_query():
    """Keys and values of every head expanded from the latent, one query at a time over an explicit list of visible
    keys; the sink counts once and is not scaled; the gate reads the mixer's input."""
    rng = np.random.RandomState(1)
    m = {"heads": 3, "dim": 4, "vdim": 5, "q_rank": 6, "kv_rank": 7, "scale": 0.8, "mask": {"size": 4}}
    D, T, eps = 9, 11, 1e-5
    W = {"dq": rng.randn(6, D), "dq.norm": 1 + 0.2 * rng.randn(6), "uq": rng.randn(12, 6), "dkv": rng.randn(7, D),
         "dkv.norm": 1 + 0.2 * rng.randn(7), "uk": rng.randn(12, 7), "uv": rng.randn(15, 7), "g": rng.randn(3, D),
         "sink": np.array([-3.0, 0.5, 4.0]), "o": rng.randn(D, 15)}
    h = rng.randn(T, D)
    got = pm.latent(h, W, "", m, eps)
    unit = lambda x, w: x / np.sqrt(np.mean(x * x) + eps) * w
    for i in range(T):
        heads = []
        for hd in range(3):
            q = W["uq"][hd * 4:hd * 4 + 4] @ unit(W["dq"] @ h[i], W["dq.norm"])
            seen = [j for j in range(T) if 0 <= i - j < 4]
            c = [unit(W["dkv"] @ h[j], W["dkv.norm"]) for j in seen]
            e = np.array([np.exp(0.8 * q @ (W["uk"][hd * 4:hd * 4 + 4] @ cj)) for cj in c])
            v = np.stack([W["uv"][hd * 5:hd * 5 + 5] @ cj for cj in c])
            heads.append((e @ v) / (np.exp(W["sink"][hd]) + e.sum()) * logistic(W["g"][hd] @ h[i]))
        assert np.abs(got[i] - W["o"] @ np.concatenate(heads)).max() < 1e-10


def test_mixed_scores_query_by_query():
    """Scores of all heads at a key, mixed by the matrix before the sigmoid (rows are outputs), the number per head
    added after mixing, keys just inside and just outside the window, no normalisation."""
    rng = np.random.RandomState(2)
    m = {"heads": 4, "kv_heads": 2, "dim": 6, "vdim": 3, "scale": 0.6, "mask": {"size": 5}, "rot": {"base": 9.0, "dims": 4}}
    D, T, eps = 7, 13, 1e-6
    W = {"q": rng.randn(24, D), "k": rng.randn(12, D), "v": rng.randn(6, D), "q.norm": 1 + 0.2 * rng.randn(24),
         "k.norm": 1 + 0.2 * rng.randn(12), "talk": rng.randn(4, 4), "pb": rng.randn(4), "o": rng.randn(D, 12)}
    h = rng.randn(T, D)
    got = pm.talk(h, W, "", m, eps)
    f = 9.0 ** (-np.arange(2) / 2.0)

    def turn(x, p):  # pairs (0, 2), (1, 3); 4 and 5 pass
        out = x.copy()
        out[0:2] = x[0:2] * np.cos(p * f) - x[2:4] * np.sin(p * f)
        out[2:4] = x[2:4] * np.cos(p * f) + x[0:2] * np.sin(p * f)
        return out

    whole = lambda name, x: (W[name] @ x) / np.sqrt(np.mean((W[name] @ x) ** 2) + eps) * W[name + ".norm"]
    for i in range(T):
        out = np.zeros((4, 3))
        for j in range(max(0, i - 4), i + 1):
            q, k = whole("q", h[i]).reshape(4, 6), whole("k", h[j]).reshape(2, 6)
            s = np.array([0.6 * turn(q[g], i) @ turn(k[g // 2], j) for g in range(4)])
            for g in range(4):
                out[g] += logistic(W["talk"][g] @ s + W["pb"][g]) * (W["v"] @ h[j]).reshape(2, 3)[g // 2]
        assert np.abs(got[i] - W["o"] @ out.reshape(-1)).max() < 1e-10


def test_linear_unit_equals_its_unrolled_form():
    """The recurrence against the sum it stands for (products of the decays between a write and the read), the
    convolution per token with nothing - not even the bias - before the first one, the gates' matrices block by block."""
    rng = np.random.RandomState(3)
    m = {"width": 6, "blocks": 2, "conv": 3}
    D, T = 5, 9
    W = {"y": rng.randn(6, D), "y.b": rng.randn(6), "x": rng.randn(6, D), "x.b": rng.randn(6), "conv": rng.randn(6, 3),
         "conv.b": rng.randn(6), "ra": rng.randn(2, 3, 3), "ra.b": rng.randn(2, 3), "ri": rng.randn(2, 3, 3),
         "ri.b": rng.randn(2, 3), "lam": rng.randn(6) - 2, "o": rng.randn(D, 6)}
    h = rng.randn(T, D)
    got = pm.drift(h, W, "", m)
    decay, write = np.zeros((T, 6)), np.zeros((T, 6))
    for t in range(T):
        u = W["conv.b"].copy()
        for back in range(3):
            if t >= back:
                u += W["conv"][:, 2 - back] * (W["x"] @ h[t - back] + W["x.b"])
        for b in range(2):
            part = slice(3 * b, 3 * b + 3)
            r = logistic(W["ra"][b] @ u[part] + W["ra.b"][b])
            i = logistic(W["ri"][b] @ u[part] + W["ri.b"][b])
            a = np.exp(-8.0 * r * np.log1p(np.exp(W["lam"][part])))
            decay[t, part], write[t, part] = a, np.sqrt(1 - a * a) * i * u[part]
    for t in range(T):
        S = sum(np.prod(decay[j + 1:t + 1], axis=0) * write[j] for j in range(t + 1))
        z = W["y"] @ h[t] + W["y.b"]
        y = 0.5 * z * (1 + np.tanh(np.sqrt(2 / np.pi) * (z + 0.044715 * z ** 3)))
        assert np.abs(got[t] - W["o"] @ (S * y)).max() < 1e-10


@pytest.mark.parametrize("name", ["mixed", "windows", "odd"])
def test_a_position_does_not_see_later_tokens(name):
    cfg = tm.CONFIGS[name]()
    W = {k: v.astype(np.float64) for k, v in tm.make_weights(cfg, 1).items()}
    toks = tm.tokens(cfg, 150, 3)
    whole = pm.forward(cfg, W, toks)
    for n in (1, 2, 64, 131):
        assert np.abs(pm.forward(cfg, W, toks[:n]) - whole[:n]).max() < 1e-9


def test_layer_reads_one_stream_twice():
    """x' = x + mixer(norm1(x)) + ff(norm2(x)): the feed-forward does not see the mixer's output."""
    cfg = tm.CONFIGS["latent"]()
    cfg["layers"][0]["mlp"] = {"kind": "dense", "ff": 16}
    W = {k: v.astype(np.float64) for k, v in tm.make_weights(cfg, 2).items()}
    toks = tm.tokens(cfg, 12, 1)
    _, after = pm.forward(cfg, W, toks, with_layers=True)
    x = W["embed"][toks] * cfg["embedding"]["scale"]
    mixed = pm.latent(pm.squash(x, W, "l0.norm1"), W, "l0.mix.", cfg["layers"][0]["mixer"], cfg["norm"]["eps"])
    h = pm.squash(x, W, "l0.norm2")
    gate = h @ W["l0.mlp.gate"].T
    fed = (gate * logistic(gate) * (h @ W["l0.mlp.up"].T)) @ W["l0.mlp.down"].T
    assert np.abs(after[0] - (x + mixed + fed)).max() < 1e-10


@pytest.mark.parametrize("name", list(tm.CONFIGS))
def test_configuration_round_trip_and_tensor_list(name):
    raw = tm.CONFIGS[name]()
    cfg = config_from_dict(raw)
    assert isinstance(cfg, MefolornConfig)
    again = config_from_dict(json.loads(json.dumps(cfg.to_dict())))
    assert again == cfg
    model = Model(build_mefolorn_spec(cfg), torch.float32, "cpu", max_positions=256)
    specs = {s.name: tuple(s.shape) for s in model.weight_specs() if not s.optional}
    assert specs == {k: tuple(v) for k, v in tm.tensor_shapes(raw).items()}
    assert model.capturable()
    for (_, _, need), lay in zip(model.cache_needs(), raw["layers"]):
        m = lay["mixer"] if lay["type"] == "latent_attention" else lay["mixer"]["left"]
        assert need.kv.window == (m.get("mask") or {}).get("size", 0)
        if lay["type"] == "latent_attention":  # one latent row per position, read as key and as value
            assert (need.kv.n_kv_heads, need.kv.head_dim, need.kv.v_in_k) == (1, m["kv_rank"], True) and need.state is None
        else:
            r = lay["mixer"]["right"]
            assert (need.kv.n_kv_heads, need.kv.head_dim) == (m["kv_heads"], m["dim"])
            assert dict((t[0], tuple(t[1])) for t in need.state.tensors) == {"S": (r["width"],), "conv": (r["conv"] - 1, r["width"])}


@pytest.mark.parametrize("path,value,words", [
    (("layers", 0, "type"), "attention", "type"),
    (("layers", 0, "mixer", "q_rank"), None, "q_rank"),
    (("layers", 0, "mixer", "kv_rank"), 0, "kv_rank"),
    (("layers", 0, "mixer", "mask"), {"size": 0}, "size"),
    (("layers", 0, "mlp"), {"kind": "moe"}, "moe"),
    (("layers", 1, "mixer", "left", "kv_heads"), 3, "multiple"),
    (("layers", 1, "mixer", "left", "rot"), {"base": 10.0, "dims": 3}, "even"),
    (("layers", 1, "mixer", "left", "rot"), {"base": 10.0, "dims": 18}, "at most"),
    (("layers", 1, "mixer", "right", "blocks"), 5, "equal blocks"),
    (("layers", 1, "mixer", "right", "conv"), 0, "conv"),
    (("layers", 1, "mixer", "left_scale"), "x", "left_scale"),
    (("layers",), [], "layers"),
    (("norm",), {"eps": -1.0}, "eps"),
    (("width",), None, "width"),
])
def test_faulty_configurations(path, value, words):
    raw = tm.config([tm.layer(tm.latent(), 8), tm.layer(tm.pair(tm.left(), tm.right()), 8)])
    at = raw
    for key in path[:-1]:
        at = at[key]
    at[path[-1]] = value
    with pytest.raises(ConfigError, match=words):
        config_from_dict(raw)


def test_random_folder_and_inspect(tmp_path, capsys):
    """The command line writes a folder of random weights for a configuration and lists it, without a GPU."""
    from cpp_minilamma_b200.cli import main
    src = tmp_path / "config.json"
    src.write_text(json.dumps(tm.CONFIGS["mixed"]()))
    out = tmp_path / "model"
    assert main(["random", str(out), "--config", str(src), "--seed", "5"]) == 0
    assert main(["inspect", str(out)]) == 0
    text = capsys.readouterr().out
    assert "Mefolorn" in text
    cfg, W = pm.read_folder(out)
    assert np.isfinite(pm.forward(cfg, W, tm.tokens(cfg, 9, 1))).all()
