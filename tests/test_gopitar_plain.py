"""The Gopitar oracle against the same mechanisms written the other way round, and the configuration, tensor list and
cache needs of the product - all without a GPU."""
import json

import numpy as np
import pytest
import torch

import plain_gopitar as pg
import tiny_gopitar as tg
from cpp_minilamma_b200.config.base import ConfigError, config_from_dict
from cpp_minilamma_b200.config.gopitar import GopitarConfig
from cpp_minilamma_b200.engine.model import Model
from cpp_minilamma_b200.models.gopitar import build_gopitar_spec


def logistic(z):
    return 1.0 / (1.0 + np.exp(-z))


def test_window_attention_query_by_query():
    """One query at a time over an explicit list of visible keys: bias, then the taps (nothing, not even the bias, before
    the first token), then the rotation; the gate reads the mixer's input; the output's bias."""
    rng = np.random.RandomState(2)
    m = {"heads": 4, "kv_heads": 2, "dim": 6, "vdim": 3, "conv": 3, "scale": 0.6, "mask": {"size": 5}, "rot": {"base": 9.0, "dims": 4}}
    D, T = 7, 13
    rows = {"q": 24, "k": 12, "v": 6}
    W = {"g": rng.randn(4, D), "o": rng.randn(D, 12), "o.b": rng.randn(D)}
    for p, n in rows.items():
        W.update({p: rng.randn(n, D), p + ".b": rng.randn(n), p + ".conv": rng.randn(n, 3)})
    h = rng.randn(T, D)
    got = pg.span(h, W, "", m)
    f = 9.0 ** (-np.arange(2) / 2.0)

    def filtered(p, t):
        return sum(W[p + ".conv"][:, 2 - back] * (W[p] @ h[t - back] + W[p + ".b"]) for back in range(3) if t >= back)

    def turn(x, p):  # pairs (0, 2), (1, 3); 4 and 5 pass
        out = x.copy()
        out[0:2] = x[0:2] * np.cos(p * f) - x[2:4] * np.sin(p * f)
        out[2:4] = x[2:4] * np.cos(p * f) + x[0:2] * np.sin(p * f)
        return out

    for i in range(T):
        seen = [j for j in range(T) if 0 <= i - j < 5]
        heads = []
        for g in range(4):
            q = turn(filtered("q", i).reshape(4, 6)[g], i)
            e = np.array([np.exp(0.6 * q @ turn(filtered("k", j).reshape(2, 6)[g // 2], j)) for j in seen])
            v = np.stack([filtered("v", j).reshape(2, 3)[g // 2] for j in seen])
            heads.append((e @ v) / e.sum() * logistic(W["g"][g] @ h[i]))
        assert np.abs(got[i] - (W["o"] @ np.concatenate(heads) + W["o.b"])).max() < 1e-10


def test_lightning_equals_its_unrolled_form():
    """The recurrence against the sum it stands for: o_t = sum_j a^(t - j) (q_t . k_j) v_j, normalised over all heads."""
    rng = np.random.RandomState(3)
    m = {"heads": 2, "dim": 4, "vdim": 3, "decay": [0.5, 0.9]}
    D, T, eps = 5, 9, 1e-5
    W = {"q": rng.randn(8, D), "k": rng.randn(8, D), "v": rng.randn(6, D), "g": rng.randn(6, D), "o": rng.randn(D, 6),
         "norm": 1 + 0.2 * rng.randn(6)}
    h = rng.randn(T, D)
    got = pg.glow(h, W, "", m, eps)
    act = lambda z: z * logistic(z)
    for t in range(T):
        o = np.zeros((2, 3))
        for hd in range(2):
            q = act(W["q"] @ h[t]).reshape(2, 4)[hd]
            for j in range(t + 1):
                k, v = act(W["k"] @ h[j]).reshape(2, 4)[hd], act(W["v"] @ h[j]).reshape(2, 3)[hd]
                o[hd] += m["decay"][hd] ** (t - j) * (q @ k) * v
        row = o.reshape(-1) / np.sqrt(np.mean(o ** 2) + eps) * W["norm"] * logistic(W["g"] @ h[t])
        assert np.abs(got[t] - W["o"] @ row).max() < 1e-10


def test_delta_rule_as_products_of_matrices():
    """S_t = g_t (I - beta k k^T) S_(t-1) + beta k v^T, the state's other form, token by token and head by head."""
    rng = np.random.RandomState(4)
    m = {"heads": 4, "kv_heads": 2, "dim": 3, "vdim": 5, "conv": 2}
    D, T, eps = 6, 11, 1e-6
    W = {"b": rng.randn(4, D), "a": rng.randn(4, D), "A_log": rng.randn(4), "dt_bias": rng.randn(4), "g": rng.randn(20, D),
         "norm": 1 + 0.2 * rng.randn(5), "o": rng.randn(D, 20)}
    for p, n in (("q", 6), ("k", 6), ("v", 20)):
        W.update({p: rng.randn(n, D), p + ".conv": rng.randn(n, 2)})
    h = rng.randn(T, D)
    got = pg.delta(h, W, "", m, eps)
    act = lambda z: z * logistic(z)
    filtered = lambda p, t: act(W[p + ".conv"][:, 1] * (W[p] @ h[t]) + (W[p + ".conv"][:, 0] * (W[p] @ h[t - 1]) if t else 0.0))
    S = np.zeros((4, 3, 5))
    for t in range(T):
        out = []
        for hd in range(4):
            q, k = (filtered(p, t).reshape(2, 3)[hd // 2] for p in "qk")
            q, k = q / np.sqrt(q @ q + 1e-6) / np.sqrt(3.0), k / np.sqrt(k @ k + 1e-6)
            v = filtered("v", t).reshape(4, 5)[hd]
            g = np.exp(-np.exp(W["A_log"][hd]) * np.log1p(np.exp(W["a"][hd] @ h[t] + W["dt_bias"][hd])))
            beta = logistic(W["b"][hd] @ h[t])
            S[hd] = g * (np.eye(3) - beta * np.outer(k, k)) @ S[hd] + beta * np.outer(k, v)
            o = S[hd].T @ q
            z = (W["g"] @ h[t]).reshape(4, 5)[hd]
            out.append(o / np.sqrt(np.mean(o * o) + eps) * W["norm"] * act(z))
        assert np.abs(got[t] - W["o"] @ np.concatenate(out)).max() < 1e-10


@pytest.mark.parametrize("name", ["mixed", "windows", "odd"])
def test_a_position_does_not_see_later_tokens(name):
    cfg = tg.CONFIGS[name]()
    W = {k: v.astype(np.float64) for k, v in tg.make_weights(cfg, 1).items()}
    toks = tg.tokens(cfg, 150, 3)
    whole = pg.forward(cfg, W, toks)
    for n in (1, 2, 64, 131):
        assert np.abs(pg.forward(cfg, W, toks[:n]) - whole[:n]).max() < 1e-9


def test_order_of_a_loop_and_the_embedding_again():
    """Layers outside the stretch run once; the embedding joins in front of every pass but the first, once; the
    feed-forward reads the stream with the mixer's output; the cap bends the logits."""
    cfg = tg.config([tg.layer(tg.delta(), 8), tg.layer(tg.delta(heads=2, kv_heads=1)), tg.layer(tg.delta(), 12)], cap=6.0, loop=(1, 2, 3))
    assert pg.order(cfg) == [(0, False), (1, False), (1, True), (1, True), (2, False)]
    W = {k: v.astype(np.float64) for k, v in tg.make_weights(cfg, 2).items()}
    toks = tg.tokens(cfg, 12, 1)
    logits, after = pg.forward(cfg, W, toks, with_layers=True)
    eps, x0 = cfg["norm"]["eps"], W["embed"][toks] * cfg["embedding"]["scale"]
    unit = lambda x: x / np.sqrt(np.mean(x * x, axis=1, keepdims=True) + eps)
    mix = lambda x, i: x + pg.delta(unit(x) * W[f"l{i}.norm1"], W, f"l{i}.mix.", cfg["layers"][i]["mixer"], eps)

    def feed(x, i):
        h = unit(x) * W[f"l{i}.norm2"]
        z = h @ W[f"l{i}.mlp.gate"].T
        gelu = 0.5 * z * (1 + np.tanh(np.sqrt(2 / np.pi) * (z + 0.044715 * z ** 3)))
        return x + (gelu * (h @ W[f"l{i}.mlp.up"].T)) @ W[f"l{i}.mlp.down"].T

    x = feed(mix(x0, 0), 0)
    want = [x]
    for again in range(3):
        x = mix(x + (x0 if again else 0.0), 1)
        want.append(x)
    want.append(feed(mix(x, 2), 2))
    assert np.abs(after - np.stack(want)).max() < 1e-10
    raw = (unit(want[-1]) * W["final.norm"]) @ W["head"].T
    assert np.abs(logits - 6.0 * np.tanh(raw / 6.0)).max() < 1e-10 and np.abs(logits).max() < 6.0 < np.abs(raw).max()


@pytest.mark.parametrize("name", list(tg.CONFIGS))
def test_configuration_round_trip_and_tensor_list(name):
    raw = tg.CONFIGS[name]()
    cfg = config_from_dict(raw)
    assert isinstance(cfg, GopitarConfig)
    again = config_from_dict(json.loads(json.dumps(cfg.to_dict())))
    assert again == cfg
    assert [(i, turn > 0) for i, turn in cfg.schedule()] == pg.order(raw)
    model = Model(build_gopitar_spec(cfg), torch.float32, "cpu", max_positions=256)
    specs = {s.name: tuple(s.shape) for s in model.weight_specs() if not s.optional}
    assert specs == {k: tuple(v) for k, v in tg.tensor_shapes(raw).items()}
    assert model.capturable()
    assert len(model.cache_needs()) == len(pg.order(raw))  # every pass has a cache and state of its own
    for (_, _, need), (index, _) in zip(model.cache_needs(), pg.order(raw)):
        m = raw["layers"][index]["mixer"]
        state = {t[0]: tuple(t[1]) for t in need.state.tensors}
        if raw["layers"][index]["type"] == "delta":
            channels = 2 * m["kv_heads"] * m["dim"] + m["heads"] * m["vdim"]
            assert need.kv is None
            assert state == {"S": (m["heads"], m["dim"], m["vdim"]), "conv": (m["conv"] - 1, channels)}
        else:
            l, r = m["left"], m["right"]
            channels = (l["heads"] + l["kv_heads"]) * l["dim"] + l["kv_heads"] * l["vdim"]
            assert need.kv.window == (l.get("mask") or {}).get("size", 0)
            assert (need.kv.n_kv_heads, need.kv.head_dim, need.kv.v_head_dim or l["dim"]) == (l["kv_heads"], l["dim"], l["vdim"])
            assert state == {"S": (r["heads"], r["dim"], r["vdim"]), "conv": (l["conv"] - 1, channels)}


@pytest.mark.parametrize("path,value,words", [
    (("layers", 0, "type"), "attention", "type"),
    (("layers", 0, "mixer", "dim"), None, "dim"),
    (("layers", 0, "mixer", "kv_heads"), 3, "multiple"),
    (("layers", 0, "mixer", "conv"), 0, "conv"),
    (("layers", 0, "mlp"), {"kind": "moe"}, "moe"),
    (("layers", 1, "mixer", "left", "kv_heads"), 3, "multiple"),
    (("layers", 1, "mixer", "left", "mask"), {"size": 0}, "size"),
    (("layers", 1, "mixer", "left", "rot"), {"base": 10.0, "dims": 3}, "even"),
    (("layers", 1, "mixer", "left", "rot"), {"base": 10.0, "dims": 18}, "at most"),
    (("layers", 1, "mixer", "left", "scale"), None, "scale"),
    (("layers", 1, "mixer", "right", "decay"), [0.5], "decay"),
    (("layers", 1, "mixer", "right_scale"), "x", "right_scale"),
    (("loop",), {"start": 1, "stop": 3, "times": 2}, "inside"),
    (("loop",), {"start": 0, "stop": 1, "times": 0}, "times"),
    (("logit_softcap",), -3.0, "logit_softcap"),
    (("layers",), [], "layers"),
    (("norm",), {"eps": -1.0}, "eps"),
    (("width",), None, "width"),
])
def test_faulty_configurations(path, value, words):
    raw = tg.config([tg.layer(tg.delta(), 8), tg.layer(tg.pair(tg.left(), tg.right()), 8)])
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
    src.write_text(json.dumps(tg.CONFIGS["mixed"]()))
    out = tmp_path / "model"
    assert main(["random", str(out), "--config", str(src), "--seed", "5"]) == 0
    assert main(["inspect", str(out)]) == 0
    text = capsys.readouterr().out
    assert "Gopitar" in text
    cfg, W = pg.read_folder(out)
    assert np.isfinite(pg.forward(cfg, W, tg.tokens(cfg, 9, 1))).all()
