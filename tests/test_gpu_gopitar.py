"""Gopitar through the engine against the plain oracle (`plain_gopitar`, float64, whole sequences), and its kernels
alone.

Every test makes its own small configuration and weights (`tiny_gopitar`).  float32 runs must agree with the oracle to
2e-4 of the largest logit (at least 2e-4 absolute): with the test weights a window one token off, a lost state, a tap or a
bias forgotten moves logits by percents.  bfloat16 runs are compared with the same unrounded oracle, so their bound is that
of rounding noise: mean error at most 0.5 % of the largest logit, and at most one row in twenty with an error above
3 % of it - keys of a few dimensions scaled to unit length make single rows ill-conditioned: perturbing the oracle's own
matrices by 2^-8 moves up to one row in twelve that far in a model with heads of one dimension.  The sharp test is
float32."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import cpp_minilamma_b200 as ml
import plain_gopitar as pg
import tiny_gopitar as tg
from cpp_minilamma_b200.cache.paged import PAGE
from cpp_minilamma_b200.engine.step import StepEntry, make_step_state

pytestmark = pytest.mark.gpu
DEV = torch.device("cuda:0")

_FOLDERS, _ENGINES, _ORACLE = {}, {}, {}


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    def get(name, dtype="float32", max_tokens=1024, max_positions=None):
        if name not in _FOLDERS:
            _FOLDERS[name] = tg.make_folder(name if isinstance(name, str) else tg.random_config(name),
                                            tmp_path_factory.mktemp(f"m{name}"), seed=len(_FOLDERS) + 1)
        folder, cfg, W = _FOLDERS[name]
        key = (name, dtype, max_tokens, max_positions)
        if key not in _ENGINES:
            _ENGINES[key] = ml.load(folder, dtype=dtype, max_tokens=max_tokens, max_positions=max_positions or 2048)
        return _ENGINES[key], cfg, W
    yield get
    _ENGINES.clear()


def oracle(name, cfg, W, toks):
    key = (name, tuple(toks))
    if key not in _ORACLE:
        _ORACLE[key] = pg.forward(cfg, W, toks)
    return _ORACLE[key]


def close(got, ref, dtype, what):
    got, ref = np.asarray(got, dtype=np.float64), np.asarray(ref, dtype=np.float64)
    assert got.shape == ref.shape, f"{what}: {got.shape} vs {ref.shape}"
    assert np.isfinite(got).all(), f"{what}: non-finite logits"
    err, scale = np.abs(got - ref), max(1.0, np.abs(ref).max())
    row = int(np.argmax(err.max(axis=-1))) if err.ndim == 2 else 0
    if dtype == "float32":
        assert err.max() <= 2e-4 * scale, f"{what}: err {err.max():.3e} of {scale:.2f}, first at row {row}"
        return
    rows = err.max(axis=-1).reshape(-1) > 3e-2 * scale
    assert rows.sum() <= max(1, len(rows) // 20) and err.mean() <= 5e-3 * scale, \
        f"{what}: max {err.max():.3e} mean {err.mean():.3e} of {scale:.2f}, {rows.sum()} rows over, worst row {row}"


def run_alone(llm, toks, cuts):
    """Feed one sequence in portions of the given sizes (the rest one token at a time); logits of every position."""
    slot = llm.engine.acquire(1)[0]
    rows, at = [], 0
    for n in list(cuts) + [1] * (len(toks) - sum(cuts)):
        rows.append(llm.engine.step([StepEntry(slot, toks[at:at + n], list(range(n)))]).cpu().numpy())
        at += n
    llm.engine.release(slot)
    return np.concatenate(rows)


LENGTH = {"span": 150, "glow": 150, "delta": 150, "mixed": 200, "ones": 140, "loop": 100, "windows": 260, "tensor": 300, "odd": 90}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(tg.CONFIGS))
def test_whole_prompt(models, name, dtype):
    """Every position of one prompt, the first tokens included (states and convolution inputs that start at nothing);
    prompts reach over windows and page borders."""
    llm, cfg, W = models(name, dtype)
    toks = tg.tokens(cfg, LENGTH[name], 11)
    close(run_alone(llm, toks, [len(toks)]), oracle(name, cfg, W, toks), dtype, f"{name} whole")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(tg.CONFIGS))
def test_prompt_then_token_by_token(models, name, dtype):
    """A short prompt, then a long run of single tokens through the cache and the state: windows and page borders pass
    over decoded tokens, states and convolution inputs are carried step by step."""
    llm, cfg, W = models(name, dtype)
    toks = tg.tokens(cfg, LENGTH[name], 12)
    close(run_alone(llm, toks, [7]), oracle(name, cfg, W, toks), dtype, f"{name} decode")


@pytest.mark.parametrize("name", ["mixed", "ones"])
def test_token_by_token_from_the_first_token(models, name):
    llm, cfg, W = models(name, "float32")
    toks = tg.tokens(cfg, 70, 14)
    close(run_alone(llm, toks, []), oracle(name, cfg, W, toks), "float32", f"{name} from the first token")


@pytest.mark.parametrize("name,cuts", [
    ("mixed", [2, 3, 1, 7, 2, 49, 2, 2, 64]),      # portions down to two tokens, shorter than the convolutions
    ("ones", [1, 1, 62, 2, 66]),                   # single first tokens; a cut at the page's edge and after it
    ("span", [39, 2, 39, 1, 41]),                  # portions that start just inside and just outside the window
    ("glow", [2, 2, 63, 1, 2, 64, 3]),             # the state handed from portion to portion
    ("delta", [2, 2, 31, 1, 2, 64, 33]),
    ("loop", [3, 2, 60, 2]),
    ("windows", [62, 2, 2, 60, 3, 64, 65]),
    ("tensor", [2, 65, 3, 128, 31, 33]),
    ("odd", [5, 2, 2, 60]),
])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_portions(models, name, cuts, dtype):
    llm, cfg, W = models(name, dtype)
    toks = tg.tokens(cfg, LENGTH[name], 13)
    close(run_alone(llm, toks, cuts), oracle(name, cfg, W, toks), dtype, f"{name} portions {cuts}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["mixed", "windows", "tensor", "loop"])
def test_unequal_batch_then_decoding_together(models, name, dtype):
    """Requests of 1, 37 and 90 tokens start in one step, go on by one token each, and the short ones end early; every
    logit equals that of the request alone."""
    llm, cfg, W = models(name, dtype)
    eng = llm.engine
    seqs = [tg.tokens(cfg, n, 20 + i) for i, n in enumerate((9, 50, 104))]
    first = [1, 37, 90]
    slots = eng.acquire(3)
    got = [[] for _ in seqs]
    out = eng.step([StepEntry(s, q[:n], list(range(n))) for s, q, n in zip(slots, seqs, first)]).cpu().numpy()
    at = 0
    for i, n in enumerate(first):
        got[i].append(out[at:at + n])
        at += n
    done, live = list(first), [0, 1, 2]
    while live:
        out = eng.step([StepEntry(slots[i], [seqs[i][done[i]]], [0]) for i in live]).cpu().numpy()
        for row, i in enumerate(live):
            got[i].append(out[row:row + 1])
            done[i] += 1
        for i in [i for i in live if done[i] == len(seqs[i])]:
            eng.release(slots[i])
            live.remove(i)
    for i, q in enumerate(seqs):
        close(np.concatenate(got[i]), oracle(name, cfg, W, q), dtype, f"{name} request {i} in a batch")
    eng.cache.check()


@pytest.mark.parametrize("name,pages", [("mixed", 6), ("tensor", 6)])
def test_slots_pages_and_states_used_again(models, name, pages):
    """Sequences longer than the page pool (every layer has a window, so pages come back while a sequence lives): in the
    same slot, pages and state rows a second one follows, while a short request comes and goes beside them.  A state or
    convolution input left behind by the first sequence would show in the second one's first rows."""
    llm, cfg, W = models(name, "float32", max_tokens=pages * PAGE, max_positions=10 * PAGE)
    eng = llm.engine
    for seed in (31, 32):
        toks = tg.tokens(cfg, pages * PAGE + 90, seed)
        short = tg.tokens(cfg, 20, seed + 10)
        slot = eng.acquire(1)[0]
        rows = []
        for at in range(0, len(toks), 50):
            part = toks[at:at + 50]
            rows.append(eng.step([StepEntry(slot, part, list(range(len(part))))]).cpu().numpy())
            if at == 50:
                other = eng.acquire(1)[0]
                got = eng.step([StepEntry(other, short, list(range(20)))]).cpu().numpy()
                eng.release(other)
                close(got, oracle(name, cfg, W, short), "float32", "the neighbour")
        eng.release(slot)
        eng.cache.check()
        close(np.concatenate(rows), oracle(name, cfg, W, toks), "float32", f"long sequence, seed {seed}")
    assert all(g.pool.n_free == g.pool.n_pages for g in eng.cache.groups)


def test_an_engine_cuts_a_long_step_itself(models):
    models("mixed")
    folder, cfg, W = _FOLDERS["mixed"]
    llm = ml.load(folder, dtype="float32", max_tokens=512, max_positions=512, max_step_tokens=64)
    toks = tg.tokens(cfg, 150, 41)
    close(run_alone(llm, toks, [150]), oracle("mixed", cfg, W, toks), "float32", "engine-cut step")


@pytest.mark.parametrize("seed", range(12))
def test_drawn_configurations(models, seed):
    """Two to five layers of either kind in any order: a whole prompt, then two unequal requests decoded together."""
    for dtype in ("float32", "bfloat16"):
        llm, cfg, W = models(seed, dtype)
        toks = tg.tokens(cfg, 230, 5)
        close(run_alone(llm, toks, [230]), oracle(seed, cfg, W, toks), dtype, f"seed {seed} whole")
        a, b = toks[:80], tg.tokens(cfg, 30, 6)
        s = llm.engine.acquire(2)
        llm.engine.step([StepEntry(s[0], a[:66], []), StepEntry(s[1], b[:16], [])])
        for i in range(14):
            got = llm.engine.step([StepEntry(s[0], [a[66 + i]], [0]), StepEntry(s[1], [b[16 + i]], [0])]).cpu().numpy()
            close(got, np.stack([oracle(seed, cfg, W, toks)[66 + i], oracle(seed, cfg, W, b)[16 + i]]), dtype,
                  f"seed {seed} decode {i}")
        for slot in s:
            llm.engine.release(slot)


def greedy_oracle(cfg, W, prompt, n):
    toks, out, sure = list(prompt), [], []
    for _ in range(n):
        logits = pg.forward(cfg, W, toks)[-1]
        best = int(np.argmax(logits))
        sure.append(logits[best] - np.partition(logits, -2)[-2] > 1e-3)
        out.append(best)
        toks.append(best)
    return out, sure


@pytest.mark.parametrize("name", ["mixed", "odd"])
def test_greedy_generation_through_the_entry_point(models, name):
    """`generate` (the scheduler, captured decode steps, device sampling) picks the oracle's tokens."""
    llm, cfg, W = models(name, "float32")
    prompts = [tg.tokens(cfg, n, 50 + i) for i, n in enumerate((3, 21, 66))]
    outs = llm.generate(prompts, max_new_tokens=14, ignore_eos=True)
    for prompt, got in zip(prompts, outs):
        want, sure = greedy_oracle(cfg, W, prompt, 14)
        upto = sure.index(False) if False in sure else len(sure)  # after a near-tie either token is right
        assert got[:upto] == want[:upto], (got, want)
    again = llm.generate(prompts, max_new_tokens=14, ignore_eos=True)
    assert again == outs  # slots, pages and states of finished requests serve the next ones
    llm.engine.cache.check()


def test_bfloat16_generation_replays_captured_steps(models):
    """Decode steps of the bfloat16 engine run from CUDA graphs and give the tokens of the same engine stepping eagerly."""
    llm, cfg, W = models("tensor", "bfloat16")
    assert llm.model.capturable()
    prompts = [tg.tokens(cfg, n, 80 + i) for i, n in enumerate((5, 40))]
    outs = llm.generate(prompts, max_new_tokens=24, ignore_eos=True)
    assert llm.engine.shared_decode_graphs().replays > 0
    eng = llm.engine
    for prompt, got in zip(prompts, outs):
        slot = eng.acquire(1)[0]
        logits = eng.step([StepEntry(slot, prompt, [len(prompt) - 1])])
        stepped = []
        for _ in range(24):
            top2 = torch.topk(logits[0], 2).values
            if float(top2[0] - top2[1]) < 0.05:  # a near-tie: rounding may fall either way from here on
                break
            stepped.append(int(torch.argmax(logits[0])))
            logits = eng.step([StepEntry(slot, [stepped[-1]], [0])])
        eng.release(slot)
        assert got[:len(stepped)] == stepped


def test_command_line_generates_the_oracles_tokens(models, capsys):
    from cpp_minilamma_b200.cli import main
    _, cfg, W = models("odd", "float32")
    prompt = tg.tokens(cfg, 5, 60)
    assert main(["generate", _FOLDERS["odd"][0], "-p", " ".join(map(str, prompt)), "-n", "6", "--dtype", "float32",
                 "--ignore-eos"]) == 0
    line = capsys.readouterr().out.splitlines()[0]
    want, sure = greedy_oracle(cfg, W, prompt, 6)
    upto = sure.index(False) if False in sure else len(sure)
    assert [int(t) for t in line.split()][:upto] == want[:upto]


def test_trace_replay_writes_the_wanted_logits(models, tmp_path):
    """The trace runner on a Gopitar folder: two requests start together, decode, one ends early."""
    _, cfg, W = models("mixed", "float32")
    folder = _FOLDERS["mixed"][0]
    a, b = tg.tokens(cfg, 30, 70), tg.tokens(cfg, 70, 71)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:28], "want": [0, 27]},
                                     {"id": "b", "tokens": b[:66], "want": [65]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[28:29], "want": []},
                                     {"id": "b", "tokens": b[66:67], "want": [0]}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": a[29:30], "want": [0]},
                                     {"id": "b", "tokens": b[67:68], "want": [0]}], "end": ["a"]},
             {"step": 3, "entries": [{"id": "b", "tokens": b[68:70], "want": [1]}], "end": ["b"]}]
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    out = tmp_path / "out"
    proc = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", folder, "--dtype",
                           "float32", "--out", str(out), "--max-tokens", "256"],
                          input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True,
                          timeout=600)
    assert proc.returncode == 0, proc.stderr[-2000:]
    assert [l for l in proc.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2", "done 3"]
    ra, rb = oracle("mixed", cfg, W, a), oracle("mixed", cfg, W, b)
    for n, rows in {0: [ra[0], ra[27], rb[65]], 1: [rb[66]], 2: [ra[29], rb[67]], 3: [rb[69]]}.items():
        got = np.fromfile(out / f"{n}.f32", dtype="<f4").reshape(len(rows), -1)
        close(got, np.stack(rows), "float32", f"trace step {n}")


# --------------------------------------------------------------------------------------------------------------- #
# kernels alone                                                                                                   #
# --------------------------------------------------------------------------------------------------------------- #
def _ints(values):
    return torch.tensor(values, dtype=torch.int32, device=DEV)


def _paged(gen, ctxs, G, d, dv, dtype):
    """Key and value caches with every sequence's pages in shuffled order; what no sequence owns is not a number."""
    n_pages = sum(-(-c // PAGE) for c in ctxs) + 3
    k = torch.full((n_pages, G, PAGE, d), float("nan")).to(dtype)
    v = torch.full((n_pages, G, PAGE, dv), float("nan")).to(dtype)
    order = torch.randperm(n_pages, generator=gen).tolist()
    table = torch.full((len(ctxs), max(-(-c // PAGE) for c in ctxs)), -1, dtype=torch.int32)
    at = 0
    for s, c in enumerate(ctxs):
        for b in range(-(-c // PAGE)):
            table[s, b] = order[at]
            n = min(PAGE, c - b * PAGE)
            k[order[at], :, :n] = (torch.randn((G, n, d), generator=gen) * 0.5).to(dtype)
            v[order[at], :, :n] = torch.randn((G, n, dv), generator=gen).to(dtype)
            at += 1
    return k, v, table


def _dense(cache, table, s, ctx):
    return torch.stack([cache[int(table[s, p // PAGE]), :, p % PAGE] for p in range(ctx)]).double()  # [ctx, G, d]


def _attention_reference(q, keys, values, pos0, scale, window, group):
    n, H, _ = q.shape
    i, j = pos0 + torch.arange(n)[:, None], torch.arange(keys.shape[0])[None, :]
    see = (j <= i) & ((j > i - window) if window else torch.ones_like(j, dtype=torch.bool))
    out = []
    for h in range(H):
        s = torch.where(see, scale * q[:, h] @ keys[:, h // group].T, torch.full_like(see, -float("inf"), dtype=torch.double))
        out.append(torch.softmax(s, dim=1) @ values[:, h // group])
    return torch.stack(out, dim=1)


@pytest.mark.parametrize("H,G,d,dv,window", [(4, 2, 64, 128, 70), (6, 2, 128, 64, 100), (3, 3, 64, 128, 1), (34, 2, 64, 128, 65),
                                             (8, 2, 128, 64, 64), (4, 4, 64, 128, 0), (18, 1, 128, 64, 33)])
def test_attention_with_values_of_another_size(H, G, d, dv, window):
    """The tcgen05 prompt kernel and the TMA-fed single-token kernel (one block a sequence, and the context in 2, 5 and 20
    splits) with values wider and narrower than keys.  The key just inside the last query's window and the one just outside
    it stand out; both multiply every head by its gate; a page that is not the sequence's, or rows past its end, hold no numbers."""
    from cpp_minilamma_b200.csrc import kernels as K
    gen = torch.Generator(device="cpu").manual_seed(d * 1000 + H)
    starts, lens = [0, 70, 300, 0], [150, 131, 1, 3]
    ctxs = [s + n for s, n in zip(starts, lens)]
    k_cache, v_cache, table = _paged(gen, ctxs, G, d, dv, torch.bfloat16)
    T, group, scale = sum(lens), H // G, 1.0 / d ** 0.5
    q = torch.randn((T, H * d), generator=gen).to(torch.bfloat16)
    for s in range(4):
        for edge in ((ctxs[s] - window, ctxs[s] - window - 1) if window else (0, 1)):
            if 0 <= edge < ctxs[s]:
                page, at = int(table[s, edge // PAGE]), edge % PAGE
                last_q = q[sum(lens[:s + 1]) - 1].float().view(G, group, d).mean(dim=1)
                k_cache[page, :, at] = (7.0 * d ** 0.5 * last_q / last_q.norm(dim=1, keepdim=True) / last_q.norm(dim=1, keepdim=True)).to(torch.bfloat16)
                v_cache[page, :, at] = (v_cache[page, :, at].float() * 4).to(torch.bfloat16)
    refs = {}
    for w in {window, window + 1, max(window - 1, 1)} if window else {0}:
        parts = []
        for s in range(4):
            rows = slice(sum(lens[:s]), sum(lens[:s + 1]))
            parts.append(_attention_reference(q[rows].double().view(-1, H, d), _dense(k_cache, table, s, ctxs[s]),
                                              _dense(v_cache, table, s, ctxs[s]), starts[s], scale, w, group))
        refs[w] = torch.cat(parts).view(T, H * dv)
    gate = torch.randn((T, H + 9), generator=gen).to(torch.bfloat16)  # a number per row and head, from the third column on
    for w in refs:
        refs[w] = (refs[w].view(T, H, dv) * torch.sigmoid(gate[:, 2:2 + H].double())[..., None]).reshape(T, H * dv)
    want = refs[window]
    tol = 1.5e-2 * max(1.0, want.abs().max().item())
    last = [sum(lens[:i + 1]) - 1 for i in range(4)]
    if window:  # one key more or one less is well above the tolerance
        assert all((r - want)[last].abs().max().item() > 4 * tol for w, r in refs.items() if w != window)
    state = make_step_state(DEV, [0, 1, 2, 3], starts, lens)
    kc, vc, table_dev, qd = (t.to(DEV) for t in (k_cache, v_cache, table, q))
    tiles = [(starts[s] + min(n, r + 128), s, r) for s, n in enumerate(lens) for r in range(0, n, 128)]
    tiles.sort()
    seqs, rows = _ints([s for _, s, _ in tiles]), _ints([r for _, _, r in tiles])
    out = torch.zeros((T, H * dv), dtype=torch.bfloat16, device=DEV)
    assert K.attention_prefill_takes_chunks(torch.bfloat16, d, dv)
    K.attention_prefill(qd, kc, vc, state.seq_slot, state.seq_ctx, state.seq_qstart, state.seq_qlen, seqs, rows, table_dev, out,
                        len(tiles), H, G, d, window, scale, wide_tiles=(seqs, rows), v_head_dim=dv, gate=(gate.to(DEV), 2))
    err = (out.cpu().double() - want).abs()
    assert err.max().item() <= tol, ("prompt", err.max().item(), tol, int(err.max(dim=1).values.argmax()))
    one = make_step_state(DEV, [0, 1, 2, 3], [c - 1 for c in ctxs], [1] * 4)
    assert K.attention_decode_takes_value_size(torch.bfloat16, d, dv)
    for splits in (1, 2, 5, 20):
        out = torch.zeros((4, H * dv), dtype=torch.bfloat16, device=DEV)
        scratch = torch.full((K.attention_decode_scratch_floats(4, H, dv, splits),), float("nan"), device=DEV)
        counters = torch.zeros((4 * G * -(-group // 16),), dtype=torch.int32, device=DEV)
        K.attention_decode(qd[last].contiguous(), kc, vc, one.seq_slot, one.seq_ctx, table_dev, scratch, out, 4, H, G, d, splits,
                           window, scale, counters=counters, v_head_dim=dv, gate=(gate[last].contiguous().to(DEV), 2))
        err = (out.cpu().double() - want[last]).abs().max().item()
        assert err <= tol, ("single tokens", splits, err, tol)


def _portions(lens_of_steps):
    """Steps of a batch of sequences: [(starts, lens)] where each sequence's portions follow one another."""
    at, out = [0] * len(lens_of_steps[0]), []
    for lens in lens_of_steps:
        out.append((list(at), list(lens)))
        at = [a + n for a, n in zip(at, lens)]
    return out


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,d,dv,rot,taps,interleaved", [
    (4, 2, 64, 128, 32, 3, False), (3, 1, 16, 8, 16, 4, False), (2, 2, 8, 12, 0, 2, False), (3, 3, 6, 10, 4, 3, False),
    (2, 1, 16, 16, 8, 5, False), (2, 1, 16, 16, 8, 3, True), (1, 1, 4, 4, 4, 1, False), (5, 1, 32, 4, 24, 4, False)])
def test_attention_inputs_behind_a_convolution(dtype, H, G, d, dv, rot, taps, interleaved):
    """Bias, convolution and rotation of q, k and v over portions of every kind (longer than a thread's run of rows, shorter
    than the convolution, single tokens whose kernel moves the state on itself) against the whole sequence in float64; the
    state of a sequence that starts is zero, and nothing - not even the bias - comes before the first token."""
    from cpp_minilamma_b200.csrc import kernels as K
    gen = torch.Generator(device="cpu").manual_seed(H * 100 + taps)
    steps = _portions([[1, 20, 2], [1, 1, 1], [3, 2, 70], [1, 1, 1], [1, 1, 1], [40, 1, 1]])
    total = [sum(lens[s] for _, lens in steps) for s in range(3)]
    C = (H + G) * d + G * dv
    ld = C + (-C % 8) + 8
    proj = [torch.randn((n, ld), generator=gen).to(dtype) for n in total]
    bias, w = torch.randn((C,), generator=gen), torch.randn((C, taps), generator=gen)
    cos = torch.rand((128, rot // 2), generator=gen) if rot else None
    sin = torch.rand((128, rot // 2), generator=gen) if rot else None
    want = []
    for p in proj:
        u = p[:, :C].double() + bias.double()
        y = torch.zeros_like(u)
        for back in range(taps):
            if back < len(u):
                y[back:] += w[:, taps - 1 - back].double() * u[:len(u) - back]
        qk, v = y[:, :(H + G) * d].reshape(len(u), H + G, d).clone(), y[:, (H + G) * d:]
        if rot:
            x = qk[..., :rot].clone()
            a, b = (x[..., 0::2], x[..., 1::2]) if interleaved else (x[..., :rot // 2], x[..., rot // 2:])
            c, s = cos[:len(u), None].double(), sin[:len(u), None].double()
            first, second = a * c - b * s, b * c + a * s
            if interleaved:
                qk[..., 0:rot:2], qk[..., 1:rot:2] = first, second
            else:
                qk[..., :rot // 2], qk[..., rot // 2:rot] = first, second
        want.append((qk[:, :H], qk[:, H:], v.reshape(len(u), G, dv)))
    n_pages = 6
    k_cache, v_cache = (torch.full((n_pages, G, PAGE, e), float("nan"), device=DEV).to(dtype) for e in (d, dv))
    table = torch.tensor([[3, 0], [5, 1], [2, 4]], dtype=torch.int32)
    state = torch.zeros((3, taps - 1, C), device=DEV)
    slots = [2, 0, 1]
    tol = 2e-6 if dtype == torch.float32 else 8e-3
    dev = lambda t: t.to(DEV) if t is not None else None
    got_q = [[] for _ in total]
    for starts, lens in steps:
        st = make_step_state(DEV, slots, starts, lens)
        rows = torch.cat([p[s:s + n] for p, s, n in zip(proj, starts, lens)]).to(DEV).contiguous()
        q = torch.zeros((sum(lens), H * d), dtype=dtype, device=DEV)
        advance = st.all_decode and K.conv_attention_advances(d, dv, rot, interleaved, taps, ld)
        K.conv_attention_prepare(rows, dev(bias), dev(w), state, dev(cos), dev(sin), st.tok_pos, st.tok_seq, st.seq_slot,
                                 st.seq_qstart, table.to(DEV), q, k_cache, v_cache, H, G, d, dv, rot, interleaved, taps,
                                 advance=advance)
        if taps > 1 and not advance:
            K.conv_state_update(rows, state, st.seq_slot, st.seq_qstart, st.seq_qlen, 3, C, taps, bias=dev(bias))
        for s, part in enumerate(torch.split(q.cpu(), lens)):
            got_q[s].append(part)
    for s, (q, k, v) in enumerate(want):
        scale = max(1.0, q.abs().max().item(), v.abs().max().item())
        got = torch.cat(got_q[s]).double().view(-1, H, d)
        keys, values = (_dense(c.cpu(), table[slots[s]:slots[s] + 1], 0, total[s]) for c in (k_cache, v_cache))
        for name, a, b in (("q", got, q), ("k", keys, k), ("v", values, v)):
            assert (a - b).abs().max().item() <= tol * scale, (name, s, (a - b).abs().max().item(), int((a - b).abs().flatten(1).max(1).values.argmax()))
        u = proj[s][:, :C].double() + bias.double()  # the state: the last inputs
        assert (state[slots[s]].cpu().double() - u[total[s] - (taps - 1):]).abs().max().item() <= 2e-6 * scale if taps > 1 else True


def _in_runs(q, k, v, state, out, st, lens, H, G, d, dv, **decays):
    from cpp_minilamma_b200.csrc import kernels as K
    runs = [(s, r) for s, n in enumerate(lens) for r in range(0, n, K.STATE_RUN)]
    first = [next(i for i, (s, _) in enumerate(runs) if s == which) for which in range(len(lens))]
    scratch = torch.full((K.state_chunks_scratch(len(runs), H, d, dv, "beta" in decays),), float("nan"), device=DEV)
    K.state_chunks(q, k, v, state, out, scratch, _ints([s for s, _ in runs]), _ints([r for _, r in runs]), _ints(first),
                   st.seq_slot, st.seq_qstart, st.seq_qlen, len(lens), H, G, d, dv, **decays)


def _delta_reference(q, k, v, g, beta, S, share):
    """float64, one sequence: q, k [T, G, d], v [T, H, dv], g, beta [T, H], S [H, d, dv] -> (o, S)."""
    out = []
    S = S.clone()
    for t in range(q.shape[0]):
        S = g[t][:, None, None] * S
        kt, qt = k[t][share], q[t][share]
        u = beta[t][:, None] * (v[t] - torch.einsum("hkv,hk->hv", S, kt))
        S = S + kt[:, :, None] * u[:, None, :]
        out.append(torch.einsum("hkv,hk->hv", S, qt))
    return torch.stack(out), S


@pytest.mark.parametrize("H,G,d,dv,lens", [
    (2, 1, 32, 64, [70, 1, 33]), (4, 2, 64, 64, [130]), (3, 3, 128, 128, [200, 3]), (2, 2, 128, 32, [64, 65, 63]), (6, 2, 16, 16, [5, 40]),
    (1, 1, 256, 48, [40, 40]), (3, 1, 7, 9, [20, 60]), (2, 1, 300, 20, [18]), (8, 4, 64, 128, [1] * 80), (8, 8, 128, 128, [1] * 40),
    (16, 16, 32, 128, [1] * 20), (2, 1, 96, 80, [100, 32])])
@pytest.mark.parametrize("strong", [False, True])
@pytest.mark.parametrize("runs", [False, True])
def test_delta_rule_with_a_decay_per_head(H, G, d, dv, lens, strong, runs):
    """The recurrence in every layout its sizes and token counts select, and a run of tokens at a time, twice in a row (the
    state handed on), against float64; keys that repeat (the correction is then as large as the value), decays from 1 down
    to none at all."""
    from cpp_minilamma_b200.csrc import kernels as K
    if runs and not K.state_chunks_supported(d, dv):
        pytest.skip("sizes of the token-by-token scan")
    gen = torch.Generator(device="cpu").manual_seed(d + dv + len(lens))
    n_seqs, share = len(lens), torch.arange(H) // (H // G)
    state = torch.randn((n_seqs + 1, H, d, dv), generator=gen).to(DEV)
    before = state.cpu().double()
    slots = [(i * 7 + 3) % n_seqs for i in range(n_seqs)] if n_seqs % 7 else list(range(n_seqs))
    for turn in range(2):
        T = sum(lens)
        unit = lambda x: x / x.norm(dim=-1, keepdim=True)
        q, k = unit(torch.randn((T, G, d), generator=gen)) / d ** 0.5, unit(torch.randn((T, G, d), generator=gen))
        k[1::3] = k[0:len(k[1::3]) * 3:3]
        v, beta = torch.randn((T, H, dv), generator=gen), torch.sigmoid(2 * torch.randn((T, H), generator=gen))
        log_g = -torch.exp((3.0 if strong else 1.5) * torch.randn((T, H), generator=gen) - (0.0 if strong else 3.0))
        log_g[::5] = 0.0
        if strong:
            log_g[3::11] = -200.0
        g = torch.exp(log_g)
        st = make_step_state(DEV, slots, [0] * n_seqs, lens)
        out = torch.full((T, H * dv), float("nan"), device=DEV)
        flat = lambda x: x.reshape(T, -1).contiguous().to(DEV)
        if runs:
            _in_runs(flat(q), flat(k), flat(v), state, out, st, lens, H, G, d, dv, token_decay=flat(g), beta=flat(beta))
        else:
            K.state_scan(flat(q), flat(k), flat(v), None, flat(beta), None, state, out, st.seq_slot, st.seq_qstart, st.seq_qlen,
                         n_seqs, H, G, d, dv, token_decay=flat(g))
        at = 0
        for s, n in zip(slots, lens):
            rows = slice(at, at + n)
            want, after = _delta_reference(q[rows].double(), k[rows].double(), v[rows].double(), g[rows].double(),
                                           beta[rows].double(), before[s], share)
            scale = max(1.0, want.abs().max().item())
            err = (out[rows].cpu().double().view(n, H, dv) - want).abs()
            assert err.max().item() <= 2e-5 * scale, (turn, s, err.max().item(), scale, int(err.flatten(1).max(1).values.argmax()))
            assert (state[s].cpu().double() - after).abs().max().item() <= 2e-5 * max(1.0, after.abs().max().item()), (turn, s)
            before[s] = after
            at += n
        assert torch.equal(state[n_seqs].cpu().double(), before[n_seqs])


@pytest.mark.parametrize("H,d,dv,lens", [(2, 64, 64, [70, 1, 33]), (3, 32, 128, [300]), (8, 128, 128, [257, 3]), (1, 16, 16, [64]), (2, 12, 20, [90]),
                                         (2, 128, 32, [65, 63, 128]), (3, 5, 7, [40, 2]), (4, 64, 128, [1] * 90), (2, 256, 48, [40])])
@pytest.mark.parametrize("form", ["scan", "runs", "runs, decays per token"])
def test_recurrence_with_a_fixed_decay(H, d, dv, lens, form):
    """One decay per head, from 0 (only the current token) to 1, in every layout and a run of tokens at a time, twice in a
    row, against float64."""
    from cpp_minilamma_b200.csrc import kernels as K
    if form != "scan" and not K.state_chunks_supported(d, dv):
        pytest.skip("sizes of the token-by-token scan")
    gen = torch.Generator(device="cpu").manual_seed(d + dv + len(lens))
    n_seqs, T = len(lens), sum(lens)
    decay = torch.tensor(([0.999, 0.3, 1.0, 0.97, 0.0, 0.6, 1e-8, 0.9999])[:H])
    state = torch.randn((n_seqs, H, d, dv), generator=gen).to(DEV)
    S = state.cpu().double()
    for turn in range(2):
        q, k, v = (torch.randn((T, H, e), generator=gen) / e ** 0.25 for e in (d, d, dv))
        st = make_step_state(DEV, list(range(n_seqs)), [0] * n_seqs, lens)
        out = torch.full((T, H * dv), float("nan"), device=DEV)
        flat = lambda x: x.reshape(T, -1).contiguous().to(DEV)
        if form == "scan":
            K.state_scan(flat(q), flat(k), flat(v), None, None, decay.to(DEV), state, out, st.seq_slot, st.seq_qstart, st.seq_qlen,
                         n_seqs, H, H, d, dv)
        elif form == "runs":
            _in_runs(flat(q), flat(k), flat(v), state, out, st, lens, H, H, d, dv, head_decay=decay.to(DEV))
        else:
            _in_runs(flat(q), flat(k), flat(v), state, out, st, lens, H, H, d, dv, token_decay=decay.expand(T, H).contiguous().to(DEV))
        at = 0
        for s, n in enumerate(lens):
            for t in range(at, at + n):
                S[s] = decay.double()[:, None, None] * S[s] + k[t].double()[:, :, None] * v[t].double()[:, None, :]
                want = torch.einsum("hkv,hk->hv", S[s], q[t].double())
                err = (out[t].cpu().double().view(H, dv) - want).abs().max().item()
                assert err <= 2e-5 * max(1.0, want.abs().max().item()) + 2e-6 * S[s].abs().max().item(), (turn, s, t - at, err)
            at += n
            assert (state[s].cpu().double() - S[s]).abs().max().item() <= 2e-5 * max(1.0, S[s].abs().max().item())


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,d,dv,taps,per_head", [(4, 2, 64, 64, 4, True), (3, 1, 128, 128, 3, True), (2, 2, 16, 40, 2, True), (3, 3, 7, 9, 3, True),
                                                    (2, 1, 256, 64, 4, True), (2, 1, 32, 300, 2, True), (2, 2, 32, 64, 6, True), (2, 1, 8, 8, 1, True),
                                                    (4, 2, 64, 32, 4, False), (3, 3, 9, 5, 3, False)])
def test_delta_rule_inputs(dtype, H, G, d, dv, taps, per_head):
    """Convolution, silu, unit length, beta and decays (per head and per key channel) over portions shorter and longer than
    the convolution and single tokens, against float64."""
    from cpp_minilamma_b200.csrc import kernels as K
    gen = torch.Generator(device="cpu").manual_seed(H * 100 + taps + d)
    steps = _portions([[1, 20, 2], [1, 1, 1], [3, 2, 70], [1, 1, 1], [1, 1, 1], [40, 1, 1]])
    total = [sum(lens[s] for _, lens in steps) for s in range(3)]
    C, decays = 2 * G * d + H * dv, H if per_head else H * d
    ld = C + 2 * H
    ld += -ld % 8
    proj = [torch.randn((n, ld), generator=gen).to(dtype) for n in total]
    rates = [torch.randn((n, decays), generator=gen) for n in total]
    w, a_log, dt = torch.randn((C, taps), generator=gen), torch.randn((H,), generator=gen), torch.randn((decays,), generator=gen)
    state = torch.zeros((3, taps - 1, C), device=DEV)
    slots = [1, 2, 0]
    got = [[] for _ in total]
    for starts, lens in steps:
        st = make_step_state(DEV, slots, starts, lens)
        T = sum(lens)
        pick = lambda xs: torch.cat([x[s:s + n] for x, s, n in zip(xs, starts, lens)]).to(DEV).contiguous()
        rows = pick(proj)
        outs = [torch.full((T, n), float("nan"), device=DEV) for n in (G * d, G * d, H * dv, decays, H)]
        advance = st.all_decode and K.delta_prepare_advances(H, G, d, dv, taps, ld)
        K.delta_prepare(rows, None if per_head else pick(rates), w.to(DEV), state, a_log.to(DEV), dt.to(DEV), st.tok_seq, st.seq_slot,
                        st.seq_qstart, *outs, H, G, d, dv, taps, 1e-6, advance=advance)
        if taps > 1 and not advance:
            K.conv_state_update(rows, state, st.seq_slot, st.seq_qstart, st.seq_qlen, 3, C, taps)
        for s in range(3):
            got[s].append([torch.split(o.cpu().double(), lens)[s] for o in outs])
    for s in range(3):
        u = proj[s].double()
        y = torch.zeros((total[s], C), dtype=torch.double)
        for back in range(min(taps, total[s])):
            y[back:] += w[:, taps - 1 - back].double() * u[:total[s] - back, :C]
        y = y * torch.sigmoid(y)
        q, k, v = y[:, :G * d].view(-1, G, d), y[:, G * d:2 * G * d].view(-1, G, d), y[:, 2 * G * d:]
        length = lambda x: x / (x.pow(2).sum(-1, keepdim=True) + 1e-6).sqrt()
        z = (u[:, C + H:C + 2 * H] if per_head else rates[s].double()) + dt.double()
        rate = a_log.double().exp() if per_head else a_log.double().exp().repeat_interleave(d)
        g = torch.exp(-rate * torch.nn.functional.softplus(z))
        want = [(length(q) / d ** 0.5).flatten(1), length(k).flatten(1), v, g, torch.sigmoid(u[:, C:C + H])]
        for i, name in enumerate(("q", "k", "v", "decay", "beta")):
            have = torch.cat([step[i] for step in got[s]])
            err = (have - want[i]).abs().max().item()
            assert err <= 3e-6 * max(1.0, want[i].abs().max().item()), (name, s, err)


def test_gated_activation_in_every_product_kernel():
    """gelu(gate) * up, tanh form, from the weight-streaming kernels' epilogues, from the kernel behind a library product
    (plain halves, blocks of eight, rows that still lack their norm's factor, with a bias) against float64."""
    from cpp_minilamma_b200.csrc import kernels as K
    gen = torch.Generator(device="cpu").manual_seed(5)
    gelu = lambda z: 0.5 * z * (1 + torch.tanh((2 / torch.pi) ** 0.5 * (z + 0.044715 * z ** 3)))
    for M, inter, width in ((1, 64, 128), (5, 136, 256), (16, 8704, 128), (40, 64, 64)):
        x = torch.randn((M, width), generator=gen).to(torch.bfloat16)
        w = (2.0 * torch.randn((2 * inter, width), generator=gen) / width ** 0.5).to(torch.bfloat16)
        y = x.double() @ w.double().T
        rows = y.view(M, inter // 8, 2, 8)
        want = (gelu(rows[:, :, 0]) * rows[:, :, 1]).reshape(M, inter)
        tol = 8e-3 * want.abs().max().item()
        for kernel, takes in ((K.linear_small, K.linear_small_supported), (K.linear_tma, K.linear_tma_supported), (K.linear_tc5, K.linear_tc5_supported)):
            if takes(M, 2 * inter, width, K.EPI_GEGLU):
                out = torch.zeros((M, inter), dtype=torch.bfloat16, device=DEV)
                kernel(x.to(DEV), w.to(DEV), None, out, K.EPI_GEGLU)
                assert (out.cpu().double() - want).abs().max().item() <= tol, kernel.__name__
    for dtype, tol in ((torch.float32, 2e-6), (torch.bfloat16, 8e-3)):
        for inter, block in ((64, 8), (64, 0), (10, 0)):
            gu = (3.0 * torch.randn((7, 2 * inter), generator=gen)).to(dtype)
            gu[0, 0], gu[1, 0] = 60.0, -60.0  # where the exponential of the form overflows
            bias = torch.randn((2 * inter,), generator=gen)
            for b in (None, bias):
                y = gu.double() + (b.double() if b is not None else 0.0)
                g, u = (y[:, :inter], y[:, inter:]) if not block else (y.view(7, -1, 2, 8)[:, :, 0].reshape(7, -1), y.view(7, -1, 2, 8)[:, :, 1].reshape(7, -1))
                want = gelu(g) * u
                out = torch.zeros((7, inter), dtype=dtype, device=DEV)
                K.swiglu(gu.to(DEV), out, block, bias=b.to(DEV) if b is not None else None, act=K.GATE_ACT_GELU_TANH)
                assert (out.cpu().double() - want).abs().max().item() <= tol * max(1.0, want.abs().max().item())
    gu = torch.randn((6, 128), generator=gen).to(torch.bfloat16)
    sumsq = torch.rand((6, 4), generator=gen) * 40
    f = 1.0 / torch.sqrt(sumsq.double().sum(1, keepdim=True) / 64 + 1e-5)
    y = gu.double() * f
    want = gelu(y.view(6, 8, 2, 8)[:, :, 0]) * y.view(6, 8, 2, 8)[:, :, 1]
    out = torch.zeros((6, 64), dtype=torch.bfloat16, device=DEV)
    K.swiglu(gu.to(DEV), out, 8, K.RowNorm(sumsq.to(DEV), 4, 1e-5), 64, act=K.GATE_ACT_GELU_TANH)
    assert (out.cpu().double() - want.reshape(6, 64)).abs().max().item() <= 8e-3 * max(1.0, want.abs().max().item())


@pytest.mark.parametrize("width", [64, 50, 4096, 9000])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_stream_joined_by_an_earlier_state_of_it(width, dtype):
    """The norm kernel adds none, one or two scaled outputs and the earlier stream, rewrites the stream and normalises it;
    other norms leave the addition to a kernel of its own."""
    from cpp_minilamma_b200.csrc import kernels as K
    from cpp_minilamma_b200.parts.base import BuildContext, PendingStream, PendingSum
    from cpp_minilamma_b200.parts.norm import LayerNorm, RMSNorm
    gen = torch.Generator(device="cpu").manual_seed(width)
    x, x0 = torch.randn((5, width), generator=gen), torch.randn((5, width), generator=gen)
    a, b = (torch.randn((5, width), generator=gen).to(dtype) for _ in range(2))
    w = 1 + 0.2 * torch.randn((width,), generator=gen)
    ctx = BuildContext(width, dtype, DEV, 16)
    norm = RMSNorm({"width": width, "eps": 1e-5, "name": "n"}, ctx)
    plain = LayerNorm({"width": width, "eps": 1e-5, "name": "n"}, ctx)
    norm.weight = plain.weight = w.to(DEV)
    state = make_step_state(DEV, [0], [0], [5])
    for pending, added in ((None, 0.0), (a.to(DEV), a.double()), (PendingSum(a.to(DEV), b.to(DEV), 0.7, 1.3), 0.7 * a.double() + 1.3 * b.double())):
        want = x.double() + added + x0.double()
        for part in (norm, plain):
            if part is plain and isinstance(pending, PendingSum):
                continue  # a layer norm adds its delta as it is
            stream = x.to(DEV).clone()
            got = part.forward(state, stream, PendingStream(pending, x0.to(DEV)))
            c = want - want.mean(1, keepdim=True) if part is plain else want
            out = c / (c.pow(2).mean(1, keepdim=True) + 1e-5).sqrt() * w.double()
            assert (stream.cpu().double() - want).abs().max().item() <= 1e-5
            assert (got.cpu().double() - out).abs().max().item() <= (1e-5 if dtype == torch.float32 else 8e-3) * out.abs().max().item()
            rows = _ints([3, 1])
            stream = x.to(DEV).clone()
            got = part.forward(state, stream, PendingStream(pending, x0.to(DEV)), rows=rows, out_name="gathered")
            assert (got.cpu().double() - out[[3, 1]]).abs().max().item() <= (1e-5 if dtype == torch.float32 else 8e-3) * out.abs().max().item()


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("width,first", [(64, 16), (50, 3), (5000, 8), (33, 0)])
def test_norm_of_a_row_of_heads_and_its_gate(dtype, width, first):
    from cpp_minilamma_b200.csrc import kernels as K
    gen = torch.Generator(device="cpu").manual_seed(width)
    o, w = torch.randn((9, width), generator=gen), 1 + 0.3 * torch.randn((width,), generator=gen)
    gate = torch.randn((9, first + width + (-(first + width) % 8)), generator=gen).to(dtype)
    z = gate[:, first:first + width].double()
    for act, f in ((K.GATE_SIGMOID, torch.sigmoid(z)), (K.GATE_SILU, z * torch.sigmoid(z))):
        want = o.double() / (o.double().pow(2).mean(1, keepdim=True) + 1e-5).sqrt() * w.double() * f
        out = torch.zeros((9, width), dtype=dtype, device=DEV)
        K.row_norm_gate(o.to(DEV), w.to(DEV), gate.to(DEV), out, 1e-5, act, gate_col=first)
        assert (out.cpu().double() - want).abs().max().item() <= (2e-6 if dtype == torch.float32 else 5e-3) * want.abs().max().item()


def test_capped_logits_and_product_biases():
    from cpp_minilamma_b200.csrc import kernels as K
    from cpp_minilamma_b200.parts.linear import Linear
    gen = torch.Generator(device="cpu").manual_seed(3)
    for n in (1, 7, 4096, 10001):
        x = 40 * torch.randn((n,), generator=gen)
        got = x.to(DEV).clone()
        K.softcap_(got, 30.0, 0.5)
        assert (got.cpu().double() - 30 * torch.tanh(0.5 * x.double() / 30)).abs().max().item() <= 1e-5
    for dtype in (torch.float32, torch.bfloat16):
        for rows, n, k in ((1, 64, 64), (6, 40, 96), (90, 64, 64), (90, 50, 40)):
            w, b = torch.randn((n, k), generator=gen).to(dtype), torch.randn((n,), generator=gen)
            x = torch.randn((rows, k), generator=gen).to(dtype)
            linear = Linear(w.to(DEV), "w", b.to(DEV))
            state = make_step_state(DEV, list(range(rows)), [0] * rows, [1] * rows, small_rows=64)
            got = linear.forward(state, x.to(DEV), "y").cpu().double()
            want = x.double() @ w.double().T + b.double()
            assert (got - want).abs().max().item() <= (1e-5 if dtype == torch.float32 else 1.2e-2) * want.abs().max().item()
