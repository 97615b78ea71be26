"""Mefolorn through the engine against the plain oracle (`plain_mefolorn`, float64, whole sequences), and its kernels
alone.

Every test makes its own small configuration and weights (`tiny_mefolorn`).  float32 runs must agree with the oracle to
2e-4 of the largest logit (at least 2e-4 absolute): with the test weights a sink left out, a window one token off, a lost
state, scores mixed by the transposed matrix or a bias forgotten moves logits by percents.  bfloat16 runs are compared
with the same unrounded oracle, so their bound is that of rounding noise: largest error at most 3 %, mean error at most
0.5 % of the largest logit.  The sharp test is float32."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import cpp_minilamma_b200 as ml
import plain_mefolorn as pm
import tiny_mefolorn as tm
from cpp_minilamma_b200.cache.paged import PAGE
from cpp_minilamma_b200.engine.step import StepEntry, make_step_state

pytestmark = pytest.mark.gpu
DEV = torch.device("cuda:0")

_FOLDERS, _ENGINES, _ORACLE = {}, {}, {}


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    def get(name, dtype="float32", max_tokens=1024, max_positions=None):
        if name not in _FOLDERS:
            _FOLDERS[name] = tm.make_folder(name if isinstance(name, str) else tm.random_config(name),
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
        _ORACLE[key] = pm.forward(cfg, W, toks)
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
    assert err.max() <= 3e-2 * scale and err.mean() <= 5e-3 * scale, \
        f"{what}: max {err.max():.3e} mean {err.mean():.3e} of {scale:.2f}, worst row {row}"


def run_alone(llm, toks, cuts):
    """Feed one sequence in portions of the given sizes (the rest one token at a time); logits of every position."""
    slot = llm.engine.acquire(1)[0]
    rows, at = [], 0
    for n in list(cuts) + [1] * (len(toks) - sum(cuts)):
        rows.append(llm.engine.step([StepEntry(slot, toks[at:at + n], list(range(n)))]).cpu().numpy())
        at += n
    llm.engine.release(slot)
    return np.concatenate(rows)


LENGTH = {"latent": 150, "talk": 150, "drift": 150, "mixed": 200, "ones": 140, "windows": 260, "tensor": 300, "heads": 130, "odd": 90}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(tm.CONFIGS))
def test_whole_prompt(models, name, dtype):
    """Every position of one prompt, the first tokens included (a state and convolution inputs that start at nothing,
    rows in which the sink is most of the denominator); prompts reach over windows and page borders."""
    llm, cfg, W = models(name, dtype)
    toks = tm.tokens(cfg, LENGTH[name], 11)
    close(run_alone(llm, toks, [len(toks)]), oracle(name, cfg, W, toks), dtype, f"{name} whole")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(tm.CONFIGS))
def test_prompt_then_token_by_token(models, name, dtype):
    """A short prompt, then a long run of single tokens through the cache and the state: windows and page borders pass
    over decoded tokens, the recurrent state and the convolution's inputs are carried step by step."""
    llm, cfg, W = models(name, dtype)
    toks = tm.tokens(cfg, LENGTH[name], 12)
    close(run_alone(llm, toks, [7]), oracle(name, cfg, W, toks), dtype, f"{name} decode")


@pytest.mark.parametrize("name", ["mixed", "ones"])
def test_token_by_token_from_the_first_token(models, name):
    llm, cfg, W = models(name, "float32")
    toks = tm.tokens(cfg, 70, 14)
    close(run_alone(llm, toks, []), oracle(name, cfg, W, toks), "float32", f"{name} from the first token")


@pytest.mark.parametrize("name,cuts", [
    ("mixed", [2, 3, 1, 7, 2, 49, 2, 2, 64]),      # portions down to two tokens, shorter than the convolutions
    ("ones", [1, 1, 62, 2, 66]),                   # single first tokens; a cut at the page's edge and after it
    ("latent", [8, 8, 7, 2, 39, 64]),              # portions that start just inside and just outside the window
    ("talk", [39, 2, 39, 1, 41]),
    ("drift", [2, 2, 63, 1, 2, 64, 3]),            # the state handed from portion to portion
    ("windows", [62, 2, 2, 60, 3, 64, 65]),
    ("heads", [5, 2, 45, 33]),
    ("odd", [5, 2, 2, 60]),
])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_portions(models, name, cuts, dtype):
    llm, cfg, W = models(name, dtype)
    toks = tm.tokens(cfg, LENGTH[name], 13)
    close(run_alone(llm, toks, cuts), oracle(name, cfg, W, toks), dtype, f"{name} portions {cuts}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["mixed", "windows", "tensor", "heads"])
def test_unequal_batch_then_decoding_together(models, name, dtype):
    """Requests of 1, 37 and 90 tokens start in one step, go on by one token each, and the short ones end early; every
    logit equals that of the request alone."""
    llm, cfg, W = models(name, dtype)
    eng = llm.engine
    seqs = [tm.tokens(cfg, n, 20 + i) for i, n in enumerate((9, 50, 104))]
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
        toks = tm.tokens(cfg, pages * PAGE + 90, seed)
        short = tm.tokens(cfg, 20, seed + 10)
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
    toks = tm.tokens(cfg, 150, 41)
    close(run_alone(llm, toks, [150]), oracle("mixed", cfg, W, toks), "float32", "engine-cut step")


@pytest.mark.parametrize("seed", range(12))
def test_drawn_configurations(models, seed):
    """Two to five layers of either kind in any order: a whole prompt, then two unequal requests decoded together."""
    for dtype in ("float32", "bfloat16"):
        llm, cfg, W = models(seed, dtype)
        toks = tm.tokens(cfg, 230, 5)
        close(run_alone(llm, toks, [230]), oracle(seed, cfg, W, toks), dtype, f"seed {seed} whole")
        a, b = toks[:80], tm.tokens(cfg, 30, 6)
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
        logits = pm.forward(cfg, W, toks)[-1]
        best = int(np.argmax(logits))
        sure.append(logits[best] - np.partition(logits, -2)[-2] > 1e-3)
        out.append(best)
        toks.append(best)
    return out, sure


@pytest.mark.parametrize("name", ["mixed", "odd"])
def test_greedy_generation_through_the_entry_point(models, name):
    """`generate` (the scheduler, captured decode steps, device sampling) picks the oracle's tokens."""
    llm, cfg, W = models(name, "float32")
    prompts = [tm.tokens(cfg, n, 50 + i) for i, n in enumerate((3, 21, 66))]
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
    prompts = [tm.tokens(cfg, n, 80 + i) for i, n in enumerate((5, 40))]
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
    prompt = tm.tokens(cfg, 5, 60)
    assert main(["generate", _FOLDERS["odd"][0], "-p", " ".join(map(str, prompt)), "-n", "6", "--dtype", "float32",
                 "--ignore-eos"]) == 0
    line = capsys.readouterr().out.splitlines()[0]
    want, sure = greedy_oracle(cfg, W, prompt, 6)
    upto = sure.index(False) if False in sure else len(sure)
    assert [int(t) for t in line.split()][:upto] == want[:upto]


def test_trace_replay_writes_the_wanted_logits(models, tmp_path):
    """The trace runner on a Mefolorn folder: two requests start together, decode, one ends early."""
    _, cfg, W = models("mixed", "float32")
    folder = _FOLDERS["mixed"][0]
    a, b = tm.tokens(cfg, 30, 70), tm.tokens(cfg, 70, 71)
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


def _mixed_reference(q, keys, values, pos0, scale, window, mix, bias, group):
    """q [n, H, d] at positions pos0 ..; keys [ctx, G, d], values [ctx, G, dv]."""
    n, H, _ = q.shape
    ctx = keys.shape[0]
    s = torch.stack([scale * q[:, h] @ keys[:, h // group].T for h in range(H)])  # [H, n, ctx]
    z = torch.einsum("hg,gij->hij", mix, s) + bias[:, None, None]
    i, j = pos0 + torch.arange(n)[:, None], torch.arange(ctx)[None, :]
    see = (j <= i) & ((j > i - window) if window else torch.ones_like(j, dtype=torch.bool))
    p = torch.where(see, torch.sigmoid(z), torch.zeros_like(z))
    return torch.stack([p[h] @ values[:, h // group] for h in range(H)], dim=1)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,d,dv,window", [
    (4, 2, 16, 16, 40), (8, 2, 64, 64, 70), (12, 4, 96, 80, 1), (6, 3, 24, 40, 63), (16, 4, 128, 128, 100), (3, 3, 32, 8, 65),
    (32, 8, 128, 128, 90), (24, 3, 16, 72, 0), (40, 5, 8, 16, 128), (5, 1, 6, 10, 33), (12, 1, 256, 256, 50), (1, 1, 8, 8, 17),
    (64, 8, 64, 64, 45)])
def test_mixed_attention_kernels(dtype, H, G, d, dv, window):
    """The general kernel (both dtypes), the tensor-core prompt kernel and the single-token kernel (one block a
    sequence, context split in 2 and in 7) against scores, mixing and sigmoid written out.  In every sequence the key
    just inside the last query's window and the one just outside it are scaled so that they stand out; the matrix is far
    from symmetric; a page that is not the sequence's, or rows past its end, hold no numbers."""
    from cpp_minilamma_b200.csrc import kernels as K
    gen = torch.Generator(device="cpu").manual_seed(d * 1000 + H)
    starts, lens = [0, 70, 300, 0], [150, 61, 1, 3]
    ctxs = [s + n for s, n in zip(starts, lens)]
    k_cache, v_cache, table = _paged(gen, ctxs, G, d, dv, dtype)
    T, group, scale = sum(lens), H // G, 1.2 / d ** 0.5
    q = torch.randn((T, H * d), generator=gen).to(dtype)
    mix = (0.6 * torch.eye(H) + (torch.randn((H, H), generator=gen) / H ** 0.5 if H > 1 else 0.5)).contiguous()
    if G % 2:  # half of the cases: entries that are bfloat16 numbers
        mix = mix.to(torch.bfloat16).float()
    bias = torch.linspace(-4.0, 1.0, H)
    for s in range(4):
        for edge in ((ctxs[s] - window, ctxs[s] - window - 1) if window else (0, 1)):
            if 0 <= edge < ctxs[s]:
                page, at = int(table[s, edge // PAGE]), edge % PAGE
                last_q = q[sum(lens[:s + 1]) - 1].float().view(G, group, d).mean(dim=1)
                k_cache[page, :, at] = (6.0 * last_q / last_q.norm(dim=1, keepdim=True)).to(dtype)
                v_cache[page, :, at] = (v_cache[page, :, at].float() * 4).to(dtype)
    refs = {}
    for w in {window, window + 1, max(window - 1, 1)} if window else {0}:
        parts = []
        for s in range(4):
            rows = slice(sum(lens[:s]), sum(lens[:s + 1]))
            parts.append(_mixed_reference(q[rows].double().view(-1, H, d), _dense(k_cache, table, s, ctxs[s]),
                                          _dense(v_cache, table, s, ctxs[s]), starts[s], scale, w, mix.double(),
                                          bias.double(), group))
        refs[w] = torch.cat(parts).view(T, H * dv)
    want = refs[window]
    size = max(1.0, want.abs().max().item())
    tol = (3e-5 if dtype == torch.float32 else 1.5e-2) * size
    last = [sum(lens[:i + 1]) - 1 for i in range(4)]
    if window:  # one key more or one less is well above the tolerance, in the prompts and in the last rows alone
        assert all((r - want)[last].abs().max().item() > 4 * tol for w, r in refs.items() if w != window)
    state = make_step_state(DEV, [0, 1, 2, 3], starts, lens)
    kc, vc, table_dev, qd, md, bd = (t.to(DEV) for t in (k_cache, v_cache, table, q, mix, bias))
    out = torch.zeros((T, H * dv), dtype=dtype, device=DEV)
    K.mixed_attention(qd, kc, vc, state.tok_pos, state.tok_seq, state.seq_slot, table_dev, md, bd, out, H, G, d, dv, window, scale)
    assert (out.cpu().double() - want).abs().max().item() <= tol, "general kernel"
    if K.mixed_attention_mma_supported(dtype, False, H, G, d, dv):
        tile_seq = [s for s, n in enumerate(lens) for _ in range(0, n, 2 * K.PREFILL_TILE)]
        tile_row0 = [r for n in lens for r in range(0, n, 2 * K.PREFILL_TILE)]
        for splits in (1, 2, 4, 8):  # blocks that share a tile's keys, many of them with none
            out = torch.zeros((T, H * dv), dtype=dtype, device=DEV)
            K.mixed_attention_tiles(qd, kc, vc, state.seq_slot, state.seq_ctx, state.seq_qstart, state.seq_qlen, _ints(tile_seq),
                                    _ints(tile_row0), table_dev, md, bd, out, H, G, d, dv, window, scale, n_splits=splits, narrow_mix=bool(G % 2))
            err = (out.cpu().double() - want).abs()
            assert err.max().item() <= tol, ("prompt kernel", splits, err.max().item(), tol, int(err.max(dim=1).values.argmax()))
    if K.mixed_attention_mma_supported(dtype, True, H, G, d, dv):
        one = make_step_state(DEV, [0, 1, 2, 3], [c - 1 for c in ctxs], [1] * 4)
        for splits in (1, 2, 7):
            out = torch.zeros((4, H * dv), dtype=dtype, device=DEV)
            scratch = torch.full((K.mixed_attention_single_scratch(4, H, dv, splits),), float("nan"), device=DEV)
            K.mixed_attention_single(qd[last].contiguous(), kc, vc, one.seq_slot, one.seq_ctx, one.seq_qstart, one.seq_qlen,
                                     table_dev, md, bd, out, 4, H, G, d, dv, window, scale, n_splits=splits, scratch=scratch)
            err = (out.cpu().double() - want[last]).abs().max().item()
            assert err <= tol, ("single tokens", splits, err, tol)


def test_mixed_scores_keep_float32(models):
    """Scores in the hundreds that cancel in the mixing (rows of M that add up to nothing over pairs of nearly equal heads):
    the mixed score is a small difference of large ones, which scores or a matrix rounded to bfloat16 would lose."""
    from cpp_minilamma_b200.csrc import kernels as K
    gen = torch.Generator(device="cpu").manual_seed(9)
    H, G, d, dv, T = 16, 4, 64, 64, 96
    k_cache, v_cache, table = _paged(gen, [T], G, d, dv, torch.bfloat16)
    base = torch.randn((T, H // 2, 1, d), generator=gen) * 8
    q = torch.cat([base, base], dim=2).reshape(T, H * d).to(torch.bfloat16)   # heads 2i and 2i + 1 are the same ...
    q[:, d::2 * d] += 0.25                                                    # ... but for one dimension
    mix = torch.zeros((H, H))
    for h in range(0, H, 2):
        mix[h, h], mix[h, h + 1], mix[h + 1, h], mix[h + 1, h + 1] = 1.37, -1.37, -0.913, 0.913
    want = _mixed_reference(q.double().view(-1, H, d), _dense(k_cache, table, 0, T), _dense(v_cache, table, 0, T), 0, 1.0, 40,
                            mix.double(), torch.zeros(H).double(), H // G).view(T, H * dv)
    state = make_step_state(DEV, [0], [0], [T])
    out = torch.zeros((T, H * dv), dtype=torch.bfloat16, device=DEV)
    K.mixed_attention_tiles(q.to(DEV), k_cache.to(DEV), v_cache.to(DEV), state.seq_slot, state.seq_ctx, state.seq_qstart,
                            state.seq_qlen, _ints([0]), _ints([0]), table.to(DEV), mix.to(DEV), None, out, H, G, d, dv, 40, 1.0)
    assert (out.cpu().double() - want).abs().max().item() <= 1.5e-2 * want.abs().max().item()


def test_mixing_matrix_of_float32_values(models, tmp_path):
    """A folder whose mixing matrix is stored in float32 with values bfloat16 does not have: it is not rounded."""
    import struct
    folder, cfg, W = tm.make_folder("talk", tmp_path / "m", seed=3)
    blob = (tmp_path / "m" / "model.safetensors").read_bytes()
    n, = struct.unpack("<Q", blob[:8])
    header, data = json.loads(blob[8:8 + n]), blob[8 + n:]
    values = (W["l0.mix.left.talk"] + 0.013 * np.arange(36).reshape(6, 6)).astype("<f4")
    header["l0.mix.left.talk"] = {"dtype": "F32", "shape": [6, 6], "data_offsets": [len(data), len(data) + values.nbytes]}
    # the old bytes stay behind as another tensor's: drop them by writing the file anew
    order, parts, at = {}, [], 0
    for name, info in header.items():
        lo, hi = info["data_offsets"]
        raw = values.tobytes() if info["dtype"] == "F32" else data[lo:hi]
        order[name] = dict(info, data_offsets=[at, at + len(raw)])
        parts.append(raw)
        at += len(raw)
    text = json.dumps(order).encode()
    (tmp_path / "m" / "model.safetensors").write_bytes(struct.pack("<Q", len(text)) + text + b"".join(parts))
    cfg, W = pm.read_folder(tmp_path / "m")
    toks = tm.tokens(cfg, 80, 4)
    for dtype in ("float32", "bfloat16"):
        llm = ml.load(folder, dtype=dtype, max_tokens=256, max_positions=256)
        assert not llm.model.layers[0].mixer.left.mix_narrow
        close(run_alone(llm, toks, [70]), pm.forward(cfg, W, toks), dtype, f"float32 matrix, {dtype}")


def test_mixed_attention_without_matrix_or_bias():
    from cpp_minilamma_b200.csrc import kernels as K
    gen = torch.Generator(device="cpu").manual_seed(5)
    H, G, d, dv, window, ctxs = 6, 2, 32, 16, 20, [50]
    k_cache, v_cache, table = _paged(gen, ctxs, G, d, dv, torch.bfloat16)
    q = torch.randn((50, H * d), generator=gen).to(torch.bfloat16)
    want = _mixed_reference(q.double().view(-1, H, d), _dense(k_cache, table, 0, 50), _dense(v_cache, table, 0, 50), 0, 0.3,
                            window, torch.eye(H).double(), torch.zeros(H).double(), H // G).view(50, H * dv)
    state = make_step_state(DEV, [0], [0], [50])
    qd, kc, vc, td = (t.to(DEV) for t in (q, k_cache, v_cache, table))
    for kind in ("general", "tiles"):
        out = torch.zeros((50, H * dv), dtype=torch.bfloat16, device=DEV)
        if kind == "general":
            K.mixed_attention(qd, kc, vc, state.tok_pos, state.tok_seq, state.seq_slot, td, None, None, out, H, G, d, dv, window, 0.3)
        else:
            K.mixed_attention_tiles(qd, kc, vc, state.seq_slot, state.seq_ctx, state.seq_qstart, state.seq_qlen, _ints([0]),
                                    _ints([0]), td, None, None, out, H, G, d, dv, window, 0.3)
        assert (out.cpu().double() - want).abs().max().item() <= 1.5e-2 * max(1.0, want.abs().max().item()), kind


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("W,n,taps", [(40, 2, 4), (144, 2, 3), (24, 24, 3), (30, 3, 1), (256, 1, 2), (200, 5, 5), (1024, 4, 4), (1, 1, 4)])
def test_linear_recurrent_unit_kernels(dtype, W, n, taps):
    """Gates, convolution state and scan against the recurrence walked token by token in float64: sequences of 150, 2, 1
    and 37 tokens, three of which go on from a state and convolution inputs that are not zero; portions shorter than
    the convolution; decays from almost none to at once.  Then a step of single tokens, which advances the state in
    the gates' kernel.  In bfloat16 the gates' products must be those of the float32 inputs: their error stays far below
    what rounding the convolution's result to bfloat16 would do."""
    from cpp_minilamma_b200.csrc import kernels as K
    gen = torch.Generator().manual_seed(W + n)
    bs = W // n
    rnd = lambda *shape: torch.randn(shape, generator=gen)
    ra, ri = (rnd(n, bs, bs) * 1.5 / bs ** 0.5).to(dtype), (rnd(n, bs, bs) * 1.5 / bs ** 0.5).to(dtype)
    conv_w, conv_b, xb, yb, gb, lam = rnd(W, taps) * 0.6, rnd(W) * 0.3, rnd(W) * 0.3, rnd(W) * 0.3, rnd(2, W) * 0.4, rnd(W) * 3 - 3
    rates = (8.0 * torch.nn.functional.softplus(lam.double(), threshold=40)).float()
    S0, C0 = rnd(7, W), rnd(7, taps - 1, W)
    S0[2], C0[2] = 0.0, 0.0
    mma = dtype == torch.bfloat16 and K.lru_mma_supported(dtype, bs)
    weights = [torch.cat([ra.float(), ri.float()], dim=1).transpose(1, 2).contiguous()]
    if mma:
        weights.append(torch.stack([ra, ri], dim=1).contiguous())
    sigm = torch.sigmoid
    for gate_w in weights:
        S_dev, C_dev = S0.to(DEV), C0.to(DEV)
        S, C = S0.double().clone(), C0.double().clone()
        for starts, lens, slots in (([0, 9, 20, 5], [150, 2, 1, 37], [2, 0, 3, 5]), ([150, 11, 21, 42], [1, 1, 1, 1], [2, 0, 3, 5])):
            T = sum(lens)
            proj = rnd(T, 2 * W + 3).to(dtype)
            if dtype == torch.bfloat16:
                proj = torch.cat([proj, torch.zeros(T, (-proj.shape[1]) % 8, dtype=dtype)], dim=1).contiguous()
            st = make_step_state(DEV, slots, starts, lens)
            pd = proj.to(DEV)
            consts = (xb.to(DEV), yb.to(DEV), conv_w.to(DEV), conv_b.to(DEV), C_dev, gate_w.to(DEV), gb.to(DEV), rates.to(DEV), S_dev,
                      st.tok_pos, st.tok_seq, st.seq_slot, st.seq_qstart, n)
            out = torch.zeros((T, W), dtype=dtype, device=DEV)
            single = max(lens) == 1
            decay, write = torch.zeros((T, W), device=DEV), torch.zeros((T, W), device=DEV)
            if single:
                K.lru_gates(pd, W, 0, *consts, out=out)
            else:
                K.lru_gates(pd, W, 0, *consts, decay=decay, write=write)
            if taps > 1:
                K.conv_state_update(pd, C_dev, st.seq_slot, st.seq_qstart, st.seq_qlen, 4, W, taps, first_column=W)
            if not single:
                K.lru_scan(decay, write, pd, 0, yb.to(DEV), S_dev, out, st.seq_slot, st.seq_qstart, st.seq_qlen, 4, max(lens))
            torch.cuda.synchronize()
            P, at = proj.double(), 0
            for slot, start, m in zip(slots, starts, lens):
                inputs = torch.cat([C[slot], P[at:at + m, W:2 * W]])  # [taps - 1 + m, W]
                for i in range(m):
                    u = conv_b.double().clone()
                    for back in range(taps):
                        if start + i - back >= 0:
                            u += conv_w[:, taps - 1 - back].double() * (inputs[taps - 1 + i - back] + xb.double())
                    blocks = u.view(n, bs)
                    r = sigm(torch.einsum("noi,ni->no", ra.double(), blocks).reshape(W) + gb[0].double())
                    g = sigm(torch.einsum("noi,ni->no", ri.double(), blocks).reshape(W) + gb[1].double())
                    log_a = -8.0 * r * torch.nn.functional.softplus(lam.double(), threshold=40)
                    a, w = torch.exp(log_a), torch.sqrt(-torch.expm1(2 * log_a)) * g * u
                    S[slot] = a * S[slot] + w
                    t = at + i
                    if not single:
                        assert (decay[t].cpu().double() - a).abs().max().item() < 3e-6, (slot, i)
                        assert (write[t].cpu().double() - w).abs().max().item() < 1e-5 * max(1.0, w.abs().max().item()), (slot, i)
                    y = torch.nn.functional.gelu(P[t, :W] + yb.double(), approximate="tanh")
                    tol = 3e-5 if dtype == torch.float32 else 8e-3
                    assert (out[t].cpu().double() - S[slot] * y).abs().max().item() <= tol * max(1.0, (S[slot] * y).abs().max().item()), (slot, i)
                assert (S_dev[slot].cpu().double() - S[slot]).abs().max().item() <= 3e-5 * max(1.0, S[slot].abs().max().item()), slot
                C[slot] = inputs[len(inputs) - (taps - 1):]
                assert torch.equal(C_dev[slot].cpu().double(), C[slot])
                at += m
        for other in (1, 4, 6):
            assert torch.equal(S_dev[other].cpu(), S0[other]) and torch.equal(C_dev[other].cpu(), C0[other])


@pytest.mark.parametrize("length", [1, 7, 8, 16, 17, 31, 500, 2049])
def test_linear_recurrent_scan_runs(length):
    """The scan at lengths around its runs' borders, beside a sequence of another length: every run's carry."""
    from cpp_minilamma_b200.csrc import kernels as K
    gen = torch.Generator().manual_seed(length)
    W, lens, slots = 50, [length, 3], [1, 0]
    T = sum(lens)
    decay, write = torch.rand((T, W), generator=gen) ** 0.1, torch.randn((T, W), generator=gen)
    proj, yb, S0 = torch.randn((T, W), generator=gen), torch.randn(W, generator=gen), torch.randn((2, W), generator=gen)
    st = make_step_state(DEV, slots, [4, 9], lens)
    S_dev, out = S0.to(DEV), torch.zeros((T, W), device=DEV)
    K.lru_scan(decay.to(DEV), write.to(DEV), proj.to(DEV), 0, yb.to(DEV), S_dev, out, st.seq_slot, st.seq_qstart, st.seq_qlen, 2, max(lens))
    at = 0
    for slot, m in zip(slots, lens):
        S = S0[slot].double()
        for t in range(at, at + m):
            S = decay[t].double() * S + write[t].double()
            want = S * torch.nn.functional.gelu(proj[t].double() + yb.double(), approximate="tanh")
            assert (out[t].cpu().double() - want).abs().max().item() < 3e-5 * max(1.0, want.abs().max().item()), (slot, t - at)
        assert (S_dev[slot].cpu().double() - S).abs().max().item() < 3e-5 * max(1.0, S.abs().max().item())
        at += m


@pytest.mark.parametrize("width", [40, 50, 1000, 4096])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_tanh_norm_kernel(width, dtype):
    """x += c1 d1 + c2 d2 + c3 d3, then none, one or two norms of the sum; gathered rows leave the stream alone."""
    from cpp_minilamma_b200.csrc import kernels as K
    gen = torch.Generator().manual_seed(width)
    x0 = torch.randn((9, width), generator=gen) * 3
    deltas = [((torch.randn((9, width), generator=gen) * 2).to(dtype), c) for c in (1.2, 0.5, 1.0)]
    forms = [(torch.tensor([0.3 + 0.4 * i]), 1 + 0.3 * torch.randn(width, generator=gen), torch.randn(width, generator=gen)) for i in range(2)]
    for n_deltas in (0, 1, 2, 3):
        for n_norms in (0, 1, 2):
            for rows in (None, [8, 0, 3]):
                if n_norms == 0 and (rows or not n_deltas):
                    continue
                summed = x0.double() + sum((c * d.double() for d, c in deltas[:n_deltas]), torch.zeros(1).double())
                x = x0.to(DEV)
                outs = [torch.zeros((len(rows) if rows else 9, width), dtype=dtype, device=DEV) for _ in range(n_norms)]
                K.add_dynamic_tanh(x, [(d.to(DEV), c) for d, c in deltas[:n_deltas]],
                                   [K.TanhNorm(a.to(DEV), w.to(DEV), b.to(DEV), o) for (a, w, b), o in zip(forms, outs)],
                                   _ints(rows) if rows else None)
                if rows:
                    assert torch.equal(x.cpu(), x0)
                else:
                    assert (x.cpu().double() - summed).abs().max().item() < 1e-5
                for (a, w, b), o in zip(forms, outs):
                    want = torch.tanh(a.double() * summed) * w.double() + b.double()
                    want = want[rows] if rows else want
                    # float32 arithmetic, then half a unit in the last of bfloat16's eight bits
                    assert ((o.cpu().double() - want).abs() <= 1e-5 + (0.0 if dtype == torch.float32 else 2.0 ** -8) * want.abs()).all()


def test_other_norms_behind_three_outputs():
    """A block whose outputs are three tensors in front of an RMS norm or a layer norm: all of them join the stream."""
    from cpp_minilamma_b200.parts.base import BuildContext, PendingSum, WeightStore
    from cpp_minilamma_b200.parts.norm import LayerNorm, RMSNorm
    gen = torch.Generator().manual_seed(1)
    ctx = BuildContext(24, torch.float32, DEV, 64)
    first, second, third = (torch.randn((5, 24), generator=gen).to(DEV) for _ in range(3))
    x0 = torch.randn((5, 24), generator=gen).to(DEV)
    state = make_step_state(DEV, [0], [0], [5])
    summed = (x0 + first + second + third).double()
    rms = RMSNorm({"width": 24, "eps": 1e-6, "name": "w"}, ctx)
    rms.bind(WeightStore({"w": torch.ones(24, device=DEV)}))
    x = x0.clone()
    got = rms.forward(state, x, PendingSum(first, second, third=third))
    assert (x.double() - summed).abs().max().item() < 1e-5
    assert (got.double() - summed / torch.sqrt((summed ** 2).mean(dim=1, keepdim=True) + 1e-6)).abs().max().item() < 1e-5
    layer = LayerNorm({"width": 24, "eps": 1e-6, "name": "w", "bias": None}, ctx)
    layer.bind(WeightStore({"w": torch.ones(24, device=DEV)}))
    x = x0.clone()
    got = layer.forward(state, x, PendingSum(first, second, third=third))
    c = summed - summed.mean(dim=1, keepdim=True)
    assert (got.double() - c / torch.sqrt((c ** 2).mean(dim=1, keepdim=True) + 1e-6)).abs().max().item() < 1e-5


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,rank,window", [(8, 64, 40), (5, 136, 64), (3, 20, 33), (70, 48, 100)])
def test_latent_rows_under_a_window_and_a_sink(dtype, H, rank, window):
    """The attention kernels over one latent row per position (values are the keys' leading columns) with a window and a
    sink per head, the keys just inside and outside the last query's window standing out: general kernel, prompt tiles,
    single tokens in one, three and sixteen context splits (the sink counts once)."""
    from cpp_minilamma_b200.csrc import kernels as K
    gen = torch.Generator(device="cpu").manual_seed(rank + H)
    starts, lens = [0, 70, 300], [150, 61, 1]
    ctxs = [s + n for s, n in zip(starts, lens)]
    cache, _, table = _paged(gen, ctxs, 1, rank, rank, dtype)
    T, scale = sum(lens), 0.5 / rank ** 0.5
    q = torch.randn((T, H * rank), generator=gen).to(dtype)
    for s in range(3):
        for edge in (ctxs[s] - window, ctxs[s] - window - 1):
            page, at = int(table[s, edge // PAGE]), edge % PAGE
            cache[page, 0, at] = (8.0 * q[sum(lens[:s + 1]) - 1].float().view(H, rank).mean(dim=0)).to(dtype)
    sinks = torch.linspace(-3.0, 4.0, H)
    want = []
    for s in range(3):
        keys = _dense(cache, table, s, ctxs[s])[:, 0]
        rows = q[sum(lens[:s]):sum(lens[:s + 1])].double().view(-1, H, rank)
        i, j = starts[s] + torch.arange(lens[s])[:, None], torch.arange(ctxs[s])[None, :]
        see = (j <= i) & (j > i - window)
        sc = torch.where(see[:, None], torch.einsum("nhd,jd->nhj", rows, keys) * scale, torch.tensor(-1e30).double())
        e = torch.exp(sc) * see[:, None]
        want.append(torch.einsum("nhj,jd->nhd", e / (e.sum(dim=2, keepdim=True) + torch.exp(sinks.double())[None, :, None]), keys))
    want = torch.cat(want).reshape(T, H * rank)
    size = max(1.0, want.abs().max().item())
    state = make_step_state(DEV, [0, 1, 2], starts, lens)
    qd, kc, td, sd = (t.to(DEV) for t in (q, cache, table, sinks))
    kw = dict(sink=True, sink_values=sd, v_in_k=True)
    out = torch.zeros((T, H * rank), dtype=dtype, device=DEV)
    K.local_attention(qd, kc, kc, state.tok_pos, state.tok_seq, state.seq_slot, td, out, H, 1, rank, rank, 0, window, scale, **kw)
    tol = (3e-5 if dtype == torch.float32 else 2e-2) * size
    assert (out.cpu().double() - want).abs().max().item() <= tol
    if not K.local_attention_mma_supported(dtype, rank, rank):
        return
    tile_seq = [s for s, n in enumerate(lens) for _ in range(0, n, K.PREFILL_TILE)]
    tile_row0 = [r for n in lens for r in range(0, n, K.PREFILL_TILE)]
    out.zero_()
    K.local_attention_tiles(qd, kc, kc, state.seq_slot, state.seq_ctx, state.seq_qstart, state.seq_qlen, _ints(tile_seq),
                            _ints(tile_row0), td, out, H, 1, rank, rank, 0, window, scale, **kw)
    assert (out.cpu().double() - want).abs().max().item() <= tol
    last = [sum(lens[:i + 1]) - 1 for i in range(3)]
    one = make_step_state(DEV, [0, 1, 2], [c - 1 for c in ctxs], [1, 1, 1])
    for splits in (1, 3, 16):
        single = torch.zeros((3, H * rank), dtype=dtype, device=DEV)
        scratch = torch.full((K.local_attention_heads_scratch(3, H, rank, splits),), float("nan"), device=DEV)
        K.local_attention_heads(qd[last].contiguous(), kc, kc, one.seq_slot, one.seq_ctx, one.seq_qstart, one.seq_qlen, td,
                                single, 3, H, 1, rank, rank, 0, window, scale, n_splits=splits,
                                scratch=scratch if splits > 1 else None, **kw)
        assert (single.cpu().double() - want[last]).abs().max().item() <= tol, splits
