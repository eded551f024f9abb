"""The Fabezen decoder against the plain statement of the design (oracle/fabezen.py): whole prompts, portions, token by token,
slots that are used again, long decoding, batches, and generation through the framework's loop."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

from nn_b200 import native as N
from nn_b200.blocks import bf16_bits, f32
from nn_b200.fabezen import Fabezen, FabezenConfig
from nn_b200.registry import load_model
from nn_b200.weights import write_safetensors
from oracle import fabezen as F
from tests.fabezen_models import CONFIGS, channel, config, delta, latent, weights_for, wide64

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
TOL = {N.NS_F32: 6e-5, N.NS_BF16: 0.06}
_cache = {}


def case(name, T=150, seed=3):
    """(config dict, weights, tokens, oracle logits), made once."""
    if (name, T) not in _cache:
        cfg = CONFIGS[name]
        w = weights_for(cfg, seed)
        tokens = np.random.default_rng([seed, T]).integers(0, cfg["vocab"], T)
        _cache[name, T] = (cfg, w, tokens, F.forward(tokens, wide64(w), cfg))
    return _cache[name, T]


def make(dev, cfg, w, dtype, **kw):
    return Fabezen(dev, FabezenConfig.from_dict(cfg), w, dtype=dtype, **kw)


def worst(got, want):
    d = got - want
    d = d - d.mean(-1, keepdims=True)
    return float(np.sqrt((d ** 2).mean(-1)).max() / np.sqrt(np.mean((want - want.mean(-1, keepdims=True)) ** 2)))


def fed(model, tokens, cuts, slot=None):
    s = model.open_sequence() if slot is None else slot
    out, at = [], 0
    for n in cuts:
        out.append(model.feed([s], tokens[None, at:at + n], range(n)))
        at += n
    assert at == len(tokens)
    model.close_sequence(s)
    return np.concatenate(out)


@pytest.mark.parametrize("dtype", [N.NS_F32, N.NS_BF16])
@pytest.mark.parametrize("name", list(CONFIGS))
def test_whole_prompt(dev, name, dtype):
    cfg, w, tokens, want = case(name)
    model = make(dev, cfg, w, dtype, max_prefill=len(tokens))
    assert worst(fed(model, tokens, [len(tokens)]), want) < TOL[dtype]
    model.close()


def cuts_of(kind, T):
    if kind == "single":
        return [1] * T
    if kind == "pairs":
        return [2] * (T // 2) + [1] * (T % 2)
    sizes, out, rng = [1, 2, 3, 5, 16, 31, 32, 33, 47, 64, 65], [], np.random.default_rng(T)
    while sum(out) < T:
        out.append(min(int(rng.choice(sizes)), T - sum(out)))
    return out


@pytest.mark.parametrize("dtype", [N.NS_F32, N.NS_BF16])
@pytest.mark.parametrize("kind", ["single", "pairs", "mixed"])
@pytest.mark.parametrize("name", list(CONFIGS))
def test_portions(dev, name, kind, dtype):
    cfg, w, tokens, want = case(name)
    model = make(dev, cfg, w, dtype, max_prefill=70)
    assert worst(fed(model, tokens, cuts_of(kind, len(tokens))), want) < TOL[dtype]
    model.close()


@pytest.mark.parametrize("max_prefill", [1, 7, 64])
def test_prompts_longer_than_a_pass(dev, max_prefill):
    cfg, w, tokens, want = case("mixed")
    model = make(dev, cfg, w, N.NS_F32, max_prefill=max_prefill)
    assert worst(fed(model, tokens, [130, 20]), want) < TOL[N.NS_F32]
    model.close()


def test_slots_are_used_again_and_do_not_mix(dev):
    cfg, w, tokens, want = case("mixed")
    other = (tokens * 7 + 3) % cfg["vocab"]
    want_other = F.forward(other, wide64(w), cfg)
    model = make(dev, cfg, w, N.NS_F32, max_prefill=40, slots=3)
    for round_ in range(3):
        # two sequences take turns, a third opens and closes between them
        a, b = model.open_sequence(), model.open_sequence()
        ga, gb = [], []
        for at in range(0, 150, 30):
            ga.append(model.feed([a], tokens[None, at:at + 30], range(30)))
            c = model.open_sequence()
            model.feed([c], other[None, :17])
            model.close_sequence(c)
            gb.append(model.feed([b], other[None, at:at + 30], range(30)))
        assert worst(np.concatenate(ga), want) < TOL[N.NS_F32] and worst(np.concatenate(gb), want_other) < TOL[N.NS_F32]
        for s in ((a, b) if round_ % 2 else (b, a)):
            model.close_sequence(s)
    with pytest.raises(RuntimeError):
        for _ in range(4):
            model.open_sequence()
    model.close()


@pytest.mark.parametrize("dtype", [N.NS_F32, N.NS_BF16])
def test_unequal_sequences_in_one_pass(dev, dtype):
    """Sequences at different positions step together."""
    cfg, w, tokens, want = case("mixed")
    model = make(dev, cfg, w, dtype, batch=3, max_prefill=64, slots=4)
    starts, slots = [0, 13, 64], [model.open_sequence() for _ in range(3)]
    for s, n in zip(slots, starts):
        if n:
            model.feed([s], tokens[None, :n])
    got = [[] for _ in slots]
    at = 0
    for n in (1, 1, 2, 40, 1, 5):
        ids = np.stack([tokens[p + at:p + at + n] for p in starts])
        logits = model.feed(slots, ids, [(b, i) for b in range(3) for i in range(n)]).reshape(3, n, -1)
        for b in range(3):
            got[b].append(logits[b])
        at += n
    for b, p in enumerate(starts):
        assert worst(np.concatenate(got[b]), want[p:p + at]) < TOL[dtype], b
    model.close()


@pytest.mark.parametrize("dtype", [N.NS_F32, N.NS_BF16])
def test_long_decoding_wraps_every_ring(dev, dtype):
    cfg, w, tokens, want = case("mixed", T=700)
    model = make(dev, cfg, w, dtype, max_prefill=5)
    assert worst(fed(model, tokens, [5] + [1] * 695), want) < TOL[dtype]
    model.close()


@pytest.mark.parametrize("dtype", [N.NS_F32, N.NS_BF16])
@pytest.mark.parametrize("T", [1, 2, 3, 4])
def test_first_tokens(dev, T, dtype):
    cfg, w, tokens, want = case("mixed")
    model = make(dev, cfg, w, dtype, max_prefill=8)
    assert worst(fed(model, tokens[:T], [T]), want[:T]) < TOL[dtype]
    model.close()


@pytest.mark.parametrize("size", [1, 2, 40, 63, 64, 65, 90])
def test_window_edges_in_prompts_and_decoding(dev, size):
    """Attention sharp enough that a window one token off changes the logits by more than the tolerance (checked on the oracle)."""
    cfg = config([latent(heads=16, dim=16, rot_dim=2, vdim=32, q_rank=32, kv_rank=32, size=size, base=1e9, scale=1.0, ff=None)], vocab=220, width=32, scale=1.0,
                 bigram=False, mult=1.0)
    w = weights_for(cfg, 5)
    w["l0.mix.uk"] = bf16_bits(f32(w["l0.mix.uk"]) * 2.5)
    tokens = np.random.default_rng(8).permutation(220)[:200]            # no token twice: a key has no twin inside the window
    want = F.forward(tokens, wide64(w), cfg)
    tol = {N.NS_F32: TOL[N.NS_F32], N.NS_BF16: 0.12}
    for off in (-1, 1):
        if size + off > 0:
            near = json.loads(json.dumps(cfg))
            near["layers"][0]["mixer"]["mask"]["size"] += off
            assert worst(F.forward(tokens, wide64(w), near), want) > 2 * tol[N.NS_BF16]
    for dtype in (N.NS_F32, N.NS_BF16):
        model = make(dev, cfg, w, dtype, max_prefill=200)
        for cuts in ([200], [15] + [1] * 185, [30, 2, 100, 68]):
            assert worst(fed(model, tokens, cuts), want) < tol[dtype], (dtype, cuts)
        model.close()


def greedy_check(tokens, prompt, w, cfg, tol):
    """Every generated token is a maximum of the oracle's logits after what came before it, up to tol."""
    w = wide64(w)
    for b in range(len(prompt)):
        logits = F.forward(np.concatenate([prompt[b], tokens[b][:-1]]), w, cfg)[len(prompt[b]) - 1:]
        for t, row in zip(tokens[b], logits):
            assert row.max() - row[t] <= tol * np.sqrt(np.var(row))


@pytest.mark.parametrize("dtype,tol", [(N.NS_F32, 1e-3), (N.NS_BF16, 0.5)])
def test_greedy_generation(dev, dtype, tol):
    cfg, w, _, _ = case("mixed")
    prompt = np.random.default_rng(9).integers(0, cfg["vocab"], (3, 37))
    model = make(dev, cfg, w, dtype, batch=3, max_prefill=16)
    tokens, resets = model.generate(prompt, 30)
    assert resets == 0 and tokens.shape == (3, 30) and model.launches_per_step > 0
    greedy_check(tokens, prompt, w, cfg, tol)
    again, _ = model.generate(prompt, 30)                        # the recorded step, other slots' worth of history behind it
    assert np.array_equal(tokens, again)
    plain, _ = model.generate(prompt, 30, use_graph=False)
    assert np.array_equal(tokens, plain)
    model.close()
    one = make(dev, cfg, w, dtype, batch=1, max_prefill=64)
    alone, _ = one.generate(prompt[1:2], 30)
    greedy_check(alone, prompt[1:2], w, cfg, tol)
    if dtype == N.NS_F32:
        assert np.array_equal(alone[0], tokens[1])
    one.close()


def test_generation_with_a_sampler(dev):
    from nn_b200.backend import NsB200Backend
    from nn_b200.sampling import TokenSampler

    cfg, w, _, _ = case("mixed")
    prompt = np.random.default_rng(10).integers(0, cfg["vocab"], (2, 9))
    model = make(dev, cfg, w, N.NS_F32, batch=2, max_prefill=16)
    greedy, _ = model.generate(prompt, 12)
    s = TokenSampler(NsB200Backend(dev), 2, cfg["vocab"], 64)
    s.TopK = 1
    model.set_sampler(s)
    tokens, _ = model.generate(prompt, 12)
    assert np.array_equal(tokens, greedy)
    s2 = TokenSampler(NsB200Backend(dev), 2, cfg["vocab"], 64)
    s2.Temperature, s2.Seed = 1.5, 4
    model.set_sampler(s2)
    free, _ = model.generate(prompt, 12)
    assert not np.array_equal(free, greedy) and free.min() >= 0 and free.max() < cfg["vocab"]
    model.close()


def test_weights_in_float32_are_taken_too(dev):
    cfg, w, tokens, want = case("ones", T=20)
    model = make(dev, cfg, {k: f32(v) for k, v in w.items()}, N.NS_BF16, max_prefill=20)
    assert worst(fed(model, tokens, [20]), want) < TOL[N.NS_BF16]
    model.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_replay_and_command_line(dev, tmp_path, dtype):
    cfg, w, tokens, want = case("wide", T=90)
    folder, out = tmp_path / "model", tmp_path / "out"
    folder.mkdir(), out.mkdir()
    (folder / "config.json").write_text(json.dumps(cfg))
    write_safetensors(str(folder / "model.safetensors"), w)
    t = [int(x) for x in tokens]
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": t[:50], "want": [0, 49]}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": t[:3], "want": []}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": t[50:51], "want": [0]}], "end": []},
             {"step": 3, "entries": [{"id": "a", "tokens": t[51:], "want": [38, 2]}], "end": ["a"]},
             {"step": 4, "entries": [{"id": "a", "tokens": t[:7], "want": [6]}], "end": ["a"]}]
    res = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(folder), "--dtype", dtype, "--out", str(out), "--max-tokens", "60"],
                         input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=300)
    assert res.returncode == 0, res.stderr[-2000:]
    assert [x for x in res.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(5)]
    assert not (out / "1.f32").exists()
    got = {n: np.fromfile(out / f"{n}.f32", "<f4").reshape(-1, cfg["vocab"]) for n in (0, 2, 3, 4)}
    tol = TOL[N.NS_F32 if dtype == "float32" else N.NS_BF16]
    for n, at in ((0, [0, 49]), (2, [50]), (3, [89, 53]), (4, [6])):
        assert worst(got[n], want[at]) < tol
    res = subprocess.run([sys.executable, "-m", "nn_b200", "generate", "--model", str(folder), "--dtype", dtype, "--prompt", "1,2,3", "--new", "5"], cwd=ROOT,
                         capture_output=True, text=True, timeout=300)
    assert res.returncode == 0, res.stderr[-2000:]
    line = [int(x) for x in res.stdout.split()]
    model = load_model(dev, str(folder), dtype)
    tokens, _ = model.generate(np.array([[1, 2, 3]]), 5)
    assert line == list(tokens[0])
    model.close()
