"""The Topidra decoder against the plain statement of the design (oracle/topidra.py): whole prompts, portions, token by token, slots that
are used again, long decoding, batches, and generation through the framework's loop."""
import copy
import json
import os
import subprocess
import sys

import numpy as np
import pytest

from nn_b200 import native as N
from nn_b200.blocks import bf16_bits, f32
from nn_b200.registry import load_model
from nn_b200.topidra import Topidra, TopidraConfig
from nn_b200.weights import write_safetensors
from oracle import topidra as F
from tests.fabezen_models import wide64
from tests.test_fabezen_model import cuts_of, fed, worst
from tests.topidra_models import CONFIGS, attention, config, lightning, weights_for

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
# Over all positions together, and at the worst one.  The small models are touchy at single positions (a norm over two values, scores
# close to one another): rounding activations to bf16 in the oracle moves these models' logits by 0.010 together and 0.08 at worst.
TOL = {N.NS_F32: (2e-5, 1e-4), N.NS_BF16: (0.02, 0.25)}
DTYPES = [N.NS_F32, N.NS_BF16]
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
    return Topidra(dev, TopidraConfig.from_dict(cfg), w, dtype=dtype, **kw)


def error(got, want):
    """(over all positions together, at the worst one) relative to the logits' spread."""
    d = got - want
    d = d - d.mean(-1, keepdims=True)
    spread = np.sqrt(np.mean((want - want.mean(-1, keepdims=True)) ** 2))
    return float(np.sqrt(np.mean(d ** 2)) / spread), worst(got, want)


def agree(got, want, dtype):
    e = error(got, want)
    return e[0] < TOL[dtype][0] and e[1] < TOL[dtype][1] or pytest.fail(f"differs by {e[0]:.3g}, at worst {e[1]:.3g}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(CONFIGS))
def test_whole_prompt(dev, name, dtype):
    cfg, w, tokens, want = case(name, T=310)
    model = make(dev, cfg, w, dtype, max_prefill=len(tokens))
    assert agree(fed(model, tokens, [len(tokens)]), want, dtype)
    model.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", ["single", "pairs", "mixed"])
@pytest.mark.parametrize("name", list(CONFIGS))
def test_portions(dev, name, kind, dtype):
    cfg, w, tokens, want = case(name)
    model = make(dev, cfg, w, dtype, max_prefill=70)
    assert agree(fed(model, tokens, cuts_of(kind, len(tokens))), want, dtype)
    model.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_portions_against_one_another(dev, dtype):
    """The same model, cut differently: what differs is rounding."""
    cfg, w, tokens, _ = case("mixed", T=310)
    model = make(dev, cfg, w, dtype, max_prefill=310)
    whole = fed(model, tokens, [310])
    for cuts in ([1] * 310, [2] * 155, [127, 1, 128, 2, 52], [31, 33, 32, 64, 150]):
        assert agree(fed(model, tokens, cuts), whole, dtype), cuts
    model.close()


@pytest.mark.parametrize("max_prefill", [1, 7, 64])
def test_prompts_longer_than_a_pass(dev, max_prefill):
    cfg, w, tokens, want = case("mixed")
    model = make(dev, cfg, w, N.NS_F32, max_prefill=max_prefill)
    assert agree(fed(model, tokens, [130, 20]), want, N.NS_F32)
    model.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_slots_are_used_again_and_do_not_mix(dev, dtype):
    cfg, w, tokens, want = case("mixed")
    other = (tokens * 7 + 3) % cfg["vocab"]
    want_other = F.forward(other, wide64(w), cfg)
    model = make(dev, cfg, w, dtype, max_prefill=40, slots=3)
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
        assert agree(np.concatenate(ga), want, dtype) and agree(np.concatenate(gb), want_other, dtype)
        for s in ((a, b) if round_ % 2 else (b, a)):
            model.close_sequence(s)
    model.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_unequal_sequences_in_one_pass(dev, dtype):
    """Sequences at different positions step together, as each does alone."""
    cfg, w, tokens, want = case("mixed", T=310)
    model = make(dev, cfg, w, dtype, batch=3, max_prefill=130, slots=4)
    starts, slots = [0, 13, 127], [model.open_sequence() for _ in range(3)]
    for s, n in zip(slots, starts):
        if n:
            model.feed([s], tokens[None, :n])
    got = [[] for _ in slots]
    at = 0
    for n in (1, 1, 2, 40, 1, 130, 5):
        ids = np.stack([tokens[p + at:p + at + n] for p in starts])
        logits = model.feed(slots, ids, [(b, i) for b in range(3) for i in range(n)]).reshape(3, n, -1)
        for b in range(3):
            got[b].append(logits[b])
        at += n
    alone = make(dev, cfg, w, dtype, batch=1, max_prefill=130)
    for b, p in enumerate(starts):
        assert agree(np.concatenate(got[b]), want[p:p + at], dtype), b
        assert agree(np.concatenate(got[b]), fed(alone, tokens[:p + at], ([p] if p else []) + [1, 1, 2, 40, 1, 130, 5])[p:], dtype), b
    model.close()
    alone.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding_wraps_every_ring(dev, dtype):
    cfg, w, tokens, want = case("mixed", T=700)
    model = make(dev, cfg, w, dtype, max_prefill=5)
    assert agree(fed(model, tokens, [5] + [1] * 695), want, dtype)
    model.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T", [1, 2, 3, 4])
def test_first_tokens(dev, T, dtype):
    cfg, w, tokens, want = case("mixed")
    model = make(dev, cfg, w, dtype, max_prefill=8)
    assert agree(fed(model, tokens[:T], [T]), want[:T], dtype)
    model.close()


def sharp(size, width=32, sink=None):
    """One attention layer whose scores are wide apart: (config, weights)."""
    cfg = config([attention(heads=8, kv_heads=4, dim=16, vdim=24, scale=1.4, size=size, ff=None)], vocab=230, width=width)
    w = weights_for(cfg, 5)
    w["l0.mix.sink"] = bf16_bits(np.full(8, -2.0 if sink is None else sink, np.float32))
    return cfg, w


@pytest.mark.parametrize("size", [1, 2, 40, 127, 128, 129, 140])
def test_window_edges_in_prompts_and_decoding(dev, size):
    """Attention sharp enough that a window one token off changes the logits by more than the tolerance (checked on the oracle)."""
    cfg, w = sharp(size)
    tokens = np.random.default_rng(8).permutation(230)[:200]            # no token twice: a key has no twin inside the window
    want = F.forward(tokens, wide64(w), cfg)
    for off in (-1, 1):
        if size + off > 0:
            near = copy.deepcopy(cfg)
            near["layers"][0]["mixer"]["mask"]["size"] += off
            assert worst(F.forward(tokens, wide64(w), near), want) > 0.3
    for dtype in DTYPES:
        model = make(dev, cfg, w, dtype, max_prefill=200)
        for cuts in ([200], [15] + [1] * 185, [30, 2, 100, 68]):
            assert worst(fed(model, tokens, cuts), want) < (1e-4 if dtype == N.NS_F32 else 0.12), (dtype, cuts)
        model.close()


@pytest.mark.parametrize("what", ["sink", "gate", "loop", "decay", "norm"])
def test_a_missing_mechanism_would_show(dev, what):
    """The model agrees with the oracle where an oracle without the mechanism does not."""
    cfg = config([lightning(heads=2, dim=16, vdim=16, decay=[0.9, 0.4], ff=None), attention(heads=4, kv_heads=2, dim=16, vdim=16, scale=0.2, size=30, ff=24)], vocab=120,
                 width=40, loop=(0, 2, 2))
    w = weights_for(cfg, 6)
    w["l1.mix.sink"] = bf16_bits(np.array([0.0, 2.0, 4.0, 5.0], np.float32))
    tokens = np.random.default_rng(7).integers(0, 120, 90)
    want = F.forward(tokens, wide64(w), cfg)
    other, wo = copy.deepcopy(cfg), dict(w)
    if what == "sink":
        wo["l1.mix.sink"] = bf16_bits(np.full(4, -30.0, np.float32))
    elif what == "gate":
        wo["l1.mix.g"] = bf16_bits(np.zeros((4, 40), np.float32))
    elif what == "loop":
        other["loop"]["times"] = 1
    elif what == "decay":
        other["layers"][0]["mixer"]["decay"] = [0.9, 0.9]
    else:
        wo["l1.mix.k.norm"] = bf16_bits(np.ones(32, np.float32))
    assert error(F.forward(tokens, wide64(wo), other), want)[0] > 2.5 * TOL[N.NS_BF16][0]
    for dtype in DTYPES:
        for c, x in ((cfg, w), (other, wo)):
            model = make(dev, c, x, dtype, max_prefill=90)
            want = F.forward(tokens, wide64(x), c)
            assert agree(fed(model, tokens, [90]), want, dtype)
            assert agree(fed(model, tokens, [50] + [1] * 40), want, dtype)
            model.close()


@pytest.mark.parametrize("loop", [(0, 1, 3), (1, 2, 2), (2, 3, 2), (1, 1, 4), (0, 3, 1)])
def test_loops_anywhere(dev, loop):
    cfg = config([lightning(), attention(size=9), lightning(heads=2, ff=32)], loop=loop)
    w = weights_for(cfg, 9)
    tokens = np.random.default_rng(10).integers(0, cfg["vocab"], 60)
    want = F.forward(tokens, wide64(w), cfg)
    for dtype in DTYPES:
        model = make(dev, cfg, w, dtype, max_prefill=60)
        for cuts in ([60], [20] + [1] * 10 + [30]):
            assert agree(fed(model, tokens, cuts), want, dtype)
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
    model = make(dev, cfg, w, dtype, batch=3, max_prefill=32)
    tokens, resets = model.generate(prompt, 30)
    assert resets == 0 and tokens.shape == (3, 30) and model.launches_per_step > 0
    greedy_check(tokens, prompt, w, cfg, tol)
    again, _ = model.generate(prompt, 30)                        # the recorded step, a state full of the first run's
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
    for n, at in ((0, [0, 49]), (2, [50]), (3, [89, 53]), (4, [6])):
        assert agree(got[n], want[at], N.NS_F32 if dtype == "float32" else N.NS_BF16)
    res = subprocess.run([sys.executable, "-m", "nn_b200", "generate", "--model", str(folder), "--dtype", dtype, "--prompt", "1,2,3", "--new", "5"], cwd=ROOT,
                         capture_output=True, text=True, timeout=300)
    assert res.returncode == 0, res.stderr[-2000:]
    model = load_model(dev, str(folder), dtype)
    tokens, _ = model.generate(np.array([[1, 2, 3]]), 5)
    assert [int(x) for x in res.stdout.split()] == list(tokens[0])
    model.close()


def test_weights_in_float32_are_taken_too(dev):
    cfg, w, tokens, want = case("ones", T=20)
    model = make(dev, cfg, {k: f32(v) for k, v in w.items()}, N.NS_BF16, max_prefill=20)
    assert agree(fed(model, tokens, [20]), want, N.NS_BF16)
    model.close()
