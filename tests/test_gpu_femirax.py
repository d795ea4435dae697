"""The Femirax decoder through the framework: model, cache, generation wrapper, command line; against the plain
implementation."""

import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

from oracle import femirax_oracle as O
from tests import femirax_cases as F

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
DTYPES = [torch.float32, torch.bfloat16]


def close(got, ref, dtype):
    """Rows within rounding.  In bf16 a head's output that is small by cancellation is normed up with its rounding, so a few
    rows may stand out, by less than a wrong token's logits would."""
    if dtype == torch.float32:
        return F.worst_rel(got, ref) < 1e-4
    return F.most_rel(got, ref) < 0.03 and F.worst_rel(got, ref) < 0.25


@pytest.fixture(scope="module")
def dev():
    assert torch.cuda.is_available()
    return torch.device("cuda:0")


_MODELS, _ORACLE = {}, {}


def model(name, dtype, dev):
    from glorcq_b200.femirax import FemiraxDecoder
    if (name, dtype) not in _MODELS:
        w = F.weights_of(name)
        _MODELS[name, dtype] = FemiraxDecoder(F.CONFIGS[name], w, dev, dtype), w
    return _MODELS[name, dtype]


def oracle(name, w, toks, trace=None):
    cfg = F.CONFIGS[name]
    if trace is not None:
        return O.forward(cfg, F.doubles(w), toks, O.new_state(cfg), trace)
    key = (name, tuple(toks))
    if key not in _ORACLE:
        _ORACLE[key] = O.forward(cfg, F.doubles(w), toks, O.new_state(cfg))
    return _ORACLE[key]


def run(m, rows, cuts, cache=None, trace=None):
    """Logits (B, T, vocab) of equal-length token rows, in portions."""
    dev = m.embed_tokens.device
    ids = torch.tensor(rows, device=dev)
    cache = cache or m.make_cache(ids.shape[0], ids.shape[1] + 2)
    out = [m(input_ids=ids[:, a:b], cache_position=torch.arange(a, b, device=dev), past_key_values=cache, trace=trace)[0].cpu() for a, b in cuts]
    return torch.cat(out, 1)


def portions(T, size):
    return [(a, min(T, a + size)) for a in range(0, T, size)]


@pytest.mark.parametrize("name", F.CONFIGS)
@pytest.mark.parametrize("dtype", DTYPES)
def test_prompt_and_layers(dev, name, dtype):
    m, w = model(name, dtype, dev)
    toks, tr, ref_tr = F.tokens(F.CONFIGS[name], 150), [], []
    ref = oracle(name, w, toks, ref_tr)
    got = run(m, [toks], [(0, 150)], trace=tr)
    for l, (a, b) in enumerate(zip(tr, ref_tr)):
        assert close(a, b, dtype), f"layer {l}"
    assert got.dtype == torch.float32 and close(got[0], ref, dtype)


@pytest.mark.parametrize("name", F.CONFIGS)
@pytest.mark.parametrize("dtype", DTYPES)
def test_portions_and_token_by_token(dev, name, dtype):
    m, w = model(name, dtype, dev)
    T = 140
    toks = F.tokens(F.CONFIGS[name], T, 2)
    ref = oracle(name, w, toks)
    mixed = [(0, 2), (2, 66), (66, 67), (67, 130), (130, 132), (132, 133), (133, 140)]
    for cuts in (portions(T, 1), portions(T, 2), portions(T, 9), portions(T, 64), portions(T, 65), mixed):
        assert close(run(m, [toks], cuts)[0], ref, dtype), cuts[:3]


@pytest.mark.parametrize("name", F.CONFIGS)
def test_sequences_of_a_batch_are_independent(dev, name):
    m, w = model(name, torch.float32, dev)
    mb, _ = model(name, torch.bfloat16, dev)
    rows = [F.tokens(F.CONFIGS[name], 90, s) for s in (3, 4, 5)]
    cuts = [(0, 70), (70, 71), (71, 75), (75, 90)]
    got, got16 = run(m, rows, cuts), run(mb, rows, cuts)
    for b, toks in enumerate(rows):
        ref = oracle(name, w, toks)
        assert close(got[b], ref, torch.float32) and close(got16[b], ref, torch.bfloat16)


def test_cache_is_used_again(dev):
    """A cache that held another, longer sequence gives what a fresh one gives, bit for bit."""
    for name in ("mixed", "wide"):
        for dtype in DTYPES:
            m, _ = model(name, dtype, dev)
            a, b = F.tokens(F.CONFIGS[name], 120, 6), F.tokens(F.CONFIGS[name], 77, 7)
            cuts = [(0, 40), (40, 41), (41, 77)]
            fresh = run(m, [b], cuts, m.make_cache(1, 128))
            cache = m.make_cache(1, 128)
            run(m, [a], [(0, 100), (100, 120)], cache)
            cache.reset()
            assert torch.equal(run(m, [b], cuts, cache), fresh)


def test_first_tokens(dev):
    m, w = model("mixed", torch.float32, dev)
    toks = F.tokens(F.MIXED, 3, 8)
    ref = oracle("mixed", w, toks)
    for cuts in ([(0, 3)], [(0, 1), (1, 3)], [(0, 2), (2, 3)], portions(3, 1)):
        assert close(run(m, [toks], cuts)[0], ref, torch.float32)


def test_logits_of_chosen_places(dev):
    m, _ = model("mixed", torch.bfloat16, dev)
    ids = torch.tensor([F.tokens(F.MIXED, 30, 9)], device=dev)
    pos = torch.arange(30, device=dev)

    def call(**kw):
        return m(input_ids=ids, cache_position=pos, past_key_values=m.make_cache(1, 32), **kw)[0]
    full = call()
    assert F.worst_rel(call(logits_to_keep=torch.tensor([0, 7, 29], device=dev)), full[:, [0, 7, 29]]) < 1e-5
    assert F.worst_rel(call(logits_to_keep=2), full[:, 28:]) < 1e-5


def test_the_token_row_belongs_to_its_layer_and_token(dev):
    """Changing one token's columns of one layer changes that layer at that token and nothing before it."""
    from glorcq_b200.femirax import FemiraxDecoder
    m, w = model("mixed", torch.float32, dev)
    toks, l, at = list(range(20, 50)), 2, 11
    w2 = {k: v.clone() for k, v in w.items()}
    w2["side.embed"][toks[at], 24 * l:24 * (l + 1)] += 2.0
    tr, tr2, ref = [], [], []
    run(m, [toks], [(0, 30)], trace=tr)
    run(FemiraxDecoder(F.MIXED, w2, dev, torch.float32), [toks], [(0, 30)], trace=tr2)
    O.forward(F.MIXED, F.doubles(w2), toks, O.new_state(F.MIXED), ref)
    for i, (a, b) in enumerate(zip(tr, tr2)):
        changed = (a != b).any(-1).cpu()
        assert not changed[:at].any() and bool(changed[at]) == (i >= l)
        assert close(b, ref[i], torch.float32)


def test_positions_beyond_the_cache_are_refused(dev):
    from glorcq_b200.graph_wrapper import GLoRCQGraphWrapper
    m, _ = model("mixed", torch.bfloat16, dev)
    ids = torch.zeros(1, 20, dtype=torch.long, device=dev)
    with pytest.raises(ValueError):
        m(input_ids=ids, cache_position=torch.arange(20, device=dev), past_key_values=m.make_cache(1, 16))
    w = GLoRCQGraphWrapper(m, 1, 16)
    with pytest.raises(ValueError):
        w.step(ids[:, :1], 16)


@pytest.mark.parametrize("name", ["mixed", "odd"])
def test_greedy_generation(dev, name):
    """Through the generation wrapper (eager prompt, replayed steps): every token is the plain implementation's choice."""
    from glorcq_b200.graph_wrapper import GLoRCQGraphWrapper
    m, w = model(name, torch.float32, dev)
    cfg = F.CONFIGS[name]
    wrap = GLoRCQGraphWrapper(m, max_batch_size=2, max_seq_len=96)
    prompts = [F.tokens(cfg, 13, 20), F.tokens(cfg, 13, 21)]
    for again in range(2):                                   # the second call replays the captured step on a used cache
        ids, _ = wrap.generate(torch.tensor(prompts, device=dev), max_new_tokens=40)
        for b in range(2):
            logits = oracle(name, w, ids[b, :-1].tolist())[12:]
            top = logits.max(-1).values
            chosen = logits.gather(1, ids[b, 13:].cpu()[:, None])[:, 0]
            assert (top - chosen).max() < 1e-3 * logits.std()
    assert torch.equal(m.generate(torch.tensor(prompts, device=dev), max_new_tokens=40), ids)


@pytest.mark.parametrize("name", ["mixed", "wide"])
def test_replayed_steps_in_the_middle_of_a_prompt(dev, name):
    """The step is captured at its first use, here between two portions; the state of the sequence is untouched by it.
    Then long decoding."""
    from glorcq_b200.graph_wrapper import GLoRCQGraphWrapper
    for dtype in DTYPES:
        m, w = model(name, dtype, dev)
        toks = F.tokens(F.CONFIGS[name], 300, 30)
        ref = oracle(name, w, toks)
        wrap = GLoRCQGraphWrapper(m, 1, 300)
        ids = torch.tensor([toks], device=dev)
        got = []
        for a, b in [(0, 7), (7, 8), (8, 30), (30, 31), (31, 32), (32, 100)] + [(i, i + 1) for i in range(100, 300)]:
            got.append(wrap.step(ids[:, a:b], a, torch.arange(b - a, device=dev)).clone().cpu())
        assert close(torch.cat(got, 1)[0], ref, dtype)


def test_captured_step_survives_a_longer_cache(dev):
    """A cache that needs longer rotation tables must not take the old ones from under a captured step."""
    from glorcq_b200.graph_wrapper import GLoRCQGraphWrapper
    m, w = model("mixed", torch.float32, dev)
    toks = F.tokens(F.MIXED, 40, 31)
    ids = torch.tensor([toks], device=dev)
    wrap = GLoRCQGraphWrapper(m, 1, 48)
    got = [wrap.step(ids[:, :20], 0, torch.arange(20, device=dev)).cpu(), wrap.step(ids[:, 20:21], 20).clone().cpu()]
    run(m, [toks], [(0, 40)], m.make_cache(1, 5000))
    junk = [torch.full((5000, 8), float("nan"), device=dev) for _ in range(20)]
    got += [wrap.step(ids[:, i:i + 1], i).clone().cpu() for i in range(21, 40)]
    del junk
    assert close(torch.cat(got, 1)[0], oracle("mixed", w, toks), torch.float32)


def test_trace_and_generate_programs(dev, tmp_path):
    """bin/trace_run and `python -m glorcq_b200 generate` on a checkpoint folder."""
    from glorcq_b200 import weights
    w = F.weights_of("mixed", 12)
    (tmp_path / "config.json").write_text(json.dumps(F.MIXED))
    weights.write_safetensors(str(tmp_path / "model.safetensors"), w)
    toks, toks2 = F.tokens(F.MIXED, 40, 40), F.tokens(F.MIXED, 9, 41)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": toks[:37], "want": [0, 36]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": toks[37:38], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "x", "tokens": toks[38:], "want": [1]}], "end": ["x"]},
             {"step": 3, "entries": [{"id": "y", "tokens": toks2, "want": [8]}], "end": ["y"]}]
    ref, ref2 = (O.forward(F.MIXED, F.doubles(w), t, O.new_state(F.MIXED)) for t in (toks, toks2))
    for dtype, tol in (("float32", 1e-4), ("bfloat16", 0.1)):
        p = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", dtype, "--out", str(tmp_path),
                            "--max-tokens", "64"], input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=120)
        assert p.returncode == 0, p.stderr[-2000:]
        assert [x for x in p.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(4)]
        assert not (tmp_path / "1.f32").exists()
        for n, want in ((0, ref[[0, 36]]), (2, ref[[39]]), (3, ref2[[8]])):
            got = torch.tensor(np.fromfile(str(tmp_path / f"{n}.f32"), "<f4")).view(-1, F.MIXED["vocab"])
            assert F.worst_rel(got, want) < tol
    g = subprocess.run([sys.executable, "-m", "glorcq_b200", "generate", "--model", str(tmp_path), "--tokens", ",".join(map(str, toks)),
                        "--max-new-tokens", "5", "--dtype", "float32"], capture_output=True, text=True, timeout=120, cwd=ROOT)
    assert g.returncode == 0, g.stderr[-2000:]
    out = [int(t) for t in g.stdout.split(",")]
    assert len(out) == 5 and out[0] == int(ref[-1].argmax())
