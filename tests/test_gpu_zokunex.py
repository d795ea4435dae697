"""The Zokunex decoder through the framework: model, cache, generation wrapper, command line; against the plain
implementation."""

import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

from oracle import zokunex_oracle as O
from tests import zokunex_cases as Z

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
CONFIGS = {"mixed": Z.MIXED, "odd": Z.ODD, "wide": Z.WIDE}
TOL = {torch.float32: 1e-4, torch.bfloat16: 0.1}


@pytest.fixture(scope="module")
def dev():
    assert torch.cuda.is_available()
    return torch.device("cuda:0")


_MODELS = {}


def model(name, dtype, dev):
    from glorcq_b200.zokunex import ZokunexDecoder
    if (name, dtype) not in _MODELS:
        w = Z.make_weights(CONFIGS[name], 11)
        _MODELS[name, dtype] = ZokunexDecoder(CONFIGS[name], w, dev, dtype), w
    return _MODELS[name, dtype]


def oracle(name, w, toks, trace=None):
    cfg = CONFIGS[name]
    return O.forward(cfg, Z.doubles(w), toks, O.new_state(cfg), trace)


def run(m, rows, cuts, cache=None, trace=None):
    """Logits (B, T, vocab) of equal-length token rows, in portions."""
    dev = m.embed_tokens.device
    ids = torch.tensor(rows, device=dev)
    cache = cache or m.make_cache(ids.shape[0], ids.shape[1] + 2)
    out = [m(input_ids=ids[:, a:b], cache_position=torch.arange(a, b, device=dev), past_key_values=cache, trace=trace)[0].cpu() for a, b in cuts]
    return torch.cat(out, 1)


def portions(T, size):
    return [(a, min(T, a + size)) for a in range(0, T, size)]


@pytest.mark.parametrize("name", CONFIGS)
@pytest.mark.parametrize("dtype", TOL)
def test_prompt_and_layers(dev, name, dtype):
    m, w = model(name, dtype, dev)
    toks, tr, ref_tr = Z.tokens(CONFIGS[name], 150), [], []
    ref = oracle(name, w, toks, ref_tr)
    got = run(m, [toks], [(0, 150)], trace=tr)
    for l, (a, b) in enumerate(zip(tr, ref_tr)):
        assert Z.most_rel(a, b) < TOL[dtype], f"layer {l}"
    assert got.dtype == torch.float32 and Z.most_rel(got[0], ref) < TOL[dtype]
    if dtype == torch.float32:
        assert Z.worst_rel(got[0], ref) < TOL[dtype]


@pytest.mark.parametrize("name", CONFIGS)
@pytest.mark.parametrize("dtype", TOL)
def test_portions_and_token_by_token(dev, name, dtype):
    m, w = model(name, dtype, dev)
    T = 140
    toks = Z.tokens(CONFIGS[name], T, 2)
    ref = oracle(name, w, toks)
    mixed = [(0, 2), (2, 66), (66, 67), (67, 130), (130, 132), (132, 133), (133, 140)]
    for cuts in (portions(T, 1), portions(T, 2), portions(T, 9), portions(T, 64), portions(T, 65), mixed):
        got = run(m, [toks], cuts)
        assert Z.most_rel(got[0], ref) < TOL[dtype], cuts[:3]
        if dtype == torch.float32:
            assert Z.worst_rel(got[0], ref) < TOL[dtype]


@pytest.mark.parametrize("name", CONFIGS)
def test_sequences_of_a_batch_are_independent(dev, name):
    m, w = model(name, torch.float32, dev)
    mb, _ = model(name, torch.bfloat16, dev)
    rows = [Z.tokens(CONFIGS[name], 90, s) for s in (3, 4, 5)]
    cuts = [(0, 70), (70, 71), (71, 75), (75, 90)]
    got, got16 = run(m, rows, cuts), run(mb, rows, cuts)
    for b, toks in enumerate(rows):
        assert Z.worst_rel(got[b], oracle(name, w, toks)) < TOL[torch.float32]
        assert Z.most_rel(got16[b], run(mb, [toks], cuts)[0]) < TOL[torch.bfloat16]


def test_cache_is_used_again(dev):
    """A cache that held another, longer sequence gives what a fresh one gives, bit for bit."""
    for dtype in TOL:
        m, _ = model("mixed", dtype, dev)
        a, b = Z.tokens(Z.MIXED, 120, 6), Z.tokens(Z.MIXED, 77, 7)
        cuts = [(0, 40), (40, 41), (41, 77)]
        fresh = run(m, [b], cuts, m.make_cache(1, 128))
        cache = m.make_cache(1, 128)
        run(m, [a], [(0, 100), (100, 120)], cache)
        cache.reset()
        assert torch.equal(run(m, [b], cuts, cache), fresh)


def test_first_tokens(dev):
    m, w = model("mixed", torch.float32, dev)
    toks = Z.tokens(Z.MIXED, 3, 8)
    ref = oracle("mixed", w, toks)
    for cuts in ([(0, 3)], [(0, 1), (1, 3)], [(0, 2), (2, 3)], portions(3, 1)):
        assert Z.worst_rel(run(m, [toks], cuts)[0], ref) < TOL[torch.float32]


def test_logits_of_chosen_places(dev):
    m, _ = model("mixed", torch.bfloat16, dev)
    ids = torch.tensor([Z.tokens(Z.MIXED, 30, 9)], device=dev)
    pos = torch.arange(30, device=dev)
    full = m(input_ids=ids, cache_position=pos, past_key_values=m.make_cache(1, 32))[0]
    some = m(input_ids=ids, cache_position=pos, past_key_values=m.make_cache(1, 32), logits_to_keep=torch.tensor([0, 7, 29], device=dev))[0]
    last = m(input_ids=ids, cache_position=pos, past_key_values=m.make_cache(1, 32), logits_to_keep=2)[0]
    assert Z.worst_rel(some, full[:, [0, 7, 29]]) < 1e-5 and Z.worst_rel(last, full[:, 28:]) < 1e-5


def test_positions_beyond_the_cache_are_refused(dev):
    from glorcq_b200.graph_wrapper import GLoRCQGraphWrapper
    m, _ = model("mixed", torch.bfloat16, dev)
    ids = torch.zeros(1, 20, dtype=torch.long, device=dev)
    with pytest.raises(ValueError):
        m(input_ids=ids, cache_position=torch.arange(20, device=dev), past_key_values=m.make_cache(1, 16))
    with pytest.raises(ValueError):
        m(input_ids=ids.view(2, 10), cache_position=torch.arange(10, device=dev), past_key_values=m.make_cache(1, 16))
    w = GLoRCQGraphWrapper(m, 1, 16)
    with pytest.raises(ValueError):
        w.step(ids[:, :1], 16)


@pytest.mark.parametrize("name", ["mixed", "odd"])
def test_greedy_generation(dev, name):
    """Through the generation wrapper (eager prompt, replayed steps): every token is the plain implementation's choice."""
    from glorcq_b200.graph_wrapper import GLoRCQGraphWrapper
    m, w = model(name, torch.float32, dev)
    cfg, W = CONFIGS[name], Z.doubles(w)
    wrap = GLoRCQGraphWrapper(m, max_batch_size=2, max_seq_len=96)
    prompts = [Z.tokens(cfg, 13, 20), Z.tokens(cfg, 13, 21)]
    for again in range(2):                                   # the second call replays the captured step on a used cache
        ids, _ = wrap.generate(torch.tensor(prompts, device=dev), max_new_tokens=40)
        for b in range(2):
            logits = O.forward(cfg, W, ids[b, :-1].tolist(), O.new_state(cfg))[12:]
            top = logits.max(-1).values
            chosen = logits.gather(1, ids[b, 13:].cpu()[:, None])[:, 0]
            assert (top - chosen).max() < 1e-3 * logits.std()
    eager = m.generate(torch.tensor(prompts, device=dev), max_new_tokens=40)
    assert torch.equal(eager, ids)


def test_replayed_steps_in_the_middle_of_a_prompt(dev):
    """The step is captured at its first use, here between two portions; the state of the sequence is untouched by it."""
    from glorcq_b200.graph_wrapper import GLoRCQGraphWrapper
    for dtype in TOL:
        m, w = model("mixed", dtype, dev)
        toks = Z.tokens(Z.MIXED, 260, 30)
        ref = oracle("mixed", w, toks)
        wrap = GLoRCQGraphWrapper(m, 1, 260)
        ids = torch.tensor([toks], device=dev)
        got = []
        for a, b in [(0, 7), (7, 8), (8, 30), (30, 31), (31, 32), (32, 100)] + [(i, i + 1) for i in range(100, 260)]:
            got.append(wrap.step(ids[:, a:b], a, torch.arange(b - a, device=dev)).clone().cpu())
        got = torch.cat(got, 1)[0]
        assert Z.most_rel(got, ref) < TOL[dtype]
        if dtype == torch.float32:
            assert Z.worst_rel(got, ref) < TOL[dtype]


def _write(tmp_path, cfg, w):
    from glorcq_b200 import weights
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    weights.write_safetensors(str(tmp_path / "model.safetensors"), w)


def test_trace_and_generate_programs(dev, tmp_path):
    """bin/trace_run and `python -m glorcq_b200 generate` on a checkpoint folder."""
    w = Z.make_weights(Z.MIXED, 12)
    _write(tmp_path, Z.MIXED, w)
    toks, toks2 = Z.tokens(Z.MIXED, 40, 40), Z.tokens(Z.MIXED, 9, 41)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": toks[:37], "want": [0, 36]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": toks[37:38], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "x", "tokens": toks[38:], "want": [1]}], "end": ["x"]},
             {"step": 3, "entries": [{"id": "y", "tokens": toks2, "want": [8]}], "end": ["y"]}]
    ref, ref2 = O.forward(Z.MIXED, Z.doubles(w), toks, O.new_state(Z.MIXED)), O.forward(Z.MIXED, Z.doubles(w), toks2, O.new_state(Z.MIXED))
    p = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", "float32", "--out", str(tmp_path),
                        "--max-tokens", "64"], input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=120)
    assert p.returncode == 0, p.stderr[-2000:]
    assert [x for x in p.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(4)]
    assert not (tmp_path / "1.f32").exists()
    for n, want in ((0, ref[[0, 36]]), (2, ref[[39]]), (3, ref2[[8]])):
        got = torch.tensor(np.fromfile(str(tmp_path / f"{n}.f32"), "<f4")).view(-1, Z.MIXED["vocab"])
        assert Z.worst_rel(got, want) < 1e-4
    g = subprocess.run([sys.executable, "-m", "glorcq_b200", "generate", "--model", str(tmp_path), "--tokens", ",".join(map(str, toks)),
                        "--max-new-tokens", "5", "--dtype", "float32"], capture_output=True, text=True, timeout=120, cwd=ROOT)
    assert g.returncode == 0, g.stderr[-2000:]
    out = [int(t) for t in g.stdout.split(",")]
    assert len(out) == 5 and out[0] == int(ref[-1].argmax())
