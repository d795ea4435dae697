"""Zokunex without a GPU: configuration and tensor names, the checkpoint reader, the registry, the exported symbols, and
properties of the plain implementation the GPU tests compare with."""

import ctypes
import json
import os
import re

import pytest
import torch

from glorcq_b200 import registry, weights, zokunex
from oracle import zokunex_oracle as O
from tests import zokunex_cases as Z

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


def _header():
    text = open(os.path.join(ROOT, "include", "glorcq_b200_dense.h")).read()
    return sorted(set(re.findall(r"\b(glq_[a-z0-9_]+)\s*\(", re.sub(r"/\*.*?\*/", "", text, flags=re.S))))


def test_header_is_exported_and_bound():
    from glorcq_b200 import _build, _lib
    L = ctypes.CDLL(_build.build(lib=_build.DENSE_LIB))
    assert len(_header()) >= 15
    assert not [s for s in _header() if not hasattr(L, s)]
    assert set(_header()) == set(_lib.dense_symbols())


def test_argument_errors_are_decided_on_the_host():
    from glorcq_b200 import _lib
    L = _lib.dense()
    assert L.glq_dense_matmul(ctypes.byref(_lib.DenseMM(N=0, K=8)), None) == -1
    assert L.glq_mlstm_step(ctypes.byref(_lib.MLstm(B=1, T=1, H=1, D=8, V=8, gate_cap=0.0)), None) == -1
    assert L.glq_mlstm_chunk(ctypes.byref(_lib.MLstm(dtype=_lib.DT_F32)), None) == -1
    assert L.glq_latent_prep(ctypes.byref(_lib.Latent(B=1, T=1, H=1, D=8, R=8, V=8, K=16, rot_dims=10, max_len=4)), None) == -1
    assert L.glq_route(ctypes.byref(_lib.Route(n=1, E=2, identity=0, top=3)), None) == -1
    assert L.glq_mlstm_slices(33) == 2
    for st in range(-5, 1):
        assert L.glq_dense_status_string(st)


def test_tensor_shapes():
    s = zokunex.tensor_shapes(Z.MIXED)
    assert s["l0.mix.q"] == (3 * 24, 104) and s["l0.mix.dkv"] == (56, 104) and s["l0.mix.uv"] == (72, 48)
    assert s["l0.mlp.router"] == (7, 104) and s["l0.mlp.e5.down"] == (104, 40) and "l0.mlp.e6.up" not in s
    assert s["l1.mix.norm"] == (80,) and s["l1.mix.i.b"] == (2,)
    assert "l2.norm2" not in s and not [k for k in s if k.startswith("l2.mlp")]
    with pytest.raises(ValueError):
        zokunex.tensor_shapes(dict(Z.MIXED, layers=[dict(Z.mlstm(), type="other", mlp=None)]))


def test_safetensors_round_trip(tmp_path):
    t = {"a": torch.randn(3, 5).bfloat16(), "b.c": torch.arange(7, dtype=torch.int32), "e": torch.empty(0, 4), "s": torch.tensor(2.5)}
    p = str(tmp_path / "x.safetensors")
    weights.write_safetensors(p, t)
    r = weights.read_safetensors(p)
    assert set(r) == set(t) and all(torch.equal(r[k], t[k]) and r[k].dtype == t[k].dtype for k in t)
    raw = open(p, "rb").read()
    open(p, "wb").write(raw[:-8])
    with pytest.raises(ValueError):
        weights.read_safetensors(p)


def test_registry(tmp_path):
    (tmp_path / "config.json").write_text(json.dumps(Z.ODD))
    assert registry.architecture_of(str(tmp_path)) == "Zokunex"
    (tmp_path / "config.json").write_text(json.dumps({"architectures": ["Unheard"]}))
    with pytest.raises(ValueError):
        registry.architecture_of(str(tmp_path))
    (tmp_path / "glorcq_model.pt").write_bytes(b"")
    assert registry.architecture_of(str(tmp_path)) is None
    with pytest.raises(registry.UnsupportedDtype):
        registry.load_model(str(tmp_path), dtype="float32")
    registry.register("Unheard", lambda path, device, dtype: (path, dtype))
    try:
        assert registry.load_model(str(tmp_path), dtype="bfloat16") == (str(tmp_path), torch.bfloat16)
    finally:
        del registry.ARCHITECTURES["Unheard"]


def test_missing_and_misshapen_tensors_are_errors():
    w = Z.make_weights(Z.ODD)
    bad = {k: v for k, v in w.items() if k != "l1.mix.uk"}
    with pytest.raises(KeyError, match="l1.mix.uk"):
        zokunex.ZokunexDecoder(Z.ODD, bad, device="cpu")
    with pytest.raises(ValueError, match="head"):
        zokunex.ZokunexDecoder(Z.ODD, dict(w, head=w["head"][:-1]), device="cpu")
    with pytest.raises(ValueError, match="dtype"):
        zokunex.ZokunexDecoder(Z.ODD, w, device="cpu", dtype=torch.float16)


def test_trace_runner_keeps_requests_apart():
    """The replay loop against a recording stand-in for the generation wrapper."""
    from glorcq_b200.trace import TraceRunner

    class Cache:
        resets = 0

        def reset(self):
            self.resets += 1

    class Wrapper:
        device, static_cache, calls = torch.device("cpu"), Cache(), []

        def step(self, ids, position, keep):
            self.calls.append((ids.tolist(), position, keep.tolist() if torch.is_tensor(keep) else keep))
            return torch.zeros(1, len(keep) if torch.is_tensor(keep) else 1, 4)
    r = TraceRunner.__new__(TraceRunner)
    r.wrapper, r.live, r.position = Wrapper(), None, 0
    assert r.run({"id": "a", "tokens": [1, 2, 3], "want": [0, 2]}).shape == (2, 4)
    assert r.run({"id": "a", "tokens": [4], "want": []}) is None
    with pytest.raises(ValueError):
        r.run({"id": "b", "tokens": [5], "want": []})
    r.end(["a"])
    r.run({"id": "b", "tokens": [5, 6], "want": [1]})
    assert r.wrapper.calls == [([[1, 2, 3]], 0, [0, 2]), ([[4]], 3, 1), ([[5, 6]], 0, [1])]
    assert r.wrapper.static_cache.resets == 2


# ---- the plain implementation itself -----------------------------------------------------------------------
def test_oracle_portions_equal_whole():
    W = Z.doubles(Z.make_weights(Z.MIXED, 3))
    toks = Z.tokens(Z.MIXED, 21)
    whole = O.forward(Z.MIXED, W, toks, O.new_state(Z.MIXED))
    st = O.new_state(Z.MIXED)
    parts = torch.cat([O.forward(Z.MIXED, W, toks[a:b], st) for a, b in ((0, 7), (7, 8), (8, 21))])
    assert (whole - parts).abs().max() < 1e-9


def test_oracle_recurrence_against_its_sum():
    """The unrolled recurrence: every position's weight is the product of the forget gates after it times its input gate."""
    g = torch.Generator().manual_seed(5)
    T, H, D, V = 12, 2, 6, 5
    q, k, v = (torch.randn(T, H, n, generator=g, dtype=torch.float64) for n in (D, D, V))
    i, f = torch.randn(T, H, generator=g, dtype=torch.float64) * 3, -torch.rand(T, H, generator=g, dtype=torch.float64)
    o = O.mlstm_recurrence(q, k, v, i, f, O.mlstm_state({"heads": H, "dim": D, "vdim": V}))
    for t in range(T):
        for h in range(H):
            lw = torch.stack([i[s, h] + f[s + 1:t + 1, h].sum() for s in range(t + 1)])
            start = f[:t + 1, h].sum()                       # the empty memory's weight takes part in the maximum
            m = max(lw.max().item(), start.item())
            w = torch.exp(lw - m)
            s = k[:t + 1, h] @ q[t, h]
            den = max(abs((w * s).sum().item()), torch.exp(torch.tensor(-m)).item()) + 1e-6
            assert torch.allclose((w * s) @ v[:t + 1, h] / den, o[t, h], atol=1e-10)


def test_oracle_rotation_is_a_rotation_by_position():
    x = torch.randn(9, 2, 10, dtype=torch.float64)
    r = O.rotate(x, torch.arange(9), 100.0, 8)
    assert torch.equal(r[..., 8:], x[..., 8:]) and torch.equal(r[0], x[0])
    assert torch.allclose(r.norm(dim=-1), x.norm(dim=-1))
    a = 3 * 100.0 ** (-2 / 8)
    z = torch.view_as_complex(torch.stack([x[3, 0, 1], x[3, 0, 5]])) * torch.polar(torch.tensor(1.0).double(), torch.tensor(a).double())
    assert torch.allclose(torch.view_as_real(z), torch.stack([r[3, 0, 1], r[3, 0, 5]]))


def test_oracle_routing_weights_ignore_the_correction():
    W = {"r.router": torch.zeros(4, 3, dtype=torch.float64), "r.correction": torch.tensor([0.0, 0.0, 0.3, 0.1], dtype=torch.float64)}
    sel, wt = O.route(torch.ones(1, 3, dtype=torch.float64), W, "r.", 2)
    assert sel[0].tolist() == [2, 3] and torch.allclose(wt, torch.full((1, 2), 0.25, dtype=torch.float64))
