"""Femirax without a GPU: configuration and tensor names, the registry, host-side argument errors, weight layouts, the
state objects, and properties of the plain implementation the GPU tests compare with."""

import ctypes
import json

import pytest
import torch

from glorcq_b200 import femirax, registry
from oracle import femirax_oracle as O
from tests import femirax_cases as F


def test_tensor_shapes():
    s = femirax.tensor_shapes(F.MIXED)
    assert s["side.embed"] == (160, 24 * 5) and s["l4.side.gate"] == (24, 104) and s["l4.side.proj"] == (104, 24)
    assert s["l0.mix.left.k"] == (32, 104) and s["l0.mix.left.o"] == (104, 64) and "l0.mix.left.v" not in s
    assert s["l0.mix.right.a1"] == (16, 104) and s["l0.mix.right.a2"] == (48, 16) and s["l0.mix.right.norm"] == (24,)
    assert s["l1.mix.g"] == (48, 104) and s["l1.mlp.down"] == (104, 40)
    assert "l2.norm2" not in s and not [k for k in s if k.startswith("l2.mlp")]
    with pytest.raises(ValueError):
        femirax.tensor_shapes(dict(F.MIXED, layers=[dict(F.retention(), type="other", mlp=None)]))
    with pytest.raises(ValueError):
        femirax.tensor_shapes(dict(F.MIXED, layers=[dict(F.retention(), mlp={"kind": "moe"})]))


def test_registry_and_checks(tmp_path):
    (tmp_path / "config.json").write_text(json.dumps(F.ODD))
    assert registry.architecture_of(str(tmp_path)) == "Femirax"
    w = F.weights_of("odd")
    with pytest.raises(KeyError, match="l0.side.proj"):
        femirax.FemiraxDecoder(F.ODD, {k: v for k, v in w.items() if k != "l0.side.proj"}, device="cpu")
    with pytest.raises(ValueError, match="l1.mix.right.a2 "):      # the rank is what the first factor has
        femirax.FemiraxDecoder(F.ODD, {**w, "l1.mix.right.a2": w["l1.mix.right.a2"][:, :2]}, device="cpu")
    with pytest.raises(ValueError, match="dtype"):
        femirax.FemiraxDecoder(F.ODD, w, device="cpu", dtype=torch.float16)
    m = femirax.FemiraxDecoder(F.ODD, w, device="cpu")
    assert len(m.mixers) == 4 and m.config.vocab_size == 101
    short = dict(F.ODD, layers=[dict(F.ODD["layers"][0], mixer=dict(F.ODD["layers"][0]["mixer"], decay=[0.5]))] + F.ODD["layers"][1:])
    with pytest.raises(ValueError, match="decays"):
        femirax.FemiraxDecoder(short, w, device="cpu")
    with pytest.raises(RuntimeError):                              # there is no CPU path
        m(input_ids=torch.zeros(1, 3, dtype=torch.long), past_key_values=m.make_cache(1, 8))


def test_argument_errors_are_decided_on_the_host():
    from glorcq_b200 import _lib
    L = _lib.dense()
    ref = ctypes.byref
    one = ctypes.create_string_buffer(64)
    p = ctypes.addressof(one)
    assert L.glq_decay_step(ref(_lib.Decay(B=1, T=1, H=1, D=8, V=8)), None) == -1
    assert L.glq_decay_step(ref(_lib.Decay(B=1, T=1, H=1, D=8, V=8, rot_dims=7, q=p, k=p, v=p, g=p, S=p, o=p, decay=p)), None) == -1
    assert L.glq_decay_step(ref(_lib.Decay(B=1, T=1, H=1, D=8, V=8, q=p, k=p, v=p, g=p, S=p, o=p, a=p, a2=p, a2b=p, rank=2)), None) == -1
    assert L.glq_decay_chunk(ref(_lib.Decay(dtype=_lib.DT_F32, D=8, V=8)), None) == -3
    assert L.glq_decay_slices(65) == 3
    assert L.glq_gqa(ref(_lib.Gqa(B=1, T=1, H=3, G=2, D=8, V=8, max_len=4)), None) == -1
    assert L.glq_gqa_form(ref(_lib.Gqa(B=1, T=1, H=2, G=2, D=8, V=8, max_len=4, dtype=_lib.DT_F32))) == 0
    assert L.glq_dense_matmul(ref(_lib.DenseMM(N=24, K=8, rows=1, split=24, act=_lib.ACT_SILU_GLU, x=p, W=p, y=p)), None) == -1
    assert L.glq_dense_matmul(ref(_lib.DenseMM(N=16, K=8, rows=1, split=8, residual=1, x=p, W=p, y=p, y32=p)), None) == -1
    assert L.glq_dense_rms_add(0, None, 0, None, p, 0, None, 1.0, None, 0.0, 1, 8, p, p, None) == -1


def test_gated_rows_interleave_and_pad():
    from glorcq_b200.dense import gated_rows
    g, u = torch.arange(10.0)[:, None].expand(10, 3), 100 + torch.arange(10.0)[:, None].expand(10, 3)
    w = gated_rows(g, u)
    assert w.shape == (32, 3)
    assert w[:, 0].tolist() == [*range(8), *range(100, 108), 8, 9, 0, 0, 0, 0, 0, 0, 108, 109, 0, 0, 0, 0, 0, 0]


def test_states_are_put_back():
    from glorcq_b200.cache import DecayState, KeyValueState, LayerStateCache, SideBySideState
    c = LayerStateCache([DecayState(2, 16, 3, 8, 40, "cpu"), SideBySideState(KeyValueState(2, 16, 2, 8, 8, "cpu", torch.bfloat16),
                                                                            DecayState(2, 16, 1, 8, 8, "cpu"))], 2, 16)
    parts = [c[0].S, c[1][0].k, c[1][0].v, c[1][1].S]
    assert parts[0].shape == (2, 3, 2, 8, 32)
    for t in parts:
        t.normal_()
    before = [t.clone() for t in parts]
    saved = c.snapshot(5)
    for i, t in enumerate(parts):
        if i in (1, 2):
            t[:, :5] = 7
        else:
            t.fill_(7)
    c.restore(saved)
    assert all(torch.equal(a, b) for a, b in zip(before, parts))
    c.reset()
    assert not c[0].S.any() and not c[1][1].S.any()


# ---- the plain implementation itself -----------------------------------------------------------------------
def test_oracle_portions_equal_whole():
    W = F.doubles(F.weights_of("mixed", 3))
    toks = F.tokens(F.MIXED, 21)
    whole = O.forward(F.MIXED, W, toks, O.new_state(F.MIXED))
    st = O.new_state(F.MIXED)
    parts = torch.cat([O.forward(F.MIXED, W, toks[a:b], st) for a, b in ((0, 7), (7, 8), (8, 21))])
    assert (whole - parts).abs().max() < 1e-9


def test_oracle_recurrence_against_its_sum():
    """Unrolled: position s reaches t through the product of the decays after s."""
    g = torch.Generator().manual_seed(5)
    T, H, D, V = 12, 2, 6, 5
    q, k, v = (torch.randn(T, H, n, generator=g, dtype=torch.float64) for n in (D, D, V))
    a = torch.rand(T, H, D, generator=g, dtype=torch.float64)
    o = O.decayed_recurrence(q, k, v, a, torch.zeros(H, D, V, dtype=torch.float64))
    for t in range(T):
        ref = sum(((q[t] * k[s] * a[s + 1:t + 1].prod(0)).sum(-1)[:, None] * v[s] for s in range(t + 1)))
        assert torch.allclose(ref, o[t], atol=1e-12)


def test_oracle_rotations():
    x = torch.randn(9, 2, 10, dtype=torch.float64)
    a, b = O.rotate_halves(x, torch.arange(9), 100.0, 8), O.rotate_pairs(x, torch.arange(9), 100.0, 8)
    perm = [0, 2, 4, 6, 1, 3, 5, 7, 8, 9]                          # pairs laid out as halves
    assert torch.allclose(O.rotate_halves(x[..., perm], torch.arange(9), 100.0, 8), b[..., perm])
    for r in (a, b):
        assert torch.equal(r[..., 8:], x[..., 8:]) and torch.equal(r[0], x[0]) and torch.allclose(r.norm(dim=-1), x.norm(dim=-1))
    ang = 3 * 100.0 ** (-2 / 8)
    z = torch.complex(x[3, 0, 2], x[3, 0, 3]) * torch.polar(torch.tensor(1.0).double(), torch.tensor(ang).double())
    assert torch.allclose(torch.view_as_real(z), b[3, 0, 2:4])


def test_oracle_normed_scores_ignore_the_size_of_keys_but_values_do_not():
    W = F.doubles(F.weights_of("mixed", 2))
    m = F.MIXED["layers"][0]["mixer"]["left"]
    h = torch.randn(6, 104, dtype=torch.float64)
    one = O.shared_value_attention(h, W, "l0.mix.left.", m, 0.0, O.key_state(m, torch.float64))
    W["l0.mix.left.k"] = W["l0.mix.left.k"] * 4
    assert torch.allclose(O.shared_value_attention(h, W, "l0.mix.left.", m, 0.0, O.key_state(m, torch.float64)), 4 * one)
