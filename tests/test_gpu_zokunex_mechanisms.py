"""Every mechanism of the Zokunex decoder alone, against the plain implementation (oracle/zokunex_oracle.py)."""

import math

import pytest
import torch

from oracle import zokunex_oracle as O
from tests import zokunex_cases as Z

pytestmark = pytest.mark.gpu
DTYPES = [torch.bfloat16, torch.float32]
BF16_STEP = 2.0 ** -8                      # spacing of bf16 below 2: the largest relative step a stored value can take


@pytest.fixture(scope="module")
def dev():
    assert torch.cuda.is_available()
    return torch.device("cuda:0")


@pytest.fixture(autouse=True)
def no_wait_ran_out(dev):
    yield
    from glorcq_b200 import dense
    torch.cuda.synchronize()
    assert dense.debug_error() is None


def rnd(*shape, seed=0, scale=1.0, dtype=torch.bfloat16):
    return (torch.randn(*shape, generator=torch.Generator().manual_seed(seed)) * scale).to(dtype)


# ---- products --------------------------------------------------------------------------------------------
ACT = {"none": lambda z: z, "relu2": lambda z: torch.relu(z) ** 2, "gelu_erf": O.gelu_erf}


@pytest.mark.parametrize("rows", [1, 3, 8, 9, 130, 300])
@pytest.mark.parametrize("N,K,split", [(48, 64, 48), (200, 104, 0), (270, 328, 136), (1000, 512, 995), (37, 44, 20), (600, 2080, 600)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_product(dev, rows, N, K, split, dtype):
    from glorcq_b200 import dense, layers
    x, W = rnd(rows, K, seed=rows), rnd(N, K, seed=N)
    for act, alpha in (("none", 0.5), ("relu2", 1.0), ("gelu_erf", 1.0)):
        ref = alpha * ACT[act](x.double() @ W.double().T)
        y, y32 = dense.matmul(x.to(dev, dtype), W.to(dev, dtype), split=split, act=layers.ACTIVATIONS[act], alpha=alpha)
        tol32 = 2e-5
        if split:
            assert y.dtype == dtype and y.shape == (rows, split)
            assert Z.stored(y, ref[:, :split], dtype) <= 1
        else:
            assert y is None
        if split < N:
            assert y32.dtype == torch.float32 and Z.worst_rel(y32, ref[:, split:]) < tol32


def test_product_forms(dev):
    """Each form of the product is the one that its sizes select."""
    import ctypes as C
    from glorcq_b200 import _lib
    x, W = torch.zeros(300, 128, device=dev, dtype=torch.bfloat16), torch.zeros(64, 128, device=dev, dtype=torch.bfloat16)

    def path(rows, K, dtype):
        a = _lib.DenseMM(dtype=dtype, N=64, K=K, rows=rows, ldx=128, x=x.data_ptr(), W=W.data_ptr())
        return _lib.dense().glq_dense_matmul_path(C.byref(a))
    assert [path(1, 128, 0), path(8, 128, 0), path(9, 128, 0), path(300, 128, 0)] == [1, 1, 2, 2]
    assert [path(1, 124, 0), path(300, 124, 0), path(300, 128, 1)] == [0, 0, 0]


def test_row_stride_and_rows_do_not_depend_on_the_batch(dev):
    from glorcq_b200 import dense
    x, W = rnd(400, 160, seed=1).to(dev), rnd(256, 96, seed=2).to(dev)
    whole = dense.matmul(x, W, split=0, ldx=160)[1]
    assert Z.rel(whole, x[:, :96].double().cpu() @ W.double().cpu().T) < 1e-5
    assert torch.equal(whole[:200], dense.matmul(x[:200], W, split=0, ldx=160)[1])
    few = dense.matmul(x[:5], W, split=0, ldx=160)[1]
    assert torch.equal(few[2:3], dense.matmul(x[2:3], W, split=0, ldx=160)[1])


# ---- norms -------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("rows,width", [(1, 104), (5, 50), (77, 1024), (3, 4099)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_norm_and_residual(dev, rows, width, dtype):
    from glorcq_b200 import dense
    x, y = rnd(rows, width, seed=1, dtype=torch.float32), rnd(rows, width, seed=2, dtype=torch.float32) * 3 + 7   # a mean to remove
    w, fw = rnd(width, seed=3, dtype=torch.float32), rnd(width, seed=4, dtype=torch.float32)
    for eps in (1e-5, 0.5):
        ref = x.double() + O.layer_norm(y.double(), w.double(), eps)
        xd = x.to(dev)
        h = dense.add_norm(xd, y.to(dev), w.to(dev), eps, dtype)
        assert Z.worst_rel(xd, ref) < 2e-6 and torch.equal(h, xd.to(dtype))
        xd = x.to(dev)
        h = dense.add_norm(xd, y.to(dev), w.to(dev), eps, dtype, fw.to(dev))
        assert Z.stored(h, O.layer_norm(ref, fw.double(), eps), dtype, 2e-6) <= 1


# ---- routing and experts -------------------------------------------------------------------------------------
@pytest.mark.parametrize("n", [1, 7, 33, 400, 1500])
@pytest.mark.parametrize("E,identity,top", [(6, 2, 3), (5, 0, 1), (40, 3, 8), (2, 1, 3), (300, 20, 4), (590, 10, 2)])
def test_routing(dev, n, E, identity, top):
    from glorcq_b200 import dense
    A = E + identity
    logits, corr = rnd(n, A, seed=n, dtype=torch.float32) * 2, rnd(A, seed=E, dtype=torch.float32) * 0.2
    sel, wt = O.route(logits.double(), {"r.router": torch.eye(A).double(), "r.correction": corr.double()}, "r.", top)
    p = dense.route(logits.to(dev), corr.to(dev), E, identity, top)
    assert torch.equal(p.sel.view(n, top).cpu(), sel.int())
    assert torch.allclose(p.wts.view(n, top).cpu().double(), wt, rtol=1e-5, atol=1e-7)
    te, er = p.tok_entries.cpu(), p.entry_row.cpu()
    entries = te[te >= 0]
    assert torch.equal((te >= 0).view(n, top), sel < E)                       # pass-through slots have no entry
    assert torch.equal(entries.sort().values, torch.arange(entries.numel(), dtype=torch.int32))
    assert torch.equal(er[te.clamp(min=0).long()][te >= 0], torch.arange(n).repeat_interleave(top)[te >= 0].int())
    # slots cover every entry once, with its expert
    ns = int(p.n_active[0])
    owner = torch.full((n * top,), -1)
    for s in range(ns):
        o, c = int(p.slot_offset[s]), int(p.slot_count[s])
        assert 0 < c <= p.max_slot_rows and (owner[o:o + c] == -1).all()
        owner[o:o + c] = int(p.active[s])
    assert torch.equal(owner[entries.long()], sel.reshape(-1)[te >= 0])
    assert (owner[entries.numel():] == -1).all()


@pytest.mark.parametrize("n", [1, 5, 20, 60, 700])
@pytest.mark.parametrize("E,identity,top,width,ff", [(6, 1, 3, 104, 40), (3, 2, 1, 50, 21), (16, 0, 4, 256, 96), (4, 3, 6, 64, 64)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_experts(dev, n, E, identity, top, width, ff, dtype):
    from glorcq_b200 import layers
    cfg = Z.config([(Z.mlstm(), Z.moe_mlp(E, identity, top, ff))], width=width)
    W = Z.make_weights(cfg, n + E)
    x = rnd(n, width, seed=n).float()
    # decisive choices: a router logit that is far ahead of its neighbours in a random order per token
    ff_mod = layers.RoutedFeedForward("gelu_erf", E, identity, top, lambda k: W["l0.mlp." + k], dev, dtype)
    sel, wt = O.route(x.double(), Z.doubles(W), "l0.mlp.", E + identity)
    score = torch.softmax(x.double() @ W["l0.mlp.router"].double().T, -1) + W["l0.mlp.correction"].double()
    ranked = score.sort(-1, descending=True).values
    clear = torch.ones(n, dtype=torch.bool) if top == E + identity else (ranked[:, top - 1] - ranked[:, top]) > 1e-4
    y = O.moe_ff(x.double(), Z.doubles(W), "l0.mlp.", {"experts": E, "top": top})
    norm_w = W["l0.norm2"].float()
    ref = x.double() + O.layer_norm(y, norm_w.double(), 1e-5)
    xd = x.to(dev)
    h = ff_mod.add(xd, x.to(dev, dtype), norm_w.to(dev), 1e-5)
    assert torch.equal(h, xd.to(dtype))
    assert clear.float().mean() > 0.5
    assert Z.worst_rel(xd.cpu()[clear], ref[clear]) < (0.02 if dtype == torch.bfloat16 else 2e-5)


def test_identity_experts_pass_the_layer_input_through(dev):
    """All tokens on pass-through experts: no expert runs, the sum is score times input."""
    from glorcq_b200 import layers
    cfg = Z.config([(Z.mlstm(), Z.moe_mlp(4, 2, 2, 40))])
    W = Z.make_weights(cfg, 8)
    W["l0.mlp.correction"] = torch.tensor([-9.0] * 4 + [9.0, 8.0])
    m = layers.RoutedFeedForward("gelu_erf", 4, 2, 2, lambda k: W["l0.mlp." + k], dev, torch.bfloat16)
    for n in (1, 40, 900):
        x = rnd(n, 104, seed=n).float()
        s = torch.softmax(x.double() @ W["l0.mlp.router"].double().T, -1)[:, 4:].sum(-1, keepdim=True)
        xd = x.to(dev)
        m.add(xd, x.to(dev).bfloat16(), torch.ones(104, device=dev), 1e-5)
        assert Z.worst_rel(xd, x.double() + O.layer_norm(s * x.double(), torch.ones(104).double(), 1e-5)) < 1e-4


# ---- matrix memory -------------------------------------------------------------------------------------------
def _mlstm_inputs(B, T, H, D, V, seed, f_shift=4.0):
    g = torch.Generator().manual_seed(seed)
    qkvg = torch.randn(B, T, 2 * H * (D + V), generator=g).bfloat16()
    gates = torch.randn(B, T, 2 * H, generator=g) * 3
    gates[..., H:] += f_shift
    return qkvg, gates, torch.randn(H, generator=g), torch.randn(H, generator=g), 1 + 0.2 * torch.randn(H * V, generator=g)


def _mlstm_oracle(qkvg, gates, bi, bf, nw, H, D, V, cap, eps, st):
    T = qkvg.shape[0]
    x = qkvg.double()
    q, k = x[:, :H * D].view(T, H, D) * D ** -0.5, x[:, H * D:2 * H * D].view(T, H, D)
    v, g = x[:, 2 * H * D:2 * H * D + H * V].view(T, H, V), x[:, 2 * H * D + H * V:]
    one, zero = torch.eye(H).double(), None
    i = O.log_gate_input(gates[:, :H].double(), one, bi.double(), cap)
    f = O.log_gate_forget(gates[:, H:].double(), one, bf.double(), cap)
    o = O.rms(O.mlstm_recurrence(q, k, v, i, f, st), eps).reshape(T, H * V)
    return o * nw.double() * torch.sigmoid(g)


def _run_mlstm(dev, dtype, ins, cuts, B, H, D, V, cap, eps, force_chunk=None):
    from glorcq_b200 import dense
    from glorcq_b200.cache import MatrixMemoryState
    qkvg, gates, bi, bf, nw = ins
    st = MatrixMemoryState(B, H, D, V, dev)
    outs = []
    for lo, hi in cuts:
        n = hi - lo
        chunk = force_chunk if force_chunk is not None else (n > 8 and dtype == torch.bfloat16)
        outs.append(dense.mlstm(qkvg[:, lo:hi].reshape(B * n, -1).to(dev, dtype), gates[:, lo:hi].reshape(B * n, -1).to(dev), B, n, H, D,
                                V, cap, eps, bi.to(dev), bf.to(dev), nw.to(dev), st, chunk).view(B, n, -1).cpu())
    return torch.cat(outs, 1), st


def _cuts(T, sizes):
    out, at = [], 0
    for s in sizes:
        if at < T:
            out.append((at, min(T, at + s)))
            at += s
    if at < T:
        out.append((at, T))
    return out


@pytest.mark.parametrize("H,D,V", [(2, 24, 40), (1, 8, 8), (3, 64, 64), (2, 72, 136), (1, 128, 256)])
@pytest.mark.parametrize("T,sizes", [(1, [1]), (2, [2]), (64, [64]), (65, [65]), (200, [200]), (200, [63, 2, 1, 64]), (130, [128]), (150, [9, 100])])
def test_matrix_memory_chunks_and_steps(dev, H, D, V, T, sizes):
    """Blocks of 64 positions and single steps in any mixture are the recurrence."""
    ins = _mlstm_inputs(2, T, H, D, V, T + D)
    for force in (None, True, False) if T <= 65 else (None, True):
        got, st = _run_mlstm(dev, torch.bfloat16, ins, _cuts(T, sizes), 2, H, D, V, 15.0, 1e-5, force)
        for b in range(2):
            s = O.mlstm_state({"heads": H, "dim": D, "vdim": V})
            ref = _mlstm_oracle(ins[0][b], ins[1][b], *ins[2:], H, D, V, 15.0, 1e-5, s)
            assert Z.worst_rel(got[b], ref) < 2 * BF16_STEP
            S = st.S[b].cpu().double().permute(0, 2, 1, 3).reshape(H, D, -1)[..., :V]
            assert Z.rel(S, s["S"]) < 3e-5 and Z.rel(st.n[b, :, -1], s["n"]) < 3e-5
            assert torch.allclose(st.m[b].cpu().double(), s["m"][:, None].expand_as(st.m[b].cpu()), atol=2e-4)


@pytest.mark.parametrize("H,D,V", [(3, 10, 13), (2, 40, 72), (1, 300, 33)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_matrix_memory_any_size_one_by_one(dev, H, D, V, dtype):
    ins = _mlstm_inputs(2, 40, H, D, V, D)
    got, _ = _run_mlstm(dev, dtype, ins, _cuts(40, [30, 1, 1]), 2, H, D, V, 7.5, 1e-3, False)
    for b in range(2):
        ref = _mlstm_oracle(ins[0][b], ins[1][b], *ins[2:], H, D, V, 7.5, 1e-3, O.mlstm_state({"heads": H, "dim": D, "vdim": V}))
        assert Z.worst_rel(got[b], ref) < (BF16_STEP if dtype == torch.bfloat16 else 3e-5)


@pytest.mark.parametrize("shift,spike", [(8.0, 40.0), (-30.0, 0.0), (0.0, -40.0)])
def test_matrix_memory_gate_extremes(dev, shift, spike):
    """Nothing forgotten after one strong early input; everything forgotten at once; inputs so weak that the starting
    maximum of zero decides the denominator."""
    H, D, V, T = 2, 32, 48, 190
    qkvg, gates, bi, bf, nw = _mlstm_inputs(1, T, H, D, V, 3, shift)
    if spike > 0:
        gates[..., :H] -= 12
        gates[:, 5, :H] = spike
    elif spike < 0:
        gates[..., :H] = spike
    for force in (True, False):
        got, _ = _run_mlstm(dev, torch.bfloat16, (qkvg, gates, bi, bf, nw), _cuts(T, [100]), 1, H, D, V, 15.0, 1e-5, force)
        ref = _mlstm_oracle(qkvg[0], gates[0], bi, bf, nw, H, D, V, 15.0, 1e-5, O.mlstm_state({"heads": H, "dim": D, "vdim": V}))
        assert Z.worst_rel(got[0], ref) < 2 * BF16_STEP


def test_matrix_memory_remembers_one_far_key(dev):
    """One key at position 3 that later queries match, hundreds of positions and many blocks away."""
    H, D, V, T = 1, 64, 64, 700
    qkvg, gates, bi, bf, nw = _mlstm_inputs(1, T, H, D, V, 9, 12.0)
    q, k, v = qkvg[0, :, :D], qkvg[0, :, D:2 * D], qkvg[0, :, 2 * D:2 * D + V]
    k *= 0.05
    k[3] = 4.0
    gates[..., :H] -= 6
    gates[0, 3, :H] = 6
    q[64] = q[65] = q[127] = q[699] = 1.0
    got, _ = _run_mlstm(dev, torch.bfloat16, (qkvg, gates, bi, bf, nw), _cuts(T, [3, 61, 1]), 1, H, D, V, 15.0, 1e-6)
    ref = _mlstm_oracle(qkvg[0], gates[0], bi, bf, nw, H, D, V, 15.0, 1e-6, O.mlstm_state({"heads": H, "dim": D, "vdim": V}))
    clean = qkvg.clone()
    clean[0, 3, D:2 * D] = 0
    other = _mlstm_oracle(clean[0], gates[0], bi, bf, nw, H, D, V, 15.0, 1e-6, O.mlstm_state({"heads": H, "dim": D, "vdim": V}))
    for t in (64, 65, 127, 699):
        assert Z.rel(other[t], ref[t]) > 0.3                # the key shows
        assert Z.rel(got[0, t], ref[t]) < 2 * BF16_STEP


# ---- latent attention ------------------------------------------------------------------------------------------
LATENT_SIZES = [(3, 16, 8, 24, 48), (2, 40, 16, 16, 32), (5, 24, 8, 40, 144), (4, 128, 64, 128, 512), (2, 9, 6, 11, 20), (1, 200, 24, 8, 272), (20, 8, 8, 8, 16),
                (2, 16, 8, 16, 80), (2, 16, 8, 16, 96), (1, 24, 16, 8, 112), (3, 5, 4, 7, 9)]


def _latent_mixer(dev, dtype, sizes, seed=0, width=64, scale=None, base=10000.0):
    from glorcq_b200.layers import LatentAttentionMixer
    H, D, R, V, K = sizes
    cfg = Z.config([(Z.latent(H, D, R, V, K, base, scale), None)], width=width)
    W, m = Z.make_weights(cfg, seed), cfg["layers"][0]["mixer"]
    mixer = LatentAttentionMixer(H, D, R, V, K, m["rot"]["base"], R, m["scale"], 1e-5, lambda k: W["l0.mix." + k], dev, dtype)
    return mixer, W, m


def _run_mixer(mixer, x, cuts, max_len, dev, dtype):
    """x (B, T, width)"""
    B = x.shape[0]
    st = mixer.make_state(B, max_len, dev, dtype)
    outs = []
    for lo, hi in cuts:
        y = mixer(x[:, lo:hi].reshape(-1, x.shape[-1]).to(dev, dtype), B, hi - lo, torch.arange(lo, hi, device=dev),
                  hi if hi - lo > 1 else None, st)
        outs.append(y.view(B, hi - lo, -1).cpu())
    return torch.cat(outs, 1), st


@pytest.mark.parametrize("sizes", LATENT_SIZES)
@pytest.mark.parametrize("T,parts", [(1, [1]), (8, [8]), (9, [9]), (64, [64]), (150, [150]), (150, [2, 62, 1, 64, 1, 3]), (100, [97, 1, 1, 1]), (70, [5, 1, 33, 2])])
@pytest.mark.parametrize("dtype", DTYPES)
def test_latent_attention(dev, sizes, T, parts, dtype):
    mixer, W, m = _latent_mixer(dev, dtype, sizes, seed=T)
    x = rnd(2, T, 64, seed=T)
    got, _ = _run_mixer(mixer, x, _cuts(T, parts), T + 3, dev, dtype)
    for b in range(2):
        ref = O.latent_attention_mixer(x[b].double(), Z.doubles(W), "l0.mix.", m, 1e-5, O.latent_state(m))
        assert Z.worst_rel(got[b], ref) < (0.04 if dtype == torch.bfloat16 else 3e-5)


@pytest.mark.parametrize("far", [0, 1, 31, 32, 63, 64, 127, 128])
def test_latent_attention_far_and_edge_keys(dev, far):
    """One key stands out for every query; the next and the previous position must not take its place, whichever form of
    the kernel sees it and whichever block of positions it lies in."""
    sizes, T = (2, 32, 8, 24, 64), 200
    mixer, W, m = _latent_mixer(dev, torch.bfloat16, sizes, seed=1, scale=1.0)
    W = {k: v.clone() for k, v in W.items()}
    x = rnd(1, T, 64, seed=2) * 0.02
    x[0, :, 0] = 1.0                                        # constant channel: the queries
    x[0, far, 1] = 8.0                                      # marks the key
    H, D, R, V, K = sizes
    W["l0.mix.q"].zero_()
    W["l0.mix.q"].view(H, D + R, 64)[:, 0, 0] = 4.0
    W["l0.mix.dkv"][0, 1] = 6.0
    W["l0.mix.uk"].zero_()
    W["l0.mix.uk"].view(H, D, K)[:, 0, 0] = 4.0
    from glorcq_b200.layers import LatentAttentionMixer
    mixer = LatentAttentionMixer(H, D, R, V, K, 10000.0, R, 1.0, 1e-5, lambda k: W["l0.mix." + k], dev, torch.bfloat16)
    for parts in ([T], [far + 1, 2, 1, 30], [far + 1] + [1] * 12, [max(far, 1), 3, 5]):
        got, _ = _run_mixer(mixer, x, _cuts(T, parts), 256, dev, torch.bfloat16)
        ref = O.latent_attention_mixer(x[0].double(), Z.doubles(W), "l0.mix.", m | {"scale": 1.0}, 1e-5, O.latent_state(m))
        assert Z.worst_rel(got[0], ref) < 0.03
    without = x.clone()
    without[0, far, 1] = 0.0
    other = O.latent_attention_mixer(without[0].double(), Z.doubles(W), "l0.mix.", m | {"scale": 1.0}, 1e-5, O.latent_state(m))
    assert Z.rel(other[far:], ref[far:]) > 0.5
    if far:
        assert Z.rel(other[:far], ref[:far]) < 1e-9         # nobody sees the future


def test_latent_cache_rows(dev):
    """What is stored: the normed latent and the turned shared key part, at the positions given."""
    for sizes in ((2, 16, 8, 24, 48), (2, 9, 6, 11, 20)):
        mixer, W, m = _latent_mixer(dev, torch.float32, sizes, base=50.0)
        x, st0 = rnd(1, 40, 64, seed=4), O.latent_state(m)
        O.latent_attention_mixer(x[0].double(), Z.doubles(W), "l0.mix.", m, 1e-5, st0)
        _, st = _run_mixer(mixer, x, [(0, 17), (17, 18), (18, 40)], 64, dev, torch.float32)
        assert Z.worst_rel(st.rows[0, :40, :sizes[4]], st0["c"]) < 1e-5
        assert Z.worst_rel(st.rows[0, :40, sizes[4]:sizes[4] + sizes[2]], st0["r"]) < 1e-5


def test_rotation_covers_only_the_first_dims(dev):
    """rot.dims smaller than the rotated part: the rest passes through."""
    from glorcq_b200.layers import LatentAttentionMixer
    sizes = (2, 16, 16, 24, 48)
    H, D, R, V, K = sizes
    _, W, m = _latent_mixer(dev, torch.float32, sizes)
    m = m | {"rot": {"base": 30.0, "dims": 6}}
    mixer = LatentAttentionMixer(H, D, R, V, K, 30.0, 6, m["scale"], 1e-5, lambda k: W["l0.mix." + k], dev, torch.float32)
    x = rnd(1, 50, 64, seed=4)
    got, _ = _run_mixer(mixer, x, [(0, 45), (45, 46), (46, 50)], 64, dev, torch.float32)
    ref = O.latent_attention_mixer(x[0].double(), Z.doubles(W), "l0.mix.", m, 1e-5, O.latent_state(m))
    assert Z.worst_rel(got[0], ref) < 3e-5


def test_output_projection_and_argmax(dev):
    from glorcq_b200 import dense
    for rows, width, vocab in ((1, 96, 160), (11, 64, 1000), (3, 104, 333), (100, 96, 160), (2, 2784, 200)):
        x, W = rnd(rows, width, seed=rows), rnd(vocab, width, seed=vocab)
        logits, best = dense.head(x.to(dev), W.to(dev), 0.37, {})
        ref = 0.37 * x.double() @ W.double().T
        assert Z.worst_rel(logits, ref) < 1e-5
        if width % 32 == 0 and rows <= 64:
            assert torch.equal(best.cpu(), logits.cpu().argmax(-1))
        else:
            assert best is None
