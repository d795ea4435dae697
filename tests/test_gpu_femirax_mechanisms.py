"""Every mechanism of the Femirax decoder alone, against the plain implementation (oracle/femirax_oracle.py)."""

import pytest
import torch

from oracle import femirax_oracle as O
from tests import femirax_cases as F

pytestmark = pytest.mark.gpu
DTYPES = [torch.bfloat16, torch.float32]
BF16_STEP = 2.0 ** -8


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


def cuts_of(T, sizes):
    out, at = [], 0
    for s in list(sizes) + [T]:
        if at < T:
            out.append((at, min(T, at + s)))
            at += s
    return out


# ---- products --------------------------------------------------------------------------------------------
SIZES = [(48, 64), (40, 104), (11, 44), (200, 328), (600, 2080), (21, 96)]


@pytest.mark.parametrize("rows", [1, 3, 8, 9, 130, 300])
@pytest.mark.parametrize("N,K", SIZES)
@pytest.mark.parametrize("dtype", DTYPES)
def test_gated_product(dev, rows, N, K, dtype):
    from glorcq_b200 import _lib, dense
    x, g, u = rnd(rows, K, seed=rows), rnd(N, K, seed=N, scale=K ** -0.5), rnd(N, K, seed=N + 1)
    ref = O.silu(x.double() @ g.double().T) * (x.double() @ u.double().T)
    y = dense.matmul(x.to(dev, dtype), dense.gated_rows(g, u).to(dev, dtype), act=_lib.ACT_SILU_GLU)[0]
    assert y.dtype == dtype and y.shape == (rows, (N + 7) // 8 * 8)
    assert F.stored(y[:, :N], ref, dtype) <= 1 and not y[:, N:].any()


@pytest.mark.parametrize("rows", [1, 5, 9, 200])
@pytest.mark.parametrize("N,K", SIZES)
@pytest.mark.parametrize("dtype", DTYPES)
def test_product_times_a_row_of_a_table(dev, rows, N, K, dtype):
    """The per-token factor: row ids[r] of some columns of a wider table."""
    from glorcq_b200 import _lib, dense
    x, W, table = rnd(rows, K, seed=rows), rnd(N, K, seed=N, scale=K ** -0.5), rnd(31, 3 * N + 5, seed=7)
    ids = torch.randint(0, 31, (rows,), generator=torch.Generator().manual_seed(1))
    ref = O.gelu_tanh(x.double() @ W.double().T) * table[ids, N:2 * N].double()
    y = dense.matmul(x.to(dev, dtype), W.to(dev, dtype), act=_lib.ACT_GELU_TANH, mul=table.to(dev, dtype)[:, N:2 * N], mul_row=ids.to(dev))[0]
    assert F.stored(y, ref, dtype) <= 1


@pytest.mark.parametrize("rows", [1, 8, 9, 130, 300])
@pytest.mark.parametrize("N,K", SIZES)
@pytest.mark.parametrize("dtype", DTYPES)
def test_product_added_to_the_residual(dev, rows, N, K, dtype):
    from glorcq_b200 import dense
    y, W, x = rnd(rows, K, seed=rows), rnd(N, K, seed=N), rnd(rows, N, seed=2, scale=30.0, dtype=torch.float32)
    ref = x.double() + y.double() @ W.double().T
    for copy in (False, True):
        xd = x.to(dev)
        h = dense.matmul_add(y.to(dev, dtype), W.to(dev, dtype), xd, copy)
        assert F.worst_rel(xd, ref) < 2e-5
        assert torch.equal(h, xd.to(dtype)) if copy else h is None


@pytest.mark.parametrize("heads,vdim,width", [(2, 64, 96), (1, 40, 104), (4, 256, 640), (3, 24, 48), (1, 2048, 96), (2, 600, 64)])
def test_head_norm_and_gate_inside_the_product(dev, heads, vdim, width):
    """Rows of a recurrence's output, normed per head and gated where the product stages them; values shared out to the
    warps in every way."""
    from glorcq_b200 import dense
    K = heads * vdim
    W, nw = rnd(width, K, seed=1, scale=K ** -0.5), rnd(K, seed=2, dtype=torch.float32)
    for rows in (1, 2, 5, 8):
        o, g = rnd(rows, K, seed=rows, dtype=torch.float32), rnd(rows, K, seed=9)
        n = O.rms(o.double().view(rows, heads, vdim), 1e-4).reshape(rows, K) * nw.double()
        got = dense.head_norm_matmul(o.to(dev), g.to(dev), nw.to(dev), heads, 1e-4, W.to(dev))
        assert F.worst_rel(got, (n * torch.sigmoid(g.double())) @ W.double().T) < 1.5 * BF16_STEP


# ---- norms -------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("rows,width", [(1, 104), (5, 50), (77, 1024), (3, 4099), (4, 3000), (2, 5120)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_rms_norms_around_the_residual_add(dev, rows, width, dtype):
    from glorcq_b200 import dense
    x, y, y2 = (rnd(rows, width, seed=s, dtype=torch.float32) * f + o for s, f, o in ((1, 1, 0), (2, 3, 7), (3, 0.01, 0)))
    w, w2, hw = (rnd(width, seed=s, dtype=torch.float32) for s in (4, 5, 6))
    dv = [t.to(dev) for t in (y, w, y2, w2, hw)]
    d = [t.double() for t in (y, w, y2, w2, hw)]
    strided = torch.cat([y, y], 1).to(dev)[:, :width]              # rows further apart than they are long
    for eps in (1e-6, 0.5):
        for add, got_kw in ((0 * d[0], {}), (d[0], dict(y=dv[0])), (d[0], dict(y=strided)), (O.rms(d[0], eps) * d[1], dict(y=dv[0], w=dv[1])),
                            (0.5 * (O.rms(d[0], eps) * d[1] + O.rms(d[2], eps) * d[3]), dict(y=dv[0], w=dv[1], y2=dv[2], w2=dv[3], alpha=0.5))):
            ref = x.double() + add
            xd = x.to(dev)
            h = dense.rms_add(xd, eps, dtype, **got_kw)
            assert F.worst_rel(xd, ref) < 2e-6 and torch.equal(h, xd.to(dtype))
            xd = x.to(dev)
            h = dense.rms_add(xd, eps, dtype, **got_kw, norm_w=dv[4])
            assert F.worst_rel(xd, ref) < 2e-6 and F.stored(h, O.rms(ref, eps) * d[4], dtype, 2e-6) <= 1


@pytest.mark.parametrize("dtype", DTYPES)
def test_embedding_with_the_first_norm(dev, dtype):
    from glorcq_b200 import dense
    for width in (50, 104, 2056):
        table, hw = rnd(40, width, seed=1), rnd(width, seed=2, dtype=torch.float32)
        ids = torch.tensor([0, 39, 7, 7])
        x, h = dense.embed(ids.to(dev), table.to(dev, dtype), hw.to(dev), 1e-3)
        assert torch.equal(x.cpu(), table[ids].float())
        assert F.stored(h, O.rms(table[ids].double(), 1e-3) * hw.double(), dtype, 2e-6) <= 1


# ---- linear attention with decay ---------------------------------------------------------------------------
class Linear:
    """One call's operands (columns of one row-major product) and its plain evaluation."""

    def __init__(self, B, T, H, D, V, seed=0, rank=None, tau=16.0, decay=None, rot=None, qs=1.0, ks=1.0, norm="none", gate="silu", z_shift=2.0,
                 z_scale=2.0):
        self.B, self.T, self.H, self.D, self.V, self.qs, self.ks, self.gate, self.tau, self.rot = B, T, H, D, V, qs, ks, gate, tau, rot
        self.rows = rnd(B, T, 2 * H * (D + V), seed=seed)
        self.decay = decay if decay is not None or rank else [1 - 0.4 ** (i + 1) for i in range(H)]
        self.rank = rank
        if rank:
            self.a, self.a2 = rnd(B, T, rank, seed=seed + 1, dtype=torch.float32), rnd(H * D, rank, seed=seed + 2, scale=z_scale * rank ** -0.5)
            self.a2b = z_shift + rnd(H * D, seed=seed + 3, dtype=torch.float32)
        self.norm_w = {"none": None, "shared": 1 + rnd(V, seed=4, dtype=torch.float32, scale=0.3),
                       "each": 1 + rnd(H * V, seed=4, dtype=torch.float32, scale=0.3)}[norm]

    def plain(self, b, S=None):
        T, H, D, V = self.T, self.H, self.D, self.V
        q, k, v, g = self.rows[b].double().split([H * D, H * D, H * V, H * V], 1)
        q, k, v = q.view(T, H, D), k.view(T, H, D), v.view(T, H, V)
        if self.rot:
            dims, base, pairs = self.rot
            turn = O.rotate_pairs if pairs else O.rotate_halves
            q, k = (turn(t, torch.arange(T), base, dims) for t in (q, k))
        if self.rank:
            z = self.a[b].double() @ self.a2.double().T + self.a2b.double()
            alpha = torch.exp(torch.nn.functional.logsigmoid(z) / self.tau).view(T, H, D)
        else:
            alpha = torch.tensor(self.decay, dtype=torch.float64)[None, :, None]
        self.S = torch.zeros(H, D, V, dtype=torch.float64) if S is None else S
        self.o = O.decayed_recurrence(q * self.qs, k * self.ks, v, alpha, self.S)
        n = O.rms(self.o, 1e-5)
        if self.norm_w is not None:
            n = n * self.norm_w.double().view(-1, V)
        return n.reshape(T, H * V) * (O.silu if self.gate == "silu" else torch.sigmoid)(g)

    def run(self, dev, dtype, cuts, short=None):
        from glorcq_b200 import _lib, dense
        from glorcq_b200.cache import DecayState
        from glorcq_b200.layers import Rotation
        B, H, D, V = self.B, self.H, self.D, self.V
        st = DecayState(B, self.T + 4, H, D, V, dev)
        rot = Rotation(*self.rot)(st.max_len, dev) if self.rot else None
        outs = []
        for lo, hi in cuts:
            n = hi - lo
            y = self.rows[:, lo:hi].reshape(B * n, -1).to(dev, dtype)
            q, k, v, g = y.split([H * D, H * D, H * V, H * V], 1)
            kw = dict(gates=(self.a[:, lo:hi].reshape(B * n, -1).contiguous().to(dev), self.a2.to(dev, dtype), self.a2b.to(dev), self.tau)) \
                if self.rank else dict(decay=torch.tensor(self.decay).to(dev))
            out = dense.decay_attention(q, k, v, g, B, n, H, D, V, st, None if self.norm_w is None else self.norm_w.to(dev), 1e-5,
                                        _lib.GATE_SILU if self.gate == "silu" else _lib.GATE_SIGMOID, rotation=rot,
                                        start=torch.tensor([lo], device=dev), q_scale=self.qs, k_scale=self.ks,
                                        short=n <= 8 if short is None else short, **kw)
            outs.append(out.view(B, n, -1).cpu())
        return torch.cat(outs, 1), st

    def state(self, st, b):
        return st.S[b].cpu().double().permute(0, 2, 1, 3).reshape(self.H, self.D, -1)[..., :self.V]


def check_linear(dev, case, cuts, forms, dtype=torch.bfloat16, exact=4e-5, state_tol=3e-5):
    for short in forms:
        got, st = case.run(dev, dtype, cuts, short)
        for b in range(case.B):
            ref = case.plain(b)
            assert F.stored(got[b], ref, dtype, exact) <= 1
            assert F.rel(case.state(st, b), case.S) < state_tol


LINEAR_SIZES = [(2, 24, 40), (1, 8, 8), (3, 64, 64), (2, 72, 136), (1, 128, 256), (2, 128, 128), (4, 16, 72)]
LENGTHS = [(1, [1]), (2, [2]), (16, [16]), (17, [17]), (64, [64]), (65, [65]), (200, [200]), (200, [63, 2, 1, 64]), (150, [9, 100]), (80, [2, 12, 2, 49])]


@pytest.mark.parametrize("H,D,V", LINEAR_SIZES)
@pytest.mark.parametrize("T,sizes", LENGTHS)
def test_retention_chunks_and_steps(dev, H, D, V, T, sizes):
    """Chunks of 64 and single steps in any mixture are the recurrence, with rotation and key scale."""
    case = Linear(2, T, H, D, V, seed=T + D, rot=(D, 1e4, False), ks=D ** -0.5)
    check_linear(dev, case, cuts_of(T, sizes), (None, False, True) if T <= 65 else (None, False))


@pytest.mark.parametrize("H,D,V", LINEAR_SIZES)
@pytest.mark.parametrize("T,sizes", LENGTHS)
@pytest.mark.parametrize("rank", [16, 5])
def test_gated_linear_attention_chunks_and_steps(dev, H, D, V, T, sizes, rank):
    case = Linear(2, T, H, D, V, seed=T + D, rank=rank, norm="shared", qs=D ** -0.5)
    check_linear(dev, case, cuts_of(T, sizes), (None, False, True) if T <= 65 else (None, False))


@pytest.mark.parametrize("H,D,V", [(3, 10, 13), (2, 40, 72), (1, 300, 33), (2, 16, 512), (1, 8, 530)])
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rank", [None, 1, 40])
def test_any_size_one_by_one(dev, H, D, V, dtype, rank):
    case = Linear(2, 40, H, D, V, seed=D, rank=rank, tau=3.0, norm="each", gate="sigmoid", rot=(4, 30.0, True))
    check_linear(dev, case, cuts_of(40, [30, 1, 1]), (True,), dtype)


@pytest.mark.parametrize("dims,pairs", [(2, False), (16, False), (24, False), (48, False), (64, False), (10, True), (64, True)])
def test_rotations_in_chunks(dev, dims, pairs):
    case = Linear(1, 100, 2, 64, 32, seed=dims, rot=(dims, 50.0, pairs))
    check_linear(dev, case, cuts_of(100, [37, 2, 40]), (None, False))


@pytest.mark.parametrize("decay", [[0.0, 1.0], [1e-6, 0.5], [0.03, 0.9999]])
def test_retention_decay_extremes(dev, decay):
    """Nothing kept, everything kept, and what lies far below and close to one."""
    case = Linear(1, 150, 2, 32, 48, seed=3, decay=decay)
    check_linear(dev, case, cuts_of(150, [70, 3]), (None, False, True))


@pytest.mark.parametrize("shift,scale,tau", [(-30.0, 1.0, 1.0), (20.0, 1.0, 16.0), (0.0, 12.0, 1.0), (-200.0, 50.0, 1.0), (-3.0, 3.0, 0.5), (1.0, 4.0, 64.0)])
def test_gated_decay_extremes(dev, shift, scale, tau):
    """Channels that forget at once beside channels that keep everything, in one block: no factor may overflow, and what
    is forgotten must not hide what is kept."""
    case = Linear(1, 150, 2, 32, 48, seed=3, rank=8, tau=tau, z_shift=shift, z_scale=scale)
    check_linear(dev, case, cuts_of(150, [70, 3]), (None, False, True), state_tol=1e-4)


@pytest.mark.parametrize("far", [0, 3, 15, 16, 62, 63, 64, 127, 128])
@pytest.mark.parametrize("rank", [None, 4])
def test_one_far_key(dev, far, rank):
    """One key that later queries match, at the edges of blocks and chunks, hundreds of positions away."""
    H, D, V, T = 1, 64, 64, 600
    case = Linear(1, T, H, D, V, seed=9, rank=rank, decay=None if rank else [0.9995], z_shift=9.0, z_scale=0.2)
    q, k = case.rows[0, :, :D], case.rows[0, :, D:2 * D]
    k *= 0.02
    k[far] = 4.0
    seen = [t for t in (far, far + 1, 64, 65, 129, 599) if t >= far]
    q[seen] = 1.0
    ref = case.plain(0)
    k[far] = 0.0
    other = case.plain(0)
    k[far] = 4.0
    for sizes in ([T], [max(far, 1), 61, 1], [far + 1, 2, 9]):
        got, _ = case.run(dev, torch.bfloat16, cuts_of(T, sizes))
        for t in seen:
            assert F.rel(other[t], ref[t]) > 0.3 and F.rel(got[0, t], ref[t]) < 2 * BF16_STEP
    assert torch.equal(other[:far], ref[:far])


def test_long_decoding_keeps_the_state(dev):
    """Two thousand single steps behind a prompt, the state in 32-bit all along."""
    for rank in (None, 16):
        case = Linear(1, 2100, 2, 32, 32, seed=5, rank=rank, decay=None if rank else [0.999, 0.9], rot=(32, 1e6, False), z_shift=6.0, ks=0.2)
        got, st = case.run(dev, torch.bfloat16, [(0, 90), (90, 92)] + [(i, i + 8) for i in range(92, 2092, 8)] + [(i, i + 1) for i in range(2092, 2100)])
        ref = case.plain(0)
        assert F.stored(got[0], ref, torch.bfloat16, 1e-4) <= 1 and F.rel(case.state(st, 0), case.S) < 3e-5


def test_prompts_longer_than_a_segment(dev):
    """The workspace holds 4096 positions at a time."""
    for rank in (None, 4):
        case = Linear(1, 4200, 1, 16, 16, seed=2, rank=rank, decay=None if rank else [0.998], z_shift=5.0, rot=(16, 1e4, False))
        check_linear(dev, case, [(0, 4200)], (None,), state_tol=1e-4)


# ---- grouped-query attention -------------------------------------------------------------------------------
ATTN_SIZES = [(4, 2, 16, 16), (3, 1, 24, 24), (2, 2, 64, 64), (8, 2, 128, 128), (6, 3, 8, 8), (20, 1, 40, 40), (2, 1, 256, 256), (4, 4, 72, 72), (2, 1, 64, 136)]
ODD_SIZES = [(6, 2, 9, 9), (2, 1, 12, 7), (1, 1, 300, 20)]


class Attn:
    def __init__(self, sizes, B, T, seed=0, rot=None, scale=None, norm=True, own_values=False, dtype=torch.bfloat16):
        self.H, self.G, self.D, self.V = sizes
        self.B, self.T, self.norm, self.dtype = B, T, norm, dtype
        self.rot = rot or (self.D // 4 * 2, 100.0, True)
        self.scale = scale or 3 * self.D ** -0.5
        self.own = own_values or self.V != self.D
        self.rows = rnd(B, T, (self.H + self.G) * self.D + (self.G * self.V if self.own else 0), seed=seed)

    def plain(self, b):
        T, H, G, D, V = self.T, self.H, self.G, self.D, self.V
        x = self.rows[b].double()
        q, k = x[:, :H * D].view(T, H, D), x[:, H * D:(H + G) * D].view(T, G, D)
        v = x[:, (H + G) * D:].view(T, G, V) if self.own else k
        turn = O.rotate_pairs if self.rot[2] else O.rotate_halves
        q, k = (turn(t, torch.arange(T), self.rot[1], self.rot[0]) for t in (q, k))
        if self.norm:
            q, k = O.rms(q, 1e-5), O.rms(k, 1e-5)
        self.k, self.v = k, v
        return O.causal_attention(q, k, v, self.scale, 0).reshape(T, H * V)

    def run(self, dev, cuts, max_len=None):
        from glorcq_b200 import dense
        from glorcq_b200.cache import KeyValueState
        from glorcq_b200.layers import Rotation
        B, H, G, D, V = self.B, self.H, self.G, self.D, self.V
        st = KeyValueState(B, max_len or self.T + 3, G, D, V, dev, self.dtype)
        rot = Rotation(*self.rot)(st.k.shape[1], dev)
        outs = []
        for lo, hi in cuts:
            n = hi - lo
            y = self.rows[:, lo:hi].reshape(B * n, -1).to(dev, self.dtype)
            pad = torch.zeros(B * n, dense.ceil_to(y.shape[1], 8), dtype=self.dtype, device=dev)
            pad[:, :y.shape[1]] = y
            q, k = pad[:, :H * D], pad[:, H * D:(H + G) * D]
            v = pad[:, (H + G) * D:(H + G) * D + G * V] if self.own else k
            out = dense.gqa(q, k, v, B, n, H, G, D, V, st, self.scale, 1e-5, torch.arange(lo, hi, device=dev), hi if n > 1 else None, rot, self.norm)
            outs.append(out.view(B, n, -1).cpu())
        return torch.cat(outs, 1), st


PARTS = [(1, [1]), (8, [8]), (9, [9]), (64, [64]), (150, [150]), (150, [2, 62, 1, 64, 1, 3]), (100, [97, 1, 1, 1]), (330, [300, 5, 2, 1]), (70, [5, 1, 33, 2])]


@pytest.mark.parametrize("sizes", ATTN_SIZES + ODD_SIZES)
@pytest.mark.parametrize("T,parts", PARTS)
@pytest.mark.parametrize("dtype", DTYPES)
def test_attention(dev, sizes, T, parts, dtype):
    case = Attn(sizes, 2, T, seed=T, dtype=dtype)
    got, st = case.run(dev, cuts_of(T, parts))
    for b in range(2):
        ref = case.plain(b)
        assert F.worst_rel(got[b], ref) < (0.03 if dtype == torch.bfloat16 else 3e-5)
        assert F.stored(st.k[b, :T], case.k, dtype) <= 1 and F.stored(st.v[b, :T], case.v, dtype) <= 1


def test_attention_forms(dev):
    """Each form is the one that its sizes select."""
    import ctypes as C
    from glorcq_b200 import _lib

    def form(T, D, V, dtype=0):
        t = torch.zeros(8, 4096, device=dev)
        p = t.data_ptr()
        a = _lib.Gqa(dtype=dtype, B=1, T=T, H=4, G=2, D=D, V=V, max_len=400, ldp=4096, q=p, k=p, v=p, kc=p, vc=p, out=p)
        return _lib.dense().glq_gqa_form(C.byref(a))
    assert [form(1, 64, 64), form(8, 64, 64), form(9, 64, 64), form(9, 256, 256), form(1, 256, 256)] == [1, 1, 2, 2, 1]
    assert [form(1, 64, 64, 1), form(9, 60, 64), form(9, 264, 64), form(1, 64, 264)] == [0, 0, 0, 2]


@pytest.mark.parametrize("norm,pairs,dims", [(False, False, 32), (True, False, 12), (False, True, 32), (True, True, 2)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_attention_variants(dev, norm, pairs, dims, dtype):
    """Rotation layouts and extents, without the norm, with values of their own."""
    case = Attn((6, 2, 32, 32), 1, 90, seed=dims, rot=(dims, 40.0, pairs), norm=norm, own_values=True, scale=0.3, dtype=dtype)
    got, _ = case.run(dev, cuts_of(90, [60, 1, 5, 2]))
    assert F.worst_rel(got[0], case.plain(0)) < (0.03 if dtype == torch.bfloat16 else 3e-5)


@pytest.mark.parametrize("far", [0, 1, 15, 16, 63, 64, 127, 128, 255, 256, 700])
@pytest.mark.parametrize("dtype", DTYPES)
def test_attention_far_and_edge_keys(dev, far, dtype):
    """One key that every query's score puts far ahead, in whichever block or split it lies; its neighbours must not take
    its place, and no earlier query may see it."""
    T = 760
    case = Attn((4, 2, 32, 32), 1, T, seed=2, rot=(0, 1.0, True), scale=0.6, dtype=dtype)
    x = case.rows
    x[0, :, :4 * 32] = 0.1 * x[0, :, :4 * 32] + 1.0              # queries along one direction
    keys = x[0, :, 4 * 32:].view(T, 2, 32)
    keys[..., 0] -= keys.float().sum(-1).to(keys.dtype)              # keys across it ..
    keys[far] = 1.0 + 0.1 * keys[far]                                # .. but one
    ref = case.plain(0)
    for parts in ([T], [far + 1, 2, 1, 30], [max(far, 1)] + [1] * 6 + [300]):
        got, _ = case.run(dev, cuts_of(T, parts), 1024)
        assert F.worst_rel(got[0], ref) < (0.03 if dtype == torch.bfloat16 else 3e-5)
    assert (ref[far:] - ref[far]).abs().max() < 0.2 * ref[far].abs().max()       # the key decides
    if far:
        assert F.rel(ref[:far], ref[far].expand(far, -1)) > 0.3


def test_attention_splits_of_a_long_cache(dev):
    """Single positions and short portions behind thousands of cached ones; more rows than one tile; a nearly empty cache
    of the same length."""
    for sizes in ((8, 2, 64, 64), (24, 1, 128, 128)):
        case = Attn(sizes, 2, 3010, seed=1)
        cuts = cuts_of(3010, [3, 1, 2900, 1, 1, 8, 7])
        got, _ = case.run(dev, cuts, 8192)
        for b in range(2):
            assert F.worst_rel(got[b], case.plain(b)) < 0.03


# ---- sublayers ---------------------------------------------------------------------------------------------
@pytest.mark.parametrize("name", F.CONFIGS)
@pytest.mark.parametrize("dtype", DTYPES)
def test_sublayers(dev, name, dtype):
    """Mixer, feed-forward and token input of every layer on given inputs, with and without a following norm."""
    from glorcq_b200.femirax import FemiraxDecoder
    cfg, w = F.CONFIGS[name], F.weights_of(name)
    W, m, eps = F.doubles(w), FemiraxDecoder(cfg, w, dev, dtype), cfg["norm"]["eps"]
    C = cfg["width"]
    tol = 3e-5 if dtype == torch.float32 else 0.05
    nw = rnd(C, seed=3, dtype=torch.float32)
    for l, L in enumerate(cfg["layers"]):
        for T in (1, 7, 90):
            h, x, ids = rnd(T, C, seed=T + l), rnd(T, C, seed=5, dtype=torch.float32), torch.tensor(F.tokens(cfg, T))
            mixer = {"retention": O.retention_mixer, "parallel": O.parallel_mixer}[L["type"]]
            start, kv, e = torch.arange(T, device=dev), T if T > 1 else None, W["side.embed"][ids][:, l * cfg["token_side"]["dim"]:][:, :cfg["token_side"]["dim"]]
            refs = [x.double() + mixer(h.double(), W, f"l{l}.mix.", L["mixer"], eps, O.new_state(cfg)[l])]
            calls = [lambda xd, n: m.mixers[l].add(xd, h.to(dev, dtype), 1, T, start, kv, m.make_cache(1, T + 2)[l], n)]
            if L["mlp"]:
                refs.append(x.double() + O.gated_ff(h.double(), W, f"l{l}.mlp."))
                calls.append(lambda xd, n: m.mlps[l].add(xd, h.to(dev, dtype), n))
            refs.append(O.token_side(x.double(), e, W, f"l{l}.side.", eps))
            calls.append(lambda xd, n: m.sides[l].add(xd, xd.to(dtype), ids.to(dev), n))
            for ref, call in zip(refs, calls):
                for n in (None, nw):
                    xd = x.to(dev)
                    out = call(xd, None if n is None else n.to(dev))
                    assert F.worst_rel(xd, ref) < tol, (l, T)
                    want = xd.cpu().double() if n is None else O.rms(xd.cpu().double(), eps) * n.double()
                    assert out.dtype == dtype and F.stored(out, want, dtype) <= 1
