"""Sublayers of the unquantized decoders.  Each takes its constants and weights as arguments; a model design is an
assembly of them (``zokunex``).

Mixers: ``forward(h, B, T, start, kv_len, state) -> y32`` for rows ``h`` (B*T, width) of the layer's input, positions
``start`` (device, int64) .. start + T - 1 of every sequence; ``kv_len`` = start + T on the host, or None inside a
decode step, whose position stays on the device.  Feed-forwards: ``add(x, h, norm, final) -> h'`` runs the sublayer on
``h`` and folds its output's norm and the residual add of ``x`` into the last launch.

Sublayers of designs that norm a sublayer's input (pre-norm) have ``add`` throughout: it runs the sublayer on ``h``, adds
its output to the residual stream ``x`` in place, and returns the next sublayer's input, rms(x) * ``norm_w``, or without
``norm_w`` x itself, in the products' type.
"""

from __future__ import annotations

import torch
import torch.nn as nn

from . import _lib, dense
from .cache import DecayState, KeyValueState, LatentState, MatrixMemoryState, SideBySideState

ACTIVATIONS = {"none": _lib.ACT_NONE, "relu2": _lib.ACT_RELU2, "gelu_erf": _lib.ACT_GELU_ERF}

# A pass of at most this many positions takes the one-by-one form of a mixer (recurrence, attention over the cached
# latents themselves) instead of the blockwise one.
SHORT_PASS = 8


def _param(t, device, dtype):
    return nn.Parameter(t.to(device=device, dtype=dtype).contiguous(), requires_grad=False)


def _stack(tensors, device, dtype):
    """Several (rows_i, K) matrices over one input as a single product."""
    return _param(torch.cat([t.to(device) for t in tensors]), device, dtype)


class MatrixMemoryMixer(nn.Module):
    """mLSTM: q, k, v, output gate and the two gate logits are one product; then the recurrence with its per-head RMS
    norm and output gate; then the output product.  ``w``: q k v g o (linear), i f (linear, with i.b f.b), norm."""

    def __init__(self, heads, dim, vdim, gate_cap, eps, w, device, dtype):
        super().__init__()
        self.heads, self.dim, self.vdim, self.cap, self.eps = heads, dim, vdim, float(gate_cap), float(eps)
        self.w_in = _stack([w("q"), w("k"), w("v"), w("g"), w("i"), w("f")], device, dtype)
        self.split = 2 * heads * (dim + vdim)           # the gate logits behind it stay in 32-bit
        self.bias_i, self.bias_f = _param(w("i.b"), device, torch.float32), _param(w("f.b"), device, torch.float32)
        self.norm_w = _param(w("norm"), device, torch.float32)
        self.w_out = _param(w("o"), device, dtype)

    def make_state(self, batch, max_len, device, dtype):
        return MatrixMemoryState(batch, self.heads, self.dim, self.vdim, device)

    def forward(self, h, B, T, start, kv_len, state):
        qkvg, gates = dense.matmul(h, self.w_in, split=self.split)
        chunked = T > SHORT_PASS and h.dtype == torch.bfloat16 and self.dim % 8 == 0 and self.vdim % 8 == 0
        fused = not chunked and dense.head_norm_matmul_supported(qkvg, self.w_out)
        o = dense.mlstm(qkvg, gates, B, T, self.heads, self.dim, self.vdim, self.cap, self.eps, self.bias_i, self.bias_f,
                        self.norm_w, state, chunked, state_idle=True, raw=fused)
        if fused:
            gate = qkvg[:, 2 * self.heads * self.dim + self.heads * self.vdim:]
            return dense.head_norm_matmul(o, gate, self.norm_w, self.heads, self.eps, self.w_out)
        return dense.matmul(o, self.w_out, split=0)[1]


def rotation_tables(rot_dims, max_len, base, device):
    """cos and sin of position * base^(-2i / rot_dims), float, from angles in double: (max_len, rot_dims / 2) each."""
    f = base ** (-2.0 * torch.arange(rot_dims // 2, dtype=torch.float64) / max(rot_dims, 1))
    a = torch.outer(torch.arange(max_len, dtype=torch.float64), f)
    return a.cos().float().to(device), a.sin().float().to(device)


class Rotation:
    """Angles position * base^(-2i / dims) of the first ``dims`` elements of a head, paired as (i, i + dims/2) or, with
    ``pairs``, as (2i, 2i + 1); tables are made for the longest cache asked for."""

    def __init__(self, dims, base, pairs):
        self.dims, self.base, self.pairs = int(dims), float(base), int(pairs)
        self._tables = []            # shorter ones stay: a captured step may use them

    def __call__(self, max_len, device):
        """(dims, pairs, cosines, sines)"""
        if not self._tables or self._tables[-1][0].shape[0] < max_len:
            self._tables.append(rotation_tables(self.dims, max_len, self.base, device))
        return (self.dims, self.pairs, *self._tables[-1])


class LatentAttentionMixer(nn.Module):
    """Attention whose keys and values are projections of a cached latent.  Queries, the latent and the heads' gate
    logits are one product.  Short passes attend to the latents through the key projection's transpose; longer ones
    expand keys and values of all positions first.  ``w``: q dkv dkv.norm uk uv g o."""

    def __init__(self, heads, dim, rot_dim, vdim, kv_rank, rot_base, rot_dims, scale, eps, w, device, dtype):
        super().__init__()
        self.heads, self.dim, self.rot_dim, self.vdim, self.kv_rank = heads, dim, rot_dim, vdim, kv_rank
        self.rotation, self.rot_dims, self.scale, self.eps = Rotation(rot_dims, rot_base, False), rot_dims, float(scale), float(eps)
        self.w_in = _stack([w("q"), w("dkv"), w("g")], device, dtype)
        self.split = heads * (dim + rot_dim)
        self.norm_w = _param(w("dkv.norm"), device, torch.float32)
        uk, uv = w("uk"), w("uv")
        self.w_kv = _stack([uk, uv], device, dtype)
        self.ukt = _param(uk.reshape(heads, dim, kv_rank).transpose(1, 2), device, dtype)
        self.uv = self.w_kv[heads * dim:]
        self.w_out = _param(w("o"), device, dtype)

    def make_state(self, batch, max_len, device, dtype):
        return LatentState(batch, max_len, self.kv_rank, self.rot_dim, device, dtype)

    def expand(self, state, B, S, form):
        """Keys and values of positions 0..S-1 as the prompt form of the attention takes them."""
        n_k, n_v = self.heads * self.dim, self.heads * self.vdim

        def new(rows, cols):
            return torch.empty(B, rows, dense.ceil_to(cols, 8), dtype=state.rows.dtype, device=state.rows.device)
        if form == 1:
            kv = new(S, n_k + n_v)
            for b in range(B):
                dense.matmul(state.rows[b], self.w_kv, rows=S, out=kv[b])
            return kv, S
        k, vt = new(S, n_k), new(n_v, S)
        for b in range(B):
            dense.matmul(state.rows[b], self.w_kv[:n_k], rows=S, out=k[b])
            dense.matmul(self.uv, state.rows[b, :S, :self.kv_rank], out=vt[b])
        return k, S, vt

    def forward(self, h, B, T, start, kv_len, state):
        q, rest = dense.matmul(h, self.w_in, split=self.split)
        cos, sin = self.rotation(state.rows.shape[1], h.device)[2:]
        y = torch.empty(B * T, self.heads * self.vdim, dtype=h.dtype, device=h.device)
        call = dense.Latent(q, rest, rest[:, self.kv_rank + self.rot_dim:], start, B, T, self.heads, self.dim, self.rot_dim,
                            self.vdim, self.kv_rank, self.rot_dims, self.scale, self.eps, self.norm_w, cos, sin, state, y)
        form = 0 if T <= SHORT_PASS or kv_len is None else call.prefill_form()
        if form == 0:
            call.absorbed(self.ukt, self.uv)
        else:
            call.prep()
            call.prefill(*self.expand(state, B, kv_len, form))
        return dense.matmul(y, self.w_out, split=0)[1]


class DenseFeedForward(nn.Module):
    """down . act(up . h).  ``w``: up down."""

    def __init__(self, act, w, device, dtype):
        super().__init__()
        self.act = ACTIVATIONS[act]
        self.up, self.down = _param(w("up"), device, dtype), _param(w("down"), device, dtype)

    def add(self, x, h, norm_w, eps, final=None):
        y = dense.matmul(dense.matmul(h, self.up, act=self.act)[0], self.down, split=0)[1]
        return dense.add_norm(x, y, norm_w, eps, h.dtype, final)


class RoutedFeedForward(nn.Module):
    """Mixture of experts: softmax scores over the experts and ``identity`` pass-through experts behind them, the
    ``top`` largest of score + correction, weighted by the bare scores.  ``w``: router correction, e<j>.up e<j>.down."""

    def __init__(self, act, experts, identity, top, w, device, dtype):
        super().__init__()
        self.act, self.experts, self.identity, self.top = ACTIVATIONS[act], experts, identity, top
        self.router, self.correction = _param(w("router"), device, dtype), _param(w("correction"), device, torch.float32)
        self.up = _param(torch.stack([w(f"e{e}.up").to(device) for e in range(experts)]), device, dtype)
        self.down = _param(torch.stack([w(f"e{e}.down").to(device) for e in range(experts)]), device, dtype)

    def add(self, x, h, norm_w, eps, final=None):
        logits = dense.matmul(h, self.router, split=0)[1]
        plan = dense.route(logits, self.correction, self.experts, self.identity, self.top)
        up = dense.matmul(h, self.up, act=self.act, plan=plan)[0]
        out = dense.matmul(up, self.down, plan=plan, gathered=False)[0]
        return dense.combine_norm(x, out, plan, norm_w, eps, h.dtype, final)


# ---- pre-norm sublayers ------------------------------------------------------------------------------------
def _added(x, h, norm_w, eps, dtype):
    """The next sublayer's input after a product has been added to x: ``h`` is its copy of x, or None."""
    return h if norm_w is None else dense.rms_add(x, eps, dtype, norm_w=norm_w)


class _DecayAttention(nn.Module):
    """Linear attention with decay on column ranges of a product (``dense.decay_attention``), up to the output product."""

    def __init__(self, heads, dim, vdim, eps, w, device, dtype, norm_w=None, gate="silu", q_scale=1.0, k_scale=1.0):
        super().__init__()
        self.heads, self.dim, self.vdim, self.eps = heads, dim, vdim, float(eps)
        self.gate_act, self.q_scale, self.k_scale = {"sigmoid": _lib.GATE_SIGMOID, "silu": _lib.GATE_SILU}[gate], float(q_scale), float(k_scale)
        self.norm_w = None if norm_w is None else _param(norm_w, device, torch.float32)
        self.w_out = _param(w("o"), device, dtype)

    def columns(self):
        """widths of q, k, v and the output gate"""
        return [self.heads * n for n in (self.dim, self.dim, self.vdim, self.vdim)]

    def make_state(self, batch, max_len, device, dtype):
        return DecayState(batch, max_len, self.heads, self.dim, self.vdim, device)

    def run(self, q, k, v, g, B, T, state, add=None, copy=False, **kw):
        """The mixer's output in float, or (``add``) its sum with x in place: see ``dense.matmul_add``."""
        o = dense.decay_attention(q, k, v, g, B, T, self.heads, self.dim, self.vdim, state, self.norm_w, self.eps, self.gate_act,
                                  q_scale=self.q_scale, k_scale=self.k_scale, short=T <= SHORT_PASS, **kw)
        return dense.matmul(o, self.w_out, split=0)[1] if add is None else dense.matmul_add(o, self.w_out, add, copy)


class RetentionMixer(_DecayAttention):
    """Linear attention whose state decays by a constant per head, on rotated queries and keys.  ``w``: q k v g o."""

    def __init__(self, heads, dim, vdim, decay, rotation, eps, w, device, dtype):
        super().__init__(heads, dim, vdim, eps, w, device, dtype, k_scale=dim ** -0.5)
        if len(decay) != heads:
            raise ValueError(f"{len(decay)} decays for {heads} heads")
        self.decay = _param(torch.tensor(decay, dtype=torch.float64), device, torch.float32)
        self.rotation = rotation
        self.w_in = _stack([w("q"), w("k"), w("v"), w("g")], device, dtype)

    def add(self, x, h, B, T, start, kv_len, state, norm_w=None):
        q, k, v, g = dense.matmul(h, self.w_in)[0].split(self.columns(), 1)
        hx = self.run(q, k, v, g, B, T, state, x, norm_w is None, decay=self.decay, rotation=self.rotation(state.max_len, x.device), start=start)
        return _added(x, hx, norm_w, self.eps, h.dtype)


class GatedLinearAttention(_DecayAttention):
    """Linear attention whose state decays per key channel by sigmoid(W_a2 W_a1 h + b)^(1/tau).  ``w``: q k v g o a1 a2
    a2.b norm (one vector for all heads)."""

    def __init__(self, heads, dim, vdim, tau, eps, w, device, dtype):
        super().__init__(heads, dim, vdim, eps, w, device, dtype, norm_w=w("norm"), q_scale=dim ** -0.5)
        self.tau = float(tau)
        self.a2, self.a2b = _param(w("a2"), device, dtype), _param(w("a2.b"), device, torch.float32)
        self.projections = [w("q"), w("k"), w("v"), w("g")]     # taken up into the layer's input product
        self.low_rank = w("a1")

    def forward(self, q, k, v, g, a, B, T, state):
        return self.run(q, k, v, g, B, T, state, gates=(a, self.a2, self.a2b, self.tau))


class SharedValueAttention(nn.Module):
    """Grouped-query attention whose values are the keys as projected; queries and keys are rotated, then divided by
    their root mean square.  ``w``: q k o."""

    def __init__(self, heads, kv_heads, dim, vdim, rotation, scale, eps, w, device, dtype):
        super().__init__()
        if vdim != dim or heads % kv_heads:
            raise ValueError(f"values are the keys ({dim} wide, not {vdim}); {heads} heads over {kv_heads}")
        self.heads, self.kv_heads, self.dim, self.vdim = heads, kv_heads, dim, vdim
        self.rotation, self.scale, self.eps = rotation, float(scale), float(eps)
        self.projections = [w("q"), w("k")]
        self.w_out = _param(w("o"), device, dtype)

    def columns(self):
        return [self.heads * self.dim, self.kv_heads * self.dim]

    def make_state(self, batch, max_len, device, dtype):
        return KeyValueState(batch, max_len, self.kv_heads, self.dim, self.vdim, device, dtype)

    def forward(self, q, k, B, T, start, kv_len, state):
        y = dense.gqa(q, k, k, B, T, self.heads, self.kv_heads, self.dim, self.vdim, state, self.scale, self.eps, start, kv_len,
                      self.rotation(state.k.shape[1], q.device), qk_norm=True)
        return dense.matmul(y, self.w_out, split=0)[1]


class ParallelMixer(nn.Module):
    """Attention and gated linear attention side by side on the same input, one input product for both; the output is the
    mean of the two, each with an RMS norm of its own.  ``w``: left.out right.out (norms)."""

    def __init__(self, left, right, eps, w, device, dtype):
        super().__init__()
        self.left, self.right, self.eps = left, right, float(eps)
        self.w_in = _stack(left.projections + right.projections + [right.low_rank], device, dtype)
        self.columns = left.columns() + right.columns()
        left.projections = right.projections = right.low_rank = None
        self.out_l, self.out_r = (_param(w(n), device, torch.float32) for n in ("left.out", "right.out"))

    def make_state(self, batch, max_len, device, dtype):
        return SideBySideState(*(m.make_state(batch, max_len, device, dtype) for m in (self.left, self.right)))

    def add(self, x, h, B, T, start, kv_len, state, norm_w=None):
        y, a = dense.matmul(h, self.w_in, split=sum(self.columns))      # the decays' low-rank product stays in 32-bit
        lq, lk, q, k, v, g = y.split(self.columns, 1)
        yl = self.left(lq, lk, B, T, start, kv_len, state[0])
        yr = self.right(q, k, v, g, a, B, T, state[1])
        return dense.rms_add(x, self.eps, h.dtype, yl, self.out_l, yr, self.out_r, 0.5, norm_w)


class GatedFeedForward(nn.Module):
    """down . (silu(gate . h) * up . h).  ``w``: gate up down."""

    def __init__(self, eps, w, device, dtype):
        super().__init__()
        self.eps = float(eps)
        self.w_in, self.down = _param(dense.gated_rows(w("gate"), w("up")), device, dtype), _param(w("down"), device, dtype)

    def add(self, x, h, norm_w=None):
        mid = dense.matmul(h, self.w_in, act=_lib.ACT_SILU_GLU)[0][:, :self.down.shape[1]]
        return _added(x, dense.matmul_add(mid, self.down, x, norm_w is None), norm_w, self.eps, h.dtype)


class TokenSideInput(nn.Module):
    """What a token's own row of a layer's table gives: x += rms(proj . (gelu_tanh(gate . x) * e[token])) * norm.
    ``table`` (vocab, dim): this layer's columns, shared with the other layers.  ``w``: gate proj norm."""

    def __init__(self, table, eps, w, device, dtype):
        super().__init__()
        self.table, self.eps = [table], float(eps)      # (in a list: the whole table is the model's parameter)
        self.gate, self.proj = _param(w("gate"), device, dtype), _param(w("proj"), device, dtype)
        self.norm_w = _param(w("norm"), device, torch.float32)

    def add(self, x, h, ids, norm_w=None):
        g = dense.matmul(h, self.gate, act=_lib.ACT_GELU_TANH, mul=self.table[0], mul_row=ids)[0]
        return dense.rms_add(x, self.eps, h.dtype, dense.matmul(g, self.proj, split=0)[1], self.norm_w, norm_w=norm_w)
