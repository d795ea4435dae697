"""Sublayers of the unquantized decoders.  Each takes its constants and weights as arguments; a model design is an
assembly of them (``zokunex``).

Mixers: ``forward(h, B, T, start, kv_len, state) -> y32`` for rows ``h`` (B*T, width) of the layer's input, positions
``start`` (device, int64) .. start + T - 1 of every sequence; ``kv_len`` = start + T on the host, or None inside a
decode step, whose position stays on the device.  Feed-forwards: ``add(x, h, norm, final) -> h'`` runs the sublayer on
``h`` and folds its output's norm and the residual add of ``x`` into the last launch.
"""

from __future__ import annotations

import torch
import torch.nn as nn

from . import _lib, dense
from .cache import LatentState, MatrixMemoryState

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


class LatentAttentionMixer(nn.Module):
    """Attention whose keys and values are projections of a cached latent.  Queries, the latent and the heads' gate
    logits are one product.  Short passes attend to the latents through the key projection's transpose; longer ones
    expand keys and values of all positions first.  ``w``: q dkv dkv.norm uk uv g o."""

    def __init__(self, heads, dim, rot_dim, vdim, kv_rank, rot_base, rot_dims, scale, eps, w, device, dtype):
        super().__init__()
        self.heads, self.dim, self.rot_dim, self.vdim, self.kv_rank = heads, dim, rot_dim, vdim, kv_rank
        self.rot_base, self.rot_dims, self.scale, self.eps = float(rot_base), rot_dims, float(scale), float(eps)
        self.w_in = _stack([w("q"), w("dkv"), w("g")], device, dtype)
        self.split = heads * (dim + rot_dim)
        self.norm_w = _param(w("dkv.norm"), device, torch.float32)
        uk, uv = w("uk"), w("uv")
        self.w_kv = _stack([uk, uv], device, dtype)
        self.ukt = _param(uk.reshape(heads, dim, kv_rank).transpose(1, 2), device, dtype)
        self.uv = self.w_kv[heads * dim:]
        self.w_out = _param(w("o"), device, dtype)
        self._tables = None

    def make_state(self, batch, max_len, device, dtype):
        return LatentState(batch, max_len, self.kv_rank, self.rot_dim, device, dtype)

    def tables(self, max_len, device):
        if self._tables is None or self._tables[0].shape[0] < max_len:
            self._tables = rotation_tables(self.rot_dims, max_len, self.rot_base, device)
        return self._tables

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
        cos, sin = self.tables(state.rows.shape[1], h.device)
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
