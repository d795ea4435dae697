"""Calls of the unquantized kernels (libglorcq_b200_dense.so) on torch tensors: bfloat16 or float32 storage, float
accumulation.  Outputs come from torch's allocator, so a captured CUDA graph keeps what its launches use."""

from __future__ import annotations

import ctypes as C
from types import SimpleNamespace

import torch

from . import _lib
from ._lib import ACT_NONE
from .tiled import _stream_ptr

DTYPES = {torch.bfloat16: _lib.DT_BF16, torch.float32: _lib.DT_F32}


def _need(t, name):
    if not t.is_cuda:
        raise RuntimeError(f"{name} must be a CUDA tensor (glorcq_b200 has no CPU path)")


def ceil_to(n, m):
    return (n + m - 1) // m * m


def debug_error(clear=True):
    """What a bounded wait recorded when it ran out, or None."""
    out = (C.c_ulonglong * 4)()
    _lib.check_dense(_lib.dense().glq_dense_debug_error(out, int(clear)), "debug_error")
    return None if out[0] == 0 else [int(v) for v in out]


def matmul(x, W, split=None, act=ACT_NONE, alpha=1.0, ldx=None, rows=None, plan=None, gathered=True, out=None, mul=None, mul_row=None):
    """alpha * act(x . W^T) with the first ``split`` columns in x's type and the others in float: (y or None, y32 or
    None), each (rows, columns) with a padded row stride.  ``plan`` (``route``): W is (experts, N, K) and every entry
    goes through its expert's matrix, reading its token's row of x (``gathered``) or its own.  ``out``: where y goes.
    A gated activation (W from ``gated_rows``) gives half as many columns.  ``mul``: a matrix of x's type whose row
    ``mul_row[r]`` (int64) multiplies row r of the result."""
    _need(x, "x")
    N, K = W.shape[-2], W.shape[-1]
    split = N if split is None else split
    cols = N // 2 if act == _lib.ACT_SILU_GLU else split
    rows = (plan.entries if plan is not None else x.shape[0]) if rows is None else rows
    dev = x.device
    y = out if out is not None else torch.empty(rows, ceil_to(cols, 8), dtype=x.dtype, device=dev) if split else None
    y32 = torch.empty(rows, ceil_to(N - split, 4), dtype=torch.float32, device=dev) if split < N else None
    a = _lib.DenseMM(dtype=DTYPES[x.dtype], act=act, N=N, K=K, rows=rows, n_matrices=1, split=split, alpha=alpha,
                     x=x.data_ptr(), ldx=x.stride(0) if ldx is None else ldx, W=W.data_ptr(),
                     ldw=W.stride(-2))
    if y is not None:
        a.y, a.ldy = y.data_ptr(), y.stride(0)
    if y32 is not None:
        a.y32, a.ldy32 = y32.data_ptr(), y32.stride(0)
    if mul is not None:
        a.mul, a.ldmul, a.mul_row, a.mul_rows = mul.data_ptr(), mul.stride(0), mul_row.data_ptr(), mul.shape[0]
    gather = None
    if plan is not None:
        a.n_matrices, a.max_slots, a.max_slot_rows = W.shape[0], plan.max_slots, plan.max_slot_rows
        a.slot_index, a.n_slots = plan.active.data_ptr(), plan.n_active.data_ptr()
        a.slot_count, a.slot_offset = plan.slot_count.data_ptr(), plan.slot_offset.data_ptr()
        if gathered:
            a.entry_row = plan.entry_row.data_ptr()
            if plan.max_slot_rows > 8 and x.dtype == torch.bfloat16 and K % 8 == 0:
                gather = torch.empty(rows, K, dtype=x.dtype, device=dev)
                a.gather = gather.data_ptr()
    with torch.cuda.device(dev):
        _lib.check_dense(_lib.dense().glq_dense_matmul(C.byref(a), _stream_ptr(dev)), "dense_matmul")
    return (None if y is None else y[:, :cols]), (None if y32 is None else y32[:, :N - split])


def matmul_add(y, W, x, copy=False):
    """x += y . W^T in place (x float, contiguous); returns x in y's type when ``copy`` asks for it."""
    _need(y, "y")
    N, K = W.shape
    h = torch.empty(x.shape, dtype=y.dtype, device=x.device) if copy else None
    a = _lib.DenseMM(dtype=DTYPES[y.dtype], N=N, K=K, rows=y.shape[0], n_matrices=1, alpha=1.0, x=y.data_ptr(), ldx=y.stride(0),
                     W=W.data_ptr(), ldw=W.stride(0), y32=x.data_ptr(), ldy32=x.stride(0), residual=1)
    if copy:
        a.y, a.ldy = h.data_ptr(), h.stride(0)
    with torch.cuda.device(x.device):
        _lib.check_dense(_lib.dense().glq_dense_matmul(C.byref(a), _stream_ptr(x.device)), "matmul_add")
    return h


def gated_rows(gate, up):
    """The (2 N', K) matrix of a gated activation from its (N, K) halves: 8 rows of one, 8 of the other; N' is N up to a
    multiple of 8 (the additional columns come out as zeros)."""
    N, K = gate.shape
    pad = ceil_to(N, 8) - N
    both = [torch.cat([t, t.new_zeros(pad, K)]).view(-1, 8, K) for t in (gate, up)]
    return torch.stack(both, 1).reshape(-1, K)


def embed(ids, table, norm_w=None, eps=0.0):
    """(x float residual rows, the same rows, or with ``norm_w`` rms(x) * norm_w, in the table's type)"""
    _need(table, "table")
    ids = ids.reshape(-1)
    rows, (V, Cw) = ids.numel(), table.shape
    x = torch.empty(rows, Cw, dtype=torch.float32, device=table.device)
    h = torch.empty(rows, Cw, dtype=table.dtype, device=table.device)
    with torch.cuda.device(table.device):
        _lib.check_dense(_lib.dense().glq_dense_embed(DTYPES[table.dtype], ids.data_ptr(), table.data_ptr(), rows, Cw, V,
                                                      None if norm_w is None else norm_w.data_ptr(), eps, x.data_ptr(), h.data_ptr(), _stream_ptr(table.device)), "embed")
    return x, h


def add_norm(x, y, w, eps, dtype, final=None):
    """x += layer_norm(y) * w in place; returns x, or layer_norm(x) * final, in ``dtype``."""
    _need(x, "x")
    h = torch.empty(x.shape, dtype=dtype, device=x.device)
    if y.stride(0) != x.shape[1]:
        y = y.contiguous()
    with torch.cuda.device(x.device):
        _lib.check_dense(_lib.dense().glq_dense_add_norm(DTYPES[dtype], y.data_ptr(), w.data_ptr(), final.data_ptr() if final is not None else None,
                                                         eps, x.shape[0], x.shape[1], x.data_ptr(), h.data_ptr(),
                                                         _stream_ptr(x.device)), "add_norm")
    return h


def rms_add(x, eps, dtype, y=None, w=None, y2=None, w2=None, alpha=1.0, norm_w=None):
    """x += alpha * (rms(y) * w + rms(y2) * w2) in place, where y2 may be missing, y too (nothing is added), and without
    w and w2 the rows are added as they are; returns x, or rms(x) * norm_w, in ``dtype``."""
    _need(x, "x")
    h = torch.empty(x.shape, dtype=dtype, device=x.device)

    def ptr(t):
        return None if t is None else t.data_ptr()
    with torch.cuda.device(x.device):
        _lib.check_dense(_lib.dense().glq_dense_rms_add(DTYPES[dtype], ptr(y), 0 if y is None else y.stride(0), ptr(w), ptr(y2),
                                                        0 if y2 is None else y2.stride(0), ptr(w2), alpha, ptr(norm_w), eps, x.shape[0],
                                                        x.shape[1], x.data_ptr(), h.data_ptr(), _stream_ptr(x.device)), "rms_add")
    return h


def combine_norm(x, entry_out, plan, w, eps, dtype, final=None):
    """add_norm of the weighted sum of every token's experts (pass-through slots add the token's own x)."""
    h = torch.empty(x.shape, dtype=dtype, device=x.device)
    with torch.cuda.device(x.device):
        _lib.check_dense(_lib.dense().glq_dense_combine_norm(
            DTYPES[dtype], entry_out.data_ptr(), entry_out.stride(0), plan.tok_entries.data_ptr(), plan.wts.data_ptr(), plan.top,
            w.data_ptr(), final.data_ptr() if final is not None else None, eps, x.shape[0], x.shape[1], x.data_ptr(), h.data_ptr(),
            _stream_ptr(x.device)), "combine_norm")
    return h


def route(logits, correction, experts, identity, top):
    """Chosen experts, weights and entry lists of every row of router logits."""
    _need(logits, "logits")
    L, dev, n = _lib.dense(), logits.device, logits.shape[0]
    nk = n * top
    chunk = 8 if n <= 32 else 0                # few tokens: slots of at most eight rows, for the streaming product
    ms = L.glq_route_max_slots(n, experts, top, chunk)
    sizes = [("sel", nk), ("tok_entries", nk), ("entry_row", 2 * nk), ("active", 3 * ms), ("slot_count", 3 * ms),
             ("slot_offset", 3 * ms), ("n_active", 2), ("block_counts", (nk + 511) // 512 * experts)]
    ints = torch.empty(sum(s for _, s in sizes), dtype=torch.int32, device=dev)
    fl = torch.empty(2, nk, dtype=torch.float32, device=dev)
    p, at = SimpleNamespace(top=top, entries=nk, max_slots=ms, max_slot_rows=min(n, chunk) if chunk else n, wts=fl[0]), 0
    for name, s in sizes:
        setattr(p, name, ints[at:at + s])
        at += s
    a = _lib.Route(n=n, E=experts, identity=identity, top=top, chunk=chunk, logits=logits.data_ptr(), ldl=logits.stride(0),
                   correction=correction.data_ptr(), wts=fl[0].data_ptr(), entry_scale=fl[1].data_ptr(), max_slots=ms,
                   **{name: getattr(p, name).data_ptr() for name, _ in sizes})
    with torch.cuda.device(dev):
        _lib.check_dense(L.glq_route(C.byref(a), _stream_ptr(dev)), "route")
    return p


def mlstm(qkvg, gates, B, T, heads, dim, vdim, cap, eps, bias_i, bias_f, norm_w, state, chunked, state_idle=False, raw=False):
    """Matrix-memory recurrence over T positions with per-head norm and output gate, or with ``raw`` (one-by-one form
    only) its float output before them; ``state`` is advanced."""
    _need(qkvg, "qkvg")
    L, dev = _lib.dense(), qkvg.device
    o = torch.empty(B * T, heads * vdim, dtype=torch.float32, device=dev)
    out = None if raw and not chunked else torch.empty(B * T, heads * vdim, dtype=qkvg.dtype, device=dev)
    a = _lib.MLstm(dtype=DTYPES[qkvg.dtype], B=B, T=T, H=heads, D=dim, V=vdim, state_idle=int(state_idle), gate_cap=cap, eps=eps,
                   qkvg=qkvg.data_ptr(), ldp=qkvg.stride(0), gates=gates.data_ptr(), ldg=gates.stride(0), bias_i=bias_i.data_ptr(),
                   bias_f=bias_f.data_ptr(), norm_w=norm_w.data_ptr(), S=state.S.data_ptr(), n=state.n.data_ptr(),
                   m=state.m.data_ptr(), o=o.data_ptr(), out=None if out is None else out.data_ptr())
    ws = None
    if chunked:
        ws = torch.empty(L.glq_mlstm_workspace_bytes(C.byref(a)), dtype=torch.uint8, device=dev)
        a.workspace, a.workspace_bytes = ws.data_ptr(), ws.numel()
    with torch.cuda.device(dev):
        fn = L.glq_mlstm_chunk if chunked else L.glq_mlstm_step
        _lib.check_dense(fn(C.byref(a), _stream_ptr(dev)), "mlstm")
    return o if out is None else out


def head_norm_matmul_supported(o, W):
    return W.dtype == torch.bfloat16 and o.shape[0] <= 8 and W.shape[1] % 8 == 0 and min(8, o.shape[0] + 1) * (W.shape[1] + 64) * 2 <= 200 * 1024


def head_norm_matmul(o, gate, norm_w, heads, eps, W):
    """(rms_norm of each head of o, times norm_w, times sigmoid(gate)) . W^T in float: the end of a recurrent mixer's
    decode step in one launch."""
    N, K = W.shape
    y32 = torch.empty(o.shape[0], ceil_to(N, 4), dtype=torch.float32, device=o.device)
    a = _lib.DenseMM(dtype=DTYPES[W.dtype], N=N, K=K, rows=o.shape[0], n_matrices=1, split=0, alpha=1.0, W=W.data_ptr(),
                     y32=y32.data_ptr(), ldy32=y32.stride(0), hn_o=o.data_ptr(), hn_g=gate.data_ptr(), hn_ldg=gate.stride(0),
                     hn_w=norm_w.data_ptr(), hn_heads=heads, hn_eps=eps)
    with torch.cuda.device(o.device):
        _lib.check_dense(_lib.dense().glq_dense_matmul(C.byref(a), _stream_ptr(o.device)), "head_norm_matmul")
    return y32[:, :N]


def head_stride(norm_w, heads, vdim):
    """Step between the norm weights of two heads: 0 when all heads share one vector."""
    return vdim if norm_w is not None and heads > 1 and norm_w.numel() == heads * vdim else 0


def decay_attention(q, k, v, g, B, T, heads, dim, vdim, state, norm_w, eps, gate_act, decay=None, gates=None, rotation=None, start=None,
                    q_scale=1.0, k_scale=1.0, short=False):
    """Linear attention with decay over T positions, with per-head norm and output gate; ``state`` is advanced.  q, k, v, g are column ranges of one product.  ``decay``:
    (heads,) float, or ``gates`` = (a, a2, a2_bias, tau) for a decay per key channel.  ``rotation`` = (dims, pairs, cos,
    sin) turns q and k by their position, the first of which is ``start``.  ``short`` keeps to the one-by-one form."""
    _need(q, "q")
    L, dev = _lib.dense(), q.device
    o = torch.empty(B * T, heads * vdim, dtype=torch.float32, device=dev)
    a = _lib.Decay(dtype=DTYPES[q.dtype], B=B, T=T, H=heads, D=dim, V=vdim, norm_stride=head_stride(norm_w, heads, vdim), gate=gate_act,
                   state_idle=1, q_scale=q_scale, k_scale=k_scale, eps=eps, q=q.data_ptr(), k=k.data_ptr(), v=v.data_ptr(), g=g.data_ptr(),
                   ldp=q.stride(0), norm_w=None if norm_w is None else norm_w.data_ptr(), S=state.S.data_ptr(), o=o.data_ptr())
    if decay is not None:
        a.decay = decay.data_ptr()
    else:
        r, a2, a2b, a.tau = gates
        a.a, a.lda, a.a2, a.a2b, a.rank = r.data_ptr(), r.stride(0), a2.data_ptr(), a2b.data_ptr(), a2.shape[1]
    if rotation is not None and rotation[0] > 0:
        a.rot_dims, a.rot_pairs, cos, sin = rotation
        a.cos_t, a.sin_t, a.max_len, a.start = cos.data_ptr(), sin.data_ptr(), cos.shape[0], start.data_ptr()
    chunked = not short and bool(L.glq_decay_chunk_supported(C.byref(a)))
    out = torch.empty(B * T, heads * vdim, dtype=q.dtype, device=dev)
    a.out = out.data_ptr()
    ws = None
    if chunked:
        ws = torch.empty(L.glq_decay_workspace_bytes(C.byref(a)), dtype=torch.uint8, device=dev)
        a.workspace, a.workspace_bytes = ws.data_ptr(), ws.numel()
    with torch.cuda.device(dev):
        _lib.check_dense((L.glq_decay_chunk if chunked else L.glq_decay_step)(C.byref(a), _stream_ptr(dev)), "decay_attention")
    return out


def gqa(q, k, v, B, T, heads, kv_heads, dim, vdim, state, scale, eps, start, kv_len, rotation=None, qk_norm=False):
    """Grouped-query attention of T new positions over the cache, into which their keys and values go first.  q, k, v:
    column ranges of one product (v may be k).  ``kv_len``: start + T on the host, or None inside a decode step."""
    _need(q, "q")
    L, dev = _lib.dense(), q.device
    out = torch.empty(B * T, heads * vdim, dtype=q.dtype, device=dev)
    a = _lib.Gqa(dtype=DTYPES[q.dtype], B=B, T=T, H=heads, G=kv_heads, D=dim, V=vdim, qk_norm=int(qk_norm), max_len=state.k.shape[1],
                 S=kv_len or 0, state_idle=1, scale=scale, eps=eps, start=start.data_ptr(), q=q.data_ptr(), k=k.data_ptr(), v=v.data_ptr(),
                 ldp=q.stride(0), kc=state.k.data_ptr(), vc=state.v.data_ptr(), out=out.data_ptr())
    if rotation is not None and rotation[0] > 0:
        a.rot_dims, a.rot_pairs, cos, sin = rotation
        a.cos_t, a.sin_t = cos.data_ptr(), sin.data_ptr()
    ws = None
    if L.glq_gqa_form(C.byref(a)) == 1:
        ws = torch.empty(max(16, L.glq_gqa_decode_workspace_bytes(C.byref(a))), dtype=torch.uint8, device=dev)
        a.workspace, a.workspace_bytes = ws.data_ptr(), ws.numel()
    with torch.cuda.device(dev):
        _lib.check_dense(L.glq_gqa(C.byref(a), _stream_ptr(dev)), "gqa")
    return out


class Latent:
    """One latent-attention call: the argument block of its launches."""

    def __init__(self, q, ckr, gate, start, B, T, heads, dim, rot_dim, vdim, kv_rank, rot_dims, scale, eps, norm_w, cos, sin, state, out):
        _need(q, "q")
        self.dev = q.device
        self.keep = (q, ckr, gate, start, norm_w, cos, sin, out)
        self.a = _lib.Latent(dtype=DTYPES[q.dtype], B=B, T=T, H=heads, D=dim, R=rot_dim, V=vdim, K=kv_rank, rot_dims=rot_dims,
                             max_len=state.rows.shape[1], scale=scale, eps=eps, start=start.data_ptr(), q=q.data_ptr(), ldq=q.stride(0),
                             ckr=ckr.data_ptr(), ldk=ckr.stride(0), gate=gate.data_ptr(), norm_w=norm_w.data_ptr(), cos_t=cos.data_ptr(),
                             sin_t=sin.data_ptr(), cache=state.rows.data_ptr(), ldc=state.ld, out=out.data_ptr())

    def _call(self, fn, what):
        with torch.cuda.device(self.dev):
            _lib.check_dense(fn(C.byref(self.a), _stream_ptr(self.dev)), what)

    def prep(self):
        """Rotates q in place and writes the cache rows: comes before ``prefill``; ``absorbed`` does both by itself."""
        self._call(_lib.dense().glq_latent_prep, "latent_prep")

    def prefill_form(self):
        """0: only ``absorbed`` covers these sizes; 1: ``prefill`` takes keys | values; 2: keys and transposed values."""
        return _lib.dense().glq_latent_prefill_form(C.byref(self.a))

    def absorbed(self, ukt, uv):
        L = _lib.dense()
        self.a.ukt, self.a.uv = ukt.data_ptr(), uv.data_ptr()
        ws = torch.empty(L.glq_latent_absorbed_workspace_bytes(C.byref(self.a)), dtype=torch.uint8, device=self.dev)
        self.a.workspace, self.a.workspace_bytes = ws.data_ptr(), ws.numel()
        self._call(L.glq_latent_absorbed, "latent_absorbed")

    def prefill(self, kv, S, vt=None):
        self.a.kv, self.a.ldkv, self.a.S = kv.data_ptr(), kv.stride(-2), S
        if vt is not None:
            self.a.vt, self.a.ldvt = vt.data_ptr(), vt.stride(-2)
        self._call(_lib.dense().glq_latent_prefill, "latent_prefill")


def head(x, W, scale, scratch):
    """(scale * x . W^T in float, arg-max of every row or None); ``scratch`` is a dict the caller keeps."""
    rows, H = x.shape
    V = W.shape[0]
    if not (x.dtype == torch.bfloat16 and 0 < rows <= 64 and H % 32 == 0 and H <= 8192):
        return matmul(x, W, split=0, alpha=scale)[1], None
    L, dev = _lib.dense(), x.device
    logits = torch.empty(rows, V, dtype=torch.float32, device=dev)
    best = torch.empty(rows, dtype=torch.int64, device=dev)
    key = (dev.index, _stream_ptr(dev))
    if key not in scratch:
        scratch[key] = (torch.empty(L.glq_dense_head_workspace_bytes(), dtype=torch.uint8, device=dev),
                        torch.zeros(1, dtype=torch.int32, device=dev))
    ws, ctr = scratch[key]
    with torch.cuda.device(dev):
        for r0 in range(0, rows, 8):
            _lib.check_dense(L.glq_dense_head(x[r0:].data_ptr(), x.stride(0), W.data_ptr(), min(8, rows - r0), V, H, scale,
                                              logits[r0:].data_ptr(), V, best[r0:].data_ptr(), ws.data_ptr(), ws.numel(),
                                              ctr.data_ptr(), _stream_ptr(dev)), "dense_head")
    return logits, best
