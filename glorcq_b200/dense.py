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


def matmul(x, W, split=None, act=ACT_NONE, alpha=1.0, ldx=None, rows=None, plan=None, gathered=True, out=None):
    """alpha * act(x . W^T) with the first ``split`` columns in x's type and the others in float: (y or None, y32 or
    None), each (rows, columns) with a padded row stride.  ``plan`` (``route``): W is (experts, N, K) and every entry
    goes through its expert's matrix, reading its token's row of x (``gathered``) or its own.  ``out``: where y goes."""
    _need(x, "x")
    N, K = W.shape[-2], W.shape[-1]
    split = N if split is None else split
    rows = (plan.entries if plan is not None else x.shape[0]) if rows is None else rows
    dev = x.device
    y = out if out is not None else torch.empty(rows, ceil_to(split, 8), dtype=x.dtype, device=dev) if split else None
    y32 = torch.empty(rows, ceil_to(N - split, 4), dtype=torch.float32, device=dev) if split < N else None
    a = _lib.DenseMM(dtype=DTYPES[x.dtype], act=act, N=N, K=K, rows=rows, n_matrices=1, split=split, alpha=alpha,
                     x=x.data_ptr(), ldx=x.stride(0) if ldx is None else ldx, W=W.data_ptr(),
                     ldw=W.stride(-2))
    if y is not None:
        a.y, a.ldy = y.data_ptr(), y.stride(0)
    if y32 is not None:
        a.y32, a.ldy32 = y32.data_ptr(), y32.stride(0)
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
    return (None if y is None else y[:, :split]), (None if y32 is None else y32[:, :N - split])


def embed(ids, table):
    """(x float residual rows, the same rows in the table's type)"""
    _need(table, "table")
    ids = ids.reshape(-1)
    rows, (V, Cw) = ids.numel(), table.shape
    x = torch.empty(rows, Cw, dtype=torch.float32, device=table.device)
    h = torch.empty(rows, Cw, dtype=table.dtype, device=table.device)
    with torch.cuda.device(table.device):
        _lib.check_dense(_lib.dense().glq_dense_embed(DTYPES[table.dtype], ids.data_ptr(), table.data_ptr(), rows, Cw, V, x.data_ptr(),
                                                      h.data_ptr(), _stream_ptr(table.device)), "embed")
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
