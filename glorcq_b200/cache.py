"""What a decoder carries from step to step, one entry per layer: cached positions of an attention layer, or the fixed
state of a recurrent one.

Every cache class has the interface the generation loop (``graph_wrapper``) works with: ``max_batch_size``,
``max_cache_len``, ``reset()`` between sequences, and ``snapshot(positions)`` / ``restore(saved)``, which put back what
trial steps at positions below ``positions`` overwrote (a step that is captured into a CUDA graph runs a few times
first).  Recurrent state has no positions to overwrite selectively: a snapshot holds all of it.
"""

from __future__ import annotations

import torch

from . import _lib


class LatentState:
    """Cached positions of latent attention: per position the normed latent and the rotated key part all heads share."""

    def __init__(self, batch, max_len, kv_rank, rot_dim, device, dtype):
        self.width = kv_rank + rot_dim
        self.ld = (self.width + 7) // 8 * 8            # rows start on 16-byte boundaries
        self.rows = torch.zeros(batch, max_len, self.ld, device=device, dtype=dtype)

    def reset(self):
        pass                                            # positions are written before they are read

    def snapshot(self, positions):
        return self.rows[:, :positions].clone()

    def restore(self, saved):
        self.rows[:, :saved.shape[1]].copy_(saved)


class MatrixMemoryState:
    """Matrix memory S, normaliser n and log maximum m of every head, in 32-bit, in the kernels' layout: S by slices of
    32 value columns, n and m once per slice."""

    def __init__(self, batch, heads, dim, vdim, device):
        sl = _lib.dense().glq_mlstm_slices(vdim)
        self.S = torch.zeros(batch, heads, sl, dim, 32, device=device)
        self.n = torch.zeros(batch, heads, sl, dim, device=device)
        self.m = torch.zeros(batch, heads, sl, device=device)

    def reset(self):
        self.S.zero_()
        self.n.zero_()
        self.m.zero_()

    def snapshot(self, positions):
        return self.S.clone(), self.n.clone(), self.m.clone()

    def restore(self, saved):
        for dst, src in zip((self.S, self.n, self.m), saved):
            dst.copy_(src)


class DecayState:
    """State S of linear attention with decay, in 32-bit, by slices of 32 value columns."""

    def __init__(self, batch, max_len, heads, dim, vdim, device):
        self.max_len = max_len                          # positions a sequence may reach (rotations are tabulated that far)
        self.S = torch.zeros(batch, heads, _lib.dense().glq_decay_slices(vdim), dim, 32, device=device)

    def reset(self):
        self.S.zero_()

    def snapshot(self, positions):
        return self.S.clone()

    def restore(self, saved):
        self.S.copy_(saved)


class KeyValueState:
    """Cached positions of grouped-query attention: keys (batch, position, head, dim) and values."""

    def __init__(self, batch, max_len, kv_heads, dim, vdim, device, dtype):
        self.k = torch.zeros(batch, max_len, kv_heads, dim, device=device, dtype=dtype)
        self.v = torch.zeros(batch, max_len, kv_heads, vdim, device=device, dtype=dtype)

    def reset(self):
        pass                                            # positions are written before they are read

    def snapshot(self, positions):
        return self.k[:, :positions].clone(), self.v[:, :positions].clone()

    def restore(self, saved):
        for dst, src in zip((self.k, self.v), saved):
            dst[:, :src.shape[1]].copy_(src)


class SideBySideState:
    """The states of mixers that run side by side in one layer."""

    def __init__(self, *parts):
        self.parts = parts

    def __getitem__(self, i):
        return self.parts[i]

    def reset(self):
        for s in self.parts:
            s.reset()

    def snapshot(self, positions):
        return [s.snapshot(positions) for s in self.parts]

    def restore(self, saved):
        for s, v in zip(self.parts, saved):
            s.restore(v)


class LayerStateCache:
    """One state object per layer."""

    def __init__(self, layers, max_batch_size, max_cache_len):
        self.layers = layers
        self.max_batch_size, self.max_cache_len = max_batch_size, max_cache_len

    def __getitem__(self, l):
        return self.layers[l]

    def reset(self):
        for s in self.layers:
            s.reset()

    def snapshot(self, positions):
        return [s.snapshot(positions) for s in self.layers]

    def restore(self, saved):
        for s, v in zip(self.layers, saved):
            s.restore(v)
