"""The frame of the unquantized decoders: checked weights, cache, step, greedy generation.  A design (``zokunex``,
``femirax``) names its tensors, builds its layers from ``layers`` and says how a step runs through them.
"""

from __future__ import annotations

import json
import os
from types import SimpleNamespace

import torch
import torch.nn as nn

from . import dense
from .cache import LayerStateCache
from .layers import _param
from .weights import read_safetensors


class DenseDecoder(nn.Module):
    """``weights``: {name: tensor} of ``tensor_shapes(cfg)``.  Storage and products are in ``dtype`` (bfloat16 or
    float32); residual stream, norms, routing, attention weights and recurrent state are float in both.

    A subclass gives ``tensor_shapes(cfg)``, ``build(cfg, weights, device, dtype)``, which fills ``mixers`` and whatever
    else its layers need, and ``run_layers``."""

    def __init__(self, cfg, weights, device="cuda:0", dtype=torch.bfloat16):
        super().__init__()
        if dtype not in dense.DTYPES:
            raise ValueError(f"dtype {dtype} is not supported")
        shapes = self.tensor_shapes(cfg, weights)
        for name in shapes:
            if name not in weights:
                raise KeyError(f"missing tensor {name}")
        for name, t in (weights.items() if hasattr(weights, "items") else ()):
            if name in shapes and tuple(t.shape) != tuple(shapes[name]):
                raise ValueError(f"tensor {name} has shape {tuple(t.shape)}, expected {tuple(shapes[name])}")
        device = torch.device(device)
        self.raw_config, self.eps, self.logit_scale = cfg, float(cfg["norm"]["eps"]), float(cfg.get("logit_scale", 1.0))
        self.config = SimpleNamespace(vocab_size=cfg["vocab"], hidden_size=cfg["width"], num_hidden_layers=len(cfg["layers"]),
                                      max_position_embeddings=cfg.get("max_position_embeddings", 4096))
        self.embed_tokens, self.lm_head = _param(weights["embed"], device, dtype), _param(weights["head"], device, dtype)
        self.norm = _param(weights["final.norm"], device, torch.float32)
        self.mixers = nn.ModuleList()
        self.build(cfg, weights, device, dtype)
        self._own_cache = None
        self._head_scratch = {}
        self.last_argmax = None      # greedy token of every kept row of the last forward, when the head kernel found it

    @staticmethod
    def tensor_shapes(cfg, weights=None):
        """{tensor name: shape}; ``weights`` settles sizes that only the tensors tell."""
        raise NotImplementedError

    def build(self, cfg, weights, device, dtype):
        raise NotImplementedError

    def run_layers(self, ids, B, T, start, kv_len, cache, trace):
        """Tokens ``ids`` (B*T,) through all layers: the output projection's input (B*T, width).  ``start``: their first
        position (device); ``kv_len`` = start + T on the host, or None inside a decode step; ``trace``: a list for the
        residual stream after every layer, or None."""
        raise NotImplementedError

    @classmethod
    def from_pretrained(cls, path, device="cuda:0", dtype=torch.bfloat16):
        with open(os.path.join(path, "config.json")) as f:
            cfg = json.load(f)
        return cls(cfg, read_safetensors(os.path.join(path, "model.safetensors")), device, dtype)

    def make_cache(self, max_batch_size, max_cache_len):
        dev, dt = self.embed_tokens.device, self.embed_tokens.dtype
        return LayerStateCache([m.make_state(max_batch_size, max_cache_len, dev, dt) for m in self.mixers], max_batch_size, max_cache_len)

    @torch.no_grad()
    def forward(self, input_ids=None, cache_position=None, past_key_values=None, use_cache=True, return_dict=False, logits_to_keep=0,
                trace=None, **_unused):
        """Logits (B, kept, vocab), float, of tokens (B, T) at positions ``cache_position`` (consecutive, the same for all
        rows), continuing from the cache.  ``logits_to_keep``: 0 all positions, k > 0 the last k, or a tensor of places.
        ``trace``: a list that receives the residual stream (B*T, width) after every layer."""
        B, T = input_ids.shape
        dev = self.embed_tokens.device
        fresh = cache_position is None
        if fresh:
            cache_position = torch.arange(T, device=dev)
        if past_key_values is None:
            if self._own_cache is None or self._own_cache.max_batch_size < B:
                self._own_cache = self.make_cache(B, self.config.max_position_embeddings)
            past_key_values = self._own_cache
            if fresh:
                past_key_values.reset()
        cache = past_key_values
        if B > cache.max_batch_size:
            raise ValueError(f"{B} sequences do not fit a cache of {cache.max_batch_size}")
        # a decode step keeps its position on the device (it may be captured into a graph)
        kv_len = int(cache_position[0]) + T if T > 1 else None
        if kv_len is not None and kv_len > cache.max_cache_len:
            raise ValueError(f"position {kv_len - 1} is beyond the cache's {cache.max_cache_len} positions")
        h = self.run_layers(input_ids.contiguous().view(-1), B, T, cache_position.to(torch.int64), kv_len, cache, trace)
        if torch.is_tensor(logits_to_keep):
            h = h.view(B, T, -1)[:, logits_to_keep].reshape(-1, h.shape[1])
        elif 0 < logits_to_keep < T:
            h = h.view(B, T, -1)[:, T - logits_to_keep:].reshape(-1, h.shape[1])
        logits, self.last_argmax = dense.head(h, self.lm_head, self.logit_scale, self._head_scratch)
        return (logits.reshape(B, h.shape[0] // B, -1), cache)

    @torch.no_grad()
    def generate(self, input_ids, max_new_tokens=100, do_sample=False):
        """Greedy generation without a graph."""
        B, T = input_ids.shape
        cache = self.make_cache(B, T + max_new_tokens)
        out, pos, tok = input_ids, 0, input_ids
        for _ in range(max_new_tokens):
            logits = self(input_ids=tok, cache_position=torch.arange(pos, pos + tok.shape[1], device=out.device), past_key_values=cache,
                          logits_to_keep=1)[0]
            pos += tok.shape[1]
            tok = torch.argmax(logits[:, -1, :], dim=-1, keepdim=True)
            out = torch.cat([out, tok], dim=1)
        return out
