"""Zokunex: a decoder of matrix-memory (mLSTM) and latent-attention layers in any order, each with a dense or a routed
feed-forward or none.  Sublayers read the residual stream itself; a layer norm sits on every sublayer's output.

    model = ZokunexDecoder.from_pretrained(folder, device="cuda:0", dtype=torch.bfloat16)

``config.json``: ``vocab``, ``width``, ``norm.eps``, ``logit_scale``, and ``layers``, a list of
    {"type": "mlstm", "mixer": {heads, dim, vdim, gate_cap}, "mlp": ...}
    {"type": "latent_attention", "mixer": {heads, dim, rot_dim, vdim, kv_rank, scale, rot: {base, dims}}, "mlp": ...}
with "mlp" one of {"kind": "dense", "ff"}, {"kind": "moe", "expert": {ff}, "router": {experts, identity, top}}, null.
The dense feed-forward's activation is the squared relu, the experts' the erf form of gelu.
"""

from __future__ import annotations

import json
import os
from types import SimpleNamespace

import torch
import torch.nn as nn

from . import dense
from .cache import LayerStateCache
from .layers import DenseFeedForward, LatentAttentionMixer, MatrixMemoryMixer, RoutedFeedForward, _param
from .weights import read_safetensors

DENSE_ACT, EXPERT_ACT = "relu2", "gelu_erf"


def tensor_shapes(cfg):
    """{tensor name: shape} of a configuration."""
    C, V = cfg["width"], cfg["vocab"]
    out = {"embed": (V, C), "head": (V, C), "final.norm": (C,)}
    for l, layer in enumerate(cfg["layers"]):
        m, p = layer["mixer"], f"l{l}.mix."
        H, D, vd = m["heads"], m["dim"], m["vdim"]
        out[f"l{l}.norm1"] = (C,)
        if layer["type"] == "mlstm":
            out.update({p + "q": (H * D, C), p + "k": (H * D, C), p + "v": (H * vd, C), p + "g": (H * vd, C), p + "o": (C, H * vd),
                        p + "norm": (H * vd,), p + "i": (H, C), p + "i.b": (H,), p + "f": (H, C), p + "f.b": (H,)})
        elif layer["type"] == "latent_attention":
            R, K = m["rot_dim"], m["kv_rank"]
            out.update({p + "q": (H * (D + R), C), p + "dkv": (K + R, C), p + "dkv.norm": (K,), p + "uk": (H * D, K),
                        p + "uv": (H * vd, K), p + "g": (H, C), p + "o": (C, H * vd)})
        else:
            raise ValueError(f"layer {l}: unknown type {layer['type']!r}")
        mlp, p = layer.get("mlp"), f"l{l}.mlp."
        if not mlp:
            continue
        out[f"l{l}.norm2"] = (C,)
        if mlp["kind"] == "dense":
            out.update({p + "up": (mlp["ff"], C), p + "down": (C, mlp["ff"])})
        elif mlp["kind"] == "moe":
            r, ff = mlp["router"], mlp["expert"]["ff"]
            n = r["experts"] + r.get("identity", 0)
            out.update({p + "router": (n, C), p + "correction": (n,)})
            for e in range(r["experts"]):
                out.update({f"{p}e{e}.up": (ff, C), f"{p}e{e}.down": (C, ff)})
        else:
            raise ValueError(f"layer {l}: unknown feed-forward {mlp['kind']!r}")
    return out


def _mixer(layer, eps, w, device, dtype):
    m = layer["mixer"]
    if layer["type"] == "mlstm":
        return MatrixMemoryMixer(m["heads"], m["dim"], m["vdim"], m["gate_cap"], eps, w, device, dtype)
    return LatentAttentionMixer(m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], m["rot"]["base"], m["rot"]["dims"],
                                m["scale"], eps, w, device, dtype)


def _feed_forward(mlp, w, device, dtype):
    if mlp["kind"] == "dense":
        return DenseFeedForward(DENSE_ACT, w, device, dtype)
    r = mlp["router"]
    return RoutedFeedForward(EXPERT_ACT, r["experts"], r.get("identity", 0), r["top"], w, device, dtype)


class ZokunexDecoder(nn.Module):
    """``weights``: {name: tensor} of ``tensor_shapes(cfg)``.  Storage and products are in ``dtype`` (bfloat16 or
    float32); residual stream, norms, routing, attention weights and recurrent state are float in both."""

    def __init__(self, cfg, weights, device="cuda:0", dtype=torch.bfloat16):
        super().__init__()
        if dtype not in dense.DTYPES:
            raise ValueError(f"dtype {dtype} is not supported")
        shapes = tensor_shapes(cfg)
        for name in shapes:
            if name not in weights:
                raise KeyError(f"missing tensor {name}")
        for name, t in (weights.items() if hasattr(weights, "items") else ()):
            if name in shapes and tuple(t.shape) != tuple(shapes[name]):
                raise ValueError(f"tensor {name} has shape {tuple(t.shape)}, expected {tuple(shapes[name])}")
        device = torch.device(device)
        self.raw_config, self.eps, self.logit_scale = cfg, float(cfg["norm"]["eps"]), float(cfg["logit_scale"])
        self.config = SimpleNamespace(vocab_size=cfg["vocab"], hidden_size=cfg["width"], num_hidden_layers=len(cfg["layers"]),
                                      max_position_embeddings=cfg.get("max_position_embeddings", 4096))
        self.embed_tokens, self.lm_head = _param(weights["embed"], device, dtype), _param(weights["head"], device, dtype)
        self.norm = _param(weights["final.norm"], device, torch.float32)
        self.mixers, self.norm1, self.mlps, self.norm2 = nn.ModuleList(), nn.ParameterList(), nn.ModuleList(), nn.ParameterList()
        for l, layer in enumerate(cfg["layers"]):
            self.mixers.append(_mixer(layer, self.eps, lambda n, p=f"l{l}.mix.": weights[p + n], device, dtype))
            self.norm1.append(_param(weights[f"l{l}.norm1"], device, torch.float32))
            mlp = layer.get("mlp")
            self.mlps.append(_feed_forward(mlp, lambda n, p=f"l{l}.mlp.": weights[p + n], device, dtype) if mlp else nn.Identity())
            self.norm2.append(_param(weights[f"l{l}.norm2"] if mlp else torch.empty(0), device, torch.float32))
        self._own_cache = None
        self._head_scratch = {}
        self.last_argmax = None      # greedy token of every kept row of the last forward, when the head kernel found it

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
        start = cache_position.to(torch.int64)
        x, h = dense.embed(input_ids.contiguous(), self.embed_tokens)
        last = len(self.mixers) - 1
        for l, (mixer, mlp) in enumerate(zip(self.mixers, self.mlps)):
            has_mlp = not isinstance(mlp, nn.Identity)
            final = self.norm if l == last else None
            y = mixer(h, B, T, start, kv_len, cache[l])
            h = dense.add_norm(x, y, self.norm1[l], self.eps, h.dtype, None if has_mlp else final)
            if has_mlp:
                h = mlp.add(x, h, self.norm2[l], self.eps, final)
            if trace is not None:
                trace.append(x.clone())
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
