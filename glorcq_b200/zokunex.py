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

import torch
import torch.nn as nn

from . import dense
from .dense_decoder import DenseDecoder
from .layers import DenseFeedForward, LatentAttentionMixer, MatrixMemoryMixer, RoutedFeedForward, _param

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


class ZokunexDecoder(DenseDecoder):
    @staticmethod
    def tensor_shapes(cfg, weights=None):
        return tensor_shapes(cfg)

    def build(self, cfg, weights, device, dtype):
        self.norm1, self.mlps, self.norm2 = nn.ParameterList(), nn.ModuleList(), nn.ParameterList()
        for l, layer in enumerate(cfg["layers"]):
            self.mixers.append(_mixer(layer, self.eps, lambda n, p=f"l{l}.mix.": weights[p + n], device, dtype))
            self.norm1.append(_param(weights[f"l{l}.norm1"], device, torch.float32))
            mlp = layer.get("mlp")
            self.mlps.append(_feed_forward(mlp, lambda n, p=f"l{l}.mlp.": weights[p + n], device, dtype) if mlp else nn.Identity())
            self.norm2.append(_param(weights[f"l{l}.norm2"] if mlp else torch.empty(0), device, torch.float32))

    def run_layers(self, ids, B, T, start, kv_len, cache, trace):
        x, h = dense.embed(ids, self.embed_tokens)
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
        return h
