"""Femirax: a pre-norm decoder whose layers mix by retention, or by attention and gated linear attention side by side, each
with a gated feed-forward or none and, at its end, an input of the token's own row of a per-layer table.

    model = FemiraxDecoder.from_pretrained(folder, device="cuda:0", dtype=torch.bfloat16)

``config.json``: ``vocab``, ``width``, ``norm.eps``, ``token_side.dim``, and ``layers``, a list of
    {"type": "retention", "mixer": {heads, dim, vdim, decay: [one per head], rot: {base, dims}}, "mlp": ...}
    {"type": "parallel", "mixer": {"left": {heads, kv_heads, dim, vdim, scale, rot: {base, dims}},
                                   "right": {heads, dim, vdim, tau}}, "mlp": ...}
with "mlp" one of {"kind": "dense", "ff"}, null.  Retention pairs the halves of a head in its rotation, the attention
neighbouring elements.  The rank of the right side's decay projection is that of its tensors.
"""

from __future__ import annotations

import torch
import torch.nn as nn

from . import dense
from .dense_decoder import DenseDecoder
from .layers import (GatedFeedForward, GatedLinearAttention, ParallelMixer, RetentionMixer, Rotation, SharedValueAttention, TokenSideInput,
                     _param)

DEFAULT_RANK = 16


def tensor_shapes(cfg, rank=DEFAULT_RANK):
    """{tensor name: shape} of a configuration; ``rank``: of the decay projections, one for all layers or {layer: rank}."""
    C, V, side = cfg["width"], cfg["vocab"], cfg["token_side"]["dim"]
    out = {"embed": (V, C), "side.embed": (V, side * len(cfg["layers"])), "head": (V, C), "final.norm": (C,)}
    for l, layer in enumerate(cfg["layers"]):
        m, p = layer["mixer"], f"l{l}.mix."
        out[f"l{l}.norm1"] = (C,)

        def linear_attention(p, m):
            qk, v = m["heads"] * m["dim"], m["heads"] * m["vdim"]
            return {p + "q": (qk, C), p + "k": (qk, C), p + "v": (v, C), p + "g": (v, C), p + "o": (C, v)}
        if layer["type"] == "retention":
            out.update(linear_attention(p, m))
        elif layer["type"] == "parallel":
            a, b = m["left"], m["right"]
            r = rank[l] if isinstance(rank, dict) else rank
            out.update({p + "left.q": (a["heads"] * a["dim"], C), p + "left.k": (a["kv_heads"] * a["dim"], C),
                        p + "left.o": (C, a["heads"] * a["vdim"]), p + "left.out": (C,), p + "right.out": (C,)})
            out.update(linear_attention(p + "right.", b))
            out.update({p + "right.norm": (b["vdim"],), p + "right.a1": (r, C), p + "right.a2": (b["heads"] * b["dim"], r),
                        p + "right.a2.b": (b["heads"] * b["dim"],)})
        else:
            raise ValueError(f"layer {l}: unknown type {layer['type']!r}")
        mlp, p = layer.get("mlp"), f"l{l}.mlp."
        if mlp:
            if mlp["kind"] != "dense":
                raise ValueError(f"layer {l}: unknown feed-forward {mlp['kind']!r}")
            out.update({f"l{l}.norm2": (C,), p + "gate": (mlp["ff"], C), p + "up": (mlp["ff"], C), p + "down": (C, mlp["ff"])})
        p = f"l{l}.side."
        out.update({p + "gate": (side, C), p + "proj": (C, side), p + "norm": (C,)})
    return out


def _mixer(layer, eps, w, device, dtype):
    m = layer["mixer"]
    if layer["type"] == "retention":
        return RetentionMixer(m["heads"], m["dim"], m["vdim"], m["decay"], Rotation(m["rot"]["dims"], m["rot"]["base"], False), eps, w, device,
                              dtype)
    a, b = m["left"], m["right"]
    left = SharedValueAttention(a["heads"], a["kv_heads"], a["dim"], a["vdim"], Rotation(a["rot"]["dims"], a["rot"]["base"], True), a["scale"],
                                eps, lambda n: w("left." + n), device, dtype)
    right = GatedLinearAttention(b["heads"], b["dim"], b["vdim"], b["tau"], eps, lambda n: w("right." + n), device, dtype)
    return ParallelMixer(left, right, eps, w, device, dtype)


class FemiraxDecoder(DenseDecoder):
    @staticmethod
    def tensor_shapes(cfg, weights=None):
        ranks = {l: weights[f"l{l}.mix.right.a1"].shape[0] for l, layer in enumerate(cfg["layers"]) if layer["type"] == "parallel"} \
            if weights is not None else DEFAULT_RANK
        return tensor_shapes(cfg, ranks)

    def build(self, cfg, weights, device, dtype):
        self.side_table = _param(weights["side.embed"], device, dtype)
        self.norm1, self.mlps, self.norm2, self.sides = nn.ParameterList(), nn.ModuleList(), nn.ParameterList(), nn.ModuleList()
        n = cfg["token_side"]["dim"]
        for l, layer in enumerate(cfg["layers"]):
            def w(name, p=f"l{l}."):
                return weights[p + name]
            self.mixers.append(_mixer(layer, self.eps, lambda name, w=w: w("mix." + name), device, dtype))
            self.norm1.append(_param(w("norm1"), device, torch.float32))
            mlp = layer.get("mlp")
            self.mlps.append(GatedFeedForward(self.eps, lambda name, w=w: w("mlp." + name), device, dtype) if mlp else nn.Identity())
            self.norm2.append(_param(w("norm2") if mlp else torch.empty(0), device, torch.float32))
            self.sides.append(TokenSideInput(self.side_table[:, l * n:(l + 1) * n], self.eps, lambda name, w=w: w("side." + name), device, dtype))

    def run_layers(self, ids, B, T, start, kv_len, cache, trace):
        x, h = dense.embed(ids, self.embed_tokens, self.norm1[0], self.eps)
        next_norm = list(self.norm1)[1:] + [self.norm]
        for l, (mixer, mlp, side) in enumerate(zip(self.mixers, self.mlps, self.sides)):
            has_mlp = not isinstance(mlp, nn.Identity)
            h = mixer.add(x, h, B, T, start, kv_len, cache[l], self.norm2[l] if has_mlp else None)
            if has_mlp:
                h = mlp.add(x, h)
            h = side.add(x, h, ids, next_norm[l])
            if trace is not None:
                trace.append(x.clone())
        return h
