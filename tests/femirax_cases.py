"""Small Femirax configurations with random weights."""

import math

import torch

from glorcq_b200.femirax import tensor_shapes
from tests.zokunex_cases import doubles, most_rel, rel, stored, tokens, worst_rel  # noqa: F401


def retention(heads=3, dim=24, vdim=16, decay=None, base=10000.0, dims=None):
    decay = decay or [1 - 0.3 * 0.2 ** i for i in range(heads)]
    return {"type": "retention", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay,
                                           "rot": {"base": base, "dims": dim if dims is None else dims}}}


def parallel(heads=4, kv_heads=2, dim=16, scale=None, base=500.0, dims=None, rheads=3, rdim=16, rvdim=24, tau=8.0):
    return {"type": "parallel", "mixer": {
        "left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale or 2.5 * dim ** -0.5,
                 "rot": {"base": base, "dims": dim if dims is None else dims}},
        "right": {"heads": rheads, "dim": rdim, "vdim": rvdim, "tau": tau}}}


def dense_mlp(ff=88):
    return {"kind": "dense", "ff": ff}


def config(layers, vocab=160, width=104, eps=1e-5, side=24):
    """layers: (mixer entry, feed-forward or None) pairs"""
    return {"architecture": "Femirax", "vocab": vocab, "width": width, "norm": {"eps": eps}, "token_side": {"dim": side},
            "layers": [dict(m, mlp=f) for m, f in layers]}


# every kind of layer with and without a feed-forward; one head of each kind, all heads on one key head, partial rotations
MIXED = config([(parallel(), dense_mlp()), (retention(), dense_mlp(40)), (retention(1, 8, 40, [0.9], 77.0, 4), None),
                (parallel(3, 1, 24, dims=10, rheads=1, rdim=40, rvdim=8, tau=1.0), None), (retention(2, 72, 24, [0.25, 1.0], 1e6, 32), None)])
# sizes that are no multiple of eight anywhere: the generic kernels
ODD = config([(retention(3, 10, 13, dims=6), dense_mlp(35)), (parallel(6, 2, 9, dims=4, rheads=2, rdim=11, rvdim=7, tau=3.0), None),
              (parallel(2, 2, 12, rheads=1, rdim=5, rvdim=12), dense_mlp(21)), (retention(1, 7, 33, [0.99], dims=2), None)],
             vocab=101, width=50, eps=1e-3, side=7)
# an odd-sized side beside a regular one, in both orders of the columns
UNEVEN = config([(parallel(2, 1, 20, rheads=2, rdim=16, rvdim=16), dense_mlp(30)), (retention(2, 16, 20), None),
                 (parallel(2, 2, 16, rheads=3, rdim=12, rvdim=8), None)], width=64, side=20)
# heads of the sizes of a large model
WIDE = config([(retention(2, 128, 256), dense_mlp(512)), (parallel(8, 2, 128, rheads=2, rdim=128, rvdim=160, tau=16.0), dense_mlp(320)),
               (parallel(2, 1, 256, rheads=1, rdim=200, rvdim=64), None)], vocab=320, width=256, side=64)
RANKS = {"mixed": {0: 16, 3: 5}, "odd": {1: 3, 2: 1}, "uneven": {0: 8, 2: 20}, "wide": {1: 24, 2: 40}}
CONFIGS = {"mixed": MIXED, "odd": ODD, "uneven": UNEVEN, "wide": WIDE}


def make_weights(cfg, seed=0, dtype=torch.bfloat16, rank=16):
    """Random tensors (bf16 values): peaked attention, decays per channel from almost one to a few per mille."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(cfg, rank).items():
        leaf = name.split(".", 1)[1] if "." in name else name
        if leaf.endswith(("norm", ".out")) or leaf in ("norm1", "norm2"):
            t = 1 + 0.3 * torch.randn(shape, generator=g)
        elif leaf == "mix.right.a2.b":
            t = 2 + 2 * torch.randn(shape, generator=g)
        elif name in ("embed", "side.embed"):
            t = torch.randn(shape, generator=g)
        else:
            gain = {"mix.right.a2": 2.0}.get(leaf, 1.0)
            t = gain * torch.randn(shape, generator=g) / math.sqrt(shape[-1])
        out[name] = t.to(dtype)
    return out


def weights_of(name, seed=11):
    return make_weights(CONFIGS[name], seed, rank=RANKS[name])
