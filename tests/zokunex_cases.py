"""Small Zokunex configurations with random weights, and comparisons against the plain implementation."""

import math

import torch

from glorcq_b200.zokunex import tensor_shapes


def mlstm(heads=2, dim=24, vdim=40, gate_cap=15.0):
    return {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": gate_cap}}


def latent(heads=3, dim=16, rot_dim=8, vdim=24, kv_rank=48, base=10000.0, scale=None):
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank,
                                                  "scale": scale or (dim + rot_dim) ** -0.5, "rot": {"base": base, "dims": rot_dim}}}


def dense_mlp(ff=88):
    return {"kind": "dense", "ff": ff}


def moe_mlp(experts=6, identity=1, top=3, ff=40):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "identity": identity, "top": top}}


def config(layers, vocab=160, width=104, eps=1e-5, logit_scale=0.25):
    """layers: (mixer entry, feed-forward or None) pairs"""
    return {"architecture": "Zokunex", "vocab": vocab, "width": width, "norm": {"eps": eps}, "logit_scale": logit_scale,
            "layers": [dict(m, mlp=f) for m, f in layers]}


MIXED = config([(latent(), moe_mlp()), (mlstm(), dense_mlp()), (mlstm(heads=1, dim=16, vdim=16), None),
                (latent(heads=2, dim=40, rot_dim=16, vdim=16, kv_rank=32), dense_mlp(40)), (mlstm(heads=3), moe_mlp(5, 2, 1))])
# sizes that are no multiple of eight anywhere: the generic kernels
ODD = config([(mlstm(heads=3, dim=10, vdim=13), moe_mlp(3, 0, 2, 21)), (latent(heads=2, dim=9, rot_dim=6, vdim=11, kv_rank=20), dense_mlp(35)),
              (latent(heads=1, dim=12, rot_dim=4, vdim=5, kv_rank=18), None)], vocab=101, width=50, eps=1e-3, logit_scale=1.0)
# heads of the sizes of a large model, one layer of each kind
WIDE = config([(mlstm(heads=2, dim=128, vdim=256), dense_mlp(512)),
               (latent(heads=4, dim=128, rot_dim=64, vdim=128, kv_rank=512), moe_mlp(8, 1, 2, 96))], vocab=320, width=256)


def make_weights(cfg, seed=0, dtype=torch.bfloat16):
    """Random tensors (bf16 values): peaked attention, input gates that differ from token to token, slow forgetting,
    and corrections that decide the routing now and then."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        leaf = name.split(".", 1)[1] if "." in name else name
        if leaf.endswith("norm") or leaf in ("norm1", "norm2"):
            t = 1 + 0.3 * torch.randn(shape, generator=g)
        elif leaf == "mix.i.b":
            t = torch.randn(shape, generator=g)
        elif leaf == "mix.f.b":
            t = 4 + torch.randn(shape, generator=g)
        elif leaf.endswith("correction"):
            t = 0.1 * torch.randn(shape, generator=g)
        else:
            gain = {"mix.i": 2.0, "mlp.router": 2.0, "mix.dkv": 2.0, "mix.q": 2.0, "embed": 3.0}.get(leaf, 1.0)
            t = gain * torch.randn(shape, generator=g) / math.sqrt(shape[-1] if leaf != "embed" else 1)
        out[name] = t.to(dtype)
    return out


def tokens(cfg, n, seed=1):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def doubles(weights):
    return {k: v.double() for k, v in weights.items()}


def rel(a, b):
    """Root mean square of the difference over that of the reference."""
    a, b = a.double().cpu(), b.double().cpu()
    return ((a - b).pow(2).mean().sqrt() / (b.pow(2).mean().sqrt() + 1e-30)).item()


def worst_rel(a, b):
    """The largest row's difference (rms) over the reference's rms: one wrong position cannot hide among many."""
    a, b = a.double().cpu(), b.double().cpu()
    a, b = a.reshape(-1, a.shape[-1]), b.reshape(-1, b.shape[-1])
    return ((a - b).pow(2).mean(-1).sqrt().max() / (b.pow(2).mean().sqrt() + 1e-30)).item()


def stored(a, b, dtype, exact=2e-5):
    """Largest difference in units of what storing the value in ``dtype`` allows (half a bf16 step of the value, or
    ``exact`` of the reference's rms): at most 1 for a correctly rounded result."""
    a, b = a.double().cpu(), b.double().cpu()
    step = 2.0 ** -8 * b.abs() if dtype == torch.bfloat16 else 0.0
    return ((a - b).abs() / (step + 10 * exact * b.pow(2).mean().sqrt() + 1e-30)).max().item()


def most_rel(a, b, share=0.9):
    """The error that ``share`` of the rows stay below: a routing choice that bf16 rounding turns may cost a few rows."""
    a, b = a.double().cpu(), b.double().cpu()
    a, b = a.reshape(-1, a.shape[-1]), b.reshape(-1, b.shape[-1])
    return (((a - b).pow(2).mean(-1) / b.pow(2).mean()).sqrt().quantile(share)).item()
