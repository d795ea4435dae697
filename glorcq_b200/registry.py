"""Which decoder a checkpoint folder holds, and how it is loaded.

``config.json`` names the design: ``architecture`` (or the first of ``architectures``) selects a loader registered here;
the quantized checkpoints of the reference (``glorcq_model.pt`` beside a transformers config) are the default.
"""

from __future__ import annotations

import json
import os

import torch

DTYPES = {"bfloat16": torch.bfloat16, "float16": torch.float16, "float32": torch.float32}


def _zokunex(path, device, dtype):
    from .zokunex import ZokunexDecoder
    return ZokunexDecoder.from_pretrained(path, device, dtype or torch.bfloat16)


def _femirax(path, device, dtype):
    from .femirax import FemiraxDecoder
    return FemiraxDecoder.from_pretrained(path, device, dtype or torch.bfloat16)


def _quantized(path, device, dtype):
    if dtype not in (None, torch.float16):
        raise UnsupportedDtype("the quantized decoders compute in float16")
    from .model_builder import load_glorcq_model
    return load_glorcq_model(path, device)


class UnsupportedDtype(ValueError):
    pass


ARCHITECTURES = {"Zokunex": _zokunex, "Femirax": _femirax}


def register(name, loader):
    """``loader(path, device, dtype or None) -> model`` for folders whose config.json names ``name``."""
    ARCHITECTURES[name] = loader


def architecture_of(path):
    """The name in config.json, or None for a quantized checkpoint."""
    with open(os.path.join(path, "config.json")) as f:
        cfg = json.load(f)
    name = cfg.get("architecture") or (cfg.get("architectures") or [None])[0]
    if name in ARCHITECTURES:
        return name
    if os.path.exists(os.path.join(path, "glorcq_model.pt")):
        return None
    raise ValueError(f"{path}: no loader for architecture {name!r} (known: {sorted(ARCHITECTURES)})")


def load_model(path, device="cuda:0", dtype=None):
    """The decoder in ``path``; ``dtype`` (torch dtype or its name) is the design's default when None."""
    if isinstance(dtype, str):
        dtype = DTYPES[dtype]
    name = architecture_of(path)
    return (ARCHITECTURES[name] if name else _quantized)(path, device, dtype)
