"""Replays a trace: given token ids go through a model step by step, and the logits of chosen places are written out.

One JSON object per input line,
    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": ["a"]}
brings the next tokens of a request ("want": places among them whose logits are written) and names the requests that
are finished after the step.  ``<out>/<step>.f32`` receives the wanted logits, [wanted, vocab], 32-bit little-endian
floats; a line ``done <step>`` follows every step.  Requests come one after the other and each keeps its state between
its steps.  Everything runs through ``GLoRCQGraphWrapper.step``, as generation does.
"""

from __future__ import annotations

import json
import os
import sys

import numpy as np
import torch

from .graph_wrapper import GLoRCQGraphWrapper
from .registry import UnsupportedDtype, load_model


class TraceRunner:
    def __init__(self, model, max_tokens):
        self.wrapper = GLoRCQGraphWrapper(model, max_batch_size=1, max_seq_len=max(16, max_tokens))
        self.live, self.position = None, 0

    def run(self, entry):
        """Logits (wanted, vocab) of one entry, on the device; None when nothing is wanted."""
        if self.live is None:
            self.live, self.position = entry["id"], 0
            self.wrapper.static_cache.reset()
        if entry["id"] != self.live:
            raise ValueError(f"request {entry['id']!r} comes while {self.live!r} is not finished")
        tokens, want = entry["tokens"], entry.get("want") or []
        if not tokens:
            return None
        dev = self.wrapper.device
        ids = torch.tensor([tokens], dtype=torch.long, device=dev)
        logits = self.wrapper.step(ids, self.position, torch.tensor(want, dtype=torch.long, device=dev) if want else 1)
        self.position += len(tokens)
        return logits[0] if want else None

    def end(self, ids):
        if self.live in ids:
            self.live, self.position = None, 0


def main(args):
    dev = torch.device("cuda:0")
    torch.backends.cuda.matmul.allow_tf32 = torch.backends.cudnn.allow_tf32 = False
    try:
        runner = TraceRunner(load_model(args.model, dev, args.dtype), args.max_tokens)
    except UnsupportedDtype as exc:
        print(exc, file=sys.stderr)
        return 3
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        parts = [runner.run(e) for e in step["entries"]]
        parts = [p for p in parts if p is not None]
        if parts:
            data = np.ascontiguousarray(torch.cat(parts).float().cpu().numpy(), dtype="<f4")
            data.tofile(os.path.join(args.out, f"{step['step']}.f32"))
        runner.end(step.get("end") or [])
        print(f"done {step['step']}", flush=True)
    torch.cuda.synchronize()
    return 0
