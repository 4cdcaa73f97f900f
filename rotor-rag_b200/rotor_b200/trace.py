"""Trace replay: token ids of a request, fed through a model portion by portion.

One request is live at a time; it runs through the model's own forward (`forward_rows_device`), which
appends to the caches at the request's length.  Ending it gives its positions back.
"""
from __future__ import annotations

import json
import os

import numpy as np


class TraceSession:
    def __init__(self, model):
        self.model = model
        self.request, self.length = None, 0

    def step(self, entries, end=()):
        """entries: [{id, tokens, want}]; returns float32 [wanted, vocab] (host) in entry order."""
        out = []
        for e in entries:
            if not e["tokens"]:
                if e.get("want"):
                    raise ValueError("logits wanted of an empty portion")
                continue
            if self.request is None:
                self.request, self.length = e["id"], 0
            if e["id"] != self.request:
                raise ValueError(f"request {e['id']} while {self.request} is live: one request at a time")
            logits = self.model.forward_rows_device(e["tokens"], self.length, e.get("want", []))
            self.length += len(e["tokens"])
            if len(e.get("want", [])):
                out.append(logits.cpu().numpy())
        for r in end:
            if r == self.request:
                self.request, self.length = None, 0
        return np.concatenate(out) if out else np.zeros((0, self.model.vocab_size), dtype=np.float32)


def replay(model, lines, out_dir, emit):
    """Runs the steps (JSON lines) and writes <step>.f32 for those that want logits."""
    from . import abi
    session = TraceSession(model)
    for line in lines:
        if not line.strip():
            continue
        s = json.loads(line)
        logits = session.step(s.get("entries", []), s.get("end", []))
        abi.device_status()
        if len(logits):
            with open(os.path.join(out_dir, f"{s['step']}.f32"), "wb") as f:
                f.write(np.ascontiguousarray(logits, dtype="<f4").tobytes())
        emit(f"done {s['step']}")
