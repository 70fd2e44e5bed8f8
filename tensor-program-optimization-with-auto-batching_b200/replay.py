"""Trace replay: feeds given tokens through a model step by step and writes the logits that are asked for.

The steps come as JSON lines; every step runs through the engine calls that generation uses -- ``EngineBase.extend`` for a
portion of a prompt, ``EngineBase.decode`` for one token of a sequence under way -- over the model's paged cache.
"""
from __future__ import annotations

import json
import os
import sys

import numpy as np
import torch

from . import build, registry

MAX_ROWS = 2048      # rows of one pass
MAX_SEQUENCES = 64   # live at a time


class TraceRunner:
    def __init__(self, model, max_tokens: int, page_size: int = 16):
        max_tokens = max(int(max_tokens), 1)
        # (every live sequence may leave a page partly filled: the cache accounts for that itself)
        self.kv = model.new_cache(MAX_SEQUENCES, max_tokens, MAX_ROWS, page_size)
        self.engine = model.new_engine(self.kv, min(MAX_ROWS, max(max_tokens, MAX_SEQUENCES)))
        self.ids = {}
        self._next = 0

    def _sid(self, name):
        if name not in self.ids:
            self.ids[name] = self._next
            self._next += 1
            self.kv.add_sequence(self.ids[name])
        return self.ids[name]

    def step(self, entries, end=()):
        """Logits [wanted, vocab] (fp32, host) of one step, or None when nothing is wanted."""
        sids = [self._sid(e["id"]) for e in entries]
        toks, want = [e["tokens"] for e in entries], [e.get("want", []) for e in entries]
        out = None
        if sids and all(len(t) == 1 for t in toks) and all(self.kv.length(s) > 0 for s in sids):
            lg, _ = self.engine.decode(sids, [t[0] for t in toks], [-1] * len(sids))
            rows = [i for i, w in enumerate(want) for _ in w]
            out = lg[rows] if rows else None
            self.engine.check_status()
        elif sids:
            out, _ = self.engine.extend(sids, toks, want=want)
        out = out.cpu().numpy().astype("<f4") if out is not None and out.shape[0] else None
        for name in end:
            if name in self.ids:
                self.kv.remove_sequence(self.ids.pop(name))
        return out


def main(args, stdin=None, stdout=None) -> int:
    stdin, stdout = stdin or sys.stdin, stdout or sys.stdout
    dtype = getattr(torch, args.dtype)
    torch.backends.cuda.matmul.allow_tf32 = False
    build.build()
    try:
        model = registry.load_model(args.model, device="cuda", dtype=dtype)
    except registry.UnsupportedPrecision as e:
        print(e, file=sys.stderr)
        return 3
    runner = TraceRunner(model, args.max_tokens)
    for line in stdin:
        if not line.strip():
            continue
        s = json.loads(line)
        out = runner.step(s["entries"], s.get("end", ()))
        if out is not None:
            out.tofile(os.path.join(args.out, f"{s['step']}.f32"))
        print(f"done {s['step']}", file=stdout, flush=True)
    return 0
