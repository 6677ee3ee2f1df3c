"""Replays a trace of token ids through a model, step by step, and writes the logits a step asks for.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N  < steps.jsonl

A step is one JSON object a line: ``{"step": n, "entries": [{"id", "tokens", "want"}, ...], "end": [ids]}``.  Every entry
brings the next tokens of a request; ``want`` are the places among them whose logits go to ``DIR/n.f32`` (little-endian fp32
``[wanted, vocab]``, in order).  Requests named by ``end`` give back what they hold.  After each step ``done n`` is printed.
The model class is chosen by ``config.json``; steps run through the model's packed forward and its state cache, exactly as
``generate`` runs them.
"""
from __future__ import annotations

import argparse
import json
import os
import sys


class TraceSession:
    """The requests of a trace on one model and one cache."""

    def __init__(self, model, max_tokens: int = 0):
        if not hasattr(model, "forward_packed"):
            raise TypeError(f"{type(model).__name__} keeps no requests of unequal length in one batch; traces need that")
        self.model, self.cache = model, model.new_cache(capacity_tokens=min(max_tokens, 1 << 16))
        self.order = []                    # request ids in the cache's row order

    def step(self, entries, end=()):
        """Runs one step; returns the wanted logits ``[wanted, vocab]`` (fp32, device), None if nothing is wanted."""
        logits = self._run(entries) if entries else None
        gone = [self.order.index(r) for r in end if r in self.order]
        if gone:
            self.cache.close(gone)
            self.order = [r for i, r in enumerate(self.order) if i not in set(gone)]
        return logits

    def _run(self, entries):
        import torch
        new = [e["id"] for e in entries if e["id"] not in self.order]
        if new:
            self.cache.open(len(new))
            self.order += new
        ids, want, at = [], [], 0
        for e in entries:
            ids += e["tokens"]
            want += [at + w for w in e["want"]]
            at += len(e["tokens"])
        rows = [self.order.index(e["id"]) for e in entries]
        whole = rows == list(range(len(self.order)))
        logits = self.model.forward_packed(torch.tensor(ids, dtype=torch.int64).to(self.model.device), self.cache,
                                           [len(e["tokens"]) for e in entries], None if whole else rows, want)
        return logits if want else None


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(description="Replay a trace of token ids from standard input and write logits.")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", choices=["bfloat16", "float32"], default="bfloat16")
    ap.add_argument("--out", required=True, help="folder for <step>.f32")
    ap.add_argument("--max-tokens", type=int, default=0, help="most tokens live requests hold at any time")
    args = ap.parse_args(argv)
    from . import build
    build.build()                          # compiles in a fresh checkout, returns at once otherwise
    import numpy as np
    import torch
    from .registry import load_model
    torch.backends.cuda.matmul.allow_tf32 = False
    session = TraceSession(load_model(args.model, dtype=getattr(torch, args.dtype), device="cuda"), args.max_tokens)
    with torch.inference_mode():
        for line in sys.stdin:
            if not line.strip():
                continue
            step = json.loads(line)
            logits = session.step(step["entries"], step.get("end", ()))
            if logits is not None:
                logits.cpu().numpy().astype("<f4").tofile(os.path.join(args.out, f"{step['step']}.f32"))
            session.cache.check_status()
            print(f"done {step['step']}", flush=True)
    return 0


if __name__ == "__main__":
    sys.exit(main())
