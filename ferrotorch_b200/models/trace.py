"""Replay of a request trace: given token ids through a model, step by step, logits to files.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N < steps.jsonl

The model is chosen by its ``config.json`` (:mod:`~ferrotorch_b200.models.registry`) and runs on the step function,
cache and kernels that serve it (:class:`~ferrotorch_b200.models.serving.PagedStepper`); nothing is sampled.  Every
input line is one step, ``{"step": 0, "entries": [{"id": "a", "tokens": [5, 17], "want": [1]}], "end": ["a"]}``: all
entries run as one batch, a sequence is admitted at its first entry and continues from its cached tokens later, the
sequences listed in ``end`` give their pages and slot back after the step.  When places are wanted, ``OUT/<step>.f32``
receives their logits (little-endian 32-bit floats, entry after entry); after every step ``done <step>`` is printed.

The cache pool holds ``--max-tokens`` tokens (sequences rounded up to whole pages) and four sequences."""
from __future__ import annotations

import argparse
import json
import os
import sys

PAGE_TOKENS = 16
MAX_SEQUENCES = 4


class TraceReplayer:
    """Maps request ids to sequence slots of a stepper and feeds it one step after another."""

    def __init__(self, stepper):
        self.stepper = stepper
        self._slots: dict = {}

    def step(self, entries: list, end: list):
        """Logits ``[wanted, vocab]`` of one step (entries as in the input format), then the ends."""
        parts = []
        for e in entries:
            rid = e["id"]
            if rid not in self._slots:
                self._slots[rid] = self.stepper.admit()
            tokens = [int(t) for t in e["tokens"]]
            if tokens:
                parts.append((self._slots[rid], tokens, [int(w) for w in e.get("want", ())]))
        logits = self.stepper.feed(parts) if parts else None
        for rid in end:
            slot = self._slots.pop(rid, None)
            if slot is not None:
                self.stepper.release(slot)
        return logits


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="Replay a request trace; logits to files.")
    ap.add_argument("--model", required=True, help="directory with config.json and model.safetensors")
    ap.add_argument("--dtype", choices=("bfloat16", "float32"), default="bfloat16")
    ap.add_argument("--out", required=True, help="directory for <step>.f32")
    ap.add_argument("--max-tokens", type=int, required=True, help="tokens the cache pool holds")
    ap.add_argument("--device", default="cuda")
    args = ap.parse_args(argv)

    import torch

    from .registry import load_causal_lm
    from .serving import PagedStepper

    model = load_causal_lm(args.model, getattr(torch, args.dtype), args.device)
    pages = (args.max_tokens + PAGE_TOKENS - 1) // PAGE_TOKENS
    replayer = TraceReplayer(PagedStepper(model, pages, PAGE_TOKENS, MAX_SEQUENCES, pages * PAGE_TOKENS))
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        logits = replayer.step(step["entries"], step.get("end", []))
        if logits is not None and logits.shape[0]:
            data = logits.float().cpu().numpy().astype("<f4", copy=False).tobytes()
            with open(os.path.join(args.out, "%d.f32" % step["step"]), "wb") as f:
                f.write(data)
        elif args.device != "cpu":
            torch.cuda.synchronize()
        print("done %d" % step["step"], flush=True)
    return 0


if __name__ == "__main__":
    raise SystemExit(main())
