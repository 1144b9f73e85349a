"""Replays a recorded trace of requests through a model, step by step, and writes logits.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR [--max-tokens N] < steps.jsonl

Every line of standard input is one step: ``{"step": n, "entries": [{"id": ..., "tokens": [...], "want": [...]}], "end":
[...]}``.  An entry brings a request's next tokens; ``want`` are the places among them whose logits go to
``OUT/<step>.f32`` (little-endian fp32, entries in order).  Requests named in ``end`` give their cache back.  After each
step ``done <n>`` is printed.  Nothing is sampled: the tokens come from the trace, and the model's own ``step`` and cache
pool, the ones its generation uses, process them.  Exit code 3: the model's family does not run in that dtype or has no
``step``.
"""
from __future__ import annotations

import argparse
import json
import os
import sys
from typing import Dict

DTYPES = ("bfloat16", "float32")


def add_arguments(ap) -> None:
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", choices=DTYPES, default="bfloat16")
    ap.add_argument("--out", required=True, help="folder for the logits")
    ap.add_argument("--max-tokens", type=int, default=0, help="most tokens live requests hold at a time")


class TraceRunner:
    """Requests by name over one model; each holds a cache of the model's pool until it ends."""

    def __init__(self, model, max_tokens: int = 0):
        self.model, self.max_tokens = model, max_tokens
        self.live: Dict[str, object] = {}

    def step(self, entries, end):
        """Wanted logits ``[n, vocab]`` (fp32, CPU) of one step, or None when nothing is wanted."""
        import torch
        wanted = []
        for e in entries:
            tokens, want = e["tokens"], list(e.get("want") or [])
            if not tokens:
                continue
            cache = self.live.get(e["id"])
            if cache is None:
                cache = self.live[e["id"]] = self.model.new_cache(max(self.max_tokens, len(tokens)))
            t = torch.tensor([tokens], dtype=torch.long, device=self.model.device)
            out = self.model.step(cache, t, want)
            if want:
                wanted.append(out.float().cpu())
        for name in end:
            cache = self.live.pop(name, None)
            if cache is not None:
                self.model.free_cache(cache)
        return torch.cat(wanted, 0) if wanted else None

    def run(self, lines, out_dir: str, report=print) -> None:
        for line in lines:
            if not line.strip():
                continue
            rec = json.loads(line)
            logits = self.step(rec.get("entries", []), rec.get("end", []))
            if logits is not None:
                path = os.path.join(out_dir, f"{rec['step']}.f32")
                logits.numpy().astype("<f4").tofile(path)
            report(f"done {rec['step']}")


def main(args) -> int:
    import torch
    from .. import _native
    from .servers import load_hf_model
    _native.load(required=True)
    dtype = getattr(torch, args.dtype)
    model, _, _ = load_hf_model("auto", args.model, device="cuda", dtype=dtype)
    if not hasattr(model, "step"):
        print(f"{type(model).__name__} has no step function", file=sys.stderr)
        raise SystemExit(3)
    model.eval()
    TraceRunner(model, args.max_tokens).run(sys.stdin, args.out, lambda s: print(s, flush=True))
    _native.raise_on_device_error()
    return 0


def cli(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="Replay a trace of requests and write logits.")
    add_arguments(ap)
    return main(ap.parse_args(argv))
