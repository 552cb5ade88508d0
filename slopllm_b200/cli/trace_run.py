"""Replay a token trace: feed given token ids through a model step by step and write the logits that are asked for.

Nothing is sampled.  The steps go through `Engine.step`, that is the model, cache, state slots, batch layout, kernels and
captured decode graphs that generation uses.  Standard input has one JSON object a line,

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

where `entries` holds each request's next tokens (all entries of a step are one batch) with the places whose logits are
wanted, and `end` names the requests that are finished after the step.  The logits of step N go to OUT/N.f32 (little-endian
fp32, [wanted, vocab]); "done N" is printed after every step.
"""
from __future__ import annotations

import argparse
import json
import os
import sys
from typing import Dict

import torch

MAX_REQUESTS = 4


class TraceRunner:
    """Applies trace steps to an engine; one sequence per live request."""

    def __init__(self, engine):
        self.engine = engine
        self.live: Dict[str, object] = {}

    def run_step(self, step: dict):
        """Logits [wanted, vocab] of one step (None when nothing is wanted)."""
        eng = self.engine
        seqs, tokens, want = [], [], []
        for e in step.get("entries", []):
            rid, toks = e["id"], [int(x) for x in e["tokens"]]
            if not toks:
                continue
            if rid not in self.live:
                self.live[rid] = eng.kv.new_sequence()
            if any(not 0 <= w < len(toks) for w in e.get("want", [])):
                raise ValueError(f"request {rid}: a wanted place lies outside its {len(toks)} tokens")
            seqs.append(self.live[rid])
            tokens.append(toks)
            want.append(list(e.get("want", [])))
        out = eng.step(seqs, tokens, want) if seqs else None
        for rid in step.get("end", []):
            s = self.live.pop(rid, None)
            if s is not None:
                eng.finish(s)
        return out


def build_engine(model_dir: str, dtype: str, max_tokens: int, device: torch.device):
    from ..config import PAGE_SIZE
    from ..models.registry import inspect_model, load_registered
    from ..ops import native
    from ..parallel.dist import ParallelContext
    from ..runtime.engine import Engine
    name, reg, _ = inspect_model(model_dir)
    if dtype == "float32" and not reg.float32:
        print(f"{name} does not run in float32", file=sys.stderr)
        raise SystemExit(3)
    if device.type == "cuda":
        from .. import build_native
        native.use_library(build_native.ensure_kernels(name, reg.kernel_sources))
        torch.backends.cuda.matmul.allow_tf32 = False
        torch.cuda.set_device(device)
    cfg, model = load_registered(reg, model_dir, ParallelContext(device=device), dtype=dtype)
    pages = max(1, -(-max_tokens // PAGE_SIZE))
    return Engine(cfg, model, num_pages=pages, max_batch=MAX_REQUESTS, max_seq_len=pages * PAGE_SIZE, max_states=MAX_REQUESTS)


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description=__doc__.split("\n")[0])
    ap.add_argument("--model", required=True, help="folder with config.json and safetensors shards")
    ap.add_argument("--dtype", choices=("bfloat16", "float32"), default="bfloat16")
    ap.add_argument("--out", required=True, help="folder for the logits")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens that live requests hold at any time")
    ap.add_argument("--cpu", action="store_true", help="fp32 reference ops on the CPU (plumbing / debugging)")
    args = ap.parse_args(argv)
    if not args.cpu and not torch.cuda.is_available():
        print("trace_run needs a GPU (--cpu runs the reference ops)", file=sys.stderr)
        return 2
    device = torch.device("cpu") if args.cpu else torch.device("cuda", 0)
    os.makedirs(args.out, exist_ok=True)
    runner = TraceRunner(build_engine(args.model, "float32" if args.cpu else args.dtype, args.max_tokens, device))
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        with torch.inference_mode():
            logits = runner.run_step(step)
        if logits is not None:
            logits.to(torch.float32).cpu().contiguous().numpy().astype("<f4").tofile(os.path.join(args.out, f"{step['step']}.f32"))
        print(f"done {step['step']}", flush=True)
    return 0


if __name__ == "__main__":
    raise SystemExit(main())
