"""Replay a trace: feed given token ids through a model step by step and write the logits (``bin/trace_run``).

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR [--max-tokens N]

Reads one JSON object per line from standard input,

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

and runs all entries of a line as one batch: either the first tokens of new requests, or one more token for requests
that started together. ``want`` lists the places among the line's tokens whose logits go to ``OUT/<step>.f32`` (little
endian float32, ``[wanted, vocab]``, in the order of the entries); ``end`` names the requests that are finished after the
line. ``done <step>`` on standard output answers every line. Nothing is sampled.

The model class follows from ``config.json``; the steps are ``generation.BatchSteps``, i.e. the padding, cache, state and
kernels of ``generate()``. In a checkout without built kernels the first call builds them.
"""
from __future__ import annotations

import argparse
import json
import os
import sys
from typing import Dict, List, TextIO


def _kernels() -> None:
    """Build the kernel extension when it is missing or older than its sources (one process at a time)."""
    import fcntl

    from . import build
    with open(os.path.join(build.HERE, ".build.lock"), "w") as lock:
        fcntl.flock(lock, fcntl.LOCK_EX)
        build.build_kernels(verbose=False)


class TraceRunner:
    def __init__(self, model, out_dir: str) -> None:
        self.model, self.out_dir = model, out_dir
        self.where: Dict[str, "Batch"] = {}

    def step(self, line: Dict) -> None:
        import torch
        entries = line.get("entries", [])
        rows: List = []
        if entries:
            known = [e["id"] in self.where for e in entries]
            if any(known) and not all(known):
                raise ValueError(f"step {line['step']}: no request joins a batch that has started")
            want = [e.get("want", []) for e in entries]
            if all(known):
                rows = self._advance(line["step"], entries, want)
            else:
                batch = Batch(self.model, [e["id"] for e in entries])
                for e in entries:
                    self.where[e["id"]] = batch
                last_only = all(i == len(e["tokens"]) - 1 for e, w in zip(entries, want) for i in w)
                logits = batch.steps.start([e["tokens"] for e in entries], last_only=last_only)
                for r, w in enumerate(want):
                    rows += [logits[r, -1 if last_only else batch.steps.pad[r] + i] for i in w]
        if rows:
            path = os.path.join(self.out_dir, f"{line['step']}.f32")
            torch.stack(rows).to(torch.float32).cpu().numpy().astype("<f4").tofile(path)
        for name in line.get("end", []):
            batch = self.where.pop(name, None)
            if batch is not None:
                batch.drop([name])

    def _advance(self, step, entries, want) -> List:
        batch = self.where[entries[0]["id"]]
        given = {e["id"]: e for e in entries}
        if any(self.where[n] is not batch for n in given) or any(len(e["tokens"]) != 1 for e in entries):
            raise ValueError(f"step {step}: a step continues one batch by one token per request")
        batch.drop([n for n in batch.names if n not in given])       # whoever is not continued has ended
        logits = batch.steps.advance([given[n]["tokens"][0] for n in batch.names])
        row_of = {n: r for r, n in enumerate(batch.names)}
        return [logits[row_of[e["id"]], 0] for e, w in zip(entries, want) for _ in w]


class Batch:
    def __init__(self, model, names: List[str]) -> None:
        from .generation import BatchSteps
        self.names, self.steps = list(names), BatchSteps(model)

    def drop(self, names: List[str]) -> None:
        rows = [r for r, n in enumerate(self.names) if n not in names]
        self.names = [self.names[r] for r in rows]
        if rows:
            self.steps.keep(rows)
        else:
            self.steps = None


def replay(model, out_dir: str, lines: TextIO, answers: TextIO) -> None:
    runner = TraceRunner(model, out_dir)
    for text in lines:
        if not text.strip():
            continue
        line = json.loads(text)
        runner.step(line)
        print(f"done {line['step']}", file=answers, flush=True)


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="Feed given token ids through a model and write logits.")
    ap.add_argument("--model", required=True, help="directory with config.json and the weights")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="directory for <step>.f32")
    ap.add_argument("--max-tokens", type=int, default=None,
                    help="most tokens that live requests hold at a time (the cache grows as needed; accepted as a hint)")
    ap.add_argument("--device", default="cuda", choices=["cuda", "cpu"], help="cpu: the PyTorch statements of the ops (for tests)")
    args = ap.parse_args(argv)
    import torch
    if args.device == "cuda":
        if not torch.cuda.is_available():
            raise SystemExit("trace_run: no CUDA device")
        _kernels()
    from .models import load_causal_lm
    torch.backends.cuda.matmul.allow_tf32 = False
    model = load_causal_lm(args.model, torch_dtype=getattr(torch, args.dtype))
    if args.device == "cuda":
        model = model.cuda().fuse()
    replay(model.eval(), args.out, sys.stdin, sys.stdout)
    return 0


if __name__ == "__main__":
    sys.exit(main())
