"""Replay a trace: feed given token ids through a checkpoint step by step and write logits.  Nothing is sampled.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N < steps.jsonl

One JSON object per line on standard input:

    {"step": 7, "entries": [{"id": "q1", "tokens": [12, 40], "want": [1]}, {"id": "q2", "tokens": [9], "want": []}], "end": ["q2"]}

An entry appends its tokens to its request (a new name takes a slot) and lists the rows whose logits are to be written; a
request in ``end`` gives its slot and pages back once the step has run.  The entries of a step form one batch of the
runtime that the loader builds for serving.  Logits go to OUT/<step>.f32 as little-endian fp32 rows of vocabulary length,
entry by entry; each step is acknowledged with ``done <step>``, whether or not it wrote a file.

The page pool has room for N tokens, shared by up to ``--slots`` requests.  Exit codes: 0 when the input ends, 2 for a model
that cannot be replayed, 3 when its family does not serve the asked dtype.
"""
from __future__ import annotations

import argparse
import json
import os
import sys
from typing import Iterable, TextIO

PAGE = 64


class TraceSession:
    """Request names -> slots of a runtime; one call per step of the trace."""

    def __init__(self, runtime):
        self.rt = runtime
        self.slots: dict[str, int] = {}

    def step(self, record: dict):
        """Runs the record's entries as one batch; returns the wanted logits (fp32 [wanted, vocab] or None)."""
        batch = []
        for e in record.get("entries", []):
            name = e["id"]
            if name not in self.slots:
                self.slots[name] = self.rt.allocate()
            batch.append((self.slots[name], [int(t) for t in e["tokens"]], [int(w) for w in e.get("want", [])]))
        logits = self.rt.step(batch) if batch else None
        for name in record.get("end", []):
            self.rt.free(self.slots.pop(name))
        return logits


def replay(runtime, lines: Iterable[str], out_dir: str, done: TextIO, check=lambda: None) -> None:
    session = TraceSession(runtime)
    for line in lines:
        if not line.strip():
            continue
        record = json.loads(line)
        logits = session.step(record)
        if logits is not None:
            data = logits.float().cpu().contiguous().numpy().astype("<f4", copy=False).tobytes()
            path = os.path.join(out_dir, f"{int(record['step'])}.f32")
            with open(path + ".part", "wb") as f:
                f.write(data)
            os.replace(path + ".part", path)
        check()
        print(f"done {record['step']}", file=done, flush=True)


def main(argv: list[str] | None = None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="replay a trace of token ids and write the wanted logits")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", choices=("bfloat16", "float32"), default="bfloat16")
    ap.add_argument("--out", required=True)
    ap.add_argument("--max-tokens", type=int, required=True, help="size of the page pool in tokens")
    ap.add_argument("--slots", type=int, default=4, help="requests that may be open together")
    a = ap.parse_args(argv)
    import torch
    from ..ops import _lib
    from ..runtime import loader
    raw, spec = loader.checkpoint_family(a.model)
    if spec is None:
        print(f"{a.model}: no registered model family claims this configuration", file=sys.stderr)
        return 2
    if a.dtype not in spec.dtypes:
        print(f"the {spec.name} family does not run in {a.dtype}", file=sys.stderr)
        return 3
    pages = (a.max_tokens + PAGE - 1) // PAGE
    device = torch.device("cuda", 0)
    torch.cuda.set_device(device)
    _, rt = loader.build_family(spec, raw, a.model, device, dtype=a.dtype, max_slots=a.slots, max_context=pages * PAGE,
                                num_blocks=pages + 1)            # page 0 is never handed out
    if not hasattr(rt, "step"):
        print(f"the {spec.name} runtime has no batched step", file=sys.stderr)
        return 2
    replay(rt, sys.stdin, a.out, sys.stdout, _lib.check_status)
    return 0


if __name__ == "__main__":
    sys.exit(main())
