"""Replays a trace of batch steps through the engine and writes logits (``bin/trace_run``).

Steps come as JSON lines on standard input: ``{"step": n, "entries": [{"id", "tokens", "want"}], "end": [ids]}``. The wanted
logits of step n go to ``<out>/n.f32`` (little-endian f32, entry order), then ``done n`` is printed; the sequences under
"end" give back what they hold.
"""
from __future__ import annotations

import argparse
import itertools
import json
import os
import sys


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="Replay a trace of batch steps and write logits.")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", choices=("bfloat16", "float32"), default="bfloat16")
    ap.add_argument("--out", required=True, help="folder for the <step>.f32 files")
    ap.add_argument("--max-tokens", type=int, required=True, help="tokens live sequences hold at most, in whole pages")
    ap.add_argument("--max-seqs", type=int, default=4, help="sequences live at any time")
    a = ap.parse_args(argv)

    from . import build
    build.ensure_built(oracle=False)
    from . import models
    from .backend import CudaBackend
    from .engine import Engine

    module = models.load_module(a.model, a.dtype)
    engine = Engine(CudaBackend((0,)).prepare(module), a.max_tokens, a.max_seqs)
    names, fresh = {}, itertools.count()
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        for e in step["entries"]:
            if e["id"] not in names:
                names[e["id"]] = next(fresh)
        entries = [(names[e["id"]], e["tokens"], e["want"]) for e in step["entries"]]
        if entries:
            logits = engine.forward(entries)
            if len(logits):
                with open(os.path.join(a.out, f"{step['step']}.f32"), "wb") as f:
                    f.write(logits.astype("<f4").tobytes())
        for name in step.get("end", []):
            engine.release(names.pop(name))
        print(f"done {step['step']}", flush=True)
    return 0


if __name__ == "__main__":
    sys.exit(main())
