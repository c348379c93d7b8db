"""Replays a trace of steps through the engine and writes logits (``bin/trace_run``).

Steps come as JSON lines on standard input,
``{"step": n, "entries": [{"id", "tokens", "want"}], "end": [ids]}``: every entry appends its tokens to its
sequence and asks for the logits at some of them; ``end`` names the sequences to give back.  Wanted logits of
step n go to ``OUT/n.f32`` ([wanted, vocab] little-endian fp32), then ``done n`` is printed.
"""
from __future__ import annotations

import argparse
import json
import os
import sys

from . import build
from .models import DTYPES, LayeredConfig, read_config


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="replay a trace of steps and write logits")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", choices=sorted(DTYPES), default="bfloat16")
    ap.add_argument("--out", required=True, help="folder for the logits")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens live sequences hold at any time")
    ap.add_argument("--max-batch", type=int, default=1, help="most live sequences")
    ap.add_argument("--device", type=int, default=0)
    a = ap.parse_args(argv)
    cfg = read_config(a.model)
    if not isinstance(cfg, LayeredConfig):
        if a.dtype == "float32":
            return 3
        raise SystemExit("trace_run needs a model with sequence slots (described layer by layer)")
    build.build()
    from .backend import CudaBackend
    from .models import load_model

    with CudaBackend(device=a.device) as be:
        eng = load_model(be, a.model, dtype=a.dtype, max_seq=a.max_tokens, max_batch=a.max_batch)
        live = {}
        for line in sys.stdin:
            if not line.strip():
                continue
            step = json.loads(line)
            entries = []
            for e in step["entries"]:
                if e["id"] not in live:
                    live[e["id"]] = eng.open_sequence()
                entries.append((live[e["id"]], e["tokens"], e["want"]))
            logits = eng.extend(entries)
            if len(logits):
                logits.astype("<f4").tofile(os.path.join(a.out, f"{step['step']}.f32"))
            for i in step["end"]:
                eng.close_sequence(live.pop(i))
            print(f"done {step['step']}", flush=True)
        eng.close()
    return 0


if __name__ == "__main__":
    sys.exit(main())
