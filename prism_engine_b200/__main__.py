"""Command line: ``python -m prism_engine_b200 {info,generate,trace} ...``."""
from __future__ import annotations

import argparse
import json
import sys


def _ids(text: str):
    return [int(t) for t in text.replace(",", " ").split()]


def cmd_info(a) -> int:
    from .models import LayeredConfig, read_config

    cfg = read_config(a.model)
    if isinstance(cfg, LayeredConfig):
        n = sum(int(s[0]) * (int(s[1]) if len(s) == 2 else 1) for s in cfg.tensor_shapes().values())
        print(json.dumps({"kind": "layered", "layers": len(cfg.layers), "width": cfg.width, "vocab": cfg.vocab, "parameters": n}))
    else:
        print(json.dumps({"kind": "palettized", "layers": cfg.num_layers, "width": cfg.hidden_size, "vocab": cfg.vocab_size}))
    return 0


def cmd_generate(a) -> int:
    from . import build
    from .backend import CudaBackend
    from .models import load_model

    build.build()
    prompts = [_ids(p) for p in a.prompt]
    if len({len(p) for p in prompts}) != 1:
        raise SystemExit("prompts of one call must have the same number of tokens")
    with CudaBackend(device=a.device) as be:
        eng = load_model(be, a.model, dtype=a.dtype, max_seq=len(prompts[0]) + a.max_new, max_batch=len(prompts))
        for row in eng.generate(prompts, a.max_new):
            print(" ".join(str(int(t)) for t in row))
        eng.close()
    return 0


def main(argv=None) -> int:
    argv = sys.argv[1:] if argv is None else list(argv)
    if argv and argv[0] == "trace":
        from .trace import main as trace_main

        return trace_main(argv[1:])
    ap = argparse.ArgumentParser(prog="prism_engine_b200")
    sub = ap.add_subparsers(dest="cmd", required=True)
    p = sub.add_parser("info", help="what a model folder holds")
    p.add_argument("--model", required=True)
    p.set_defaults(fn=cmd_info)
    p = sub.add_parser("generate", help="greedy generation from token ids")
    p.add_argument("--model", required=True)
    p.add_argument("--prompt", required=True, action="append", metavar="IDS", help="token ids, separated by commas (repeat for a batch)")
    p.add_argument("--max-new", type=int, default=16)
    p.add_argument("--dtype", choices=["bfloat16", "float32"], default="bfloat16")
    p.add_argument("--device", type=int, default=0)
    p.set_defaults(fn=cmd_generate)
    sub.add_parser("trace", help="replay a trace of steps (see bin/trace_run --help)")
    a = ap.parse_args(argv)
    return a.fn(a)


if __name__ == "__main__":
    sys.exit(main())
