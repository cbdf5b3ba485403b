"""Command line: ``python -m hf2q_b200 generate`` (greedy continuation of token ids) and ``trace`` (replay of given
token ids, logits to files)."""
from __future__ import annotations

import argparse
import json
import sys
from pathlib import Path


def _model(args, max_seq: int, n_slots: int):
    from . import build
    build.build()
    import torch
    from . import ops, registry
    ctx = ops.GpuContext(0)
    return ctx, registry.load_model(ctx, args.model, dtype=getattr(torch, args.dtype), max_seq=max_seq, n_slots=n_slots)


def generate(args) -> int:
    from .engine import Engine
    prompts = [[int(t) for t in p.split(",")] for p in args.prompt]
    ctx, model = _model(args, args.max_seq, min(len(prompts), args.slots))
    for ids in Engine(model).generate(prompts, args.new):
        print(json.dumps(ids))
    ctx.check_status()
    return 0


def trace(args) -> int:
    """Reads one JSON object a line: {"step": n, "entries": [{"id", "tokens", "want"}], "end": [ids]}; writes the wanted
    logits of a step to OUT/<step>.f32 (little-endian f32) and answers "done <step>"."""
    from .engine import Engine, Entry
    ctx, model = _model(args, args.max_tokens, 4)
    engine, out = Engine(model), Path(args.out)
    for line in sys.stdin:
        if not line.strip():
            continue
        req = json.loads(line)
        logits = engine.step([Entry(e["id"], e["tokens"], e.get("want", [])) for e in req.get("entries", [])], req.get("end", []))
        ctx.check_status()
        if logits is not None:
            (out / f"{req['step']}.f32").write_bytes(logits.float().cpu().numpy().astype("<f4").tobytes())
        print(f"done {req['step']}", flush=True)
    return 0


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="hf2q_b200")
    sub = ap.add_subparsers(dest="cmd", required=True)
    g = sub.add_parser("generate", help="greedy continuation of prompts given as token ids")
    g.add_argument("--prompt", action="append", required=True, help="comma-separated token ids; may be given several times")
    g.add_argument("--new", type=int, default=16, help="tokens to generate per prompt")
    g.add_argument("--max-seq", type=int, default=32768)
    g.add_argument("--slots", type=int, default=4, help="sequences held at a time")
    g.set_defaults(run=generate)
    t = sub.add_parser("trace", help="replay token ids read from standard input, step by step")
    t.add_argument("--out", required=True, help="folder for <step>.f32")
    t.add_argument("--max-tokens", type=int, default=32768, help="most tokens live requests hold at any time")
    t.set_defaults(run=trace)
    for p in (g, t):
        p.add_argument("--model", required=True, help="folder with config.json and model.safetensors, or a .gguf file")
        p.add_argument("--dtype", choices=["bfloat16", "float32"], default="bfloat16")
    args = ap.parse_args(argv)
    return args.run(args)


if __name__ == "__main__":
    sys.exit(main())
