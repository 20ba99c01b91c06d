"""Command line: `python -m densecore_b200 generate` runs greedy generation of token ids through the scheduler."""
from __future__ import annotations

import argparse
import sys


def parser() -> argparse.ArgumentParser:
    ap = argparse.ArgumentParser(prog="python -m densecore_b200")
    sub = ap.add_subparsers(dest="command", required=True)
    g = sub.add_parser("generate", help="greedy generation; prints one line of new token ids per prompt")
    g.add_argument("--model", required=True, help="folder with config.json and model.safetensors, or a .gguf file")
    g.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"], help="arithmetic of a layer-list decoder")
    g.add_argument("--tokens", default=None, help="one prompt's token ids, comma or space separated (default: one prompt a line from stdin)")
    g.add_argument("--max-new", type=int, default=32)
    g.add_argument("--max-ctx", type=int, default=4096)
    g.add_argument("--eos", type=int, default=-1)
    g.add_argument("--device", type=int, default=0)
    return ap


def prompts(args) -> list[list[int]]:
    lines = [args.tokens] if args.tokens else sys.stdin.read().splitlines()
    return [[int(t) for t in ln.replace(",", " ").split()] for ln in lines if ln.strip()]


def main(argv=None) -> int:
    args = parser().parse_args(argv)
    todo = prompts(args)
    from . import Context, Model, Scheduler
    ctx = Context(args.device)
    if args.model.endswith(".gguf"):
        model = Model.from_gguf(ctx, args.model, 4, args.max_ctx)
    else:
        model = Model.from_dir(ctx, args.model, args.dtype, 4, args.max_ctx)
    model.finalize()
    sched = Scheduler(model, eos_token=args.eos)
    ids = [sched.add(p, args.max_new) for p in todo]
    out = sched.run()
    for i in ids:
        print(" ".join(str(t) for t in out[i]))
    sched.close()
    model.close()
    ctx.close()
    return 0


if __name__ == "__main__":
    sys.exit(main())
