"""Command line: `python kronos_2t_b200.py build | models | generate` (see `generate --help`)."""
import argparse


def main(argv=None):
    ap = argparse.ArgumentParser(prog="kronos_2t_b200")
    sub = ap.add_subparsers(dest="cmd", required=True)
    b = sub.add_parser("build", help="compile the library")
    b.add_argument("--force", action="store_true")
    sub.add_parser("models", help="list the registered architectures")
    g = sub.add_parser("generate", help="greedy continuation of a prompt of token ids")
    g.add_argument("--model", required=True, help="folder with config.json and the weights")
    g.add_argument("--tokens", required=True, help="prompt: comma-separated token ids")
    g.add_argument("--steps", type=int, default=32)
    g.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    g.add_argument("--device", type=int, default=0)
    args = ap.parse_args(argv)
    from . import ffi, models
    from .build import build
    if args.cmd == "models":
        print("\n".join(sorted(models.READERS)))
        return
    path = build(force=getattr(args, "force", False))
    if args.cmd == "build":
        print(path)
        return
    prompt = [int(t) for t in args.tokens.split(",")]
    ctx = ffi.Context(args.device)
    engine = models.load_engine(ctx, args.model, args.dtype, max_seq=len(prompt) + args.steps)
    print(",".join(str(int(t)) for t in models.generate(engine, prompt, args.steps)))
    engine.close()
    ctx.close()
