"""Command line: python -m meganeura_b200 generate --model DIR --prompt 1,2,3 [--max-new N]."""
import argparse
import sys


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="meganeura_b200")
    sub = ap.add_subparsers(dest="command", required=True)
    gen = sub.add_parser("generate", help="greedy continuation of token ids")
    gen.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    gen.add_argument("--prompt", required=True, help="token ids, separated by commas")
    gen.add_argument("--max-new", type=int, default=32)
    gen.add_argument("--dtype", choices=["bfloat16", "float32"], default="bfloat16")
    args = ap.parse_args(argv)
    from .engine import Engine
    from .registry import load_model
    prompt = [int(t) for t in args.prompt.split(",")]
    model = load_model(args.model, dtype=args.dtype, max_rows=min(1024, len(prompt)), max_tokens=len(prompt) + args.max_new)
    print(",".join(str(t) for t in Engine(model).generate(prompt, args.max_new)))
    return 0


if __name__ == "__main__":
    sys.exit(main())
