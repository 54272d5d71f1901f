"""Command line: python -m lumen_b200 generate --model DIR --ids "5 17 3" [--max-new 32] [--temperature 0]

Generates from token ids with the chat session (caches, scheduling of prefill and decode steps, device sampler) of any
registered model; with --text the prompt goes through DIR/tokenizer.json instead.  `trace` is bin/trace_run.
"""
from __future__ import annotations

import argparse
import sys


def generate(args) -> int:
    from .chat import ChatSession
    from .registry import load_model
    model = load_model(args.model, args.max_seq_len, {"bfloat16": "bf16", "float32": "f32"}[args.dtype])
    tok = None
    if args.text is not None:
        from .tokenizer import LlamaTokenizer
        tok = LlamaTokenizer.from_file(f"{args.model}/tokenizer.json")
        ids = tok.encode(args.text, True)
    else:
        ids = [int(t) for t in args.ids.replace(",", " ").split()]
    session = ChatSession(model, lambda p: p, lambda p: p, stop_ids=args.stop or (), temperature=args.temperature, top_p=args.top_p,
                          repetition_penalty=args.repetition_penalty, max_gen=args.max_new)
    out = session.turn(ids)
    print(tok.decode(out, True) if tok else " ".join(str(t) for t in out))
    return 0


def main(argv=None) -> int:
    argv = sys.argv[1:] if argv is None else argv
    if argv[:1] == ["trace"]:
        from .replay import main as trace
        return trace(argv[1:])
    ap = argparse.ArgumentParser(prog="python -m lumen_b200", description=__doc__.splitlines()[0])
    sub = ap.add_subparsers(dest="cmd", required=True)
    g = sub.add_parser("generate", help="generate token ids from a prompt")
    g.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    src = g.add_mutually_exclusive_group(required=True)
    src.add_argument("--ids", help="prompt as token ids")
    src.add_argument("--text", help="prompt as text")
    g.add_argument("--dtype", choices=["bfloat16", "float32"], default="bfloat16")
    g.add_argument("--max-new", type=int, default=32)
    g.add_argument("--max-seq-len", type=int, default=2048)
    g.add_argument("--temperature", type=float, default=0.0, help="0: the most likely token")
    g.add_argument("--top-p", type=float, default=1.0)
    g.add_argument("--repetition-penalty", type=float, default=1.0)
    g.add_argument("--stop", type=int, nargs="*", help="stop token ids")
    sub.add_parser("trace", help="replay a trace (see bin/trace_run)", add_help=False)
    args = ap.parse_args(argv)
    return generate(args)


if __name__ == "__main__":
    sys.exit(main())
