"""Command line.

    python -m msa_b200 generate --model DIR --prompt TEXT [--prompt TEXT ...] [--tokens 5,17,3 ...]
                                [--max-new-tokens N] [--temperature T --top-p P --seed S] [--dtype float32] [--memory FILE] [--gpus N]
    python -m msa_b200 designs            # the model designs the package serves
    python -m msa_b200 trace ...          # bin/trace_run
"""
from __future__ import annotations

import argparse
import json
import sys


def _generate(args) -> int:
    from .engine import GenerateConfig, MSAEngine
    from .memory import MemoryConfig, ModelConfig
    from .registry import design_of
    prompts = list(args.prompt) + [[int(t) for t in row.replace(",", " ").split()] for row in args.tokens]
    if not prompts:
        print("nothing to generate: give --prompt or --tokens", file=sys.stderr)
        return 2
    if design_of(args.model).serves == "memory" and (not args.memory or args.tokens):
        print("this model answers text prompts over a document memory: give --memory FILE and --prompt", file=sys.stderr)
        return 2
    cfg = GenerateConfig(devices=list(range(args.gpus)), max_generate_tokens=args.max_new_tokens, temperature=args.temperature,
                         top_p=args.top_p, seed=args.seed, max_context=args.max_context)
    with MSAEngine(cfg, ModelConfig(model_path=args.model, dtype=args.dtype), MemoryConfig(memory_file_path=args.memory or "")) as engine:
        texts, _, _ = engine.generate(prompts)
    for prompt, text in zip(prompts, texts):
        print(json.dumps({"prompt": prompt, "text": text}, ensure_ascii=False))
    return 0


def main(argv=None) -> int:
    argv = list(sys.argv[1:] if argv is None else argv)
    if argv[:1] == ["trace"]:
        from .trace import main as trace_main
        return trace_main(argv[1:])
    ap = argparse.ArgumentParser(prog="msa_b200")
    sub = ap.add_subparsers(dest="command", required=True)
    g = sub.add_parser("generate", help="generate from a checkpoint")
    g.add_argument("--model", required=True)
    g.add_argument("--prompt", action="append", default=[])
    g.add_argument("--tokens", action="append", default=[], help="a prompt as token ids, separated by commas or blanks")
    g.add_argument("--max-new-tokens", type=int, default=32)
    g.add_argument("--max-context", type=int, default=8192)
    g.add_argument("--temperature", type=float, default=0.0)
    g.add_argument("--top-p", type=float, default=0.9)
    g.add_argument("--seed", type=int, default=None)
    g.add_argument("--memory", default="", help="document file (memory models)")
    g.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"], help="models on state slots")
    g.add_argument("--gpus", type=int, default=1)
    sub.add_parser("designs", help="list the model designs")
    sub.add_parser("trace", help="replay a trace (see bin/trace_run)")
    args = ap.parse_args(argv)
    if args.command == "designs":
        from .registry import designs
        for d in designs().values():
            print(f"{d.name}\tserved from {d.serves}\t{', '.join(str(t).split('.')[-1] for t in d.dtypes)}")
        return 0
    return _generate(args)


if __name__ == "__main__":
    sys.exit(main())
