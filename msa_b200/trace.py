"""Replays a trace of token portions through a model and writes the logits that are asked for.

Steps come as JSON lines on standard input,

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

``entries``: the next tokens of each request and the places among them whose logits are wanted; ``end``: the requests
that are finished after the step.  Wanted logits go to ``<out>/<step>.f32`` (little-endian fp32, ``[wanted, vocab]``, in
the order of the entries), and every step is answered by a line ``done <step>``.  The model runs as in serving: its
packed step, its state cache, its kernels; nothing is sampled."""
from __future__ import annotations

import argparse
import json
import os
import sys

import torch

UNSUPPORTED_DTYPE = 3      # exit code


def replay(model, cache, lines, out_dir: str, reply) -> None:
    for line in lines:
        line = line.strip()
        if not line:
            continue
        msg = json.loads(line)
        entries = []
        for e in msg.get("entries", []):
            if e["id"] not in cache:
                cache.acquire(e["id"])
            entries.append((e["id"], e["tokens"], e.get("want", [])))
        if entries:
            logits = model.run(entries, cache)
            if logits.shape[0]:
                data = logits.to(torch.float32).cpu().numpy().astype("<f4")
                model.check_status()
                path = os.path.join(out_dir, f"{msg['step']}.f32")
                with open(path + ".part", "wb") as f:
                    f.write(data.tobytes())
                os.replace(path + ".part", path)
        for name in msg.get("end", []):
            if name in cache:
                cache.release(name)
        reply(f"done {msg['step']}")


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="feed token portions through a model, write logits")
    ap.add_argument("--model", required=True)
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True)
    ap.add_argument("--max-tokens", type=int, default=8192, help="most tokens that live requests hold at any time")
    ap.add_argument("--max-requests", type=int, default=8, help="most requests that are live at any time")
    args = ap.parse_args(argv)
    from .registry import design_of
    dtype = getattr(torch, args.dtype)
    design = design_of(args.model)
    if design.serves != "states":
        print(f"{design.name} is served over a document bank, not from traces", file=sys.stderr)
        return 2
    if dtype not in design.dtypes:
        return UNSUPPORTED_DTYPE
    from .build import build
    build(only="lm")
    torch.backends.cuda.matmul.allow_tf32 = False
    torch.backends.cudnn.allow_tf32 = False
    torch.set_float32_matmul_precision("highest")
    model = design.load(args.model, "cuda:0", dtype)
    cache = model.new_cache(args.max_requests, max(args.max_tokens, 1))

    def reply(text):
        print(text, flush=True)
    replay(model, cache, sys.stdin, args.out, reply)
    return 0


if __name__ == "__main__":
    sys.exit(main())
