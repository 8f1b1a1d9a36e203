"""Command line:  python -m sharpmind_b200 generate --model PATH --tokens 1,2,3 [--tokens ...] --max-new 16
                  python -m sharpmind_b200 info --model PATH
                  python -m sharpmind_b200 trace --model DIR --dtype bfloat16 --out DIR --max-tokens N  (see trace.py)

PATH is a GGUF file or a folder with config.json and model.safetensors.  Token ids in, token ids out (no tokenizer)."""
from __future__ import annotations

import argparse
import sys


def main(argv=None) -> int:
    argv = list(sys.argv[1:] if argv is None else argv)
    if argv[:1] == ["trace"]:
        from . import trace

        return trace.main(argv[1:])
    ap = argparse.ArgumentParser(prog="sharpmind_b200")
    sub = ap.add_subparsers(dest="cmd", required=True)
    g = sub.add_parser("generate", help="continue prompts of token ids")
    g.add_argument("--model", required=True)
    g.add_argument("--tokens", action="append", required=True, help="one prompt: ids with commas between them; repeat for a batch")
    g.add_argument("--max-new", type=int, default=16)
    g.add_argument("--max-seq", type=int, default=0, help="positions to hold per sequence (0: what the prompts need)")
    g.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    g.add_argument("--device", type=int, default=0)
    g.add_argument("--temperature", type=float, default=0.0)
    g.add_argument("--top-k", type=int, default=0)
    g.add_argument("--top-p", type=float, default=1.0)
    g.add_argument("--min-p", type=float, default=0.0)
    g.add_argument("--repetition-penalty", type=float, default=1.0)
    g.add_argument("--seed", type=int, default=0)
    i = sub.add_parser("info", help="what a model file or folder holds")
    i.add_argument("--model", required=True)
    sub.add_parser("trace", help="replay a trace of requests")
    a = ap.parse_args(argv)

    from . import ops, registry
    from .session import Sampling, generate

    if a.cmd == "info":
        print(registry.describe(a.model))
        return 0
    prompts = [[int(x) for x in p.replace(" ", ",").split(",") if x] for p in a.tokens]
    ctx = ops.CudaContext(a.device)
    model = registry.load_model(ctx, a.model, max_seq=a.max_seq or max(map(len, prompts)) + a.max_new, max_batch=len(prompts), act=a.dtype)
    out = generate(model, prompts, a.max_new, Sampling(a.temperature, a.top_k, a.top_p, a.min_p, a.repetition_penalty, seed=a.seed))
    for row in out:
        print(",".join(map(str, row)))
    model.close()
    ctx.close()
    return 0


if __name__ == "__main__":
    sys.exit(main())
