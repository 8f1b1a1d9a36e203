"""Replays a trace: given token ids go through a model step by step and the logits that are asked for are written out.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N  < steps

Every input line is one step, {"step": n, "entries": [{"id": ..., "tokens": [...], "want": [...]}], "end": [...]}: each
entry's tokens continue that request, `want` names places among them, `end` the requests that give their slot back.
DIR/<n>.f32 receives the wanted rows as little-endian fp32; "done <n>" follows on standard output.  The model, its state
slots and its passes are the ones generation uses (session.Session).
"""
from __future__ import annotations

import argparse
import json
import os
import sys

SLOTS = 8  # requests that may be open together


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run")
    ap.add_argument("--model", required=True)
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True)
    ap.add_argument("--max-tokens", type=int, required=True, help="upper bound on the tokens of all open requests together")
    ap.add_argument("--device", type=int, default=0)
    a = ap.parse_args(argv)

    from . import ops, registry
    from .session import Session

    ctx = ops.CudaContext(a.device)
    model = registry.load_model(ctx, a.model, max_seq=max(1, a.max_tokens), max_batch=SLOTS, act=a.dtype)
    session = Session(model)
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        parts = []
        for e in step["entries"]:
            if e["id"] not in session:
                session.open(e["id"])
            logits = session.feed(e["id"], e["tokens"], e.get("want", ()))
            if logits is not None:
                parts.append(logits)
        if parts:
            rows = model.torch.cat(parts).cpu().numpy().astype("<f4")
            path = os.path.join(a.out, f"{step['step']}.f32")
            with open(path + ".part", "wb") as f:
                f.write(rows.tobytes())
            os.replace(path + ".part", path)
        model.torch.cuda.synchronize()
        for name in step.get("end", ()):
            if name in session:
                session.close(name)
        print(f"done {step['step']}", flush=True)
    ctx.device_status()
    model.close()
    ctx.close()
    return 0
