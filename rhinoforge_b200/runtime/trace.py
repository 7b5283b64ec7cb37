"""Replay of a request trace: token ids go through a served model step by step and logits come out.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N

Steps are read from standard input, one JSON object per line::

    {"step": 4, "entries": [{"id": "r1", "tokens": [11, 48], "want": [1]}, {"id": "r2", "tokens": [7], "want": []}], "end": ["r1"]}

All entries of a step run as one batch through the request scheduler and the engine's step; nothing is sampled.  The logits at
the wanted places go to ``OUT/<step>.f32`` (little-endian fp32, ``[wanted, vocab]``, in the order of the entries), then
``done <step>`` is printed.  Requests named in ``end`` return their slot and pages after the step.
"""
from __future__ import annotations

import argparse
import json
import sys
from pathlib import Path
from typing import Optional, Sequence

MAX_LIVE = 4


def parse_args(argv: Optional[Sequence[str]] = None) -> argparse.Namespace:
    ap = argparse.ArgumentParser(prog="trace_run", description="replay a request trace through a served model")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"], help="activation dtype of the engine")
    ap.add_argument("--out", required=True, help="folder the logits files are written to")
    ap.add_argument("--max-tokens", type=int, required=True, help="cached tokens that live requests hold together at most")
    return ap.parse_args(argv)


def main(argv: Optional[Sequence[str]] = None) -> int:
    args = parse_args(argv)
    import torch
    from ..api.causal_lm import RPUModelForCausalLM
    from ..api.errors import RPUUnsupportedDtypeError
    from .kv_cache import PAGE_TOKENS
    from .scheduler import RequestScheduler
    torch.backends.cuda.matmul.allow_tf32 = False
    pool = (args.max_tokens + PAGE_TOKENS - 1) // PAGE_TOKENS * PAGE_TOKENS
    try:
        model = RPUModelForCausalLM.from_pretrained(args.model, dtype=getattr(torch, args.dtype), device="rpu", max_batch=MAX_LIVE)
    except RPUUnsupportedDtypeError as e:
        print(f"trace_run: {e}", file=sys.stderr)
        return 3
    model.bind_cache(batch_size=MAX_LIVE, max_seq_len=pool, pool_tokens=pool)
    sched = RequestScheduler(model.engine)
    out = Path(args.out)
    for line in sys.stdin:
        if not line.strip():
            continue
        msg = json.loads(line)
        entries = [(e["id"], torch.tensor(e["tokens"], dtype=torch.int32), list(e.get("want", ()))) for e in msg["entries"]]
        if entries:
            _, logits = sched.step(entries)
            rows = torch.cat([lg.float() for lg in logits]) if any(w for _, _, w in entries) else None
            model.engine.check_status()
            if rows is not None:
                rows.cpu().numpy().astype("<f4").tofile(out / f"{msg['step']}.f32")
        for r in msg.get("end", ()):
            sched.finish(r)
        print(f"done {msg['step']}", flush=True)
    model.close()
    return 0


__all__ = ["main", "parse_args"]
