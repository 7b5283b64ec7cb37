#!/usr/bin/env python3
"""Batched generation from token-id prompts with a Vabarax checkpoint."""
from __future__ import annotations

import sys
from pathlib import Path

sys.path.insert(0, str(Path(__file__).resolve().parent))
from _config import check_execution, load_toml, ok, parse_args, require_model, resolve_checkpoint

DTYPES = ("float16", "bfloat16", "float32")


def _ids(rows) -> bool:
    good = lambda x: isinstance(x, int) and not isinstance(x, bool) and x >= 0
    return isinstance(rows, list) and bool(rows) and all(isinstance(r, list) and r and all(good(x) for x in r) for r in rows)


def load_config(path) -> dict:
    config = load_toml(path)
    require_model(config)
    gen = config.get("generation")
    if not isinstance(gen, dict) or not _ids(gen.get("prompt_tokens")):
        raise ValueError("[generation].prompt_tokens must be a non-empty list of non-empty lists of token ids")
    for key, default in (("max_new_tokens", None), ("slots", 1), ("top_k", 1)):
        v = gen.get(key, default)
        if not isinstance(v, int) or isinstance(v, bool) or v < 1:
            raise ValueError(f"[generation].{key} must be a positive integer")
    if not isinstance(gen.get("do_sample", False), bool):
        raise ValueError("[generation].do_sample must be a boolean")
    if config["model"].get("dtype", "bfloat16") not in DTYPES:
        raise ValueError(f"[model].dtype must be one of {', '.join(DTYPES)}")
    check_execution(config, {"prefill"})
    return config


def main(default: str = "vabarax.toml", doc=__doc__) -> int:
    args = parse_args(default, doc)
    config = load_config(args.config)
    if args.check_config:
        return ok(args.config, require_model(config))
    sys.path.insert(0, str(Path(__file__).resolve().parents[1]))
    import torch
    from rpu_backend import RPUModelForCausalLM

    gen = config["generation"]
    prompts = [torch.tensor(p, dtype=torch.int64) for p in gen["prompt_tokens"]]
    slots = min(gen.get("slots", len(prompts)), len(prompts))
    model = RPUModelForCausalLM.from_pretrained(resolve_checkpoint(config), dtype=getattr(torch, config["model"].get("dtype", "bfloat16")),
                                                device="rpu", rpu_execution=config.get("rpu_execution"), max_batch=slots)
    if gen.get("do_sample", False):
        for p in prompts:
            out = model.generate(p[None], max_new_tokens=gen["max_new_tokens"], do_sample=True,
                                 temperature=float(gen.get("temperature", 1.0)), top_k=gen.get("top_k", 50))
            print(" ".join(map(str, out[0, len(p):].tolist())))
        return 0
    for new in model.generate_batch(prompts, gen["max_new_tokens"], slots=slots):
        print(" ".join(map(str, new)))
    return 0


if __name__ == "__main__":
    raise SystemExit(main())
