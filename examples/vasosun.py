#!/usr/bin/env python3
"""Batched generation from token-id prompts with a Vasosun checkpoint."""
from __future__ import annotations

import sys
from pathlib import Path

sys.path.insert(0, str(Path(__file__).resolve().parent))
from vabarax import load_config, main  # noqa: F401  (the same configuration keys)

if __name__ == "__main__":
    raise SystemExit(main("vasosun.toml", __doc__))
