"""Kuzupel adapter: distance-biased window attention and rotary window attention (convolved projections, kept first tokens, gates per
head) in any order, clipped gated feed-forwards or mixtures of them, an embedding of token pairs, fp32 residual stream.

    model = RPUModelForCausalLM.from_pretrained(folder, dtype=torch.bfloat16, device="rpu")
    ids = model.generate(prompt, max_new_tokens=32)

Checkpoints (``"architecture": "Kuzupel"``) and dtypes: :mod:`rhinoforge_b200.adapters.mixed_base`.
"""
from __future__ import annotations

from ...models.mixed import MixedConfig
from ..mixed_base import MixedAdapter


class KuzupelAdapter(MixedAdapter):
    ARCH = "Kuzupel"
    FAMILY = "Kuzupel"
    read_config = staticmethod(MixedConfig.from_kuzupel)


__all__ = ["KuzupelAdapter"]
