"""Vabarax adapter: latent-attention and HGRN2 layers in any order, fp32 residual stream, token shift, per-token side input.

    model = RPUModelForCausalLM.from_pretrained(folder, dtype=torch.bfloat16, device="rpu")
    ids = model.generate(prompt, max_new_tokens=32)

Checkpoints (``"architecture": "Vabarax"``) and dtypes: :mod:`rhinoforge_b200.adapters.mixed_base`.
"""
from __future__ import annotations

from ...models.mixed import MixedConfig
from ..mixed_base import MixedAdapter


class VabaraxAdapter(MixedAdapter):
    ARCH = "Vabarax"
    FAMILY = "Vabarax"
    read_config = staticmethod(MixedConfig.from_vabarax)


config_from_dict = VabaraxAdapter.config_from_dict
mixed_config = VabaraxAdapter.mixed_config

__all__ = ["VabaraxAdapter", "config_from_dict", "mixed_config"]
