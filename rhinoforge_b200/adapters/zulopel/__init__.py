"""Zulopel adapter: grouped attention (chunks, sinks, output gates, value mixing) and selective-scan layers in any order, a mixture
of experts behind each, norms and layer scales on the sublayers' outputs, fp32 residual stream.

    model = RPUModelForCausalLM.from_pretrained(folder, dtype=torch.bfloat16, device="rpu")
    ids = model.generate(prompt, max_new_tokens=32)

Checkpoints (``"architecture": "Zulopel"``) and dtypes: :mod:`rhinoforge_b200.adapters.mixed_base`.
"""
from __future__ import annotations

from ...models.mixed import MixedConfig
from ..mixed_base import MixedAdapter


class ZulopelAdapter(MixedAdapter):
    ARCH = "Zulopel"
    FAMILY = "Zulopel"
    read_config = staticmethod(MixedConfig.from_zulopel)


__all__ = ["ZulopelAdapter"]
