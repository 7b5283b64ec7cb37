"""Vasosun adapter: gated delta-rule layers, window attention with a logarithmic distance bias and latent attention (query latents, a
rotated key part, caches shared between layers) in any order, SwiGLU feed-forwards or mixtures with identity experts, a convolution in
front of every sublayer, scalar norms on both sides of it, an embedding of token pairs, fp32 residual stream.

    model = RPUModelForCausalLM.from_pretrained(folder, dtype=torch.bfloat16, device="rpu")
    ids = model.generate(prompt, max_new_tokens=32)

Checkpoints (``"architecture": "Vasosun"``) and dtypes: :mod:`rhinoforge_b200.adapters.mixed_base`.
"""
from __future__ import annotations

from ...models.mixed import MixedConfig
from ..mixed_base import MixedAdapter


class VasosunAdapter(MixedAdapter):
    ARCH = "Vasosun"
    FAMILY = "Vasosun"
    read_config = staticmethod(MixedConfig.from_vasosun)


__all__ = ["VasosunAdapter"]
