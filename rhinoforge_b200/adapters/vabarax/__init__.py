"""Vabarax adapter: latent-attention and HGRN2 layers in any order, fp32 residual stream, token shift, per-token side input.

    model = RPUModelForCausalLM.from_pretrained(folder, dtype=torch.bfloat16, device="rpu")
    ids = model.generate(prompt, max_new_tokens=32)

A checkpoint is a folder with ``config.json`` (``"architecture": "Vabarax"``, not a Hugging Face config) and
``model.safetensors``.  Every size, layer order and constant comes from the config; activations are float16, bfloat16 or
float32.
"""
from __future__ import annotations

from typing import Callable, Optional

import torch

from ...api._execution import prefill_chunk_rows
from ...api.errors import RPUUnsupportedDtypeError, WeightShapeMismatchError
from ...models.mixed import MixedConfig, weight_shapes
from ..causal_base import CausalLMAdapter


def config_from_dict(raw: dict):
    """The configuration object of a ``config.json`` mapping: the fields Hugging Face's generation loop looks at, and the parsed
    :class:`MixedConfig` as ``mixed``."""
    from transformers import PretrainedConfig
    mixed = MixedConfig.from_vabarax(raw)
    cfg = PretrainedConfig(architectures=["Vabarax"], vocab_size=mixed.vocab_size, hidden_size=mixed.hidden_size,
                           num_hidden_layers=mixed.num_layers, tie_word_embeddings=True)
    object.__setattr__(cfg, "model_type", "vabarax")
    object.__setattr__(cfg, "_mixed", mixed)
    return cfg


class VabaraxAdapter(CausalLMAdapter):
    ARCH = "Vabarax"
    FAMILY = "Vabarax"
    SUPPORTED_DTYPES = (torch.float16, torch.bfloat16, torch.float32)

    @classmethod
    def config_from_dict(cls, raw: dict):
        return config_from_dict(raw)

    @classmethod
    def check_profile(cls, config) -> None:
        """Any sizes: the kernels are not tied to released profiles."""
        mixed_config(config)

    @classmethod
    def preflight(cls, config) -> None:
        cls.check_profile(config)

    def _validate_shapes(self, cfg: MixedConfig, get: Callable[[str], torch.Tensor]) -> None:
        names = getattr(get, "names", None)
        if names is None:
            return
        missing = [n for n, _, _ in weight_shapes(cfg) if n not in names]
        if missing:
            raise WeightShapeMismatchError(f"checkpoint is missing {missing[:8]}")
        shape_of = getattr(get, "shape", None)
        for name, shape, _ in weight_shapes(cfg):
            got = tuple(shape_of(name)) if shape_of is not None else tuple(shape)
            if got != tuple(shape):
                raise WeightShapeMismatchError(f"{name!r} has shape {got}, the config says {tuple(shape)}")

    def decoder_config(self) -> MixedConfig:
        return mixed_config(self.config)

    def _check_dtype(self) -> None:
        if self._dtype not in self.SUPPORTED_DTYPES:
            raise RPUUnsupportedDtypeError(f"Vabarax runs in float16, bfloat16 or float32, got {self._dtype}")

    def _build_engine(self, cfg: MixedConfig, get, *, max_batch: int, tp=None, quant: Optional[str] = None):
        from ...runtime.mixed_engine import MixedDecoderEngine
        return MixedDecoderEngine(cfg, get, dtype=self._dtype, max_batch=max_batch, max_seq_len=16,
                                  max_prefill_tokens=prefill_chunk_rows(self._rpu_execution), tp=tp)


def mixed_config(config) -> MixedConfig:
    m = getattr(config, "_mixed", None)
    return m if m is not None else MixedConfig.from_vabarax(config if isinstance(config, dict) else config.to_dict())


__all__ = ["VabaraxAdapter", "config_from_dict", "mixed_config"]
