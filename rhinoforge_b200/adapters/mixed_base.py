"""Shared adapter logic of the decoders with per-layer mixers (:mod:`rhinoforge_b200.models.mixed`).

A checkpoint is a folder with ``config.json`` (the design named under ``"architecture"``, not a Hugging Face config) and
``model.safetensors``.  Every size, layer order and constant comes from the config; activations are float16, bfloat16 or float32.
"""
from __future__ import annotations

from typing import Callable, Mapping, Optional

import torch

from ..api._execution import prefill_chunk_rows
from ..api.errors import RPUUnsupportedDtypeError, WeightShapeMismatchError
from ..models.mixed import MixedConfig, weight_shapes
from .causal_base import CausalLMAdapter


class MixedAdapter(CausalLMAdapter):
    SUPPORTED_DTYPES = (torch.float16, torch.bfloat16, torch.float32)

    @staticmethod
    def read_config(raw: Mapping) -> MixedConfig:
        """The design's reader of its ``config.json`` mapping."""
        raise NotImplementedError

    @classmethod
    def config_from_dict(cls, raw: dict):
        """The configuration object of a ``config.json`` mapping: the fields Hugging Face's generation loop looks at, and the parsed
        :class:`MixedConfig` behind it."""
        from transformers import PretrainedConfig
        mixed = cls.read_config(raw)
        cfg = PretrainedConfig(architectures=[cls.ARCH], vocab_size=mixed.vocab_size, hidden_size=mixed.hidden_size,
                               num_hidden_layers=mixed.num_layers, tie_word_embeddings=mixed.tied_head)
        object.__setattr__(cfg, "model_type", mixed.model_type)
        object.__setattr__(cfg, "_mixed", mixed)
        return cfg

    @classmethod
    def mixed_config(cls, config) -> MixedConfig:
        m = getattr(config, "_mixed", None)
        return m if m is not None else cls.read_config(config if isinstance(config, dict) else config.to_dict())

    @classmethod
    def check_profile(cls, config) -> None:
        """Any sizes: the kernels are not tied to released profiles."""
        cls.mixed_config(config)

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
        return self.mixed_config(self.config)

    def _check_dtype(self) -> None:
        if self._dtype not in self.SUPPORTED_DTYPES:
            raise RPUUnsupportedDtypeError(f"{self.FAMILY} runs in float16, bfloat16 or float32, got {self._dtype}")

    def _build_engine(self, cfg: MixedConfig, get, *, max_batch: int, tp=None, quant: Optional[str] = None):
        from ..runtime.mixed_engine import MixedDecoderEngine
        return MixedDecoderEngine(cfg, get, dtype=self._dtype, max_batch=max_batch, max_seq_len=16,
                                  max_prefill_tokens=prefill_chunk_rows(self._rpu_execution), tp=tp)


__all__ = ["MixedAdapter"]
