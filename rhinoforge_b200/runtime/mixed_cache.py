"""Per-sequence state of decoders with per-layer mixers: paged latent rows of the attention layers, fp32 recurrent states of
the linear-attention layers and the token-shift rows of every layer.

Latent rows live in 16-token pages addressed through the page table of :class:`PagedSequences`; a layer's pool is
``[pages, 16, rank]`` and all layers share the page numbers.  Recurrent and shift state belong to the sequence SLOT: nothing
has to be cleared when a slot is given to another request, because a row at position 0 starts from an empty state in every
kernel.
"""
from __future__ import annotations

from typing import List, Optional

import torch

from ..models.mixed import HGRN2, LatentAttention, MixedConfig
from .kv_cache import PAGE_TOKENS, PagedSequences


def pad_to(n: int, m: int) -> int:
    return (n + m - 1) // m * m


class MixedCache(PagedSequences):
    def __init__(self, cfg: MixedConfig, batch_size: int, max_seq_len: int, *, device="cuda", dtype=torch.bfloat16,
                 pool_tokens: Optional[int] = None):
        for name, v in (("batch_size", batch_size), ("max_seq_len", max_seq_len)):
            if isinstance(v, bool) or not isinstance(v, int) or v <= 0:
                raise ValueError(f"cache {name} must be a positive integer, got {v!r}")
        self.cfg, self.dtype, self.num_layers = cfg, dtype, cfg.num_layers
        self._init_pages(batch_size, max_seq_len, device, pool_tokens)
        self.latent: List[Optional[torch.Tensor]] = []
        self.recurrent: List[Optional[torch.Tensor]] = []
        for layer in cfg.layers:
            m = layer.mixer
            self.latent.append(torch.zeros((self.num_pages, PAGE_TOKENS, pad_to(m.kv_rank, 16)), dtype=dtype, device=self.device)
                               if isinstance(m, LatentAttention) else None)
            self.recurrent.append(torch.zeros((batch_size, m.heads, pad_to(m.dim, 8), pad_to(m.vdim, 8)), dtype=torch.float32,
                                              device=self.device) if isinstance(m, HGRN2) else None)
        self.shift = torch.zeros((cfg.num_layers, batch_size, pad_to(cfg.hidden_size, 8)), dtype=torch.float32, device=self.device)

    def layer_ptrs(self, layer: int):
        """Device addresses ``(latent pool, recurrent state, shift rows)`` of one layer; None where it has none."""
        ptr = lambda t: None if t is None else t.data_ptr()
        return ptr(self.latent[layer]), ptr(self.recurrent[layer]), self.shift[layer].data_ptr()

    def state_tensors(self) -> List[torch.Tensor]:
        """Everything a step advances in place (latent pages are only ever written at new positions)."""
        return [t for t in self.recurrent if t is not None] + [self.shift]

    def zero_(self) -> None:
        for t in self.latent + self.recurrent + [self.shift]:
            if t is not None:
                t.zero_()

    def nbytes(self) -> int:
        return sum(t.numel() * t.element_size() for t in self.latent + self.recurrent + [self.shift] if t is not None)


__all__ = ["MixedCache", "pad_to"]
