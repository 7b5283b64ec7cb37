"""Per-sequence state of decoders with per-layer mixers: paged latent rows or keys and values of the attention layers, fp32
recurrent states, convolution inputs, and the token-shift rows, input-convolution rows and last tokens of designs that have them.

Latent rows, keys and values live in 16-token pages addressed through the page table of :class:`PagedSequences`; a layer's pool
is ``[pages, 16, rank + rotated part]`` (latent; a layer that attends over another one's cache has none) or ``[pages, kv_heads, 16, head size]`` and all layers share the page numbers.  Recurrent,
convolution, shift and last-token state belong to the sequence SLOT: nothing has to be cleared when a slot is given to another request,
because a row at position 0 starts from an empty state in every kernel.
"""
from __future__ import annotations

from typing import List, Optional

import torch

from .. import _native as N
from ..models.mixed import HGRN2, DeltaRule, GroupedAttention, LatentAttention, Mamba1, MixedConfig
from .kv_cache import PAGE_TOKENS, PagedSequences


def pad_to(n: int, m: int) -> int:
    return (n + m - 1) // m * m


def head_layout(m: GroupedAttention, dtype: torch.dtype):
    """``(stored head size, runs on the tensor cores)`` of a grouped-attention layer: heads of keys and values are padded to one of
    the tensor-core kernels' sizes where those take the layer, else to eight values."""
    big = max(m.dim, m.vdim)
    hd = next((x for x in (64, 128, 256) if big <= x), 0) if dtype != torch.float32 and m.scale > 0 else 0
    return (hd, True) if hd else (pad_to(big, 8), False)


def latent_layout(m: LatentAttention):
    """``(columns of the latent, columns of the rotated part)`` of a cached row."""
    return pad_to(m.kv_rank, 16), pad_to(m.rot.dims, 16) if m.rot is not None else 0


def delta_layout(m: DeltaRule, dtype: torch.dtype):
    """``(dim, vdim)`` of a stored delta-rule state: padded to the tensor-core form's sizes where that takes the layer, else to eight."""
    dim = next((x for x in (64, 128) if m.dim <= x), 0) if dtype != torch.float32 else 0
    return (dim, pad_to(m.vdim, 32)) if dim else (pad_to(m.dim, 8), pad_to(m.vdim, 8))


class MixedCache(PagedSequences):
    def __init__(self, cfg: MixedConfig, batch_size: int, max_seq_len: int, *, device="cuda", dtype=torch.bfloat16,
                 pool_tokens: Optional[int] = None):
        for name, v in (("batch_size", batch_size), ("max_seq_len", max_seq_len)):
            if isinstance(v, bool) or not isinstance(v, int) or v <= 0:
                raise ValueError(f"cache {name} must be a positive integer, got {v!r}")
        self.cfg, self.dtype, self.num_layers = cfg, dtype, cfg.num_layers
        self._init_pages(batch_size, max_seq_len, device, pool_tokens)
        self.latent: List[Optional[torch.Tensor]] = []
        self.kv: List[Optional[torch.Tensor]] = []                # [2, pages, kv_heads, 16, head size]
        self.recurrent: List[Optional[torch.Tensor]] = []
        self.conv: List[Optional[torch.Tensor]] = []
        zeros = lambda *shape, dt=dtype: torch.zeros(shape, dtype=dt, device=self.device)
        for layer in cfg.layers:
            m = layer.mixer
            latent = kv = rec = conv = None
            if isinstance(m, LatentAttention):
                latent = zeros(self.num_pages, PAGE_TOKENS, sum(latent_layout(m))) if m.kv_from is None else None
            elif isinstance(m, DeltaRule):
                D, V = delta_layout(m, dtype)
                rec = zeros(batch_size, m.heads, D, V, dt=torch.float32)
                conv = zeros(batch_size, m.conv, 2 * m.kv_heads * D + m.heads * V)
            elif isinstance(m, GroupedAttention):
                hd = head_layout(m, dtype)[0]
                kv = zeros(2, self.num_pages, m.kv_heads, PAGE_TOKENS, hd)
                conv = zeros(batch_size, m.conv - 1, (m.heads + 2 * m.kv_heads) * hd) if m.conv > 1 else None
            elif isinstance(m, HGRN2):
                rec = zeros(batch_size, m.heads, pad_to(m.dim, 8), pad_to(m.vdim, 8), dt=torch.float32)
            elif isinstance(m, Mamba1):
                rec = zeros(batch_size, pad_to(m.inner, 8), pad_to(m.state, 8), dt=torch.float32)
                conv = zeros(batch_size, m.conv - 1, pad_to(m.inner, 8)) if m.conv > 1 else None
            self.latent.append(latent)
            self.kv.append(kv)
            self.recurrent.append(rec)
            self.conv.append(conv)
        self.shift = zeros(cfg.num_layers, batch_size, pad_to(cfg.hidden_size, 8), dt=torch.float32) if cfg.token_shift else None
        self.inputs = zeros(cfg.num_layers, 2, batch_size, cfg.input_taps - 1, pad_to(cfg.hidden_size, 8)) if cfg.input_taps > 1 else None
        self.last_token = zeros(batch_size, dt=torch.int32) if cfg.pairs is not None else None

    def layer_state(self, layer: int) -> N.RfMixedState:
        """Device addresses of one layer's memory; null where it has none."""
        ptr = lambda t: None if t is None else t.data_ptr()
        st = N.RfMixedState()
        st.latent_pool, st.rec_state, st.conv_state = (ptr(x[layer]) for x in (self.latent, self.recurrent, self.conv))
        if self.kv[layer] is not None:
            st.k_pool, st.v_pool, st.pool_pages = self.kv[layer][0].data_ptr(), self.kv[layer][1].data_ptr(), self.num_pages
        of = getattr(self.cfg.layers[layer].mixer, "kv_from", None)
        if of is not None:
            st.latent_pool = self.latent[of].data_ptr()
        if self.inputs is not None:
            st.input_state[0], st.input_state[1] = (t.data_ptr() for t in self.inputs[layer])
        st.shift_state = None if self.shift is None else self.shift[layer].data_ptr()
        st.last_token = None if self.last_token is None else self.last_token.data_ptr()
        return st

    def state_tensors(self) -> List[torch.Tensor]:
        """Everything a step advances in place (pages are only ever written at new positions)."""
        return [t for t in self.recurrent + self.conv + [self.shift, self.inputs, self.last_token] if t is not None]

    def _tensors(self) -> List[torch.Tensor]:
        return [t for t in self.latent + self.kv if t is not None] + self.state_tensors()

    def zero_(self) -> None:
        for t in self._tensors():
            t.zero_()

    def nbytes(self) -> int:
        return sum(t.numel() * t.element_size() for t in self._tensors())


__all__ = ["MixedCache", "head_layout", "latent_layout", "delta_layout", "pad_to"]
