"""Decoders whose layers name their own mixer: configuration records and weight tables.

A :class:`MixedConfig` is a list of layers, each with one mixer (:class:`LatentAttention`, :class:`HGRN2`) and an optional
feed-forward (:class:`DenseMLP`), over what the layers share: the width of an fp32 residual stream, RMSNorm epsilon, tied
embedding, a token shift in front of every mixer and a gated per-token side input behind every layer.  The native executor
is ``csrc/models/mixed_stack.cu``, the engine :mod:`rhinoforge_b200.runtime.mixed_engine`.

Reader of Vabarax's ``config.json``: :meth:`MixedConfig.from_vabarax`.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Dict, Iterator, Mapping, Optional, Tuple, Union

import torch

from ..runtime.errors import UnsupportedModelError


@dataclass(frozen=True)
class LatentAttention:
    """Attention over one cached latent row per token; keys and values of a head are linear maps of it.  ``window``: how many
    positions a query sees, its own included (None: all of them)."""
    heads: int
    dim: int
    vdim: int
    kv_rank: int
    scale: float
    window: Optional[int] = None


@dataclass(frozen=True)
class HGRN2:
    """Linear attention with one gate per key channel for keeping and adding (state ``[heads, dim, vdim]``)."""
    heads: int
    dim: int
    vdim: int


@dataclass(frozen=True)
class DenseMLP:
    """``down(relu(up h)^2)``."""
    ff: int


@dataclass(frozen=True)
class MixedLayer:
    mixer: Union[LatentAttention, HGRN2]
    mlp: Optional[DenseMLP] = None


def _int(d: Mapping[str, Any], key: str, where: str) -> int:
    v = d.get(key)
    if isinstance(v, bool) or not isinstance(v, int) or v <= 0:
        raise UnsupportedModelError(f"{where}: {key!r} must be a positive integer, got {v!r}")
    return v


def _known(d: Mapping[str, Any], keys, where: str) -> None:
    extra = sorted(set(d) - set(keys))
    if extra:
        raise UnsupportedModelError(f"{where}: unsupported key(s) {extra}")


@dataclass(frozen=True)
class MixedConfig:
    name: str
    vocab_size: int
    hidden_size: int
    rms_eps: float
    layers: Tuple[MixedLayer, ...]
    side_dim: int
    model_type: str = "vabarax"
    raw: Optional[Mapping[str, Any]] = field(default=None, compare=False, repr=False)

    @property
    def num_layers(self) -> int:
        return len(self.layers)

    @classmethod
    def from_vabarax(cls, c: Mapping[str, Any]) -> "MixedConfig":
        """The mapping of a Vabarax ``config.json``.  Keys that the reader does not know are refused rather than ignored."""
        if not isinstance(c.get("layers"), list) or not c["layers"]:
            raise UnsupportedModelError("Vabarax: 'layers' must be a non-empty list")
        layers = []
        for i, entry in enumerate(c["layers"]):
            where = f"Vabarax layer {i}"
            _known(entry, ("type", "mixer", "mlp"), where)
            kind, m = entry.get("type"), entry.get("mixer")
            if not isinstance(m, Mapping):
                raise UnsupportedModelError(f"{where}: 'mixer' must be a mapping")
            if kind == "latent_attention":
                _known(m, ("heads", "dim", "vdim", "kv_rank", "scale", "mask"), where)
                mask = m.get("mask") or {}
                _known(mask, ("size",), where + " mask")
                mixer: Union[LatentAttention, HGRN2] = LatentAttention(
                    _int(m, "heads", where), _int(m, "dim", where), _int(m, "vdim", where), _int(m, "kv_rank", where),
                    float(m["scale"]), _int(mask, "size", where + " mask") if mask else None)
            elif kind == "hgrn2":
                _known(m, ("heads", "dim", "vdim"), where)
                mixer = HGRN2(_int(m, "heads", where), _int(m, "dim", where), _int(m, "vdim", where))
            else:
                raise UnsupportedModelError(f"{where}: mixer type {kind!r} is not built")
            mlp = None
            if entry.get("mlp") is not None:
                _known(entry["mlp"], ("kind", "ff"), where + " mlp")
                if entry["mlp"].get("kind") != "dense":
                    raise UnsupportedModelError(f"{where}: feed-forward kind {entry['mlp'].get('kind')!r} is not built")
                mlp = DenseMLP(_int(entry["mlp"], "ff", where + " mlp"))
            layers.append(MixedLayer(mixer, mlp))
        return cls(name="vabarax", vocab_size=_int(c, "vocab", "Vabarax"), hidden_size=_int(c, "width", "Vabarax"),
                   rms_eps=float(c["norm"]["eps"]), layers=tuple(layers), side_dim=_int(c["token_side"], "dim", "Vabarax token_side"),
                   raw=c)

    def to_vabarax(self) -> Dict[str, Any]:
        """The inverse of :meth:`from_vabarax`."""
        out = []
        for layer in self.layers:
            m = layer.mixer
            d: Dict[str, Any] = {"heads": m.heads, "dim": m.dim, "vdim": m.vdim}
            if isinstance(m, LatentAttention):
                d.update(kv_rank=m.kv_rank, scale=m.scale)
                if m.window is not None:
                    d["mask"] = {"size": m.window}
            out.append({"type": "latent_attention" if isinstance(m, LatentAttention) else "hgrn2", "mixer": d,
                        "mlp": None if layer.mlp is None else {"kind": "dense", "ff": layer.mlp.ff}})
        return {"architecture": "Vabarax", "vocab": self.vocab_size, "width": self.hidden_size, "norm": {"eps": self.rms_eps},
                "token_side": {"dim": self.side_dim}, "layers": out}


def weight_shapes(cfg: MixedConfig) -> Iterator[Tuple[str, Tuple[int, ...], str]]:
    """(tensor name, shape, kind) of a checkpoint; kind is 'linear', 'embed', 'norm', 'unit' (values in [0, 1)) or 'bias'."""
    H, P = cfg.hidden_size, cfg.side_dim
    yield "embed", (cfg.vocab_size, H), "embed"
    yield "side.embed", (cfg.vocab_size, cfg.num_layers * P), "embed"
    for i, layer in enumerate(cfg.layers):
        p, m = f"l{i}.", layer.mixer
        qd, vd = m.heads * m.dim, m.heads * m.vdim
        yield p + "norm1", (H,), "norm"
        yield p + "shift", (H,), "unit"
        yield p + "mix.q", (qd, H), "linear"
        if isinstance(m, LatentAttention):
            yield p + "mix.dkv", (m.kv_rank, H), "linear"
            yield p + "mix.dkv.norm", (m.kv_rank,), "norm"
            yield p + "mix.uk", (qd, m.kv_rank), "linear"
            yield p + "mix.uv", (vd, m.kv_rank), "linear"
        else:
            yield p + "mix.f", (qd, H), "linear"
            yield p + "mix.f.b", (qd,), "bias"
            yield p + "mix.lower", (qd,), "unit"
            yield p + "mix.v", (vd, H), "linear"
            yield p + "mix.norm", (m.vdim,), "norm"
        yield p + "mix.o", (H, vd), "linear"
        if layer.mlp is not None:
            yield p + "norm2", (H,), "norm"
            yield p + "mlp.up", (layer.mlp.ff, H), "linear"
            yield p + "mlp.down", (H, layer.mlp.ff), "linear"
        yield p + "side.gate", (P, H), "linear"
        yield p + "side.proj", (H, P), "linear"
        yield p + "side.norm", (H,), "norm"
    yield "final.norm", (H,), "norm"


def random_weights(cfg: MixedConfig, *, seed: int = 0, dtype=torch.bfloat16, device="cpu", gain: float = 1.0):
    """Weight getter with random values generated on demand (one seeded generator per tensor): linears and embeddings scaled by
    ``gain / sqrt(columns)`` so that activations stay of order one, norms around one, units uniform in [0, 1)."""
    table = {name: (idx, shape, kind) for idx, (name, shape, kind) in enumerate(weight_shapes(cfg))}
    dev = torch.device(device)

    def get(name: str) -> torch.Tensor:
        idx, shape, kind = table[name]
        g = torch.Generator(device=dev)
        g.manual_seed(seed * 1_000_003 + idx)
        t = torch.empty(shape, dtype=torch.float32, device=dev)
        if kind == "unit":
            return t.uniform_(0, 1, generator=g).to(dtype)
        t.normal_(0.0, 1.0, generator=g)
        if kind == "norm":
            return (1.0 + 0.1 * t).to(dtype)
        if kind == "linear":
            t *= gain / shape[1] ** 0.5
        return t.to(dtype)

    get.names = frozenset(table)  # type: ignore[attr-defined]
    return get


__all__ = ["MixedConfig", "MixedLayer", "LatentAttention", "HGRN2", "DenseMLP", "weight_shapes", "random_weights"]
