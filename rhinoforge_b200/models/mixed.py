"""Decoders whose layers name their own mixer: configuration records and weight tables.

A :class:`MixedConfig` is a list of layers, each with one mixer (:class:`LatentAttention`, :class:`HGRN2`,
:class:`GroupedAttention`, :class:`Mamba1`, :class:`DeltaRule`) and an optional feed-forward (:class:`DenseMLP`, :class:`GatedMLP`,
:class:`ClippedGLU`, :class:`MoE`), over what the layers share: the width of an fp32 residual stream, RMSNorm epsilon, where the norms
sit, and optionally an embedding of token pairs, a factor on the sublayers' outputs, a token shift in front of every mixer, a
convolution in front of every sublayer, a gated per-token side input behind every layer and a soft cap of the logits.  The native executor is ``csrc/models/mixed_stack.cu``, the engine
:mod:`rhinoforge_b200.runtime.mixed_engine`.

Readers of ``config.json``: :meth:`MixedConfig.from_vabarax`, :meth:`MixedConfig.from_zulopel`, :meth:`MixedConfig.from_kuzupel`,
:meth:`MixedConfig.from_vasosun`.
"""
from __future__ import annotations

import math
from dataclasses import dataclass, field
from typing import Any, Dict, Iterator, Mapping, Optional, Tuple, Union

import torch

from ..runtime.errors import UnsupportedModelError


@dataclass(frozen=True)
class LatentAttention:
    """Attention over one cached latent row per token; keys and values of a head are linear maps of it.  ``window``: how many
    positions a query sees, its own included (None: all of them).  ``q_rank`` > 0: queries go through a normalised latent of this size.
    ``rot``: every query head has ``rot.dims`` more dimensions, rotated in neighbouring pairs, against one rotated key part per token that
    all heads share and that is cached behind the latent.  ``kv_from``: the layer whose cache this one attends over (None: its own)."""
    heads: int
    dim: int
    vdim: int
    kv_rank: int
    scale: float
    window: Optional[int] = None
    q_rank: int = 0
    rot: Optional["Rotary"] = None
    kv_from: Optional[int] = None


@dataclass(frozen=True)
class HGRN2:
    """Linear attention with one gate per key channel for keeping and adding (state ``[heads, dim, vdim]``)."""
    heads: int
    dim: int
    vdim: int


@dataclass(frozen=True)
class YarnScaling:
    """Stretch of a rotation made for ``original`` positions by ``factor``: pairs of dimensions that turn more than ``fast`` times
    over the original length keep their frequency, those that turn less than ``slow`` times are divided by the factor."""
    factor: float
    original: int
    fast: float
    slow: float


@dataclass(frozen=True)
class Rotary:
    """Rotation of ``dims`` dimensions of a head: the first ones, dimension i paired with i + dims / 2 (:class:`GroupedAttention`), or a
    part of their own, dimension 2 i paired with 2 i + 1 (:class:`LatentAttention`)."""
    dims: int
    base: float
    scaling: Optional[YarnScaling] = None

    def frequencies(self) -> torch.Tensor:
        """float64 ``[dims / 2]``, stretch applied."""
        f = torch.tensor([self.base ** (-2.0 * i / self.dims) for i in range(self.dims // 2)], dtype=torch.float64)
        y = self.scaling
        if y is None:
            return f
        pair = lambda turns: self.dims * math.log(y.original / (2.0 * math.pi * turns)) / (2.0 * math.log(self.base))
        lo, hi = max(math.floor(pair(y.fast)), 0), min(math.ceil(pair(y.slow)), self.dims - 1)
        ramp = ((torch.arange(self.dims // 2, dtype=torch.float64) - lo) / max(hi - lo, 0.001)).clamp(0.0, 1.0)
        return f / y.factor * ramp + f * (1.0 - ramp)

    def tables(self, positions: int, device) -> Tuple[torch.Tensor, torch.Tensor]:
        """fp32 cos and sin ``[positions, dims / 2]`` of positions 0, 1, ..., the stretch's magnitude factor included."""
        amp = 1.0 if self.scaling is None else 0.1 * math.log(self.scaling.factor) + 1.0
        angle = torch.arange(positions, dtype=torch.float64, device=device)[:, None] * self.frequencies().to(device)[None]
        return (angle.cos() * amp).float().contiguous(), (angle.sin() * amp).float().contiguous()


@dataclass(frozen=True)
class GroupedAttention:
    """Softmax attention with ``heads // kv_heads`` query heads per key / value head.

    What a position sees: ``chunk``, its own chunk of this many positions; ``window``, the last this many positions, its own
    included, and then also the first ``keep_first`` ones (both None: everything before it).  ``distance_bias``: head h's scores
    lose ``2^(-8 (h + 1) / heads)`` per token of distance.  ``sink``: one more learned term in every head's softmax denominator;
    ``unit_sink``: that term is exp(0) in every head.  ``v_mix``: values are mixed with those of the first layer that says so.
    ``qk_norm``: RMSNorm of every query and key head, or with ``norm_all`` one over all query heads and one over all key heads.
    ``conv`` > 0: causal convolution of this many taps on the projected queries, keys and values.  ``gate``: sigmoid gate on the
    heads' outputs, element by element, or with ``gate_by_head`` one number per head.  ``log_bias``: head h's scores lose
    ``r1[h] ln(1 + r2[h] distance)`` with learned r1 and r2.  ``growth_every`` > 0: queries of position p are multiplied by
    ``1 + growth ln(floor((p + 1) / growth_every) + 1)``."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    chunk: Optional[int] = None
    rot: Optional[Rotary] = None
    v_mix: bool = False
    qk_norm: bool = True
    sink: bool = True
    gate: bool = True
    window: Optional[int] = None
    keep_first: int = 0
    distance_bias: bool = False
    unit_sink: bool = False
    norm_all: bool = False
    conv: int = 0
    gate_by_head: bool = False
    log_bias: bool = False
    growth: float = 0.0
    growth_every: int = 0

    def slopes(self) -> Optional[torch.Tensor]:
        """float64 ``[heads]``: what the scores lose per token of distance."""
        if not self.distance_bias:
            return None
        return torch.tensor([2.0 ** (-8.0 * (h + 1) / self.heads) for h in range(self.heads)], dtype=torch.float64)


@dataclass(frozen=True)
class Mamba1:
    """Selective scan over ``inner`` channels with ``state`` states each, behind a causal convolution of ``conv`` taps."""
    inner: int
    state: int
    dt_rank: int
    conv: int


@dataclass(frozen=True)
class DeltaRule:
    """Gated delta rule (state ``[heads, dim, vdim]``) over ``kv_heads`` query / key heads, behind a causal convolution of ``conv`` taps
    with silu on queries, keys and values; the outputs are normalised per head and gated."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int


@dataclass(frozen=True)
class GatedMLP:
    """``down(silu(gate h) * up h)``."""
    ff: int


@dataclass(frozen=True)
class DenseMLP:
    """``down(relu(up h)^2)``."""
    ff: int


@dataclass(frozen=True)
class ClippedGLU:
    """``down(g sigmoid(alpha g) (u + 1))`` with ``g = min(gate h, limit)`` and ``u = clamp(up h, -limit, limit)``."""
    ff: int
    limit: float
    alpha: float = 1.702


@dataclass(frozen=True)
class MoE:
    """``top`` of ``experts`` gated experts of width ``ff`` per token; ``shared_ff`` > 0: one more expert that every token uses.

    ``router`` "corrected": chosen among the ``keep`` best of ``groups`` groups by softmax score plus correction, weighted by
    normalised score.  "chosen": the logits have a bias, the largest are chosen, weights are the softmax over the chosen ones.
    ``limit``: experts are clipped (:class:`ClippedGLU`), the shared one with ``shared_limit``; None: SwiGLU.  ``shared_gate``: the
    shared expert is weighted by a sigmoid of one number per token.  ``gated`` False: experts are ``down(gelu(up h))``.  ``identity``: this
    many more experts behind the others whose output is their input.  ``renormalise`` False: the weights of "corrected" stay the
    chosen experts' scores."""
    experts: int
    top: int
    ff: int
    groups: int = 1
    keep: int = 1
    shared_ff: int = 0
    router: str = "corrected"
    limit: Optional[float] = None
    shared_limit: Optional[float] = None
    alpha: float = 1.702
    shared_gate: bool = False
    gated: bool = True
    identity: int = 0
    renormalise: bool = True


@dataclass(frozen=True)
class TokenPairs:
    """Embedding row of (previous token, token): ``(previous * mul_prev + token * mul_cur) % buckets``, row ``buckets`` for a
    sequence's first token."""
    buckets: int
    mul_prev: int
    mul_cur: int


@dataclass(frozen=True)
class MixedLayer:
    mixer: Union[LatentAttention, HGRN2, GroupedAttention, Mamba1, DeltaRule]
    mlp: Optional[Union[DenseMLP, GatedMLP, ClippedGLU, MoE]] = None


def _int(d: Mapping[str, Any], key: str, where: str, least: int = 1) -> int:
    v = d.get(key)
    if isinstance(v, bool) or not isinstance(v, int) or v < least:
        raise UnsupportedModelError(f"{where}: {key!r} must be an integer of at least {least}, got {v!r}")
    return v


def _float(d: Mapping[str, Any], key: str, where: str, positive: bool = False) -> float:
    v = d.get(key)
    if isinstance(v, bool) or not isinstance(v, (int, float)) or not math.isfinite(v) or (positive and v <= 0):
        raise UnsupportedModelError(f"{where}: {key!r} must be a {'positive ' if positive else ''}number, got {v!r}")
    return float(v)


def _map(d: Mapping[str, Any], key: str, where: str) -> Mapping[str, Any]:
    v = d.get(key)
    if not isinstance(v, Mapping):
        raise UnsupportedModelError(f"{where}: {key!r} must be a mapping, got {v!r}")
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
    side_dim: int = 0              # width of the per-token side input behind every layer (0: none)
    token_shift: bool = True       # mix every token's normalised row with the one before, in front of every mixer
    norm_after: bool = False       # norms on the sublayers' outputs instead of their inputs
    norm_both: bool = False        # norms on the sublayers' outputs as well as on their inputs
    scalar_norms: bool = False     # the norms around the sublayers and the last one have one weight for all coordinates
    input_taps: int = 0            # > 0: h + convolution of this many taps over h in front of every sublayer
    layer_scale: bool = False      # element-wise factors on the sublayers' outputs
    tied_head: bool = True
    embed_scale: float = 1.0
    pairs: Optional[TokenPairs] = None     # embedding of token pairs, added to the tokens' own
    residual_mult: float = 1.0             # factor of the sublayers' outputs
    logit_softcap: Optional[float] = None  # logits <- cap * tanh(logits / cap)
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

    @classmethod
    def zulopel(cls, name: str, vocab: int, width: int, eps: float, layers, embed_scale: float = 1.0, **kw) -> "MixedConfig":
        """A decoder of the Zulopel design: grouped attention and selective-scan layers in any order, mixture-of-experts
        feed-forwards, norms and layer scales on the sublayers' outputs, an untied head."""
        cfg = cls(name, vocab, width, eps, tuple(layers), 0, token_shift=False, norm_after=True, layer_scale=True, tied_head=False,
                  embed_scale=embed_scale, model_type="zulopel", **kw)
        widths = {(i, m.kv_heads * m.vdim) for i, m in enumerate(x.mixer for x in cfg.layers) if isinstance(m, GroupedAttention) and m.v_mix}
        if len({w for _, w in widths}) > 1:
            raise UnsupportedModelError(f"{name}: layers that mix values need values of one size, got (layer, size) {sorted(widths)}")
        return cfg

    @classmethod
    def from_zulopel(cls, c: Mapping[str, Any]) -> "MixedConfig":
        """The mapping of a Zulopel ``config.json``.  Keys that the reader does not know are refused rather than ignored."""
        _known(c, ("architecture", "embedding", "layers", "norm", "vocab", "width"), "Zulopel")
        if not isinstance(c.get("layers"), list) or not c["layers"]:
            raise UnsupportedModelError("Zulopel: 'layers' must be a non-empty list")
        layers = []
        for i, entry in enumerate(c["layers"]):
            where = f"Zulopel layer {i}"
            if not isinstance(entry, Mapping):
                raise UnsupportedModelError(f"{where}: must be a mapping")
            _known(entry, ("type", "mixer", "mlp"), where)
            kind, m = entry.get("type"), _map(entry, "mixer", where)
            if kind == "attention":
                mixer: Union[GroupedAttention, Mamba1] = _zulopel_attention(m, where)
            elif kind == "mamba1":
                _known(m, ("inner", "state", "dt_rank", "conv"), where)
                mixer = Mamba1(*(_int(m, k, where) for k in ("inner", "state", "dt_rank", "conv")))
            else:
                raise UnsupportedModelError(f"{where}: mixer type {kind!r} is not built")
            layers.append(MixedLayer(mixer, None if entry.get("mlp") is None else _zulopel_experts(_map(entry, "mlp", where), where + " mlp")))
        norm = _map(c, "norm", "Zulopel")
        _known(norm, ("eps",), "Zulopel norm")
        emb = c.get("embedding") or {}
        _known(emb, ("scale",), "Zulopel embedding")
        return cls.zulopel("zulopel", _int(c, "vocab", "Zulopel"), _int(c, "width", "Zulopel"), _float(norm, "eps", "Zulopel norm"), layers,
                           _float(emb, "scale", "Zulopel embedding") if "scale" in emb else 1.0, raw=c)

    def to_zulopel(self) -> Dict[str, Any]:
        """The inverse of :meth:`from_zulopel`."""
        out = []
        for layer in self.layers:
            m, f = layer.mixer, layer.mlp
            if isinstance(m, Mamba1):
                d: Dict[str, Any] = {"inner": m.inner, "state": m.state, "dt_rank": m.dt_rank, "conv": m.conv}
            else:
                d = {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "scale": m.scale, "v_mix": m.v_mix}
                if m.chunk is not None:
                    d["mask"] = {"size": m.chunk}
                if m.rot is not None:
                    d["rot"] = {"dims": m.rot.dims, "base": m.rot.base}
                    if m.rot.scaling is not None:
                        y = m.rot.scaling
                        d["rot"]["scaling"] = {"factor": y.factor, "original": y.original, "fast": y.fast, "slow": y.slow}
            mlp = None
            if f is not None:
                mlp = {"kind": "moe", "expert": {"ff": f.ff},
                       "router": {"experts": f.experts, "top": f.top, "groups": {"count": f.groups, "keep": f.keep}}}
                if f.shared_ff:
                    mlp["shared"] = {"ff": f.shared_ff}
            out.append({"type": "mamba1" if isinstance(m, Mamba1) else "attention", "mixer": d, "mlp": mlp})
        return {"architecture": "Zulopel", "vocab": self.vocab_size, "width": self.hidden_size, "norm": {"eps": self.rms_eps},
                "embedding": {"scale": self.embed_scale}, "layers": out}

    @classmethod
    def kuzupel(cls, name: str, vocab: int, width: int, eps: float, layers, *, pairs: Optional[TokenPairs] = None, embed_scale: float = 1.0,
                residual_mult: float = 1.0, logit_softcap: Optional[float] = None, **kw) -> "MixedConfig":
        """A decoder of the Kuzupel design: distance-biased and rotary window attention in any order, clipped gated feed-forwards or
        mixtures of them, an embedding of token pairs, an untied head with a soft cap."""
        return cls(name, vocab, width, eps, tuple(layers), 0, token_shift=False, tied_head=False, embed_scale=embed_scale, pairs=pairs,
                   residual_mult=residual_mult, logit_softcap=logit_softcap, model_type="kuzupel", **kw)

    @classmethod
    def from_kuzupel(cls, c: Mapping[str, Any]) -> "MixedConfig":
        """The mapping of a Kuzupel ``config.json``.  Keys that the reader does not know are refused rather than ignored."""
        _known(c, ("architecture", "embedding", "layers", "logit_softcap", "norm", "residual_mult", "vocab", "width"), "Kuzupel")
        if not isinstance(c.get("layers"), list) or not c["layers"]:
            raise UnsupportedModelError("Kuzupel: 'layers' must be a non-empty list")
        layers = []
        for i, entry in enumerate(c["layers"]):
            where = f"Kuzupel layer {i}"
            if not isinstance(entry, Mapping):
                raise UnsupportedModelError(f"{where}: must be a mapping")
            _known(entry, ("type", "mixer", "mlp"), where)
            read = {"attention": _kuzupel_biased, "attention_2": _kuzupel_rotary}.get(entry.get("type"))
            if read is None:
                raise UnsupportedModelError(f"{where}: mixer type {entry.get('type')!r} is not built")
            mlp = None if entry.get("mlp") is None else _kuzupel_mlp(_map(entry, "mlp", where), where + " mlp")
            layers.append(MixedLayer(read(_map(entry, "mixer", where), where), mlp))
        norm, emb = _map(c, "norm", "Kuzupel"), c.get("embedding") or {}
        _known(norm, ("eps",), "Kuzupel norm")
        _known(emb, ("scale", "bigram"), "Kuzupel embedding")
        number = lambda d, key, default, where: default if d.get(key) is None else _float(d, key, where, True)
        cap = c.get("logit_softcap")
        return cls.kuzupel("kuzupel", _int(c, "vocab", "Kuzupel"), _int(c, "width", "Kuzupel"), _float(norm, "eps", "Kuzupel norm"), layers,
                           pairs=_token_pairs(emb, "Kuzupel"), embed_scale=number(emb, "scale", 1.0, "Kuzupel embedding"),
                           residual_mult=number(c, "residual_mult", 1.0, "Kuzupel"),
                           logit_softcap=None if cap is None else _float(c, "logit_softcap", "Kuzupel", True), raw=c)

    def to_kuzupel(self) -> Dict[str, Any]:
        """The inverse of :meth:`from_kuzupel`."""
        out = []
        for layer in self.layers:
            m, f = layer.mixer, layer.mlp
            d: Dict[str, Any] = {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "scale": m.scale}
            if m.window is not None:
                d["mask"] = {"size": m.window} if m.distance_bias else {"size": m.window, "keep_first": m.keep_first}
            if not m.distance_bias:
                d["conv"] = m.conv
                if m.rot is not None:
                    d["rot"] = {"dims": m.rot.dims, "base": m.rot.base}
            mlp: Optional[Dict[str, Any]] = None
            if isinstance(f, MoE):
                mlp = {"kind": "moe", "expert": {"ff": f.ff, "limit": f.limit}, "router": {"experts": f.experts, "top": f.top}}
                if f.shared_ff:
                    mlp["shared"] = {"ff": f.shared_ff, "limit": f.shared_limit}
            elif f is not None:
                mlp = {"kind": "dense", "ff": f.ff, "limit": f.limit}
            out.append({"type": "attention" if m.distance_bias else "attention_2", "mixer": d, "mlp": mlp})
        emb: Dict[str, Any] = {"scale": self.embed_scale}
        if self.pairs is not None:
            emb["bigram"] = {"buckets": self.pairs.buckets, "mul_prev": self.pairs.mul_prev, "mul_cur": self.pairs.mul_cur}
        top = {"architecture": "Kuzupel", "vocab": self.vocab_size, "width": self.hidden_size, "norm": {"eps": self.rms_eps},
               "embedding": emb, "residual_mult": self.residual_mult, "layers": out}
        return top if self.logit_softcap is None else {**top, "logit_softcap": self.logit_softcap}

    @classmethod
    def vasosun(cls, name: str, vocab: int, width: int, eps: float, layers, *, input_taps: int = 0, pairs: Optional[TokenPairs] = None,
                logit_softcap: Optional[float] = None, **kw) -> "MixedConfig":
        """A decoder of the Vasosun design: delta-rule, window-attention and latent-attention layers in any order, SwiGLU feed-forwards
        or mixtures with identity experts, scalar norms on both sides of the sublayers, a convolution in front of each."""
        cfg = cls(name, vocab, width, eps, tuple(layers), 0, token_shift=False, norm_both=True, scalar_norms=True, input_taps=input_taps,
                  tied_head=False, pairs=pairs, logit_softcap=logit_softcap, model_type="vasosun", **kw)
        for i, m in enumerate(layer.mixer for layer in cfg.layers):
            if getattr(m, "kv_from", None) is None:
                continue
            of = cfg.layers[m.kv_from].mixer if 0 <= m.kv_from < i else None
            if not isinstance(of, LatentAttention) or of.kv_from is not None or (of.kv_rank, of.rot) != (m.kv_rank, m.rot):
                raise UnsupportedModelError(f"{name} layer {i}: layer {m.kv_from} has no cache of its own with the same latent and rotation")
        return cfg

    @classmethod
    def from_vasosun(cls, c: Mapping[str, Any]) -> "MixedConfig":
        """The mapping of a Vasosun ``config.json``.  Keys that the reader does not know are refused rather than ignored."""
        _known(c, ("architecture", "canon", "embedding", "layers", "logit_softcap", "norm", "vocab", "width"), "Vasosun")
        if not isinstance(c.get("layers"), list) or not c["layers"]:
            raise UnsupportedModelError("Vasosun: 'layers' must be a non-empty list")
        layers = []
        for i, entry in enumerate(c["layers"]):
            where = f"Vasosun layer {i}"
            if not isinstance(entry, Mapping):
                raise UnsupportedModelError(f"{where}: must be a mapping")
            _known(entry, ("type", "mixer", "mlp"), where)
            read = {"attention": _vasosun_window, "latent_attention": _vasosun_latent, "delta": _vasosun_delta}.get(entry.get("type"))
            if read is None:
                raise UnsupportedModelError(f"{where}: mixer type {entry.get('type')!r} is not built")
            mlp = None if entry.get("mlp") is None else _vasosun_mlp(_map(entry, "mlp", where), where + " mlp")
            layers.append(MixedLayer(read(_map(entry, "mixer", where), where), mlp))
        norm, taps = _map(c, "norm", "Vasosun"), 0
        _known(norm, ("eps",), "Vasosun norm")
        if c.get("canon") is not None:
            _known(_map(c, "canon", "Vasosun"), ("taps",), "Vasosun canon")
            taps = _int(c["canon"], "taps", "Vasosun canon")
        emb = c.get("embedding") or {}
        _known(emb, ("bigram",), "Vasosun embedding")
        return cls.vasosun("vasosun", _int(c, "vocab", "Vasosun"), _int(c, "width", "Vasosun"), _float(norm, "eps", "Vasosun norm"), layers,
                           input_taps=taps, pairs=_token_pairs(emb, "Vasosun"),
                           logit_softcap=None if c.get("logit_softcap") is None else _float(c, "logit_softcap", "Vasosun", True), raw=c)

    def to_vasosun(self) -> Dict[str, Any]:
        """The inverse of :meth:`from_vasosun`."""
        out = []
        for layer in self.layers:
            m, f = layer.mixer, layer.mlp
            d: Dict[str, Any] = {"heads": m.heads, "dim": m.dim, "vdim": m.vdim}
            if isinstance(m, DeltaRule):
                kind = "delta"
                d.update(kv_heads=m.kv_heads, conv=m.conv)
            elif isinstance(m, GroupedAttention):
                kind = "attention"
                d.update(kv_heads=m.kv_heads, scale=m.scale)
                if m.window is not None:
                    d["mask"] = {"size": m.window}
                if m.growth_every:
                    d["q_temp"] = {"coef": m.growth, "every": m.growth_every}
            else:
                kind = "latent_attention"
                d.update(kv_rank=m.kv_rank, q_rank=m.q_rank, rot_dim=m.rot.dims, scale=m.scale, rot={"dims": m.rot.dims, "base": m.rot.base})
                if m.rot.scaling is not None:
                    y = m.rot.scaling
                    d["rot"]["scaling"] = {"factor": y.factor, "original": y.original, "fast": y.fast, "slow": y.slow}
                if m.kv_from is not None:
                    d["kv_from"] = m.kv_from
            mlp: Optional[Dict[str, Any]] = None
            if isinstance(f, MoE):
                mlp = {"kind": "moe", "expert": {"ff": f.ff}, "router": {"experts": f.experts, "identity": f.identity, "top": f.top}}
            elif f is not None:
                mlp = {"kind": "dense", "ff": f.ff}
            out.append({"type": kind, "mixer": d, "mlp": mlp})
        top: Dict[str, Any] = {"architecture": "Vasosun", "vocab": self.vocab_size, "width": self.hidden_size, "norm": {"eps": self.rms_eps},
                               "embedding": {}, "layers": out}
        if self.pairs is not None:
            top["embedding"]["bigram"] = {"buckets": self.pairs.buckets, "mul_prev": self.pairs.mul_prev, "mul_cur": self.pairs.mul_cur}
        if self.input_taps:
            top["canon"] = {"taps": self.input_taps}
        if self.logit_softcap is not None:
            top["logit_softcap"] = self.logit_softcap
        return top

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


def _token_pairs(emb: Mapping[str, Any], design: str) -> Optional[TokenPairs]:
    if emb.get("bigram") is None:
        return None
    b, w = _map(emb, "bigram", design + " embedding"), design + " bigram"
    _known(b, ("buckets", "mul_prev", "mul_cur"), w)
    return TokenPairs(_int(b, "buckets", w), _int(b, "mul_prev", w, 0), _int(b, "mul_cur", w, 0))


def _yarn(r: Mapping[str, Any], where: str) -> Optional[YarnScaling]:
    if not r.get("scaling"):
        return None
    sc, w = _map(r, "scaling", where), where + " scaling"
    _known(sc, ("factor", "original", "fast", "slow"), w)
    return YarnScaling(*(_float(sc, k, w, True) for k in ("factor", "original", "fast", "slow")))


def _zulopel_attention(m: Mapping[str, Any], where: str) -> GroupedAttention:
    _known(m, ("heads", "kv_heads", "dim", "vdim", "scale", "mask", "rot", "v_mix"), where)
    mask, rot = m.get("mask") or {}, None
    _known(mask, ("size",), where + " mask")
    if m.get("rot"):
        r, w = _map(m, "rot", where), where + " rot"
        _known(r, ("dims", "base", "scaling"), w)
        rot = Rotary(_int(r, "dims", w), _float(r, "base", w, True), _yarn(r, w))
    a = GroupedAttention(_int(m, "heads", where), _int(m, "kv_heads", where), _int(m, "dim", where), _int(m, "vdim", where),
                         _float(m, "scale", where), _int(mask, "size", where + " mask") if mask else None, rot, bool(m.get("v_mix", False)))
    if a.heads % a.kv_heads:
        raise UnsupportedModelError(f"{where}: {a.heads} heads do not share {a.kv_heads} key / value heads evenly")
    if rot is not None and (rot.dims % 2 or rot.dims > a.dim):
        raise UnsupportedModelError(f"{where}: rotation of {rot.dims} of {a.dim} dimensions")
    return a


def _zulopel_experts(f: Mapping[str, Any], where: str) -> MoE:
    _known(f, ("kind", "expert", "router", "shared"), where)
    if f.get("kind") != "moe":
        raise UnsupportedModelError(f"{where}: feed-forward kind {f.get('kind')!r} is not built")
    expert, r = _map(f, "expert", where), _map(f, "router", where)
    _known(expert, ("ff",), where + " expert")
    _known(r, ("experts", "top", "groups"), where + " router")
    groups = r.get("groups") or {"count": 1, "keep": 1}
    _known(groups, ("count", "keep"), where + " groups")
    shared = f.get("shared") or {}
    _known(shared, ("ff",), where + " shared")
    e = MoE(_int(r, "experts", where), _int(r, "top", where), _int(expert, "ff", where), _int(groups, "count", where), _int(groups, "keep", where),
            _int(shared, "ff", where + " shared") if shared else 0)
    if e.experts % e.groups or e.keep > e.groups or e.top > e.experts // e.groups * e.keep:
        raise UnsupportedModelError(f"{where}: {e.top} of {e.experts} experts in {e.keep} of {e.groups} groups")
    if e.experts > 256 or e.top > 32:
        raise UnsupportedModelError(f"{where}: the router takes up to 256 experts and 32 choices")
    return e


def _kuzupel_sizes(m: Mapping[str, Any], where: str, keys, mask_keys) -> Dict[str, Any]:
    _known(m, ("heads", "kv_heads", "dim", "vdim", "scale", "mask") + keys, where)
    mask = m.get("mask") or {}
    _known(mask, mask_keys, where + " mask")
    a = {k: _int(m, k, where) for k in ("heads", "kv_heads", "dim", "vdim")}
    if a["heads"] % a["kv_heads"]:
        raise UnsupportedModelError(f"{where}: {a['heads']} heads do not share {a['kv_heads']} key / value heads evenly")
    a.update(scale=_float(m, "scale", where), sink=False, window=_int(mask, "size", where + " mask") if mask else None)
    return a


def _kuzupel_biased(m: Mapping[str, Any], where: str) -> GroupedAttention:
    return GroupedAttention(**_kuzupel_sizes(m, where, (), ("size",)), gate=False, distance_bias=True, norm_all=True)


def _kuzupel_rotary(m: Mapping[str, Any], where: str) -> GroupedAttention:
    a = _kuzupel_sizes(m, where, ("conv", "rot"), ("size", "keep_first"))
    mask, rot = m.get("mask") or {}, None
    if m.get("rot"):
        r, w = _map(m, "rot", where), where + " rot"
        _known(r, ("dims", "base"), w)
        rot = Rotary(_int(r, "dims", w), _float(r, "base", w, True))
        if rot.dims % 2 or rot.dims > a["dim"]:
            raise UnsupportedModelError(f"{where}: rotation of {rot.dims} of {a['dim']} dimensions")
    return GroupedAttention(**a, rot=rot, unit_sink=True, gate_by_head=True, conv=_int(m, "conv", where),
                            keep_first=_int(mask, "keep_first", where + " mask", 0) if "keep_first" in mask else 0)


def _kuzupel_mlp(f: Mapping[str, Any], where: str) -> Union[ClippedGLU, MoE]:
    if f.get("kind") == "dense":
        _known(f, ("kind", "ff", "limit"), where)
        return ClippedGLU(_int(f, "ff", where), _float(f, "limit", where, True))
    if f.get("kind") != "moe":
        raise UnsupportedModelError(f"{where}: feed-forward kind {f.get('kind')!r} is not built")
    _known(f, ("kind", "expert", "router", "shared"), where)
    expert, r, shared = _map(f, "expert", where), _map(f, "router", where), f.get("shared") or {}
    for d, keys, what in ((expert, ("ff", "limit"), " expert"), (r, ("experts", "top"), " router"), (shared, ("ff", "limit"), " shared")):
        _known(d, keys, where + what)
    e = MoE(_int(r, "experts", where), _int(r, "top", where), _int(expert, "ff", where), router="chosen",
            limit=_float(expert, "limit", where + " expert", True), shared_ff=_int(shared, "ff", where + " shared") if shared else 0,
            shared_limit=_float(shared, "limit", where + " shared", True) if shared else None, shared_gate=bool(shared))
    if e.top > e.experts or e.experts > 256 or e.top > 32:
        raise UnsupportedModelError(f"{where}: {e.top} of {e.experts} experts (the router takes up to 32 of 256)")
    return e


def _shares(a: Mapping[str, int], where: str) -> None:
    if a["heads"] % a["kv_heads"]:
        raise UnsupportedModelError(f"{where}: {a['heads']} heads do not share {a['kv_heads']} key / value heads evenly")


def _vasosun_window(m: Mapping[str, Any], where: str) -> GroupedAttention:
    _known(m, ("heads", "kv_heads", "dim", "vdim", "scale", "mask", "q_temp"), where)
    mask, t = m.get("mask") or {}, m.get("q_temp") or {}
    _known(mask, ("size",), where + " mask")
    _known(t, ("coef", "every"), where + " q_temp")
    a = {k: _int(m, k, where) for k in ("heads", "kv_heads", "dim", "vdim")}
    _shares(a, where)
    return GroupedAttention(**a, scale=_float(m, "scale", where), qk_norm=False, sink=False, gate=False, log_bias=True,
                            window=_int(mask, "size", where + " mask") if mask else None,
                            growth=_float(t, "coef", where + " q_temp") if t else 0.0, growth_every=_int(t, "every", where + " q_temp") if t else 0)


def _vasosun_latent(m: Mapping[str, Any], where: str) -> LatentAttention:
    _known(m, ("heads", "dim", "vdim", "kv_rank", "q_rank", "rot_dim", "rot", "scale", "kv_from"), where)
    a = {k: _int(m, k, where) for k in ("heads", "dim", "vdim", "kv_rank", "q_rank")}
    r, w = _map(m, "rot", where), where + " rot"
    _known(r, ("dims", "base", "scaling"), w)
    rot = Rotary(_int(r, "dims", w), _float(r, "base", w, True), _yarn(r, w))
    if rot.dims % 2 or rot.dims != _int(m, "rot_dim", where):
        raise UnsupportedModelError(f"{where}: rotation of {rot.dims} of {m['rot_dim']} rotated dimensions")
    return LatentAttention(**a, scale=_float(m, "scale", where), rot=rot, kv_from=None if m.get("kv_from") is None else _int(m, "kv_from", where, 0))


def _vasosun_delta(m: Mapping[str, Any], where: str) -> DeltaRule:
    _known(m, ("heads", "kv_heads", "dim", "vdim", "conv"), where)
    a = {k: _int(m, k, where) for k in ("heads", "kv_heads", "dim", "vdim", "conv")}
    _shares(a, where)
    if a["dim"] > 256 or a["vdim"] > 512:
        raise UnsupportedModelError(f"{where}: the delta rule takes states of up to 256 x 512, got {a['dim']} x {a['vdim']}")
    return DeltaRule(**a)


def _vasosun_mlp(f: Mapping[str, Any], where: str) -> Union[GatedMLP, MoE]:
    if f.get("kind") == "dense":
        _known(f, ("kind", "ff"), where)
        return GatedMLP(_int(f, "ff", where))
    if f.get("kind") != "moe":
        raise UnsupportedModelError(f"{where}: feed-forward kind {f.get('kind')!r} is not built")
    _known(f, ("kind", "expert", "router"), where)
    expert, r = _map(f, "expert", where), _map(f, "router", where)
    _known(expert, ("ff",), where + " expert")
    _known(r, ("experts", "identity", "top"), where + " router")
    e = MoE(_int(r, "experts", where), _int(r, "top", where), _int(expert, "ff", where), gated=False, renormalise=False,
            identity=_int(r, "identity", where, 0) if r.get("identity") is not None else 0)
    if e.top > e.experts + e.identity or e.experts + e.identity > 256 or e.top > 32:
        raise UnsupportedModelError(f"{where}: {e.top} of {e.experts} + {e.identity} experts (the router takes up to 32 of 256)")
    return e


def weight_shapes(cfg: MixedConfig) -> Iterator[Tuple[str, Tuple[int, ...], str]]:
    """(tensor name, shape, kind) of a checkpoint; kind is 'linear', 'embed', 'norm', 'unit' (values in [0, 1)), 'bias', 'scale'
    (positive factors), 'log_a' (logarithms of decay rates), 'dt_bias' (step sizes before softplus) or 'correction'."""
    H, P = cfg.hidden_size, cfg.side_dim
    around = () if cfg.scalar_norms else (H,)
    yield "embed", (cfg.vocab_size, H), "embed"
    if cfg.pairs is not None:
        yield "bigram", (cfg.pairs.buckets + 1, H), "embed"
    if P:
        yield "side.embed", (cfg.vocab_size, cfg.num_layers * P), "embed"
    for i, layer in enumerate(cfg.layers):
        p, m = f"l{i}.", layer.mixer
        yield p + "norm1", around, "norm"
        if cfg.norm_both:
            yield p + "norm1b", around, "norm"
        if cfg.input_taps:
            yield p + "canon1", (H, cfg.input_taps), "linear"
        if cfg.token_shift:
            yield p + "shift", (H,), "unit"
        if isinstance(m, Mamba1):
            yield p + "mix.in", (2 * m.inner, H), "linear"
            yield p + "mix.conv", (m.inner, m.conv), "linear"
            yield p + "mix.conv.b", (m.inner,), "bias"
            yield p + "mix.x", (m.dt_rank + 2 * m.state, m.inner), "linear"
            yield p + "mix.dt", (m.inner, m.dt_rank), "linear"
            yield p + "mix.dt.b", (m.inner,), "dt_bias"
            yield p + "mix.A_log", (m.inner, m.state), "log_a"
            yield p + "mix.D", (m.inner,), "norm"
            vd = m.inner
        elif isinstance(m, DeltaRule):
            vd = m.heads * m.vdim
            for name, rows in (("q", m.kv_heads * m.dim), ("k", m.kv_heads * m.dim), ("v", vd)):
                yield f"{p}mix.{name}", (rows, H), "linear"
                yield f"{p}mix.{name}.conv", (rows, m.conv), "linear"
            yield p + "mix.g", (vd, H), "linear"
            yield p + "mix.b", (m.heads, H), "linear"
            yield p + "mix.a", (m.heads, H), "linear"
            yield p + "mix.A_log", (m.heads,), "log_a"
            yield p + "mix.dt_bias", (m.heads,), "dt_bias"
            yield p + "mix.norm", (m.vdim,), "norm"
        elif getattr(m, "q_rank", 0):
            qd, vd = m.heads * (m.dim + (m.rot.dims if m.rot else 0)), m.heads * m.vdim
            yield p + "mix.dq", (m.q_rank, H), "linear"
            yield p + "mix.dq.norm", (m.q_rank,), "norm"
            yield p + "mix.uq", (qd, m.q_rank), "linear"
        else:
            qd, vd = m.heads * m.dim, m.heads * m.vdim
            yield p + "mix.q", (qd, H), "linear"
        if isinstance(m, GroupedAttention):
            yield p + "mix.k", (m.kv_heads * m.dim, H), "linear"
            yield p + "mix.v", (m.kv_heads * m.vdim, H), "linear"
            if m.qk_norm:
                yield p + "mix.q.norm", (qd if m.norm_all else m.dim,), "norm"
                yield p + "mix.k.norm", (m.kv_heads * m.dim if m.norm_all else m.dim,), "norm"
            if m.conv:
                for name, rows in (("q", qd), ("k", m.kv_heads * m.dim), ("v", m.kv_heads * m.vdim)):
                    yield f"{p}mix.{name}.conv", (rows, m.conv), "linear"
            if m.v_mix:
                yield p + "mix.vmix", (), "unit"
            if m.sink:
                yield p + "mix.sink", (m.heads,), "bias"
            if m.log_bias:
                yield p + "mix.r1", (m.heads,), "scale"
                yield p + "mix.r2", (m.heads,), "scale"
            if m.gate:
                yield p + "mix.g", (m.heads if m.gate_by_head else vd, H), "linear"
        elif isinstance(m, LatentAttention):
            if m.kv_from is None:
                yield p + "mix.dkv", (m.kv_rank + (m.rot.dims if m.rot else 0), H), "linear"
                yield p + "mix.dkv.norm", (m.kv_rank,), "norm"
            yield p + "mix.uk", (m.heads * m.dim, m.kv_rank), "linear"
            yield p + "mix.uv", (vd, m.kv_rank), "linear"
        elif isinstance(m, HGRN2):
            yield p + "mix.f", (qd, H), "linear"
            yield p + "mix.f.b", (qd,), "bias"
            yield p + "mix.lower", (qd,), "unit"
            yield p + "mix.v", (vd, H), "linear"
            yield p + "mix.norm", (m.vdim,), "norm"
        yield p + "mix.o", (H, vd), "linear"
        if layer.mlp is not None:
            yield p + "norm2", around, "norm"
            if cfg.norm_both:
                yield p + "norm2b", around, "norm"
            if cfg.input_taps:
                yield p + "canon2", (H, cfg.input_taps), "linear"
        if isinstance(layer.mlp, MoE):
            f = layer.mlp
            for e, ff in [(f"e{j}", f.ff) for j in range(f.experts)] + ([("shared", f.shared_ff)] if f.shared_ff else []):
                if f.gated:
                    yield f"{p}mlp.{e}.gate", (ff, H), "linear"
                yield f"{p}mlp.{e}.up", (ff, H), "linear"
                yield f"{p}mlp.{e}.down", (H, ff), "linear"
            yield p + "mlp.router", (f.experts + f.identity, H), "linear"
            yield p + ("mlp.router.b" if f.router == "chosen" else "mlp.correction"), (f.experts + f.identity,), "bias" if f.router == "chosen" else "correction"
            if f.shared_gate:
                yield p + "mlp.shared.sg", (1, H), "linear"
        elif layer.mlp is not None:
            if isinstance(layer.mlp, (ClippedGLU, GatedMLP)):
                yield p + "mlp.gate", (layer.mlp.ff, H), "linear"
            yield p + "mlp.up", (layer.mlp.ff, H), "linear"
            yield p + "mlp.down", (H, layer.mlp.ff), "linear"
        if cfg.layer_scale:
            yield p + "ls1", (H,), "scale"
            if layer.mlp is not None:
                yield p + "ls2", (H,), "scale"
        if P:
            yield p + "side.gate", (P, H), "linear"
            yield p + "side.proj", (H, P), "linear"
            yield p + "side.norm", (H,), "norm"
    yield "final.norm", around, "norm"
    if not cfg.tied_head:
        yield "head", (cfg.vocab_size, H), "linear"


def random_weights(cfg: MixedConfig, *, seed: int = 0, dtype=torch.bfloat16, device="cpu", gain: float = 1.0):
    """Weight getter with random values generated on demand (one seeded generator per tensor): linears and embeddings scaled by
    ``gain / sqrt(columns)`` so that activations stay of order one, norms around one, units uniform in [0, 1), layer scales around
    one half, decay rates from 1 to 16 and step sizes from 0.001 to 0.1 (both spread evenly in their logarithms)."""
    table = {name: (idx, shape, kind) for idx, (name, shape, kind) in enumerate(weight_shapes(cfg))}
    dev = torch.device(device)

    def get(name: str) -> torch.Tensor:
        idx, shape, kind = table[name]
        g = torch.Generator(device=dev)
        g.manual_seed(seed * 1_000_003 + idx)
        t = torch.empty(shape, dtype=torch.float32, device=dev)
        if kind == "unit":
            return t.uniform_(0, 1, generator=g).to(dtype)
        if kind == "scale":
            return t.uniform_(0.25, 0.75, generator=g).to(dtype)
        if kind == "log_a":
            return t.uniform_(0.0, math.log(16.0), generator=g).to(dtype)
        if kind == "dt_bias":
            step = t.uniform_(math.log(1e-3), math.log(1e-1), generator=g).exp_()
            return (step + torch.log(-torch.expm1(-step))).to(dtype)
        t.normal_(0.0, 1.0, generator=g)
        if kind == "correction":
            return (t * (0.25 / shape[0])).to(dtype)           # of the order of a softmax score
        if kind == "norm":
            return (1.0 + 0.1 * t).to(dtype)
        if kind == "linear":
            t *= gain / shape[1] ** 0.5
        return t.to(dtype)

    get.names = frozenset(table)  # type: ignore[attr-defined]
    return get


__all__ = ["MixedConfig", "MixedLayer", "LatentAttention", "HGRN2", "GroupedAttention", "Mamba1", "DeltaRule", "Rotary", "YarnScaling", "DenseMLP",
           "GatedMLP", "ClippedGLU", "MoE", "TokenPairs", "weight_shapes", "random_weights"]
