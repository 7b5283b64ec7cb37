"""Serving engine of decoders with per-layer mixers (:mod:`rhinoforge_b200.models.mixed`).

The engine interface is :class:`DecoderEngine`'s: ``prefill`` / ``extend`` / ``run_step`` pack portions of any sequences into one
launch, ``decode`` replays a captured graph, ``generate`` strings them together.  What differs is behind it: the native
executor is the mixed stack (fp32 residual stream, one mixer per layer), the cache a :class:`MixedCache`, and the decode graph
addresses sequences through a slot array, so a scheduler step of single tokens replays it for any subset of the live requests.

Weights are padded once at load to the granularity of the kernels (rows of 8 / 16 values, attention heads to 64 / 128 / 256
for the tcgen05 prefill attention, expert widths to 128 inside the expert banks); padding rows and columns are zero.
"""
from __future__ import annotations

import ctypes as C
import math
import os
from typing import Dict, List, Optional, Sequence

import torch

from .. import _native as N
from ..models.mixed import HGRN2, ClippedGLU, DeltaRule, GatedMLP, GroupedAttention, LatentAttention, Mamba1, MixedConfig, MoE
from ..ops import kernels as K
from ..parallel.tp import TPContext
from .engine import DecoderEngine, WeightGetter
from .errors import RPUBackendError
from .mixed_cache import MixedCache, delta_layout, head_layout, latent_layout, pad_to


def _pad2(w: torch.Tensor, rows: int, cols: int) -> torch.Tensor:
    if tuple(w.shape) == (rows, cols):
        return w
    out = w.new_zeros((rows, cols))
    out[:w.shape[0], :w.shape[1]] = w
    return out


def _pad_heads(w: torch.Tensor, heads: int, true: int, padded: int) -> torch.Tensor:
    """``[heads * true, K]`` -> ``[heads * padded, K]`` with zero rows behind every head."""
    if true == padded:
        return w
    out = w.new_zeros((heads, padded, w.shape[1]))
    out[:, :true] = w.view(heads, true, w.shape[1])
    return out.view(heads * padded, w.shape[1])


class MixedDecoderEngine(DecoderEngine):
    LONG_MIN = 16          # portions of at least this many tokens take the prefill forms of the mixers
    HEAD_ROWS = 64         # rows one logits launch takes

    def __init__(self, cfg: MixedConfig, get_weight: WeightGetter, *, device="cuda", dtype=torch.bfloat16, max_batch: int = 1,
                 max_seq_len: int = 2048, max_prefill_tokens: int = 8192, tp: Optional[TPContext] = None, hist_steps: int = 4096,
                 kv_cache: Optional[MixedCache] = None, kv_pool_tokens: Optional[int] = None):
        if not torch.cuda.is_available():
            raise RPUBackendError("MixedDecoderEngine needs a CUDA device")
        if tp is not None and tp.enabled:
            raise RPUBackendError(f"{cfg.name}: tensor parallelism is not built for decoders with per-layer mixers")
        if dtype not in (torch.float16, torch.bfloat16, torch.float32):
            raise RPUBackendError(f"{cfg.name}: activations are float16, bfloat16 or float32, got {dtype}")
        self.cfg, self.dtype = cfg, dtype
        self.tp = tp or TPContext.single(device)
        self.device = torch.device(self.tp.device if self.tp.device is not None else device)
        self.comm, self.quant = None, None
        self.max_batch = max_batch
        self.max_tokens = max(max_prefill_tokens, max_batch)
        self.fp32 = dtype == torch.float32
        experts = any(isinstance(layer.mlp, MoE) for layer in cfg.layers)      # expert banks exist in the tile-major form only
        self.packed = not self.fp32 and (experts or os.environ.get("RF_PACKED_WEIGHTS", "1") != "0")
        self.long_min = (1 << 30) if self.fp32 else self.LONG_MIN
        self.H = pad_to(cfg.hidden_size, 8)
        self.vocab_local = cfg.vocab_size
        self.vocab_ld = pad_to(cfg.vocab_size, 8)
        self.head_rows = max(max_batch, self.HEAD_ROWS)
        self._keep: List[torch.Tensor] = []
        self.cache = kv_cache if kv_cache is not None else MixedCache(cfg, max_batch, max_seq_len, device=self.device, dtype=dtype,
                                                                      pool_tokens=kv_pool_tokens)
        self._check_cache(self.cache)
        self.handle = None
        self._max_context = max(max_seq_len, self.cache.max_seq_len)
        self._load(get_weight, self._max_context)
        self._bind_arena()
        # ---- decode state, advanced on the device
        i32 = dict(dtype=torch.int32, device=self.device)
        self.ids, self.out_ids = torch.zeros(max_batch, **i32), torch.zeros(self.head_rows, **i32)
        self.out_vals = torch.zeros(self.head_rows, dtype=torch.float32, device=self.device)
        self.pos_stride = 1
        self.pos, self.kv_len = torch.zeros((max_batch, 1), **i32), torch.zeros(max_batch, **i32)
        self.slot = torch.arange(max_batch, **i32)
        self.logits = torch.zeros((max_batch, self.vocab_ld), dtype=dtype, device=self.device)
        self.step = torch.zeros(1, **i32)
        self.hist_steps = hist_steps
        self.hist = torch.zeros((hist_steps, max_batch), **i32)
        self.graphs: Dict[int, torch.cuda.CUDAGraph] = {}
        self.batch = 0
        self._hb = self._host_steps = 0
        self.heartbeat_every = 0

    def _bind_arena(self) -> None:
        lib = N.lib()
        nbytes = lib.rf_mixed_arena_bytes(self.handle)
        self.arena = torch.zeros(nbytes + 1024, dtype=torch.uint8, device=self.device)
        base = (self.arena.data_ptr() + 1023) // 1024 * 1024
        N.check(lib.rf_mixed_bind_arena(self.handle, C.c_void_p(base), C.c_uint64(nbytes)), "rf_mixed_bind_arena")
        off = lib.rf_mixed_status_ptr(self.handle) - self.arena.data_ptr()
        self.status = self.arena[off:off + 32].view(torch.int32)

    # ------------------------------------------------------------------ weights
    def _f32(self, t: torch.Tensor, n: int, fill: float = 0.0) -> torch.Tensor:
        out = torch.full((n,), fill, dtype=torch.float32, device=self.device)
        out[:t.numel()] = t.reshape(-1).to(self.device, torch.float32)
        self._keep.append(out)
        return out

    def _linear(self, w: torch.Tensor, sections: int = 1) -> torch.Tensor:
        t = w.to(self.device, self.dtype).contiguous()
        if self.packed:
            t = K.pack_weight(t, sections)
        self._keep.append(t)
        return t

    def _plain(self, w: torch.Tensor) -> torch.Tensor:
        t = w.to(self.device, self.dtype).contiguous()
        self._keep.append(t)
        return t

    def _load(self, get: WeightGetter, max_context: int) -> None:
        cfg, lib, H = self.cfg, N.lib(), self.H
        g = lambda name: get(name).to(self.device)
        P = pad_to(cfg.side_dim, 8)
        V, L = cfg.vocab_size, cfg.num_layers
        self.embed = self._plain(_pad2(g("embed"), V, H))
        self.side_table = None
        if P:
            side = g("side.embed").view(V, L, cfg.side_dim)
            if P != cfg.side_dim:
                wide = side.new_zeros((V, L, P))
                wide[:, :, :cfg.side_dim] = side
                side = wide
            self.side_table = self._plain(side.reshape(V, L * P))
        # norms with one weight for all coordinates are spread over the row
        weight = lambda name: g(name).reshape(-1).expand(cfg.hidden_size) if cfg.scalar_norms else g(name)
        self.final_norm = self._f32(weight("final.norm"), H)
        lm = self._linear(_pad2(self.embed if cfg.tied_head else g("head"), self.vocab_ld, H))
        self._rotations: Dict[object, tuple] = {}
        self._v_mixing = False                  # has a value-mixing layer been loaded already?
        sc = N.RfMixedConfig()
        sc.layers, sc.hidden, sc.hidden_true, sc.vocab, sc.vocab_ld = L, H, cfg.hidden_size, V, self.vocab_ld
        sc.dtype = 2 if self.fp32 else K.dtype_code(self.dtype)
        sc.max_tokens, sc.max_seqs, sc.max_seq_len = self.max_tokens, self.max_batch, max_context
        sc.side_dim, sc.side_ld, sc.eps = P, L * P, cfg.rms_eps
        sc.weights_packed, sc.long_min = int(self.packed), self.long_min
        sc.embed, sc.final_norm, sc.w_lm = (t.data_ptr() for t in (self.embed, self.final_norm, lm))
        sc.side_table = None if self.side_table is None else self.side_table.data_ptr()
        sc.embed_scale, sc.norm_after = cfg.embed_scale, int(cfg.norm_after)
        sc.residual_mult, sc.logit_softcap = cfg.residual_mult, cfg.logit_softcap or 0.0
        if cfg.pairs is not None:
            b = cfg.pairs
            sc.pair_table = self._plain(_pad2(g("bigram"), b.buckets + 1, H)).data_ptr()
            sc.pair_buckets, sc.pair_mul_prev, sc.pair_mul_cur = b.buckets, b.mul_prev, b.mul_cur
        sc.input_taps = cfg.input_taps
        h = lib.rf_mixed_create(C.byref(sc))
        if h < 0:
            N.check(-1, "rf_mixed_create")
        self.handle = C.c_int64(h)
        for i, layer in enumerate(cfg.layers):
            m, p = layer.mixer, f"l{i}."
            lw = N.RfMixedLayer()
            lw.heads = getattr(m, "heads", 0)
            # layer scales act on the normalised outputs: one factor with the norm's weight
            norm = lambda name, scale: g(p + name).float() * g(p + scale).float() if cfg.layer_scale else weight(p + name)
            lw.norm1 = self._f32(norm("norm1", "ls1"), H).data_ptr()
            if cfg.token_shift:
                lw.shift = self._f32(g(p + "shift"), H).data_ptr()
            sublayers = 1 if layer.mlp is None else 2
            if cfg.norm_both:
                for n in range(sublayers):
                    setattr(lw, f"norm{n + 1}b", self._f32(weight(f"{p}norm{n + 1}b"), H).data_ptr())
            if cfg.input_taps:
                for n in range(sublayers):
                    taps = _pad2(g(f"{p}canon{n + 1}").t().float(), cfg.input_taps, H)
                    lw.input_conv[n] = self._f32(taps, taps.numel()).data_ptr()
            load = {DeltaRule: self._load_delta, LatentAttention: self._load_latent, HGRN2: self._load_hgrn2, GroupedAttention: self._load_grouped, Mamba1: self._load_mamba1}
            load[type(m)](lw, m, g, p + "mix.")
            lw.st = self.cache.layer_state(i)
            if layer.mlp is not None:
                lw.norm2 = self._f32(norm("norm2", "ls2"), H).data_ptr()
            if isinstance(layer.mlp, MoE):
                self._load_moe(lw, layer.mlp, g, p + "mlp.")
            elif isinstance(layer.mlp, (ClippedGLU, GatedMLP)):
                f = layer.mlp
                lw.inter, lw.act = pad_to(f.ff, 8), 2
                if isinstance(f, ClippedGLU):
                    lw.act, lw.act_limit, lw.act_alpha = 1, f.limit, f.alpha
                lw.w_up = self._linear(torch.cat([_pad2(g(f"{p}mlp.{x}"), lw.inter, H) for x in ("gate", "up")], 0), 2).data_ptr()
                lw.w_down = self._linear(_pad2(g(p + "mlp.down"), H, lw.inter)).data_ptr()
            elif layer.mlp is not None:
                lw.inter, lw.act = pad_to(layer.mlp.ff, 8), 0
                lw.w_up = self._linear(_pad2(g(p + "mlp.up"), lw.inter, H)).data_ptr()
                lw.w_down = self._linear(_pad2(g(p + "mlp.down"), H, lw.inter)).data_ptr()
            if P:
                lw.side_gate = self._linear(_pad2(g(p + "side.gate"), P, H)).data_ptr()
                lw.side_proj = self._linear(_pad2(g(p + "side.proj"), H, P)).data_ptr()
                lw.side_norm = self._f32(g(p + "side.norm"), H).data_ptr()
            N.check(lib.rf_mixed_set_layer(self.handle, i, C.byref(lw)), "rf_mixed_set_layer")
        torch.cuda.empty_cache()

    def _load_latent(self, lw, m: LatentAttention, g, p: str) -> None:
        H = self.H
        R, P = latent_layout(m)
        rot, plain = m.rot.dims if m.rot is not None else 0, pad_to(m.dim, 8)
        key = plain + pad_to(rot, 8)                          # a head: plain dimensions, then rotated ones
        # heads of the tcgen05 prefill attention; without one (fp32, very wide heads) every row attends in the latent space
        hd, hv = K.latent_heads(key, m.vdim) if not self.fp32 and m.scale > 0 else (0, 0)
        D, VD = hd or key, hv or pad_to(m.vdim, 8)
        lw.mixer, lw.dim, lw.vdim, lw.vdim_true = 0, D, VD, m.vdim
        lw.rank, lw.rank_true, lw.window, lw.scale, lw.expand_hd = R, m.kv_rank, m.window or 0, m.scale, hd
        lw.plain, lw.rot, lw.rot_pad, lw.shares = plain, rot, P, int(m.kv_from is not None)
        QR = lw.q_rank = pad_to(m.q_rank, 8)
        q = g(p + ("uq" if QR else "q"))
        q = _pad2(q, q.shape[0], QR or H).view(m.heads, m.dim + rot, QR or H)
        heads = q.new_zeros((m.heads, D, QR or H))
        heads[:, :m.dim], heads[:, plain:plain + rot] = q[:, :m.dim], q[:, m.dim:]
        q = heads.view(m.heads * D, QR or H)
        if QR:
            lw.q_rank_true, lw.q_latent_norm, lw.w_uq = m.q_rank, self._f32(g(p + "dq.norm"), QR).data_ptr(), self._linear(q).data_ptr()
            q = _pad2(g(p + "dq"), QR, H)
        parts = [q]
        if m.kv_from is None:
            dkv = g(p + "dkv")
            parts += [_pad2(dkv[:m.kv_rank], R, H)] + ([_pad2(dkv[m.kv_rank:], P, H)] if rot else [])
            lw.latent_norm = self._f32(g(p + "dkv.norm"), R).data_ptr()
        w_in = torch.cat(parts, 0)
        lw.in_dim = w_in.shape[0]
        lw.w_in = self._linear(w_in).data_ptr()
        if rot:
            cos, sin = self._rotation(m.rot)
            lw.cos, lw.sin = cos.data_ptr(), sin.data_ptr()
        uk = _pad_heads(_pad2(g(p + "uk"), m.heads * m.dim, R), m.heads, m.dim, plain)
        uv = _pad_heads(_pad2(g(p + "uv"), m.heads * m.vdim, R), m.heads, m.vdim, VD)
        lw.w_absorb = self._plain(uk.view(m.heads, plain, R).transpose(1, 2)).data_ptr()
        lw.w_unabsorb = self._plain(uv).data_ptr()
        if hd:
            # keys of a head are a map of the latent and a copy of the rotated part, values a map of the latent
            keys = uk.new_zeros((m.heads, hd, R + P))
            keys[:, :plain, :R] = uk.view(m.heads, plain, R)
            for i in range(rot):
                keys[:, plain + i, R + i] = 1.0
            lw.w_expand = self._linear(torch.cat((keys.view(m.heads * hd, R + P), _pad2(uv, m.heads * hv, R + P)), 0)).data_ptr()
        o = g(p + "o")
        o = _pad_heads(o.t().contiguous(), m.heads, m.vdim, VD).t()
        lw.w_o, lw.out_dim = self._linear(_pad2(o, H, m.heads * VD)).data_ptr(), m.heads * VD

    def _rotation(self, rot):
        """cos and sin tables over the longest context, one pair per distinct rotation."""
        if rot not in self._rotations:
            self._rotations[rot] = rot.tables(self._max_context, self.device)
        return self._rotations[rot]

    def _load_grouped(self, lw, m: GroupedAttention, g, p: str) -> None:
        H = self.H
        hd, tensor_core = head_layout(m, self.dtype)
        lw.mixer, lw.dim, lw.vdim, lw.dim_true, lw.vdim_true = 2, hd, hd, m.dim, m.vdim
        lw.kv_heads, lw.tensor_core, lw.chunk, lw.scale = m.kv_heads, int(tensor_core), m.chunk or 0, m.scale
        lw.window, lw.keep_first, lw.norm_all, lw.gate_by_head, lw.conv_taps = m.window or 0, m.keep_first, int(m.norm_all), int(m.gate_by_head), m.conv
        rows = lambda name, heads, true: _pad_heads(_pad2(g(p + name), heads * true, H), heads, true, hd)
        parts = [rows("q", m.heads, m.dim), rows("k", m.kv_heads, m.dim), rows("v", m.kv_heads, m.vdim)]
        if m.gate:
            parts.append(_pad2(g(p + "g"), pad_to(m.heads, 8), H) if m.gate_by_head else rows("g", m.heads, m.vdim))
            lw.gated = 1
        w_in = torch.cat(parts, 0)
        lw.in_dim = w_in.shape[0]
        lw.w_in = self._linear(w_in).data_ptr()
        if m.qk_norm:
            heads = (m.heads, m.kv_heads) if m.norm_all else (1, 1)
            lw.q_norm, lw.k_norm = (self._f32(_fill_heads(g(p + x).float(), n, m.dim, hd, 0.0), n * hd).data_ptr()
                                    for x, n in zip(("q.norm", "k.norm"), heads))
        if m.sink or m.unit_sink:
            lw.sink = self._f32(g(p + "sink") if m.sink else torch.zeros(m.heads), m.heads).data_ptr()
        if m.distance_bias:
            lw.slopes = self._f32(m.slopes(), m.heads).data_ptr()
        if m.log_bias:
            lw.slopes, lw.rates = self._f32(g(p + "r1"), m.heads).data_ptr(), self._f32(g(p + "r2"), m.heads).data_ptr()
        lw.growth, lw.growth_every = m.growth, m.growth_every
        if m.conv:
            taps = torch.cat([_pad_heads(g(f"{p}{x}.conv").float(), n, d, hd)
                              for x, n, d in (("q", m.heads, m.dim), ("k", m.kv_heads, m.dim), ("v", m.kv_heads, m.vdim))], 0)
            lw.conv_w = self._f32(taps.t().contiguous(), taps.numel()).data_ptr()
        if m.rot is not None:
            cos, sin = self._rotation(m.rot)
            lw.rot_dims, lw.cos, lw.sin = m.rot.dims, cos.data_ptr(), sin.data_ptr()
        if m.v_mix:
            lw.v_role = 2 if self._v_mixing else 1
            lw.v_lambda = float(g(p + "vmix")) if self._v_mixing else 0.0
            self._v_mixing = True
        o = _pad_heads(g(p + "o").t().contiguous(), m.heads, m.vdim, hd).t()
        lw.w_o, lw.out_dim = self._linear(_pad2(o, H, m.heads * hd)).data_ptr(), m.heads * hd

    def _load_delta(self, lw, m: DeltaRule, g, p: str) -> None:
        H = self.H
        D, V = delta_layout(m, self.dtype)
        lw.mixer, lw.dim, lw.vdim, lw.dim_true, lw.vdim_true, lw.kv_heads, lw.taps = 4, D, V, m.dim, m.vdim, m.kv_heads, m.conv
        parts = (("q", m.kv_heads, m.dim, D), ("k", m.kv_heads, m.dim, D), ("v", m.heads, m.vdim, V), ("g", m.heads, m.vdim, V))
        w_in = [_pad_heads(_pad2(g(p + x), n * true, H), n, true, padded) for x, n, true, padded in parts]
        w_in += [_pad2(g(p + x), pad_to(m.heads, 8), H) for x in ("b", "a")]
        w_in = torch.cat(w_in, 0)
        lw.w_in, lw.in_dim = self._linear(w_in).data_ptr(), w_in.shape[0]
        taps = torch.cat([_pad_heads(g(f"{p}{x}.conv").float(), n, true, padded) for x, n, true, padded in parts[:3]], 0)
        lw.conv_w = self._f32(taps.t().contiguous(), taps.numel()).data_ptr()
        lw.rate = self._f32(g(p + "A_log").double().exp(), m.heads).data_ptr()
        lw.dt_bias, lw.head_norm = self._f32(g(p + "dt_bias"), m.heads).data_ptr(), self._f32(g(p + "norm"), V).data_ptr()
        o = _pad_heads(g(p + "o").t().contiguous(), m.heads, m.vdim, V).t()
        lw.w_o, lw.out_dim = self._linear(_pad2(o, H, m.heads * V)).data_ptr(), m.heads * V

    def _load_mamba1(self, lw, m: Mamba1, g, p: str) -> None:
        H, I, S, R = self.H, pad_to(m.inner, 8), pad_to(m.state, 8), pad_to(m.dt_rank, 8)
        lw.mixer, lw.inner, lw.states, lw.dt_rank, lw.taps = 3, I, S, R, m.conv
        w_in = g(p + "in")
        w_in = torch.cat([_pad2(w_in[:m.inner], I, H), _pad2(w_in[m.inner:], I, H)], 0)
        lw.w_in, lw.in_dim = self._linear(w_in).data_ptr(), 2 * I
        lw.conv_w = self._f32(_pad2(g(p + "conv").t().float(), m.conv, I), m.conv * I).data_ptr()
        lw.conv_b = self._f32(g(p + "conv.b"), I).data_ptr()
        dt, b, c = g(p + "x").split((m.dt_rank, m.state, m.state), 0)
        lw.w_x = self._linear(torch.cat((_pad2(dt, R, I), _pad2(b, S, I), _pad2(c, S, I)), 0)).data_ptr()
        w_dt = _pad2(g(p + "dt"), I, R)
        lw.w_dt, lw.w_dt_rows = self._linear(w_dt).data_ptr(), self._plain(w_dt).data_ptr()
        lw.dt_bias = self._f32(g(p + "dt.b"), I).data_ptr()
        a2 = g(p + "A_log").double().exp() * (-1.0 / math.log(2.0))       # the kernels raise two to these
        lw.a2 = self._f32(_pad2(a2.float(), I, S), I * S).data_ptr()
        lw.d_skip = self._f32(g(p + "D"), I).data_ptr()
        lw.w_o, lw.out_dim = self._linear(_pad2(g(p + "o"), H, I)).data_ptr(), I

    def _load_moe(self, lw, f: MoE, g, p: str) -> None:
        """Expert banks: gates then ups of all experts stacked along the rows; downs one behind the other along the columns in
        16 bits (tile-major image), along the rows in 32."""
        H, I = self.H, pad_to(f.ff, 8)
        B = I if self.fp32 else pad_to(f.ff, 128)
        lw.inter, lw.bank_inter, lw.act = I, B, 0
        lw.experts, lw.top, lw.groups, lw.keep = f.experts, f.top, f.groups, f.keep
        lw.score_fn, lw.norm_topk, lw.route_scale = {"corrected": 1, "chosen": 2}[f.router], int(f.renormalise), 1.0
        lw.identity = f.identity
        if f.limit is not None:
            lw.act, lw.act_limit, lw.act_alpha, lw.shared_limit = 1, f.limit, f.alpha, f.shared_limit or 0.0
        if not f.gated:
            lw.act = 3
        names = ("gate", "up") if f.gated else ("up",)
        up = torch.zeros((len(names), f.experts, B, H), dtype=self.dtype, device=self.device)
        down = torch.zeros((f.experts, H, B), dtype=self.dtype, device=self.device)
        for e in range(f.experts):
            for i, name in enumerate(names):
                w = g(f"{p}e{e}.{name}")
                up[i, e, :f.ff, :w.shape[1]] = w
            w = g(f"{p}e{e}.down")
            down[e, :w.shape[0], :f.ff] = w
        lw.w_up = self._linear(up.view(len(names) * f.experts * B, H), len(names)).data_ptr()
        lw.w_down = self._linear(down.view(f.experts * H, B) if self.fp32 else down.transpose(0, 1).reshape(H, f.experts * B)).data_ptr()
        router = _pad2(g(p + "router"), f.experts + f.identity, H)
        if f.shared_gate:
            router, lw.shared_gate = torch.cat((router, _pad2(g(p + "shared.sg"), 1, H)), 0), 1
        lw.router = self._plain(router).data_ptr()
        lw.correction = self._f32(g(p + ("router.b" if f.router == "chosen" else "correction")), f.experts + f.identity).data_ptr()
        if f.shared_ff:
            S = lw.shared_inter = pad_to(f.shared_ff, 8)
            gate_up = torch.cat((_pad2(g(p + "shared.gate"), S, H), _pad2(g(p + "shared.up"), S, H)), 0)
            lw.shared_up = self._linear(gate_up, 2).data_ptr()
            lw.shared_down = self._linear(_pad2(g(p + "shared.down"), H, S)).data_ptr()

    def _load_hgrn2(self, lw, m: HGRN2, g, p: str) -> None:
        H, D, VD = self.H, pad_to(m.dim, 8), pad_to(m.vdim, 8)
        lw.mixer, lw.dim, lw.vdim, lw.vdim_true = 1, D, VD, m.vdim
        head_rows = lambda name, true, padded: _pad_heads(_pad2(g(p + name), m.heads * true, H), m.heads, true, padded)
        w_in = torch.cat((head_rows("q", m.dim, D), head_rows("f", m.dim, D), head_rows("v", m.vdim, VD)), 0)
        lw.in_dim = w_in.shape[0]
        lw.w_in = self._linear(w_in).data_ptr()
        per_head = lambda t, fill: _fill_heads(t.float(), m.heads, m.dim, D, fill)
        lw.f_bias = self._f32(per_head(g(p + "f.b"), 0.0), m.heads * D).data_ptr()
        lw.lower = self._f32(per_head(g(p + "lower"), 1.0), m.heads * D).data_ptr()    # padding channels keep their (zero) state
        lw.head_norm = self._f32(g(p + "norm"), VD).data_ptr()
        o = _pad_heads(g(p + "o").t().contiguous(), m.heads, m.vdim, VD).t()
        lw.w_o, lw.out_dim = self._linear(_pad2(o, H, m.heads * VD)).data_ptr(), m.heads * VD

    # ------------------------------------------------------------------ cache
    def _check_cache(self, cache) -> None:
        if not isinstance(cache, MixedCache) or cache.cfg != self.cfg or cache.dtype != self.dtype or cache.batch_size > self.max_batch:
            raise RPUBackendError(f"{self.cfg.name}: the cache was not made for this model (dtype {getattr(cache, 'dtype', None)}, batch "
                                  f"{getattr(cache, 'batch_size', None)}; engine {self.dtype}, max_batch {self.max_batch})")

    def make_cache(self, batch_size: int, max_seq_len: int, *, pool_tokens: Optional[int] = None):
        """A cache object for this model (``RPUCache.from_model`` ends here)."""
        from ..api.cache import RPUMixedCache
        return RPUMixedCache(self.cfg, batch_size, max_seq_len, device=self.device, dtype=self.dtype, pool_tokens=pool_tokens)

    def bind_cache(self, cache) -> None:
        if cache is self.cache:
            return
        self._check_cache(cache)
        for i in range(self.cfg.num_layers):
            N.check(N.lib().rf_mixed_set_state(self.handle, i, C.byref(cache.layer_state(i))), "rf_mixed_set_state")
        self.cache = cache
        self.graphs.clear()
        self.batch = 0
        if cache.max_seq_len > self._max_context:
            # attention without a window may have to expand every cached row of a portion's sequence
            self._max_context = cache.max_seq_len
            if self._rotations:
                torch.cuda.synchronize()
                self._rotations.clear()
                for i, layer in enumerate(self.cfg.layers):
                    if getattr(layer.mixer, "rot", None) is not None:
                        N.check(N.lib().rf_mixed_set_rotation(self.handle, i, *(C.c_void_p(t.data_ptr()) for t in self._rotation(layer.mixer.rot))),
                                "rf_mixed_set_rotation")
            if any(isinstance(layer.mixer, LatentAttention) and layer.mixer.window is None for layer in self.cfg.layers):
                torch.cuda.synchronize()
                N.check(N.lib().rf_mixed_set_context(self.handle, self._max_context), "rf_mixed_set_context")
                self._bind_arena()

    def reset(self) -> None:
        for s in range(self.cache.batch_size):
            self.cache.release(s)
        self.step.zero_()
        self.batch = 0

    # ------------------------------------------------------------------ launches
    def _rows(self, r: "N.RfRows", num_seqs: int) -> None:
        r.page_table, r.pt_stride, r.num_seqs = self.cache.page_table.data_ptr(), self.cache.page_table.stride(0), num_seqs

    def _logits_of(self, row_idx: Optional[torch.Tensor], rows: int, out: torch.Tensor) -> None:
        N.check(N.lib().rf_mixed_head(self.handle, C.c_void_p(None if row_idx is None else row_idx.data_ptr()), rows,
                                      C.c_void_p(self.out_ids.data_ptr()), C.c_void_p(self.out_vals.data_ptr()),
                                      C.c_void_p(out.data_ptr()), self._stream()), "rf_mixed_head")

    def _prefill_chunk(self, ch, prompts, lens, starts, first, logits_all, inputs_embeds, positions3, deepstack=None,
                       row_logits=None, slots=None, taps: Optional[torch.Tensor] = None) -> None:
        if inputs_embeds is not None or positions3 is not None or deepstack is not None:
            raise RPUBackendError(f"{self.cfg.name} takes token ids only")
        ch = sorted(ch, key=lambda c: c[2] >= self.long_min)          # short portions first (stable)
        T, n = sum(c[2] for c in ch), len(ch)
        seq_meta = torch.empty((4, n), dtype=torch.int32)             # q_start, q_len, first position, slot
        tok_meta = torch.empty((3, T), dtype=torch.int32)             # sequence, position, token id
        o = 0
        for j, (s, off, cnt) in enumerate(ch):
            pos0 = starts[s] + off
            seq_meta[0, j], seq_meta[1, j], seq_meta[2, j], seq_meta[3, j] = o, cnt, pos0, slots[s]
            tok_meta[0, o:o + cnt] = j
            tok_meta[1, o:o + cnt] = torch.arange(pos0, pos0 + cnt, dtype=torch.int32)
            tok_meta[2, o:o + cnt] = prompts[s][off:off + cnt].to("cpu", torch.int32)
            o += cnt
        sm, tm = seq_meta.pin_memory().to(self.device, non_blocking=True), tok_meta.pin_memory().to(self.device, non_blocking=True)
        short = [c for c in ch if c[2] < self.long_min]
        f = N.RfMixedForward()
        f.rows.q_start, f.rows.q_len, f.rows.slot = sm[0].data_ptr(), sm[1].data_ptr(), sm[3].data_ptr()
        f.rows.seq_of_row, f.rows.pos, f.ids = tm[0].data_ptr(), tm[1].data_ptr(), tm[2].data_ptr()
        self._rows(f.rows, n)
        f.tokens, f.short_seqs, f.short_rows, f.decode = T, len(short), sum(c[2] for c in short), 0
        f.max_kv = max(starts[s] + off + cnt for s, off, cnt in (short or ch))
        f.h_q_len, f.h_pos0 = seq_meta[1].data_ptr(), seq_meta[2].data_ptr()
        f.taps = None if taps is None else taps.data_ptr()
        N.check(N.lib().rf_mixed_forward(self.handle, C.byref(f), self._stream()), "rf_mixed_forward")
        # rows whose logits are wanted, then the last rows of the prompts that end in this chunk (for the next token)
        jobs, row0 = [], {}
        o = 0
        for (s, off, cnt) in ch:
            row0[s] = o
            if row_logits is not None:
                jobs += [(o + r, s, True) for r in self._wanted_rows(row_logits, s, off, cnt, lens[s])]
            if off + cnt == lens[s]:
                jobs.append((o + cnt - 1, s, False))
            o += cnt
        for b0 in range(0, len(jobs), self.head_rows):
            sub = jobs[b0:b0 + self.head_rows]
            idx = torch.tensor([r for r, _, _ in sub], dtype=torch.int32).pin_memory().to(self.device, non_blocking=True)
            lg = torch.empty((len(sub), self.vocab_ld), dtype=self.dtype, device=self.device)
            self._logits_of(idx, len(sub), lg)
            for k, (_, s, wanted) in enumerate(sub):
                if wanted:
                    row_logits["out"][s].append(lg[k:k + 1, :self.vocab_local])
                else:
                    first[s:s + 1].copy_(self.out_ids[k:k + 1])
                    if logits_all is not None:
                        logits_all[s].copy_(lg[k, :self.vocab_local])

    @torch.no_grad()
    def residual_taps(self, tokens: torch.Tensor) -> torch.Tensor:
        """The fp32 residual stream after every layer ``[layers, tokens, hidden]`` of one prompt run from position 0 in slot 0
        (diagnostics and tests)."""
        n = int(tokens.numel())
        self.reset()
        self.cache.ensure(0, n)
        self.cache.sync_table()
        taps = torch.zeros((self.cfg.num_layers, n, self.H), dtype=torch.float32, device=self.device)
        first = torch.zeros(1, dtype=torch.int32, device=self.device)
        self._prefill_chunk([(0, 0, n)], [tokens], [n], [0], first, None, None, None, slots=[0], taps=taps)
        self.cache.release(0)
        return taps[:, :, :self.cfg.hidden_size]

    def _decode_step(self, B: int, logits_out: Optional[torch.Tensor] = None) -> None:
        f = N.RfMixedForward()
        f.ids, f.rows.pos, f.rows.slot = self.ids.data_ptr(), self.pos.data_ptr(), self.slot.data_ptr()
        self._rows(f.rows, B)
        f.tokens = f.short_seqs = f.short_rows = B
        f.decode, f.max_kv = 1, self.cache.max_seq_len
        N.check(N.lib().rf_mixed_forward(self.handle, C.byref(f), self._stream()), "rf_mixed_forward")
        self._logits_of(None, B, self.logits)
        N.check(N.lib().rf_decode_advance(C.c_void_p(self.pos.data_ptr()), 1, C.c_void_p(self.kv_len.data_ptr()), B,
                                          C.c_void_p(self.out_ids.data_ptr()), C.c_void_p(self.ids.data_ptr()),
                                          C.c_void_p(self.hist.data_ptr()), C.c_void_p(self.step.data_ptr()),
                                          self.hist_steps, self._stream()), "rf_decode_advance")

    def _decode_state(self) -> List[torch.Tensor]:
        return [self.pos, self.kv_len, self.ids, self.step] + self.cache.state_tensors()

    # ------------------------------------------------------------------ scheduler step
    @torch.no_grad()
    def run_step(self, tokens: Sequence[torch.Tensor], slots: Sequence[int], want: Sequence[Sequence[int]]):
        """See :meth:`DecoderEngine.run_step`.  A step of single tokens replays the decode graph of its batch size."""
        if any(int(t.numel()) != 1 for t in tokens) or len(tokens) > self.max_batch:
            return super().run_step(tokens, slots, want)
        cache, B = self.cache, len(tokens)
        slots = [int(s) for s in slots]
        if len(set(slots)) != B or any(not 0 <= s < cache.batch_size for s in slots):
            raise RPUBackendError(f"slots {slots} are not {B} different slots of a cache with {cache.batch_size}")
        for s in slots:
            cache.check_fits(s, 1)
        for s in slots:
            cache.ensure(s, int(cache.lengths[s]) + 1)
        cache.sync_table()
        host = torch.tensor([[int(t) for t in tokens], [int(cache.lengths[s]) for s in slots], slots], dtype=torch.int32).pin_memory()
        dev = host.to(self.device, non_blocking=True)
        self.ids[:B].copy_(dev[0])
        self.pos[:B, 0].copy_(dev[1])
        self.slot[:B].copy_(dev[2])
        self.batch = 0
        self.capture(B)
        self.graphs[B].replay()
        for s in slots:
            cache.lengths[s] += 1
        lg = self.logits[:B, :self.vocab_local].clone()
        return self.out_ids[:B].clone(), [lg[i:i + 1].expand(len(w), -1) for i, w in enumerate(want)]

    def extend(self, tokens, **kw):
        out = super().extend(tokens, **kw)
        if self.batch:
            self.slot.copy_(torch.arange(self.max_batch, dtype=torch.int32, device=self.device))
        return out

    def close(self) -> None:
        torch.cuda.synchronize()
        self.graphs.clear()
        if getattr(self, "handle", None) is not None:
            N.lib().rf_mixed_destroy(self.handle)
            self.handle = None
        if getattr(self, "cache", None) is not None:
            self.cache.close()


def _fill_heads(t: torch.Tensor, heads: int, true: int, padded: int, fill: float) -> torch.Tensor:
    out = torch.full((heads, padded), fill, dtype=t.dtype, device=t.device)
    out[:, :true] = t.view(heads, true)
    return out.reshape(-1)


__all__ = ["MixedDecoderEngine"]
