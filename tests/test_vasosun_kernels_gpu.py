"""Kernels of the Vasosun decoders, each against the plain formulation of its mechanism."""
import math

import pytest
import torch

import _vasosun_oracle as oracle
from rhinoforge_b200.models.mixed import Rotary, YarnScaling
from test_kuzupel_kernels_gpu import BF16, DTYPES, F16, F32, K, attend, cached, close, gen, i32, pack, page_table, widen

pytestmark = pytest.mark.gpu


# ------------------------------------------------------------------------------------------------ residual stream
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H", [40, 1024, 4096, 8200])
@pytest.mark.parametrize("n", [3, 700])
def test_identity_weights_add_the_input_to_the_picked_rows(dtype, H, n):
    rnd, picks = gen(1), 3
    x, y, own, sw = rnd(n, H).float(), rnd(n * picks, H).to(dtype), rnd(n, H).to(dtype), rnd(n).float()
    yw, w = rnd(H).float(), rnd(H).float()
    slots = torch.randperm(n * picks, generator=torch.Generator().manual_seed(3)).to(torch.int32).view(n, picks)
    slots[1] = -1                                                                      # a token whose picks are all identities
    total = torch.where((slots >= 0)[..., None], y.double()[slots.clamp(min=0).long()], torch.zeros((), dtype=torch.float64)).sum(1)
    total = total + sw.double()[:, None] * own.double()
    r = K().rows(torch.arange(n, dtype=torch.int32, device="cuda"))
    xo, h, _ = K().stream_norm(x.cuda(), r, dtype=dtype, eps=1e-4, norm_w=w.cuda(), y=y.cuda(), y_norm_w=yw.cuda(), y_slots=slots.cuda(),
                               y_self=(own.cuda(), sw.cuda()))
    want = x.double() + oracle.rms(total, 1e-4, yw.double())
    close(xo, want, F32, 8.0)
    close(h, oracle.rms(want, 1e-4, w.double()), dtype, 4.0)


@pytest.mark.parametrize("taps", [1, 2, 3, 4, 7, 19])
@pytest.mark.parametrize("H", [40, 1024, 8192])
def test_input_convolution_fused_and_behind_the_norm(taps, H):
    """Portions convolve behind the stream step, decode rows inside it, over the same carried rows; both against whole sequences."""
    rnd, eps, slots, total = gen(2), 1e-4, [2, 0], (61, 33)
    w, cw = (1 + 0.1 * rnd(H)).float(), (rnd(H, taps) / taps).float()
    x = [rnd(n, H).float() for n in total]
    state = torch.full((3, max(taps - 1, 1), H), 9.0, dtype=BF16, device="cuda")       # left over by earlier requests
    taps_first, got, at = cw.t().contiguous().cuda(), [[], []], [0, 0]
    for lens in ([1, 1], [1, 2], [17, 1], [1, 1], [1, 0], [2, 20], [1, 1], [1, 1], [30, 3]):
        live = [i for i in range(2) if lens[i]]
        d, _, _ = pack([lens[i] for i in live], [at[i] for i in live], [slots[i] for i in live])
        rows = torch.cat([x[i][at[i]:at[i] + lens[i]] for i in live]).cuda()
        if max(lens) == 1:
            _, h, _ = K().stream_norm(rows, K().rows(pos=d["pos"], slot=d["slot"]), dtype=BF16, eps=eps, norm_w=w.cuda(), conv=(taps_first, state))
        else:
            _, h, _ = K().stream_norm(rows, K().rows(**d), dtype=BF16, eps=eps, norm_w=w.cuda())
            h = K().conv_silu(h, taps_first, None, state, K().rows(**d), max_q_len=max(lens), add=True)
        o = 0
        for i in live:
            got[i].append(h[o:o + lens[i]])
            at[i], o = at[i] + lens[i], o + lens[i]
    for i in range(2):
        h = oracle.rms(x[i][:at[i]].double(), eps, w.double())
        close(torch.cat(got[i]), h + oracle.causal_convolution(h, cw.double()), BF16, 3.0)
    assert (state[1] == 9.0).all()


# ------------------------------------------------------------------------------------------------ window attention
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("coef,every", [(0.7, 1), (0.5, 16), (2.0, 100), (-0.1, 40)])
def test_queries_grow_with_their_position(dtype, coef, every):
    lens, pos0, slots, heads, kv, dim, hd = [1, 9, 2, 17], [99, 0, 15, 30], [3, 1, 0, 4], 4, 2, 20, 24
    d, pos, _ = pack(lens, pos0, slots)
    n, rnd = sum(lens), gen(3)
    q, k, v = rnd(n, heads, dim).to(dtype), rnd(n, kv, dim).to(dtype), rnd(n, kv, dim).to(dtype)
    rows = torch.cat([widen(t, hd).reshape(n, -1) for t in (q, k, v)], 1).to("cuda", dtype)
    pt = page_table(5, 8)
    kp, vp = (torch.zeros(40, kv, 16, hd, dtype=dtype, device="cuda") for _ in range(2))
    K().qkv_insert(rows, K().rows(**d, page_table=pt), kp, vp, heads=heads, kv_heads=kv, hd=hd, eps=1e-5, dim=dim, vdim=dim, growth=coef, growth_every=every)
    factor = torch.tensor([oracle.query_factor(p, {"coef": coef, "every": every}) for p in pos], dtype=torch.float64)
    close(rows[:, :heads * hd].view(n, heads, hd)[..., :dim], q.double() * factor[:, None, None], dtype, 4.0)
    assert torch.equal(kp[int(pt[3, 99 // 16]), :, 99 % 16, :dim].cpu(), k[0])


SHAPES = [(6, 1, 64, 64, 64), (4, 4, 40, 64, 64), (20, 1, 128, 96, 128), (34, 2, 64, 64, 64), (4, 2, 256, 130, 256)]


@pytest.mark.parametrize("form", ["f32", "rows-bf16", "tensor", "prefill"])
@pytest.mark.parametrize("size", [0, 1, 5, 16, 64, 100, 500])
@pytest.mark.parametrize("heads,kv,dim,vdim,hd", SHAPES)
def test_windows_with_logarithmic_fall(form, size, heads, kv, dim, vdim, hd):
    dtype = F32 if form == "f32" else BF16
    lens, total, slots = [40, 3, 1, 130], [40, 80, 101, 255], [2, 0, 3, 1]
    d, pos, seq = pack(lens, [t - n for t, n in zip(total, lens)], slots)
    n, rnd = sum(lens), gen(5)
    pt = page_table(4, 16, seed=1)
    k, v, kp, vp = cached(rnd, slots, total, kv, hd, dim, vdim, dtype, pt, 64)
    q, scale, r1, r2 = rnd(n, heads, dim).to(dtype), 2.0 / math.sqrt(dim), rnd(heads).abs().float(), rnd(heads).abs().float() * 3
    out = attend(form, widen(q, hd).reshape(n, -1).cuda(), d, pt, kp, vp, total, lens, Hq=heads, Hkv=kv, hd=hd, scale=scale, window=size,
                 slopes=r1.cuda(), rates=r2.cuda())
    got, share = out.view(n, heads, hd)[..., :vdim].double().cpu(), heads // kv
    for i in range(0, n, 9):
        js = torch.arange(0 if not size else max(0, pos[i] - size + 1), pos[i] + 1)
        kk, vv = k[seq[i]].double(), v[seq[i]].double()
        want = [oracle.softmax(kk[js, a // share] @ q[i, a].double() * scale - oracle.log_bias(r1[a].double(), r2[a].double(), (pos[i] - js).double()))
                @ vv[js, a // share] for a in range(heads)]
        close(got[i], torch.stack(want), dtype)


@pytest.mark.parametrize("form", ["f32", "tensor", "prefill"])
def test_a_far_key_loses_to_the_logarithm_of_its_distance(form):
    """Two equal keys with opposite values, the older one far away: how much of it is left is the bias's doing, head by head."""
    dtype, n, heads = F32 if form == "f32" else BF16, 200, 8
    pt, rnd = page_table(1, 13), gen(8)
    _, _, kp, vp = cached(rnd, [0], [n], 1, 64, 64, 64, dtype, pt, 13)
    kp.zero_(), vp.zero_()
    for at, sign in ((3, 1.0), (199, -1.0)):
        kp[int(pt[0, at // 16]), 0, at % 16], vp[int(pt[0, at // 16]), 0, at % 16] = 4.0, sign
    r1, r2 = torch.tensor([0.0, 0.1, 0.5, 1.0, 2.0, 0.5, 0.5, 4.0]), torch.tensor([1.0, 1.0, 0.01, 0.5, 3.0, 10.0, 0.0, 100.0])
    d, _, _ = pack([1], [n - 1], [0])
    out = attend(form, torch.ones(1, heads * 64, dtype=dtype, device="cuda"), d, pt, kp, vp, [n], [1], Hq=heads, Hkv=1, hd=64, scale=0.125,
                 slopes=r1.cuda(), rates=r2.cuda())
    left = (1 + 196.0 * r2.double()) ** -r1.double()
    close(out.view(heads, 64)[:, 0], (left - 1) / (left + 1), dtype)


# ------------------------------------------------------------------------------------------------ latent attention
ROT = Rotary(20, 1000.0, YarnScaling(4.0, 100, 8.0, 1.0))


def raw(rot):
    y = rot.scaling
    return {"dims": rot.dims, "base": rot.base, "scaling": y and {"factor": y.factor, "original": y.original, "fast": y.fast, "slow": y.slow}}


def turned(x, pos, rot):
    """``x [rows, heads, dims]`` at the given positions."""
    wide = torch.zeros(max(pos) + 1, len(pos), x.shape[1], x.shape[2], dtype=torch.float64)
    for i, p in enumerate(pos):
        wide[p, i] = x[i]
    return torch.stack([oracle.rotate(wide[:, i], raw(rot))[p] for i, p in enumerate(pos)])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rot", [ROT, Rotary(2, 10.0), Rotary(64, 1e6, YarnScaling(2.0, 64, 32.0, 1.0))])
def test_rotation_in_neighbouring_pairs(dtype, rot):
    rnd, pos = gen(6), [0, 1, 5, 33, 120, 7]
    pad = (rot.dims + 7) // 8 * 8
    buf = rnd(6, 3, 16 + pad).to("cuda", dtype)
    x = buf[..., 16:16 + rot.dims]
    want, before = turned(x.double().cpu(), pos, rot), buf[..., :16].clone()
    K().head_rotate(x, i32(*pos), *rot.tables(128, "cuda"))
    close(x, want, dtype, 2.0)
    assert torch.equal(buf[..., :16], before) and not buf[..., 16 + rot.dims:].any()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rank,rot", [(41, ROT), (16, Rotary(64, 1e4)), (512, Rotary(64, 1e6)), (300, Rotary(2, 10.0))])
def test_cached_rows_hold_the_latent_and_the_rotated_part(dtype, rank, rot):
    lens, pos0, slots = [3, 18, 1], [14, 0, 31], [2, 0, 1]
    d, pos, seq = pack(lens, pos0, slots)
    n, rnd, pt = sum(lens), gen(7), page_table(3, 3)
    R, P, Q = (rank + 15) // 16 * 16, (rot.dims + 15) // 16 * 16, 40
    x, c, q = torch.zeros(n, Q + R + P), rnd(n, rank).to(dtype), rnd(n, 37).to(dtype)
    t = rnd(n, rot.dims).to(dtype)
    x[:, :37], x[:, Q:Q + rank], x[:, Q + R:Q + R + rot.dims] = q, c, t
    x = x.to("cuda", dtype)
    nw, qw = rnd(rank).float(), rnd(37).float()
    pool = torch.full((9, 16, R + P), 7.0, device="cuda", dtype=dtype)
    K().latent_insert(x[:, Q:], widen(nw, R).cuda().contiguous(), pool, K().rows(**d, page_table=pt), 1e-4, rank=rank, cos=rot.tables(64, "cuda")[0],
                      sin=rot.tables(64, "cuda")[1], q=x, q_norm=widen(qw, Q).cuda().contiguous(), q_rank=37)
    rows = torch.stack([pool[int(pt[slots[s], p // 16]), p % 16] for s, p in zip(seq, pos)])
    close(rows[:, :rank], oracle.rms(c.double(), 1e-4, nw.double()), dtype, 4.0)
    close(rows[:, R:R + rot.dims], turned(t.double()[:, None], pos, rot)[:, 0], dtype, 2.0)
    assert not rows[:, rank:R].any() and not rows[:, R + rot.dims:].any()
    close(x[:, :37], oracle.rms(q.double(), 1e-4, qw.double()), dtype, 4.0)
    before = pool.clone()
    K().latent_insert(None, None, None, K().rows(**d, page_table=pt), 1e-4, q=x, q_norm=widen(qw, Q).cuda().contiguous(), q_rank=37)
    assert torch.equal(pool, before)


@pytest.mark.parametrize("dtype", [BF16, F16])
@pytest.mark.parametrize("size", [0, 70])
def test_prefill_attention_with_keys_wider_than_values(dtype, size):
    """Keys of 192 and values of 128 as column blocks of one buffer, ragged sequences with cached rows ahead of the portion."""
    lens, total, heads, rnd = [130, 1, 64, 40], [200, 33, 64, 41], 3, gen(10)
    q, kv = rnd(sum(lens), heads * 192).to("cuda", dtype), rnd(sum(total), heads * (192 + 128)).to("cuda", dtype)
    starts, kv_starts = [sum(lens[:i]) for i in range(4)], [sum(total[:i]) for i in range(4)]
    out, status = torch.zeros(sum(lens), heads * 128, dtype=dtype, device="cuda"), torch.zeros(8, dtype=torch.int32, device="cuda")
    K().attention_prefill(q, out, Hq=heads, Hkv=heads, hd=192, vd=128, q_start=i32(*starts), q_len=i32(*lens), kv_len=i32(*total), max_q_len=130,
                          kv_start=i32(*kv_starts), k=kv[:, :heads * 192], v=kv[:, heads * 192:], window=size, scale=0.1, status=status)
    assert int(status[0]) == 0
    kk, vv = (t.double().cpu().view(sum(total), heads, -1) for t in (kv[:, :heads * 192], kv[:, heads * 192:]))
    for s, (n, t) in enumerate(zip(lens, total)):
        for i in range(0, n, 7):
            at, lo = t - n + i, max(0, t - n + i - size + 1) if size else 0
            rows = slice(kv_starts[s] + lo, kv_starts[s] + at + 1)
            p = torch.softmax(torch.einsum("hd,jhd->hj", q[starts[s] + i].double().cpu().view(heads, 192), kk[rows]) * 0.1, -1)
            close(out[starts[s] + i].view(heads, 128), torch.einsum("hj,jhd->hd", p, vv[rows]), dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads", [1, 17, 40])
@pytest.mark.parametrize("rank,vrank", [(48, 32), (128, 64), (176, 160), (192, 128), (320, 256), (512, 448), (576, 512), (640, 512)])
def test_latent_attention_with_key_columns_that_are_no_values(dtype, heads, rank, vrank):
    lens, total, slots = [2, 1, 3], [150, 40, 3], [1, 0, 2]
    d, pos, seq = pack(lens, [t - n for t, n in zip(total, lens)], slots)
    n, rnd, pt = sum(lens), gen(8), page_table(3, 10)
    pool = rnd(30, 16, rank).to("cuda", dtype)
    q, scale = (rnd(n, heads, rank) * 2).to("cuda", dtype), rank ** -0.5
    got = K().latent_attention(q, pool, K().rows(**d, page_table=pt), window=0, scale=scale, max_kv=150, vrank=vrank)
    assert got.shape == (n, heads, vrank)
    for i in range(n):
        c = torch.stack([pool[int(pt[slots[seq[i]], j // 16]), j % 16] for j in range(pos[i] + 1)]).double().cpu()
        s = q[i].double().cpu() @ c.T * scale
        close(got[i], torch.softmax(s, -1) @ c[:, :vrank], dtype)


# ------------------------------------------------------------------------------------------------ delta rule
class Layer:
    """Random weights and inputs of one delta-rule layer, heads padded as asked, and the plain results."""

    def __init__(self, heads, kv, dim, vdim, D, V, taps, dtype, total, seed=9, slow=False):
        rnd = gen(seed)
        self.heads, self.kv, self.dim, self.vdim, self.D, self.V, self.taps, self.dtype, self.total = heads, kv, dim, vdim, D, V, taps, dtype, total
        self.x = [[rnd(n, c, d).to(dtype) for c, d in ((kv, dim), (kv, dim), (heads, vdim))] for n in total]
        self.w = [(rnd(c, d, taps) / math.sqrt(taps)).float() for c, d in ((kv, dim), (kv, dim), (heads, vdim))]
        self.b, self.a, self.z = ([rnd(n, heads, *s).to(dtype) for n in total] for s in ((), (), (vdim,)))
        self.rate = torch.exp(rnd(heads)).float() * (0.02 if slow else 1.0)
        self.dt_bias, self.norm = rnd(heads).float() - 1.0, rnd(vdim).float()
        self.state = torch.full((4, heads, D, V), 5.0, device="cuda")
        self.ring = torch.full((4, taps, self.channels()), 5.0, device="cuda", dtype=dtype)
        self.conv_w = torch.cat([self.flat(w.permute(2, 0, 1), p) for w, p in zip(self.w, (D, D, V))], 1).cuda().contiguous()

    def channels(self):
        return 2 * self.kv * self.D + self.heads * self.V

    def flat(self, t, padded):
        """``[n, heads, d]`` -> ``[n, heads * padded]``"""
        out = torch.zeros(t.shape[0], t.shape[1], padded, dtype=t.dtype)
        out[..., :t.shape[2]] = t
        return out.flatten(1)

    def conv(self, s, k):
        n, c, d = self.x[s][k].shape
        y = oracle.causal_convolution(self.x[s][k].double().reshape(n, -1), self.w[k].double().reshape(c * d, -1))
        return oracle.silu(y).view(n, c, d)

    def want(self, s, eps):
        share = self.heads // self.kv
        q, k, v = (self.conv(s, i) for i in range(3))
        q, k = ((oracle.unit(t) * f).repeat_interleave(share, 1) for t, f in ((q, self.dim ** -0.5), (k, 1.0)))
        decay = torch.exp(-self.rate.double() * oracle.softplus(self.a[s].double() + self.dt_bias.double()))
        o, last = oracle.delta_rule(q, k, v, oracle.sigmoid(self.b[s].double()), decay)
        return oracle.rms(o, eps, self.norm.double()) * oracle.silu(self.z[s].double()), last

    def run(self, parts, slots, at, *, eps, form):
        """``parts``: (sequence, rows) of one launch; ``form``: fused decode step, recurrence or chunks."""
        d, _, _ = pack([n for _, n in parts], [at[s] for s, _ in parts], [slots[s] for s, _ in parts])
        cat = lambda get: torch.cat([get(s)[at[s]:at[s] + n] for s, n in parts])
        rows = torch.cat([self.flat(cat(lambda s: self.x[s][k]), p) for k, p in enumerate((self.D, self.D, self.V))], 1).to("cuda", self.dtype)
        gates = torch.cat([cat(lambda s: self.b[s]), cat(lambda s: self.a[s])], 1)
        gates = widen(gates, (2 * self.heads + 7) // 8 * 8).to("cuda", self.dtype)
        z = self.flat(cat(lambda s: self.z[s]), self.V).to("cuda", self.dtype)
        kw = dict(kv_heads=self.kv, eps=eps, dim=self.dim, vdim=self.vdim)
        common = (gates, gates[:, self.heads:], z, self.rate.cuda(), self.dt_bias.cuda(), widen(self.norm, self.V).cuda().contiguous(), self.state)
        if form == "fused":
            out = K().delta_rule(rows, *common, K().rows(pos=d["pos"], slot=d["slot"]), conv=(self.conv_w, self.ring), **kw)
        else:
            r = K().rows(**d)
            x = K().conv_silu(rows, self.conv_w, None, self.ring, r, max_q_len=max(n for _, n in parts), ring=True)
            out = K().delta_rule(x, *common, r, chunked=form == "chunks", **kw)
        out = out.view(-1, self.heads, self.V)
        assert not out[..., self.vdim:].any()
        return list(out[..., :self.vdim].split([n for _, n in parts]))


def loose(got, want, dtype):
    """16-bit queries and keys of a long recurrence, whose small products the norm behind it makes large: the bound is on the root mean
    square, with room for single values (the test of the digits below is the sharp one)."""
    got = got.double().cpu()
    err = (got - want).pow(2).mean().sqrt() / want.pow(2).mean().sqrt()
    assert float(err) < (2e-5 if dtype == F32 else 2.5e-2), float(err)
    assert float((got - want).abs().max()) < (2e-3 if dtype == F32 else 0.15) * float(want.abs().max())


SIZES = [(4, 2, 24, 40, 24, 40, 3), (3, 3, 64, 32, 64, 32, 4), (4, 1, 100, 90, 128, 96, 2), (2, 1, 7, 5, 8, 8, 1), (2, 2, 128, 128, 128, 128, 5), (2, 1, 256, 200, 256, 200, 4),
         (1, 1, 40, 512, 40, 512, 9)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("size", SIZES)
def test_delta_rule_token_by_token_in_portions_and_fused(dtype, size):
    """Decode steps with the convolution inside, and portions behind the convolution kernel, over the same carried state."""
    layer, slots, at, got = Layer(*size, dtype, (60, 37)), [2, 0], [0, 0], [[], []]
    for lens in ([1, 1], [1, 1], [2, 1], [1, 1], [15, 0], [1, 1], [3, 9], [1, 1], [1, 1], [30, 2], [1, 0], [0, 1], [1, 15]):
        parts = [(s, n) for s, n in enumerate(lens) if n]
        for (s, n), o in zip(parts, layer.run(parts, slots, at, eps=1e-5, form="fused" if max(lens) == 1 else "rows")):
            got[s].append(o)
            at[s] += n
    for s in range(2):
        want, _ = layer.want(s, 1e-5)
        loose(torch.cat(got[s]), want[:at[s]], dtype)
    assert (layer.state[[1, 3]] == 5.0).all() and (layer.ring[[1, 3]] == 5.0).all()


@pytest.mark.parametrize("dtype", [BF16, F16])
@pytest.mark.parametrize("slow", [False, True])
@pytest.mark.parametrize("size", [(4, 2, 64, 32, 64, 32, 4), (3, 1, 40, 60, 64, 64, 3), (2, 2, 128, 128, 128, 128, 4), (4, 1, 100, 90, 128, 96, 2)])
def test_delta_rule_in_chunks(dtype, slow, size):
    """Portions that start and end anywhere in a chunk, several sequences; the state against the plain one."""
    total = (64, 200, 331, 1)
    layer, slots, at, got = Layer(*size, dtype, total, slow=slow), [2, 0, 3, 1], [0] * 4, [[] for _ in total]
    for lens in ([64, 17, 100, 1], [0, 64, 65, 0], [0, 1, 2, 0], [0, 118, 164, 0]):
        parts = [(s, n) for s, n in enumerate(lens) if n]
        for (s, n), o in zip(parts, layer.run(parts, slots, at, eps=1e-5, form="chunks")):
            got[s].append(o)
            at[s] += n
    assert at == list(total)
    for s in range(4):
        want, last = layer.want(s, 1e-5)
        loose(torch.cat(got[s]), want, dtype)
        state = layer.state[slots[s]].double().cpu()
        assert not state[:, layer.dim:].any() and not state[..., layer.vdim:].any()
        err = (state[:, :layer.dim, :layer.vdim] - last).pow(2).mean().sqrt() / last.pow(2).mean().sqrt()
        assert float(err) < (1.2e-2 if dtype == BF16 else 2e-3), float(err)


@pytest.mark.parametrize("dtype", [BF16, F16])
def test_chunks_lose_no_digits_of_the_state(dtype):
    """Inputs that 16 bits hold exactly: what is left is the arithmetic, which is 32-bit; a state that decays slowly for long."""
    g = torch.Generator().manual_seed(4)
    n, heads, D, V = 512, 2, 64, 32
    x = (torch.randint(-8, 9, (n, 2 * heads * D + heads * V), generator=g) / 8).to("cuda", dtype)
    gates = (torch.randint(-16, 17, (n, 8), generator=g) / 8).to("cuda", dtype)
    z, rate, dt, w = torch.ones(n, heads * V, dtype=dtype, device="cuda"), torch.tensor([1e-3, 0.3]), torch.zeros(heads), torch.ones(V)
    q, k, v = x.double().cpu().split([heads * D, heads * D, heads * V], 1)
    q, k, v = q.view(n, heads, D), k.view(n, heads, D), v.view(n, heads, V)
    decay = torch.exp(-rate.double() * oracle.softplus(gates[:, 4:6].double().cpu()))
    _, want = oracle.delta_rule(oracle.unit(q) * D ** -0.5, oracle.unit(k), v, oracle.sigmoid(gates[:, :2].double().cpu()), decay)
    for chunked, bound in ((False, 2e-6), (True, 2e-5)):
        state = torch.zeros(1, heads, D, V, device="cuda")
        K().delta_rule(x, gates, gates[:, 4:], z, rate.cuda(), dt.cuda(), w.cuda(), state, K().rows(torch.arange(n, dtype=torch.int32, device="cuda"),
                       seq_of_row=torch.zeros(n, dtype=torch.int32, device="cuda"), q_start=i32(0), q_len=i32(n)), kv_heads=heads, eps=1e-6, chunked=chunked)
        err = (state[0].double().cpu() - want).pow(2).mean().sqrt() / want.pow(2).mean().sqrt()
        assert float(err) < bound, (chunked, float(err))


# ------------------------------------------------------------------------------------------------ experts
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("E,identity,k", [(12, 4, 4), (5, 1, 6), (1, 3, 2), (60, 4, 6), (200, 56, 32), (8, 0, 2), (30, 40, 1)])
@pytest.mark.parametrize("T,H", [(1, 40), (37, 328), (300, 1024)])
def test_choice_with_identity_experts(dtype, E, identity, k, T, H):
    rnd, n = gen(12), E + identity
    x, w, bias = rnd(T, H).to(dtype), (rnd(n, H) * 2 / math.sqrt(H)).to(dtype), (rnd(n) / n).float()
    for scatter in (True, False):
        b = K().RoutedBatch(x.cuda(), w.cuda(), k, correction=bias.cuda(), norm_topk=False, tile_rows=16, scatter=scatter, identity=identity)
        for _ in range(2):
            b.route()
        if not scatter:
            b.gather()
        assert not b.counters.any()
        slot, ids, sw, own = b.slot_of.cpu(), b.ids.cpu(), b.slot_w.double().cpu(), b.self_w.double().cpu()
        z = x.double() @ w.double().T
        for t in range(0, T, 1 if T < 100 else 7):
            picks, a = oracle.choose(z[t], bias.double(), k)
            if ids[t].tolist() != [e if e < E else -1 for e in picks]:                 # only ever between near-ties
                s = torch.sort(oracle.softmax(z[t]) + bias.double(), descending=True).values
                assert float((s[:-1] - s[1:])[:k].min()) < 1e-5, (t, ids[t].tolist(), picks)
                continue
            assert float(own[t]) == pytest.approx(sum(float(v) for e, v in zip(picks, a) if e >= E), rel=1e-4, abs=1e-7)
            for j, e in enumerate(picks):
                assert (int(slot[t, j]) >= 0) == (e < E)
                if e < E:
                    assert float(sw[int(slot[t, j])]) == pytest.approx(float(a[j]), rel=1e-4, abs=1e-7)
        used = slot[slot >= 0].tolist()
        assert sorted(used) == list(range(len(used))) and int(b.tiles[0]) == sum(-(-int((ids == e).sum()) // 16) for e in range(E))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("E,identity,k,ff,H", [(6, 2, 2, 24, 72), (4, 1, 4, 136, 200), (3, 0, 1, 8, 8), (16, 8, 3, 256, 640)])
@pytest.mark.parametrize("T,tile", [(1, 16), (40, 16), (130, 32), (600, 128)])
def test_single_operand_experts(dtype, E, identity, k, ff, H, T, tile):
    fp32 = dtype == F32
    rnd, grouped, n = gen(13), tile == 128 and not fp32, E + identity
    x, router, bias = rnd(T, H).to(dtype), (rnd(n, H) / math.sqrt(H)).to(dtype), (rnd(n) / n).float()
    w = {}
    for e in range(E):
        w[f"e{e}.up"], w[f"e{e}.down"] = (rnd(ff, H) / math.sqrt(H)).to(dtype), (rnd(H, ff) / math.sqrt(ff)).to(dtype)
    pad = ff if fp32 else (ff + 127) // 128 * 128
    b = K().moe_router(x.cuda(), router.cuda(), k, correction=bias.cuda(), norm_topk=False, tile_rows=64 if fp32 else tile, scatter=not grouped, identity=identity)
    up, down = torch.zeros(E, pad, H, dtype=dtype), torch.zeros(E, H, pad, dtype=dtype)
    for e in range(E):
        up[e, :ff], down[e, :, :ff] = w[f"e{e}.up"], w[f"e{e}.down"]
    img = lambda t: t.cuda().contiguous() if fp32 else K().pack_weight(t.cuda().contiguous())
    up, down = img(up.view(-1, H)), img(down.view(E * H, pad) if fp32 else down.transpose(0, 1).reshape(H, E * pad))
    if grouped:
        h = K().moe_grouped_gemm(b.gather(), up, b.tiles[3:], n=pad, k=H, bank_rows=E * pad, bank_k=H, expert_rows=pad, act="gelu_erf")
        y = K().moe_grouped_gemm(h, down, b.tiles[3:], n=H, k=pad, bank_rows=H, bank_k=E * pad, expert_k=pad, row_scale=b.slot_w[:T * k].contiguous())
    else:
        h = K().moe_experts(b, x.cuda(), up, n=ff, k=H, experts=E, expert_pad=pad, act="gelu_erf", stacked=True)
        y = K().moe_experts(b, h, down, n=H, k=ff, experts=E, expert_pad=pad, gathered=False, weighted=True)
    slot, wd = b.slot_of.long().cpu(), {a: t.double() for a, t in w.items()}
    got = torch.where((slot >= 0)[..., None], y.double().cpu()[slot.clamp(min=0)], torch.zeros((), dtype=torch.float64)).sum(1)
    ids, ws = b.ids.cpu().tolist(), b.weights.double().cpu()
    for t in range(0, T, 1 if T < 50 else 5):
        want = sum((ws[t, j] * oracle.expert(x[t].double(), wd, f"e{e}.") for j, e in enumerate(ids[t]) if e >= 0), torch.zeros(H, dtype=torch.float64))
        close(got[t], want, dtype, 2.0)


@pytest.mark.parametrize("M", [4, 200, 700])
def test_exact_gelu_of_the_gemms_keeps_its_small_values(M):
    """The negative side, where one plus the error function cancels: relative error down to where results vanish."""
    x = torch.linspace(-5.0, 5.0, M * 64).view(M, 64).to("cuda", BF16)
    w = torch.eye(64).repeat(4, 1).to("cuda", BF16)
    got = K().gemm(x, K().pack_weight(w), packed_shape=(256, 64), act="gelu_erf").double().cpu()
    want = (x.double().cpu() * 0.5 * torch.erfc(-x.double().cpu() / math.sqrt(2.0))).repeat(1, 4)
    torch.testing.assert_close(got, want, rtol=2e-2, atol=2e-7)


def test_invalid_options_are_refused_on_the_host():
    from rhinoforge_b200.api.errors import RPUBackendError
    pt = page_table(1, 1)
    r = K().rows(i32(0), page_table=pt)
    x = torch.zeros(1, 64, device="cuda", dtype=BF16)
    with pytest.raises(RPUBackendError):                                               # rates without slopes
        pool = torch.zeros(1, 1, 16, 64, device="cuda", dtype=BF16)
        K().attention_rows(x, r, pool, pool, Hq=1, Hkv=1, hd=64, scale=1.0, max_kv=1, rates=torch.ones(1, device="cuda"))
    with pytest.raises(RPUBackendError):                                               # the fused convolution takes decode rows
        K().stream_norm(torch.zeros(2, 64, device="cuda"), K().rows(i32(0, 1), seq_of_row=i32(0, 0), q_start=i32(0), q_len=i32(2)), dtype=BF16, eps=1e-6,
                        norm_w=torch.ones(64, device="cuda"), conv=(torch.ones(2, 64, device="cuda"), torch.zeros(1, 1, 64, device="cuda", dtype=BF16)))
    with pytest.raises(RPUBackendError):                                               # chunks of a head size they do not take
        z = torch.zeros(1, 8, device="cuda", dtype=BF16)
        K().delta_rule(torch.zeros(1, 72, device="cuda", dtype=BF16), z, z, torch.zeros(1, 24, device="cuda", dtype=BF16), *(torch.ones(24, device="cuda"),) * 3,
                       torch.zeros(1, 1, 24, 24, device="cuda"), r, kv_heads=1, eps=1e-6, chunked=True)
    with pytest.raises(RPUBackendError):                                               # more value columns than the cache has
        K().latent_attention(torch.zeros(1, 1, 64, device="cuda", dtype=BF16), torch.zeros(1, 16, 64, device="cuda", dtype=BF16), r, window=0, scale=1.0,
                             max_kv=1, vrank=80)
    with pytest.raises(RPUBackendError):                                               # nothing but identity experts
        K().RoutedBatch(x, torch.zeros(2, 64, device="cuda", dtype=BF16), 1, identity=2).route()
