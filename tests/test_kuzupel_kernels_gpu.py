"""Kernels of the Kuzupel decoders, each against the plain formulation of its mechanism."""
import math

import pytest
import torch

import _kuzupel_oracle as oracle
from rhinoforge_b200.models.mixed import GroupedAttention, Rotary

pytestmark = pytest.mark.gpu
F32, BF16, F16 = torch.float32, torch.bfloat16, torch.float16
DTYPES = [F32, BF16]
ALPHA = 1.702


def K():
    from rhinoforge_b200.ops import kernels
    return kernels


def i32(*v):
    return torch.tensor(v, dtype=torch.int32, device="cuda")


def pack(lens, pos0, slots):
    q_start = [sum(lens[:i]) for i in range(len(lens))]
    seq = [s for s, n in enumerate(lens) for _ in range(n)]
    pos = [pos0[s] + i for s, n in enumerate(lens) for i in range(n)]
    return dict(pos=i32(*pos), seq_of_row=i32(*seq), q_start=i32(*q_start), q_len=i32(*lens), slot=i32(*slots)), pos, seq


def page_table(slots, per_slot, seed=0):
    return torch.randperm(slots * per_slot, generator=torch.Generator().manual_seed(seed)).to(torch.int32).view(slots, per_slot).cuda()


def close(got, want, dtype, scale=1.0):
    tol = 2e-5 if dtype == F32 else 1.5e-2
    torch.testing.assert_close(got.double().cpu(), want.double().cpu(), rtol=tol, atol=tol * scale)


def gen(seed):
    g = torch.Generator().manual_seed(seed)
    return lambda *s: torch.randn(*s, generator=g, dtype=torch.float64)


def widen(t, width):
    return torch.nn.functional.pad(t, (0, width - t.shape[-1]))


# ------------------------------------------------------------------------------------------------ embedding and residual stream
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,dim", [(40, 37), (1024, 1024), (8200, 8200)])
@pytest.mark.parametrize("buckets,mul_prev,mul_cur", [(1, 5, 3), (13, 1, 0), (50, 1_000_003, 2_147_483_647)])
def test_pair_embedding_carries_the_last_token(dtype, H, dim, buckets, mul_prev, mul_cur):
    vocab, rnd = 211, gen(1)
    table, pair, w = (widen(rnd(n, dim), H).to(dtype) for n in (vocab, buckets + 1, 1))
    last = torch.full((4,), 99, dtype=torch.int32, device="cuda")                     # left over by earlier requests
    toks = [torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(n)) for n in (30, 7, 2)]
    b = {"buckets": buckets, "mul_prev": mul_prev, "mul_cur": mul_cur}
    want = [oracle.embed(t, {"embed": table.double(), "bigram": pair.double()}, {"scale": 0.75, "bigram": b}) for t in toks]
    slots, at = [2, 0, 3], [0, 0, 0]
    for lens in ([1, 2, 0], [17, 1, 1], [1, 1, 0], [1, 0, 1], [10, 3, 0]):
        live = [i for i in range(3) if lens[i]]
        d, _, _ = pack([lens[i] for i in live], [at[i] for i in live], [slots[i] for i in live])
        ids = torch.cat([toks[i][at[i]:at[i] + lens[i]] for i in live]).to(torch.int32).cuda()
        if max(lens) == 1:                                                             # single tokens: rows are sequences
            d = dict(pos=d["pos"], slot=d["slot"])
        x, h, _ = K().stream_norm(None, K().rows(**d), dtype=dtype, eps=1e-4, norm_w=w[0].float().cuda(), table=table.cuda(), ids=ids, dim=dim,
                                  embed_scale=0.75, pairs=(pair.cuda(), last, mul_prev, mul_cur))
        exp = torch.cat([want[i][at[i]:at[i] + lens[i]] for i in live])[:, :dim]
        close(x[:, :dim], exp, F32, 4.0)
        close(h[:, :dim], oracle.rms(exp, 1e-4, w[0, :dim].double()), dtype, 4.0)
        at = [a + n for a, n in zip(at, lens)]
        assert all(int(last[slots[i]]) == int(toks[i][at[i] - 1]) for i in live)
    assert int(last[1]) == 99


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H", [40, 1024, 8200])
@pytest.mark.parametrize("n", [3, 700])
@pytest.mark.parametrize("picks", [0, 3])
def test_stream_multiplies_what_it_adds(dtype, H, n, picks):
    rnd = gen(2)
    x, y, w = rnd(n, H).float(), rnd(n * max(picks, 1), H).to(dtype), rnd(H).float()
    slots = torch.randperm(n * picks, generator=torch.Generator().manual_seed(3)).to(torch.int32).view(n, picks) if picks else None
    total = y.double()[slots.long()].sum(1) if picks else y.double()
    r = K().rows(torch.arange(n, dtype=torch.int32, device="cuda"))
    xo, h, xc = K().stream_norm(x.cuda(), r, dtype=dtype, eps=1e-4, norm_w=w.cuda(), y=y.cuda(), y_mult=0.37, cast=True,
                                y_slots=None if slots is None else slots.cuda())
    want = x.double() + 0.37 * total
    close(xo, want, F32, 4.0)
    close(xc, want, dtype, 4.0)
    close(h, oracle.rms(want, 1e-4, w.double()), dtype, 4.0)


# ------------------------------------------------------------------------------------------------ between projection and attention
HEADS = [(4, 2, 20, 13, 24), (3, 1, 64, 64, 64), (8, 8, 100, 128, 128), (2, 1, 16, 200, 256), (2, 2, 300, 31, 304), (1, 1, 16, 9, 16), (40, 5, 128, 128, 128)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,kv,dim,vdim,hd", HEADS)
@pytest.mark.parametrize("rot", [None, Rotary(12, 1e4)])
def test_one_norm_over_all_heads(dtype, heads, kv, dim, vdim, hd, rot):
    lens, pos0, slots = [1, 9, 2, 17], [33, 0, 15, 7], [3, 1, 0, 4]
    d, pos, seq = pack(lens, pos0, slots)
    n, rnd, eps = sum(lens), gen(3), 1e-3
    q, k, v = rnd(n, heads, dim).to(dtype), (rnd(n, kv, dim) * 3).to(dtype), rnd(n, kv, vdim).to(dtype)
    q[:, 0] *= 5                                                                       # one head far larger than the others
    qn, kn = rnd(heads, dim).float(), rnd(kv, dim).float()
    pt = page_table(5, 4)
    cos, sin = rot.tables(64, "cuda") if rot else (None, None)
    raw = None if rot is None else {"dims": rot.dims, "base": rot.base}

    def normed(x, w):
        x = oracle.rms(x.double().reshape(n, -1), eps, w.double().reshape(-1)).view(x.shape)
        return torch.cat([oracle.rotate(x[i:i + 1], pos[i], raw) for i in range(n)])
    rows = torch.cat([widen(t, hd).reshape(n, -1) for t in (q, k, v)], 1).to("cuda", dtype)
    kp, vp = (torch.zeros(20, kv, 16, hd, dtype=dtype, device="cuda") for _ in range(2))
    K().qkv_insert(rows, K().rows(**d, page_table=pt), kp, vp, heads=heads, kv_heads=kv, hd=hd, eps=eps, dim=dim, vdim=vdim,
                   q_norm=widen(qn, hd).cuda().contiguous(), k_norm=widen(kn, hd).cuda().contiguous(), cos=cos, sin=sin, norm_all=True)
    got = lambda pool: torch.stack([pool[int(pt[slots[seq[i]], pos[i] // 16]), :, pos[i] % 16] for i in range(n)])
    close(rows[:, :heads * hd].view(n, heads, hd)[..., :dim], normed(q, qn), dtype, 4.0)
    close(got(kp)[..., :dim], normed(k, kn), dtype, 4.0)
    close(got(vp)[..., :vdim], v.double(), dtype)
    assert not got(kp)[..., dim:].any() and not rows[:, :heads * hd].view(n, heads, hd)[..., dim:].any()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,kv,dim,vdim,hd", HEADS)
@pytest.mark.parametrize("taps", [1, 2, 3, 4, 5, 20])
def test_convolved_projections_carry_their_inputs(dtype, heads, kv, dim, vdim, hd, taps):
    rot, eps, rnd, slots = Rotary(min(dim, 12), 1e4), 1e-3, gen(4), [2, 0, 3]
    if heads > 8 and taps not in (1, 4):
        return
    total = (70, 41, 9)
    cols = [(heads, dim), (kv, dim), (kv, vdim)]
    x = [[rnd(n, c, d).to(dtype) for c, d in cols] for n in total]
    w = [(rnd(c, d, taps) / taps).float() for c, d in cols]
    qn, kn = rnd(dim).float(), rnd(dim).float()
    raw = {"dims": rot.dims, "base": rot.base}

    def conv(u, t):
        return oracle.causal_convolution(u.double().reshape(u.shape[0], -1), t.double().reshape(-1, taps)).view(u.shape)
    want = []
    for parts in x:
        cq, ck, cv = (conv(u, t) for u, t in zip(parts, w))
        want.append((oracle.rotate(oracle.rms(cq, eps, qn.double()), 0, raw), oracle.rotate(oracle.rms(ck, eps, kn.double()), 0, raw), cv))
    cw = torch.cat([torch.nn.functional.pad(t, (0, 0, 0, hd - t.shape[1])).permute(2, 0, 1).reshape(taps, -1) for t in w], 1).contiguous().cuda()
    width = (heads + 2 * kv) * hd
    state = rnd(4, max(taps - 1, 1), width).to("cuda", dtype)                          # left over by earlier requests
    pt = page_table(4, 5)
    kp, vp = (torch.zeros(20, kv, 16, hd, dtype=dtype, device="cuda") for _ in range(2))
    cos, sin = rot.tables(80, "cuda")
    tables = dict(heads=heads, kv_heads=kv, hd=hd, eps=eps, dim=dim, vdim=vdim, q_norm=widen(qn, hd).cuda(), k_norm=widen(kn, hd).cuda(), cos=cos, sin=sin,
                  conv_w=cw, conv_state=state if taps > 1 else None)
    at = [0, 0, 0]
    for lens in ([1, 2, 0], [40, 1, 1], [2, 19, 1], [1, 1, 3], [26, 18, 3], [0, 0, 1]):
        live = [i for i in range(3) if lens[i]]
        d, _, _ = pack([lens[i] for i in live], [at[i] for i in live], [slots[i] for i in live])
        if max(lens) == 1:                                                             # single tokens: rows are sequences
            d = dict(pos=d["pos"], slot=d["slot"])
        rows = torch.cat([torch.cat([widen(u[at[i]:at[i] + lens[i]], hd).reshape(lens[i], -1) for u in x[i]], 1) for i in live]).to("cuda", dtype)
        before = rows.clone()
        q = K().qkv_insert(rows, K().rows(**d, page_table=pt), kp, vp, max_q_len=max(lens), **tables)
        assert torch.equal(rows, before)
        close(q.view(-1, heads, hd)[..., :dim], torch.cat([want[i][0][at[i]:at[i] + lens[i]] for i in live]), dtype, 4.0)
        at = [a + n for a, n in zip(at, lens)]
    assert tuple(at) == total
    for i, s in enumerate(slots):
        pages = lambda pool: torch.stack([pool[int(pt[s, p // 16]), :, p % 16] for p in range(total[i])])
        close(pages(kp)[..., :dim], want[i][1], dtype, 4.0)
        close(pages(vp)[..., :vdim], want[i][2], dtype, 4.0)


# ------------------------------------------------------------------------------------------------ attention
def cached(rnd, slots, lens, kv, hd, dim, vdim, dtype, pt, pages):
    """Random keys and values of every slot, dense and in pages."""
    k = [rnd(n, kv, dim).to(dtype) for n in lens]
    v = [rnd(n, kv, vdim).to(dtype) for n in lens]
    kp, vp = (torch.zeros(pages, kv, 16, hd, dtype=dtype, device="cuda") for _ in range(2))
    for s, a, b in zip(slots, k, v):
        for i in range(a.shape[0]):
            p = int(pt[s, i // 16])
            kp[p, :, i % 16, :dim], vp[p, :, i % 16, :vdim] = a[i].cuda(), b[i].cuda()
    return k, v, kp, vp


def attend(form, q, d, pt, kp, vp, totals, lens, **kw):
    """One of the three forms over packed query rows."""
    if form != "prefill":
        return K().attention_rows(q, K().rows(**d, page_table=pt), kp, vp, max_kv=max(totals), tensor_core=form == "tensor", **kw)
    status = torch.zeros(8, dtype=torch.int32, device="cuda")
    out = torch.zeros(q.shape[0], kw["Hq"] * kw["hd"], dtype=q.dtype, device="cuda")
    K().attention_prefill(q, out, q_start=d["q_start"], q_len=d["q_len"], kv_len=i32(*totals), max_q_len=max(lens), k_pool=kp, v_pool=vp,
                          page_table=pt, slot=d["slot"], max_kv_len=max(totals), status=status, **kw)
    assert int(status[0]) == 0
    return out


def expected(q, k, v, i, scale, mask, biased, with_one, gate):
    """One query ``[heads, dim]`` at position i."""
    js, share, heads = torch.tensor(oracle.visible(i, mask)), q.shape[0] // k.shape[1], q.shape[0]
    out = []
    for a in range(heads):
        s = (k[js, a // share] @ q[a]) * scale
        if biased:
            s = s - oracle.slope(a, heads) * (i - js).double()
        out.append(oracle.softmax(s, with_one) @ v[js, a // share])
    return torch.stack(out) * oracle.sigmoid(gate)[:, None]


SHAPES = [(6, 1, 64, 64, 64), (4, 4, 40, 64, 64), (20, 1, 128, 96, 128), (34, 2, 64, 64, 64), (4, 2, 256, 130, 256)]
MASKS = [None, {"size": 1}, {"size": 5}, {"size": 16, "keep_first": 1}, {"size": 37, "keep_first": 16}, {"size": 64}, {"size": 100, "keep_first": 70},
         {"size": 3, "keep_first": 130}, {"size": 1, "keep_first": 17}, {"size": 500, "keep_first": 9}]


@pytest.mark.parametrize("form", ["f32", "rows-bf16", "tensor", "prefill"])
@pytest.mark.parametrize("mask", range(len(MASKS)))
@pytest.mark.parametrize("heads,kv,dim,vdim,hd", SHAPES)
def test_windows_kept_tokens_slopes_and_gates(form, mask, heads, kv, dim, vdim, hd):
    mask = MASKS[mask]
    dtype = F32 if form == "f32" else BF16
    lens, total, slots = [40, 3, 1, 130], [40, 80, 101, 255], [2, 0, 3, 1]
    d, pos, seq = pack(lens, [t - n for t, n in zip(total, lens)], slots)
    n, rnd = sum(lens), gen(5)
    pt = page_table(4, 16, seed=1)
    k, v, kp, vp = cached(rnd, slots, total, kv, hd, dim, vdim, dtype, pt, 64)
    q, gate, scale = rnd(n, heads, dim).to(dtype), rnd(n, heads).to(dtype), 2.0 / math.sqrt(dim)
    qq, gg = widen(q, hd).reshape(n, -1).cuda(), widen(gate, (heads + 7) // 8 * 8).cuda()
    slopes = torch.tensor([oracle.slope(a, heads) for a in range(heads)]).float().cuda()
    for biased in (False, True):
        kw = dict(Hq=heads, Hkv=kv, hd=hd, scale=scale, window=(mask or {}).get("size", 0), keep_first=(mask or {}).get("keep_first", 0),
                  gate=gg, gate_by_head=True, **(dict(slopes=slopes) if biased else dict(sink=torch.zeros(heads, device="cuda"))))
        out = attend(form, qq, d, pt, kp, vp, total, lens, **kw)
        got = out.view(n, heads, hd)[..., :vdim]
        if form == "tensor":
            one = attend(form, qq, d, pt, kp, vp, total, lens, split=False, **kw).view(n, heads, hd)[..., :vdim]
            close(one, got, dtype)
        got = got.double().cpu()
        for i in range(0, n, 9):
            s = seq[i]
            close(got[i], expected(q[i].double(), k[s].double(), v[s].double(), pos[i], scale, mask, biased, not biased, gate[i].double()), dtype)


@pytest.mark.parametrize("form", ["f32", "tensor", "prefill"])
@pytest.mark.parametrize("window,keep", [(16, 0), (17, 16), (64, 20), (65, 64), (70, 63), (128, 1)])
def test_one_key_that_stands_out_is_seen_inside_its_window_only(form, window, keep):
    """A key that every query likes, at page and block borders, among the kept ones and just behind them: the result is its value
    as long as it is visible."""
    dtype, n = F32 if form == "f32" else BF16, 230
    pt, rnd = page_table(1, 15), gen(7)
    like = torch.ones(64, dtype=torch.float64)
    q = (rnd(n, 1, 64) * 0.1 + like).to(dtype)
    d, _, _ = pack([n], [0], [0])
    for at in sorted({0, 15, 16, 63, 64, 80, max(keep - 1, 0), keep, keep + 1}):
        k, v, kp, vp = cached(rnd, [0], [n], 1, 64, 64, 64, dtype, pt, 15)
        kp[int(pt[0, at // 16]), 0, at % 16] = (like * 4).to("cuda", dtype)
        kw = dict(Hq=1, Hkv=1, hd=64, scale=0.125, window=window, keep_first=keep, sink=torch.zeros(1, device="cuda"))
        out = attend(form, q.view(n, 64).cuda(), d, pt, kp, vp, [n], [n], **kw).double().cpu()
        for i in range(at, n):
            seen = float((out[i] - v[0][at, 0].double()).abs().max()) < 0.05
            assert seen == (i - at < window or at < keep), (at, i)


@pytest.mark.parametrize("form", ["f32", "tensor", "prefill"])
def test_a_far_key_loses_to_its_distance(form):
    """Two equal keys with opposite values, the older one far away: how much of it is left is the slope's doing, head by head."""
    dtype, n, heads = F32 if form == "f32" else BF16, 200, 16
    pt, rnd = page_table(1, 13), gen(8)
    k, v, kp, vp = cached(rnd, [0], [n], 1, 64, 64, 64, dtype, pt, 13)
    kp.zero_(), vp.zero_()
    for at, sign in ((3, 1.0), (199, -1.0)):
        kp[int(pt[0, at // 16]), 0, at % 16], vp[int(pt[0, at // 16]), 0, at % 16] = 4.0, sign
    q = torch.ones(1, heads * 64, dtype=dtype, device="cuda")
    slopes = GroupedAttention(heads, 1, 64, 64, 1.0, distance_bias=True).slopes()
    d, _, _ = pack([1], [n - 1], [0])
    out = attend(form, q, d, pt, kp, vp, [n], [1], Hq=heads, Hkv=1, hd=64, scale=0.125, slopes=slopes.float().cuda())
    got = out.view(heads, 64)[:, 0].double().cpu()
    score = torch.zeros(heads, n, dtype=torch.float64)
    score[:, [3, 199]] = 4.0 * 64 * 0.125
    score -= slopes[:, None] * (199 - torch.arange(n, dtype=torch.float64))
    p = torch.softmax(score, -1)
    close(got, p[:, 3] - p[:, 199], dtype)
    assert float(got[-1]) > -0.7 and float(got[0]) < -0.99                             # nearly level for the last head, all lost for the first


@pytest.mark.parametrize("form", ["f32", "tensor", "prefill"])
def test_the_one_in_the_denominator(form):
    """Scores far below zero leave nothing, far above zero everything; at one key with score zero exactly one half."""
    dtype, n = F32 if form == "f32" else BF16, 20
    pt, rnd = page_table(1, 2), gen(9)
    k, v, kp, vp = cached(rnd, [0], [n], 1, 64, 64, 64, dtype, pt, 2)
    kp.zero_()
    kp[:, :, :, 0] = 8.0
    q = torch.zeros(n, 3, 64, dtype=dtype)
    q[:, 0, 0], q[:, 1, 0] = -30.0, 30.0
    d, _, _ = pack([n], [0], [0])
    out = attend(form, q.view(n, -1).cuda(), d, pt, kp, vp, [n], [n], Hq=3, Hkv=1, hd=64, scale=0.5, sink=torch.zeros(3, device="cuda"))
    got, vv = out.view(n, 3, 64).double().cpu(), v[0][:, 0].double()
    for i in range(n):
        mean = vv[:i + 1].mean(0)
        close(got[i, 0], torch.zeros(64), dtype)
        close(got[i, 1], mean, dtype)
        close(got[i, 2], mean * (i + 1) / (i + 2), dtype)


# ------------------------------------------------------------------------------------------------ feed-forward
@pytest.mark.parametrize("dtype", [BF16, F16, F32])
@pytest.mark.parametrize("M,N,KK", [(1, 40, 72), (16, 1024, 512), (64, 4096, 4096), (200, 136, 1000), (300, 256, 320), (1100, 4096, 1024), (5000, 1536, 768)])
@pytest.mark.parametrize("limit", [0.4, 7.0])
def test_clipped_pair_in_every_gemm(dtype, M, N, KK, limit):
    rnd = gen(10)
    x, w = rnd(M, KK).to(dtype), (rnd(2 * N, KK) / math.sqrt(KK)).to(dtype)
    g, u = (x.double().cuda() @ w.double().cuda().T).split((N, N), 1)
    g, u = torch.clamp(g, max=limit), torch.clamp(u, -limit, limit)
    want = g * torch.sigmoid(ALPHA * g) * (u + 1)
    if dtype == F32:
        got = K().gemm_f32(x.cuda(), w.cuda(), "clipped_glu", dual=True, limit=limit, alpha=ALPHA)
    else:
        wp = K().pack_weight(w.cuda(), 2)
        got = K().gemm(x.cuda(), wp, packed_shape=(2 * N, KK), act="clipped_glu", dual=True, limit=limit, alpha=ALPHA)
    close(got, want, dtype, 1.0 if limit > 1 else 0.3)


@pytest.mark.parametrize("dtype", [BF16, F32])
@pytest.mark.parametrize("M,N", [(1, 640), (64, 32768), (3, 80000)])
def test_soft_cap_of_the_logits(dtype, M, N):
    rnd, KK, cap = gen(11), 256, 5.0
    x, w = (rnd(M, KK) * torch.linspace(0.1, 30, M)[:, None]).to(dtype), (rnd(N, KK) / 16).to(dtype)
    want = oracle.soft_cap(x.double().cuda() @ w.double().cuda().T, cap)
    got = K().gemm_f32(x.cuda(), w.cuda(), "soft_cap", limit=cap) if dtype == F32 else \
        K().gemm(x.cuda(), K().pack_weight(w.cuda()), packed_shape=(N, KK), act="soft_cap", limit=cap)
    close(got, want, dtype, 5.0)
    assert float(got.abs().max()) <= cap


ROUTERS = [(15, 4), (8, 1), (5, 5), (64, 6), (160, 8), (256, 32), (1, 1), (64, 1), (65, 2)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("E,k", ROUTERS)
@pytest.mark.parametrize("T,H", [(1, 40), (37, 328), (300, 1024), (1100, 520)])
def test_choice_by_biased_logits_and_the_shared_weight(dtype, E, k, T, H):
    rnd = gen(12)
    x, w, bias = rnd(T, H).to(dtype), (rnd(E + 1, H) * 2 / math.sqrt(H)).to(dtype), (rnd(E) * 3).float()
    for scatter in (True, False):
        b = K().RoutedBatch(x.cuda(), w.cuda(), k, correction=bias.cuda(), score_fn="chosen", tile_rows=16, shared=True, scatter=scatter, shared_gate=True)
        for _ in range(2):
            b.route()
        if not scatter:
            b.gather()
        assert not b.counters.any()
        ids, weights = b.ids.cpu(), b.weights.double().cpu()
        z = x.double() @ w.double().T
        for t in range(0, T, 1 if T < 100 else 7):
            want, a = oracle.choose(z[t, :E] + bias.double(), k)
            if ids[t].tolist() != want:                                                # only ever between near-ties
                s = torch.sort(z[t, :E] + bias.double(), descending=True).values
                assert float((s[:-1] - s[1:])[:k].min()) < 1e-5, (t, ids[t].tolist(), want)
                continue
            torch.testing.assert_close(weights[t], a, rtol=1e-4, atol=1e-7)
        torch.testing.assert_close(weights.sum(1), torch.ones(T, dtype=torch.float64), rtol=1e-5, atol=0)
        slot, sw = b.slot_of.long().cpu(), b.slot_w.double().cpu()
        assert slot[:, k].tolist() == [T * k + t for t in range(T)] and sorted(slot[:, :k].reshape(-1).tolist()) == list(range(T * k))
        torch.testing.assert_close(sw[slot[:, :k]], weights, rtol=1e-6, atol=0)
        torch.testing.assert_close(sw[T * k:], torch.sigmoid(z[:, E]), rtol=1e-4, atol=1e-6)


def banks(w, E, ff, H, pad, dtype, fp32):
    up, down = torch.zeros(2, E, pad, H, dtype=dtype), torch.zeros(E, H, pad, dtype=dtype)
    for e in range(E):
        up[0, e, :ff], up[1, e, :ff], down[e, :, :ff] = w[f"e{e}.gate"], w[f"e{e}.up"], w[f"e{e}.down"]
    img = lambda t, n=1: t.cuda().contiguous() if fp32 else K().pack_weight(t.cuda().contiguous(), n)
    return img(up.view(-1, H), 2), img(down.view(E * H, pad) if fp32 else down.transpose(0, 1).reshape(H, E * pad)), img


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("E,k,ff,shared,H", [(6, 2, 24, 40, 72), (4, 4, 136, 0, 200), (3, 1, 8, 8, 8), (16, 3, 256, 512, 640)])
@pytest.mark.parametrize("T,tile", [(1, 16), (40, 16), (130, 32), (600, 128)])
def test_clipped_experts(dtype, E, k, ff, shared, H, T, tile):
    fp32 = dtype == F32
    rnd, grouped, limit, shared_limit = gen(13), tile == 128 and not fp32, 0.8, 0.3
    x, router, bias = rnd(T, H).to(dtype), (rnd(E + bool(shared), H) / math.sqrt(H)).to(dtype), rnd(E).float() * 0.1
    w = {}
    for name, f in [(f"e{e}", ff) for e in range(E)] + ([("shared", shared)] if shared else []):
        w[name + ".gate"], w[name + ".up"], w[name + ".down"] = ((rnd(a, b) / math.sqrt(b)).to(dtype) for a, b in ((f, H), (f, H), (H, f)))
    pad = ff if fp32 else (ff + 127) // 128 * 128
    b = K().moe_router(x.cuda(), router.cuda(), k, correction=bias.cuda(), tile_rows=64 if fp32 else tile, shared=bool(shared), score_fn="chosen",
                       shared_gate=bool(shared), scatter=not grouped)
    up, down, img = banks(w, E, ff, H, pad, dtype, fp32)
    act = dict(act="clipped_glu", limit=limit, alpha=ALPHA)
    if grouped:
        tiles = b.tiles[3:]
        h = K().moe_grouped_gemm(b.gather(), up, tiles, n=pad, k=H, bank_rows=E * pad, bank_k=H, expert_rows=pad, dual=True, **act)
        y = K().moe_grouped_gemm(h, down, tiles, n=H, k=pad, bank_rows=H, bank_k=E * pad, expert_k=pad, row_scale=b.slot_w[:T * k].contiguous())
        if shared:
            hs = K().gemm(x.cuda(), img(torch.cat((w["shared.gate"], w["shared.up"])), 2), packed_shape=(2 * shared, H), dual=True,
                          act="clipped_glu", limit=shared_limit, alpha=ALPHA)
            y = torch.cat((y, K().gemm(hs, img(w["shared.down"]), packed_shape=(H, shared), row_scale=b.slot_w[T * k:].contiguous())))
    else:
        sh_up = img(torch.cat((w["shared.gate"], w["shared.up"])), 2) if shared else None
        sh_down = img(w["shared.down"]) if shared else None
        h = K().moe_experts(b, x.cuda(), up, n=ff, k=H, experts=E, expert_pad=pad, dual=True, shared=sh_up, shared_n=shared, shared_k=H if shared else 0,
                            shared_limit=shared_limit, **act)
        y = K().moe_experts(b, h, down, n=H, k=ff, experts=E, expert_pad=pad, gathered=False, weighted=True, shared=sh_down,
                            shared_n=H if shared else 0, shared_k=shared)
    got = y.double().cpu()[b.slot_of.long().cpu()].sum(1)
    wd = {n: t.double() for n, t in w.items()}
    ids, ws = b.ids.cpu().tolist(), b.weights.double().cpu()
    sg = torch.sigmoid(x.double() @ router.double().T[:, -1:])
    for t in range(0, T, 1 if T < 50 else 5):
        want = sum(ws[t, j] * oracle.clipped_glu(x[t].double(), wd, f"e{e}.", limit) for j, e in enumerate(ids[t]))
        if shared:
            want = want + sg[t] * oracle.clipped_glu(x[t].double(), wd, "shared.", shared_limit)
        close(got[t], want, dtype, 2.0)


def test_invalid_options_are_refused_on_the_host():
    from rhinoforge_b200.api.errors import RPUBackendError
    x, w = torch.zeros(2, 64, device="cuda", dtype=BF16), torch.zeros(16, 64, device="cuda", dtype=BF16)
    with pytest.raises(RPUBackendError):
        K().gemm(x, w, act="clipped_glu", dual=True)                                   # no limit
    with pytest.raises(RPUBackendError):
        K().gemm(x, w, act="soft_cap")
    with pytest.raises(RPUBackendError):
        K().RoutedBatch(x, w, 2, shared_gate=True).route()                             # a weight for a shared expert that is not there
    pool, pt = torch.zeros(1, 1, 16, 24, device="cuda"), page_table(1, 1)
    with pytest.raises(RPUBackendError):
        K().qkv_insert(torch.zeros(1, 72, device="cuda"), K().rows(i32(0), page_table=pt), pool, pool, heads=1, kv_heads=1, hd=24, eps=1e-6, dim=20,
                       conv_w=torch.zeros(3, 72, device="cuda"))                        # no carried inputs
    with pytest.raises(RPUBackendError):
        K().stream_norm(torch.zeros(1, 64, device="cuda"), K().rows(i32(0)), dtype=BF16, eps=1e-6, ids=i32(0),
                        pairs=(torch.zeros(4, 64, device="cuda", dtype=BF16), i32(0), 1, 1))
