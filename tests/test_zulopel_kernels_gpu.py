"""Kernels of the Zulopel decoders, each against the plain formulation of its mechanism."""
import math

import pytest
import torch

import _zulopel_oracle as oracle
from rhinoforge_b200.models.mixed import Rotary, YarnScaling

pytestmark = pytest.mark.gpu
F32, BF16 = torch.float32, torch.bfloat16
DTYPES = [F32, BF16]


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


# ------------------------------------------------------------------------------------------------ residual stream
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,dim", [(40, 37), (512, 512), (4104, 4099), (8200, 8200)])
def test_stream_adds_the_sum_of_picked_rows_and_scales_the_embedding(dtype, H, dim):
    n, picks, rnd = 21, 3, gen(1)
    pad = lambda t: torch.nn.functional.pad(t, (0, H - dim))
    y, table, w = pad(rnd(50, dim)).to(dtype), pad(rnd(9, dim)).to(dtype), pad(rnd(dim)).float()
    slots = torch.randint(0, 50, (n, picks), generator=torch.Generator().manual_seed(2)).to(torch.int32)
    slots[3, 1] = -1
    ids = torch.arange(n).to(torch.int32) % 9
    r = K().rows(torch.arange(n, dtype=torch.int32, device="cuda"))
    xo, _, xc = K().stream_norm(None, r, dtype=dtype, eps=1e-4, table=table.cuda(), ids=ids.cuda(), y=y.cuda(), y_norm_w=w.cuda(), dim=dim,
                                cast=True, embed_scale=7.25, y_slots=slots.cuda())
    total = torch.stack([sum(y[s].double() for s in row if s >= 0) for row in slots.tolist()])[:, :dim]
    want = table.double()[ids.long(), :dim] * 7.25 + oracle.rms(total, 1e-4, w.double()[:dim])
    close(xo[:, :dim], want, F32, 4.0)
    close(xc[:, :dim], want, dtype, 4.0)


# ------------------------------------------------------------------------------------------------ attention
ROTS = [None, Rotary(2, 50.0), Rotary(12, 1e4), Rotary(16, 500.0, YarnScaling(8.0, 100, 20.0, 1.0)), Rotary(16, 3e5, YarnScaling(2.0, 4096, 4.0, 4.0))]


@pytest.mark.parametrize("rot", ROTS[1:])
def test_rotation_tables(rot):
    raw = {"dims": rot.dims, "base": rot.base}
    if rot.scaling:
        raw["scaling"] = vars(rot.scaling)
    f, amp = oracle.rotation_frequencies(raw)
    cos, sin = rot.tables(3000, "cuda")
    a = torch.arange(3000, dtype=torch.float64)[:, None] * f[None]
    close(cos, a.cos() * amp, F32, 0.01)
    close(sin, a.sin() * amp, F32, 0.01)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,kv,dim,vdim,hd", [(4, 2, 20, 13, 24), (3, 1, 64, 64, 64), (8, 8, 100, 128, 128), (2, 1, 16, 200, 256), (2, 2, 300, 31, 304), (1, 1, 16, 9, 16)])
@pytest.mark.parametrize("rot", range(len(ROTS)))
def test_qkv_insert_normalises_rotates_mixes_and_pages(dtype, heads, kv, dim, vdim, hd, rot):
    rot = ROTS[rot]
    lens, pos0, slots = [1, 9, 2, 17], [33, 0, 15, 7], [3, 1, 0, 4]
    d, pos, seq = pack(lens, pos0, slots)
    n, rnd, eps = sum(lens), gen(3), 1e-3
    pad = lambda t: torch.nn.functional.pad(t, (0, hd - t.shape[-1]))
    q, k, v = rnd(n, heads, dim).to(dtype), rnd(n, kv, dim).to(dtype), rnd(n, kv, vdim).to(dtype)
    first, qn, kn = rnd(n, kv, vdim).to(dtype), rnd(dim).float(), rnd(dim).float()
    pt = page_table(5, 4)
    raw = None if rot is None else {"dims": rot.dims, "base": rot.base, **({"scaling": vars(rot.scaling)} if rot.scaling else {})}
    cos, sin = rot.tables(64, "cuda") if rot else (None, None)
    def turned(x, w):
        x = oracle.rms(x.double(), eps, w.double())
        return torch.cat([oracle.rotate(x[i:i + 1], pos[i], raw) for i in range(n)])
    for role, lam in (("none", 0.0), ("first", 0.4), ("mix", 0.3)):
        rows = torch.cat([pad(q).reshape(n, -1), pad(k).reshape(n, -1), pad(v).reshape(n, -1)], 1).to("cuda", dtype)
        kp, vp = (torch.zeros(20, kv, 16, hd, dtype=dtype, device="cuda") for _ in range(2))
        store = first.clone().reshape(n, -1).cuda()
        K().qkv_insert(rows, K().rows(**d, page_table=pt), kp, vp, heads=heads, kv_heads=kv, hd=hd, eps=eps, dim=dim, vdim=vdim,
                       q_norm=pad(qn).cuda(), k_norm=pad(kn).cuda(), cos=cos, sin=sin, v_first=store, v_role=role, v_lambda=lam)
        close(rows[:, :heads * hd].view(n, heads, hd)[..., :dim], turned(q, qn), dtype, 4.0)
        want_k, want_v = turned(k, kn), oracle.mix_values(v.double(), first.double(), lam) if role == "mix" else v.double()
        at = [(int(pt[slots[seq[i]], pos[i] // 16]), pos[i] % 16) for i in range(n)]
        got = lambda pool: torch.stack([pool[p, :, o] for p, o in at])
        close(got(kp)[..., :dim], want_k, dtype, 4.0)
        close(got(vp)[..., :vdim], want_v, dtype, 4.0)
        assert not got(kp)[..., dim:].any() and not got(vp)[..., vdim:].any()
        close(store.view(n, kv, vdim), (v if role == "first" else first).double(), dtype)


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


def expected(q, k, v, i, scale, sink, chunk, gate):
    """One query ``[heads, dim]`` at position i."""
    lo, share = oracle.first_visible(i, chunk), q.shape[0] // k.shape[1]
    o = [oracle.sink_softmax((k[lo:i + 1, a // share] @ q[a]) * scale, sink[a]) @ v[lo:i + 1, a // share] for a in range(q.shape[0])]
    return torch.stack(o) * torch.sigmoid(gate)


SHAPES = [(6, 1, 64, 64, 64), (4, 4, 40, 64, 64), (20, 1, 128, 96, 128), (34, 2, 64, 64, 64), (4, 2, 256, 130, 256)]


@pytest.mark.parametrize("form", ["f32", "rows-bf16", "tensor", "prefill"])
@pytest.mark.parametrize("chunk", [0, 1, 5, 16, 37, 64, 100])
@pytest.mark.parametrize("heads,kv,dim,vdim,hd", SHAPES)
def test_chunked_attention_with_sinks_and_gates(form, chunk, heads, kv, dim, vdim, hd):
    dtype = F32 if form == "f32" else BF16
    lens, total, slots = [40, 3, 1, 130], [40, 80, 101, 155], [2, 0, 3, 1]
    pos0 = [t - n for t, n in zip(total, lens)]
    d, pos, seq = pack(lens, pos0, slots)
    n, rnd = sum(lens), gen(5)
    pt = page_table(4, 10, seed=chunk)
    k, v, kp, vp = cached(rnd, slots, total, kv, hd, dim, vdim, dtype, pt, 40)
    pad = lambda t: torch.nn.functional.pad(t, (0, hd - t.shape[-1]))
    q, gate, sink, scale = rnd(n, heads, dim).to(dtype), rnd(n, heads, vdim).to(dtype), rnd(heads).float() * 2, 2.0 / math.sqrt(dim)
    rows = torch.cat([pad(q).reshape(n, -1), pad(gate).reshape(n, -1)], 1).to("cuda", dtype)
    qq, gg = rows[:, :heads * hd], rows[:, heads * hd:]
    kw = dict(Hq=heads, Hkv=kv, hd=hd, scale=scale, chunk=chunk, sink=sink.cuda(), gate=gg)
    if form == "prefill":
        status = torch.zeros(8, dtype=torch.int32, device="cuda")
        out = torch.zeros(n, heads * hd, dtype=dtype, device="cuda")
        K().attention_prefill(qq, out, q_start=d["q_start"], q_len=d["q_len"], kv_len=i32(*total), max_q_len=max(lens), k_pool=kp, v_pool=vp,
                              page_table=pt, slot=d["slot"], max_kv_len=max(total), status=status, **kw)
        assert int(status[0]) == 0
    else:
        r = K().rows(**d, page_table=pt)
        out = K().attention_rows(qq, r, kp, vp, max_kv=160, tensor_core=form == "tensor", **kw)
        if form == "tensor":
            one = K().attention_rows(qq, r, kp, vp, max_kv=160, split=False, **kw)
            close(one.view(n, heads, hd)[..., :vdim], out.view(n, heads, hd)[..., :vdim], dtype)
    got = out.view(n, heads, hd)[..., :vdim].double().cpu()
    for i in range(0, n, 1 if n < 50 else 3):
        s = seq[i]
        close(got[i], expected(q[i].double(), k[s].double(), v[s].double(), pos[i], scale, sink.double(), chunk, gate[i].double()), dtype)


@pytest.mark.parametrize("form", ["f32", "tensor", "prefill"])
@pytest.mark.parametrize("at", [0, 15, 16, 31, 63, 64, 79, 80])
def test_one_key_that_stands_out_is_seen_inside_its_chunk_only(form, at):
    """A key that every query likes, at page and chunk borders: the result is its value as long as it is visible."""
    dtype, chunk, n = F32 if form == "f32" else BF16, 80, 130
    pt, rnd = page_table(1, 9), gen(7)
    k, v, kp, vp = cached(rnd, [0], [n], 1, 64, 64, 64, dtype, pt, 9)
    like = torch.ones(64, dtype=torch.float64)
    kp[int(pt[0, at // 16]), 0, at % 16] = (like * 4).to("cuda", dtype)
    k[0][at, 0] = (like * 4).to(dtype)
    q = (rnd(n, 1, 64) * 0.1 + like).to(dtype)
    d, _, _ = pack([n], [0], [0])
    kw = dict(Hq=1, Hkv=1, hd=64, scale=0.125, chunk=chunk, sink=torch.zeros(1, device="cuda"))
    qq = q.view(n, 64).cuda()
    if form == "prefill":
        out = torch.zeros(n, 64, dtype=dtype, device="cuda")
        K().attention_prefill(qq, out, q_start=i32(0), q_len=i32(n), kv_len=i32(n), max_q_len=n, k_pool=kp, v_pool=vp, page_table=pt, **kw)
    else:
        out = K().attention_rows(qq, K().rows(**d, page_table=pt), kp, vp, max_kv=n, tensor_core=form == "tensor", **kw)
    for i in range(at, n):
        seen = float((out[i].double().cpu() - v[0][at, 0].double()).abs().max()) < 0.05
        assert seen == (i // chunk == at // chunk), i


@pytest.mark.parametrize("form", ["f32", "tensor", "prefill"])
def test_a_strong_sink_takes_the_weight(form):
    dtype, n = F32 if form == "f32" else BF16, 20
    pt, rnd = page_table(1, 2), gen(8)
    k, v, kp, vp = cached(rnd, [0], [n], 2, 64, 64, 64, dtype, pt, 2)
    q = rnd(n, 4, 64).to(dtype)
    sink = torch.tensor([-100.0, 200.0, 4.0, 0.0])
    d, pos, _ = pack([n], [0], [0])
    kw = dict(Hq=4, Hkv=2, hd=64, scale=0.125, sink=sink.cuda())
    qq = q.view(n, 256).cuda()
    if form == "prefill":
        out = torch.zeros(n, 256, dtype=dtype, device="cuda")
        K().attention_prefill(qq, out, q_start=i32(0), q_len=i32(n), kv_len=i32(n), max_q_len=n, k_pool=kp, v_pool=vp, page_table=pt, **kw)
    else:
        out = K().attention_rows(qq, K().rows(**d, page_table=pt), kp, vp, max_kv=n, tensor_core=form == "tensor", **kw)
    got = out.view(n, 4, 64)
    assert float(got[:, 1].abs().max()) < 1e-6 and torch.isfinite(got).all()
    ones = torch.full((4, 64), 1e9, dtype=torch.float64)
    for i in range(n):
        close(got[i], expected(q[i].double(), k[0].double(), v[0].double(), i, 0.125, sink.double(), 0, ones), dtype)


# ------------------------------------------------------------------------------------------------ selective scan
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("taps", [1, 2, 3, 4, 5, 20])
def test_convolution_carries_its_inputs(dtype, taps):
    C, slots, rnd = 1032, [2, 0, 3], gen(9)
    xs = [rnd(n, C).to(dtype) for n in (70, 41, 9)]
    w, b = rnd(taps, C).float() / taps, rnd(C).float()
    state = rnd(4, max(taps - 1, 1), C).to("cuda", dtype)                          # left over by earlier requests
    want = [oracle.silu(oracle.causal_convolution(x.double(), w.double().T, b.double())) for x in xs]
    at = [0, 0, 0]
    for lens in ([1, 2, 0], [40, 1, 1], [2, 19, 1], [1, 1, 3], [26, 18, 4]):
        live = [i for i in range(3) if lens[i]]
        d, _, _ = pack([lens[i] for i in live], [at[i] for i in live], [slots[i] for i in live])
        x = torch.cat([xs[i][at[i]:at[i] + lens[i]] for i in live]).cuda()
        y = K().conv_silu(x, w.cuda(), b.cuda(), state if taps > 1 else None, K().rows(**d), max_q_len=max(lens))
        close(y, torch.cat([want[i][at[i]:at[i] + lens[i]] for i in live]), dtype)
        at = [a + n for a, n in zip(at, lens)]
    if taps > 1:                                                                   # single tokens: rows are sequences
        y = K().conv_silu(x[-3:].contiguous(), w.cuda(), b.cuda(), state, K().rows(i32(0, 0, 0), slot=i32(*slots)))
        close(y, torch.cat([oracle.silu(oracle.causal_convolution(t[None].double().cpu(), w.double().T, b.double())) for t in x[-3:]]), dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("form", ["recurrent", "scan", "decode"])
@pytest.mark.parametrize("inner,states,rank", [(8, 8, 8), (72, 16, 24), (136, 24, 8), (64, 40, 40), (40, 104, 16), (24, 256, 8), (4096, 16, 256)])
def test_selective_scan_over_portions(dtype, form, inner, states, rank):
    small = inner < 1000
    slots, rnd, S = [2, 0, 3], gen(10), states - 3                                 # three padding states
    total = (75, 36, 5) if small else (6, 3, 2)
    n = sum(total)
    pad = lambda t: torch.nn.functional.pad(t, (0, states - S))
    xs, zs = [[rnd(m, inner).to(dtype) for m in total] for _ in range(2)]
    bs, cs = [[rnd(m, S).to(dtype) for m in total] for _ in range(2)]
    ds = [rnd(m, rank).to(dtype) for m in total]
    w_dt, bias, D = (rnd(inner, rank) / math.sqrt(rank)).to(dtype), (rnd(inner) - 2).float(), rnd(inner).float()
    A = -torch.exp(rnd(inner, S)).float()
    a2 = pad(A.double() / math.log(2)).float().cuda()
    state = rnd(4, inner, states).float().cuda()
    want, final = [], []
    for i in range(3):
        pre = ds[i].double() @ w_dt.double().T
        if form == "scan":
            pre = pre.to(dtype).double()                                           # projected by a GEMM in the activation dtype
        y, st = oracle.selective_scan(xs[i].double(), oracle.softplus(pre + bias.double()), A.double(), bs[i].double(), cs[i].double(),
                                      D.double(), torch.zeros(inner, S, dtype=torch.float64))
        want.append(y * oracle.silu(zs[i].double()))
        final.append(st)
    at = [0, 0, 0]
    for lens in ([1, 2, 0], [40, 1, 1], [2, 19, 1], [32, 14, 3]) if small else ([1, 1, 1], [5, 2, 1]):
        if form == "decode":
            lens = [1, 1, 1]
        live = [i for i in range(3) if lens[i]]
        d, _, _ = pack([lens[i] for i in live], [at[i] for i in live], [slots[i] for i in live])
        if form == "decode":                                                       # single tokens: rows are sequences
            d = dict(pos=d["pos"], slot=d["slot"])
        cut = lambda t: torch.cat([t[i][at[i]:at[i] + lens[i]] for i in live])
        bc = torch.cat([cut(ds), pad(cut(bs)), pad(cut(cs))], 1).cuda().contiguous()
        kw = dict(w_dt=w_dt.cuda()) if form != "scan" else dict(dt=(cut(ds).double() @ w_dt.double().T).to(dtype).cuda())
        out = K().mamba1(cut(xs).cuda(), cut(zs).cuda(), bc, a2, D.cuda(), bias.cuda(), state, K().rows(**d), **kw)
        close(out, cut(want), dtype, 4.0)
        at = [a + m for a, m in zip(at, lens)]
    if form == "decode":
        return
    for i, s in enumerate(slots):
        close(state[s, :, :S], final[i], F32 if dtype == F32 else BF16, 2.0)
        assert not state[s, :, S:].any()
    assert n == sum(at)


def test_scan_step_sizes_from_tiny_to_large():
    """Softplus far on both sides of zero: nothing overflows, tiny steps keep their digits."""
    inner, n = 64, 40
    bias = torch.linspace(-16, 30, inner)
    rnd = gen(11)
    x, z, B, C = rnd(n, inner).to(BF16), rnd(n, inner).to(BF16), rnd(n, 8).to(BF16), rnd(n, 8).to(BF16)
    a2, D = -torch.ones(inner, 8).cuda(), torch.zeros(inner).cuda()
    bc = torch.cat([torch.zeros(n, 8), B, C], 1).to("cuda", BF16)
    dt = oracle.softplus(bias.double())[None].expand(n, inner)
    _, want = oracle.selective_scan(x.double(), dt, -math.log(2) * torch.ones(inner, 8, dtype=torch.float64), B.double(), C.double(),
                                    torch.zeros(inner, dtype=torch.float64), torch.zeros(inner, 8, dtype=torch.float64))
    for kw in (dict(w_dt=torch.zeros(inner, 8, dtype=BF16, device="cuda")), dict(dt=torch.zeros(n, inner, dtype=BF16, device="cuda"))):
        state = torch.zeros(1, inner, 8, device="cuda")
        d, _, _ = pack([n], [0], [0])
        K().mamba1(x.cuda(), z.cuda(), bc, a2, D, bias.cuda(), state, K().rows(**d), **kw)
        err = (state[0].double().cpu() - want).norm(dim=1) / want.norm(dim=1)
        assert float(err.max()) < 2e-5


# ------------------------------------------------------------------------------------------------ experts
ROUTERS = [(15, 4, 5, 2), (8, 1, 8, 1), (5, 5, 1, 1), (64, 6, 8, 3), (160, 8, 4, 4), (256, 32, 16, 9), (1, 1, 1, 1), (200, 4, 100, 2)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("E,k,groups,keep", ROUTERS)
@pytest.mark.parametrize("T,H", [(1, 40), (37, 328), (300, 1024), (1100, 520)])
def test_router_choice_weights_and_plan(dtype, E, k, groups, keep, T, H):
    rnd = gen(12)
    x, w, corr = rnd(T, H).to(dtype), (rnd(E, H) * 2 / math.sqrt(H)).to(dtype), (rnd(E) * 0.3 - 0.4).float()    # choice scores of both signs
    for scatter in (True, False):
        b = K().RoutedBatch(x.cuda(), w.cuda(), k, correction=corr.cuda(), groups=groups, keep=keep, tile_rows=16, shared=True, scatter=scatter)
        for _ in range(2):                                                         # the counters are left clean
            b.route()
        if not scatter:
            xg = b.gather()
            torch.testing.assert_close(xg.cpu(), x[b.token_of_slot[:T * k].long().cpu()])
        assert not b.counters.any()
        ids, weights = b.ids.cpu(), b.weights.double().cpu()
        s = torch.softmax(x.double() @ w.double().T, -1)
        key = s + corr.double()
        size, wrong = E // groups, 0
        for t in range(0, T, 1 if T < 100 else 7):
            want = oracle.choose(s[t], corr.double(), k, {"count": groups, "keep": keep})
            got = ids[t].tolist()
            if got != want:                                                        # only ever between near-ties
                top = key[t].view(groups, size).max(1).values.sort(descending=True).values
                edge = [float(top[keep - 1] - top[keep])] if keep < groups else []
                order = key[t][want]
                edge += [float((order[:-1] - order[1:]).min())] if k > 1 else []
                rest = [e for e in range(E) if e not in want and e // size in {x // size for x in want}]
                edge += [float(order[-1] - key[t][rest].max())] if rest else []
                assert min(edge) < 1e-6, (t, got, want)
                wrong += 1
                continue
            torch.testing.assert_close(weights[t], s[t][want] / (s[t][want].sum() + 1e-20), rtol=1e-4, atol=1e-7)
        assert wrong <= 2
        # the plan: every pick has its own sorted row, an expert's rows are neighbours, the tiles cover exactly them
        slot = b.slot_of.cpu()
        assert sorted(slot[:, :k].reshape(-1).tolist()) == list(range(T * k)) and slot[:, k].tolist() == [T * k + t for t in range(T)]
        tos, sw = b.token_of_slot.cpu(), b.slot_w.double().cpu()
        assert (tos[slot.long()] == torch.arange(T, dtype=torch.int32)[:, None]).all() and (sw[T * k:] == 1).all()
        torch.testing.assert_close(sw[slot[:, :k].long()], weights, rtol=1e-6, atol=0)
        tiles = b.tiles.cpu().view(-1, 4)
        assert tiles[0, 0] == tiles[0, 3]
        covered = torch.full((T * (k + 1),), -1)
        for e, r0, end, _ in tiles[1:1 + int(tiles[0, 0])].tolist():
            covered[r0:min(end, r0 + 16)] = e
        if not scatter:
            covered[T * k:] = E
        assert (covered[slot[:, :k].long()] == ids).all() and (covered[T * k:] == E).all()


def expert_weights(rnd, E, ff, H, shared, dtype):
    names = [f"e{e}" for e in range(E)] + (["shared"] if shared else [])
    w = {}
    for n in names:
        f = shared if n == "shared" else ff
        w[n + ".gate"], w[n + ".up"], w[n + ".down"] = (rnd(f, H) / math.sqrt(H)).to(dtype), (rnd(f, H) / math.sqrt(H)).to(dtype), (rnd(H, f) / math.sqrt(f)).to(dtype)
    return w


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("E,k,ff,shared,H", [(6, 2, 24, 40, 72), (4, 4, 136, 0, 200), (3, 1, 8, 8, 8), (16, 3, 256, 512, 640)])
@pytest.mark.parametrize("T,tile", [(1, 16), (40, 16), (130, 32)])
def test_expert_gemms_of_few_rows(dtype, E, k, ff, shared, H, T, tile):
    rnd = gen(13)
    x, router, corr = rnd(T, H).to(dtype), (rnd(E, H) / math.sqrt(H)).to(dtype), rnd(E).float() * 0.1
    w = expert_weights(rnd, E, ff, H, shared, dtype)
    fp32 = dtype == F32
    pad = ff if fp32 else (ff + 127) // 128 * 128
    b = K().moe_router(x.cuda(), router.cuda(), k, correction=corr.cuda(), tile_rows=64 if fp32 else tile, shared=bool(shared))
    up, down = torch.zeros(2, E, pad, H, dtype=dtype), torch.zeros(E, H, pad, dtype=dtype)
    for e in range(E):
        up[0, e, :ff], up[1, e, :ff], down[e, :, :ff] = w[f"e{e}.gate"], w[f"e{e}.up"], w[f"e{e}.down"]
    img = lambda t, n=1: t.cuda().contiguous() if fp32 else K().pack_weight(t.cuda().contiguous(), n)
    up, down = img(up.view(-1, H), 2), img(down.view(E * H, pad) if fp32 else down.transpose(0, 1).reshape(H, E * pad))
    sh_up = sh_down = None
    if shared:
        sh_up, sh_down = img(torch.cat((w["shared.gate"], w["shared.up"])), 2), img(w["shared.down"])
    h = K().moe_experts(b, x.cuda(), up, n=ff, k=H, experts=E, expert_pad=pad, dual=True, shared=sh_up, shared_n=shared, shared_k=H if shared else 0)
    y = K().moe_experts(b, h, down, n=H, k=ff, experts=E, expert_pad=pad, gathered=False, weighted=True, shared=sh_down,
                        shared_n=H if shared else 0, shared_k=shared)
    got = y.double().cpu()[b.slot_of.long().cpu()].sum(1)
    wd = {n: t.double() for n, t in w.items()}
    ids, ws = b.ids.cpu().tolist(), b.weights.double().cpu()
    for t in range(0, T, 1 if T < 50 else 5):
        want = sum(ws[t, j] * oracle.glu(x[t].double(), wd, f"e{e}.") for j, e in enumerate(ids[t]))
        if shared:
            want = want + oracle.glu(x[t].double(), wd, "shared.")
        close(got[t], want, dtype, 2.0)


def test_invalid_sizes_are_refused_on_the_host():
    from rhinoforge_b200.api.errors import RPUBackendError
    x, w = torch.zeros(2, 64, device="cuda", dtype=BF16), torch.zeros(12, 64, device="cuda", dtype=BF16)
    for kw in (dict(k=13), dict(k=4, groups=5), dict(k=5, groups=3, keep=1), dict(k=2, groups=3, keep=4)):
        with pytest.raises(RPUBackendError):
            K().moe_router(x, w, **kw)
    pool, pt = torch.zeros(1, 1, 16, 24, device="cuda"), page_table(1, 1)
    with pytest.raises(RPUBackendError):
        K().qkv_insert(torch.zeros(1, 72, device="cuda"), K().rows(i32(0), page_table=pt), pool, pool, heads=1, kv_heads=1, hd=24, eps=1e-6, dim=20,
                       cos=torch.zeros(1, 11, device="cuda"), sin=torch.zeros(1, 11, device="cuda"))
    with pytest.raises(RPUBackendError):
        K().mamba1(x, x, torch.zeros(2, 8 + 2 * 264, device="cuda", dtype=BF16), torch.zeros(64, 264, device="cuda"), torch.zeros(64, device="cuda"),
                   torch.zeros(64, device="cuda"), torch.zeros(2, 64, 264, device="cuda"), K().rows(i32(0, 0)), w_dt=torch.zeros(64, 8, device="cuda", dtype=BF16))
