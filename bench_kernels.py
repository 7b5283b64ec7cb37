#!/usr/bin/env python
"""Kernel micro-benchmarks with roofline fractions (device-timed, L2 flushed between iterations).

    python bench_kernels.py gemm --m 64 --n 12288 --k 4096 --dual [--packed] [--int8]
    python bench_kernels.py attn_prefill --seqs 4 --len 2048 --heads 32 --kv-heads 8 --hd 128
    python bench_kernels.py attn_decode --seqs 64 --len 1024 --heads 32 --kv-heads 8 --hd 128
    python bench_kernels.py gdn --seqs 1 --len 1024 --hk 16 --hv 32
    python bench_kernels.py mixed            # latent attention / HGRN2 / fp32 stream beside the like kernels at equal size
    python bench_kernels.py routed           # chunked attention / selective scan / routed experts beside the like kernels
    python bench_kernels.py windowed         # window attention with slopes or kept tokens / clipped feed-forwards beside the like kernels
    python bench_kernels.py suite            # the shapes of one Qwen3-8B decode step and prefill chunk

Every line is JSON: the achieved throughput and its fraction of the measured peaks in
``MEASURED_PEAKS.json`` (copy bandwidth and cuBLAS bf16 throughput measured on this pool; the fallback
values 6.65 TB/s and 1.59 PFLOP/s are used, and labelled, when the file is absent).
"""
from __future__ import annotations

import argparse
import json
import os
import statistics
import sys
from pathlib import Path

import torch

ROOT = Path(__file__).resolve().parent


def peaks() -> dict:
    f = ROOT / "MEASURED_PEAKS.json"
    if f.is_file():
        d = json.loads(f.read_text())
        return {"hbm_gbs": float(d.get("hbm_gbs", 6650.0)), "tflops": float(d.get("bf16_tflops", 1590.0)), "src": "measured"}
    return {"hbm_gbs": 6650.0, "tflops": 1590.0, "src": "fallback"}


_flush = None


def flush_l2() -> None:
    global _flush
    if _flush is None:
        _flush = torch.empty(256 << 20, dtype=torch.uint8, device="cuda")      # 2x the 126 MB L2
    _flush.zero_()


def time_graph_us(make_fn, nbuf: int, reps: int = 24) -> float:
    """Back-to-back in-stream time per launch: ``reps`` launches captured in one CUDA graph, cycling over ``nbuf``
    operand sets (``make_fn(i)`` returns the launch closure of set ``i``) so that no launch finds its weights in L2."""
    fns = [make_fn(i) for i in range(nbuf)]
    for f in fns:
        f()
    torch.cuda.synchronize()
    s = torch.cuda.Stream()
    s.wait_stream(torch.cuda.current_stream())
    g = torch.cuda.CUDAGraph()
    with torch.cuda.graph(g, stream=s):
        for i in range(reps):
            fns[i % nbuf]()
    ts = []
    for _ in range(5):
        flush_l2()
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        torch.cuda.synchronize()
        e0.record()
        g.replay()
        e1.record()
        torch.cuda.synchronize()
        ts.append(e0.elapsed_time(e1) * 1e3 / reps)
    return statistics.median(ts)


def time_us(fn, iters: int = 20, warmup: int = 3) -> float:
    for _ in range(warmup):
        fn()
    ts = []
    for _ in range(iters):
        flush_l2()
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        torch.cuda.synchronize()
        e0.record()
        fn()
        e1.record()
        torch.cuda.synchronize()
        ts.append(e0.elapsed_time(e1) * 1e3)
    return statistics.median(ts)


def time_cold_us(fn, iters: int = 15) -> float:
    """One launch from a cold L2, replayed from a CUDA graph so that the host's launch path is not part of the time."""
    fn()
    torch.cuda.synchronize()
    s = torch.cuda.Stream()
    s.wait_stream(torch.cuda.current_stream())
    g = torch.cuda.CUDAGraph()
    with torch.cuda.graph(g, stream=s):
        fn()
    ts = []
    for _ in range(iters):
        flush_l2()
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        torch.cuda.synchronize()
        e0.record()
        g.replay()
        e1.record()
        torch.cuda.synchronize()
        ts.append(e0.elapsed_time(e1) * 1e3)
    return statistics.median(ts)


def report(name: str, us: float, *, flops: float = 0.0, bytes_: float = 0.0, **extra) -> dict:
    pk = peaks()
    out = {"kernel": name, "us": round(us, 2), **extra}
    if flops:
        out["tflops"] = round(flops / us * 1e-6, 1)
        out[f"frac_of_{pk['src']}_tflops"] = round(flops / us * 1e-6 / pk["tflops"], 3)
    if bytes_:
        out["gbs"] = round(bytes_ / us * 1e-3, 1)
        out[f"frac_of_{pk['src']}_hbm"] = round(bytes_ / us * 1e-3 / pk["hbm_gbs"], 3)
    print(json.dumps(out), flush=True)
    return out


def bench_gemm(m, n, k, *, dual=False, packed=False, int8=False, dtype=torch.float16, profile=False, splits=0):
    """In-stream time of one GEMM: launches are chained in a CUDA graph over enough weight copies to defeat L2."""
    from rhinoforge_b200.ops import kernels as K
    rows = 2 * n if dual else n
    wbytes = rows * k * (1 if int8 else 2)
    nbuf = 1 if profile else max(1, min(12, -(-(300 << 20) // wbytes)))
    x = (torch.randn(m, k, device="cuda") * 0.5).to(dtype)
    out = torch.empty(m, n, dtype=dtype, device="cuda")
    sets = []
    for _ in range(nbuf):
        if int8:
            w = torch.randint(-127, 128, (rows, k), device="cuda", dtype=torch.int8)
            sc = (torch.rand(rows, device="cuda") * 0.004 + 0.001).to(dtype)
        else:
            w, sc = (torch.randn(rows, k, device="cuda") * 0.05).to(dtype), None
        sets.append((K.pack_weight(w, 2 if dual else 1) if packed else w, sc))

    def make(i):
        w, sc = sets[i]
        kw = dict(out=out, scale=sc, act="silu_mul" if dual else None, dual=dual, force_splits=splits)
        if packed:
            return lambda: K.gemm(x, w, packed_shape=(rows, k), **kw)
        return lambda: K.gemm(x, w, **kw)
    if profile:
        fn = make(0)
        fn(); torch.cuda.synchronize()
        torch.cuda.profiler.start(); fn(); torch.cuda.synchronize(); torch.cuda.profiler.stop()
        return None
    us = time_graph_us(make, nbuf)
    return report("gemm", us, flops=2.0 * m * rows * k, bytes_=wbytes + m * k * 2 + m * n * 2, m=m, n=n, k=k, dual=dual,
                  packed=packed, int8=int8, splits=splits or "auto", plan=_plan(m, n, k, dual, packed, int8, dtype, splits))


def _plan(m, n, k, dual, packed, int8, dtype, splits):
    """The launch plan the library picks for this shape (swap-AB, tile width, splits, stages, grid, shared memory)."""
    from rhinoforge_b200.ops.kernels import gemm_plan
    try:
        return gemm_plan(m, n, k, dtype=dtype, dual=dual, packed=packed, int8=int8, force_splits=splits)
    except Exception:  # noqa: BLE001  (diagnostic only)
        return None


def bench_attn_prefill(seqs, length, heads, kv_heads, hd, *, causal=True, dtype=torch.float16, profile=False, timer=None):
    from rhinoforge_b200.ops import kernels as K
    T = seqs * length
    qkv = (torch.randn(T, (heads + 2 * kv_heads) * hd, device="cuda") * 0.5).to(dtype)
    out = torch.empty(T, heads * hd, dtype=dtype, device="cuda")
    ql = torch.full((seqs,), length, dtype=torch.int32, device="cuda")
    qs = (torch.arange(seqs, dtype=torch.int32, device="cuda") * length).contiguous()
    q, k, v = qkv[:, :heads * hd], qkv[:, heads * hd:(heads + kv_heads) * hd], qkv[:, (heads + kv_heads) * hd:]
    fn = lambda: K.attention_prefill(q, out, Hq=heads, Hkv=kv_heads, hd=hd, q_start=qs, q_len=ql, kv_len=ql, max_q_len=length,
                                     k=k, v=v, kv_start=qs, causal=causal)
    if profile:
        fn(); torch.cuda.synchronize()
        torch.cuda.profiler.start(); fn(); torch.cuda.synchronize(); torch.cuda.profiler.stop()
        return None
    us = (timer or time_us)(fn)
    flops = 4.0 * seqs * heads * length * length * hd * (0.5 if causal else 1.0)
    return report("attn_prefill", us, flops=flops, seqs=seqs, len=length, heads=heads, kv_heads=kv_heads, hd=hd, causal=causal)


def bench_attn_decode(seqs, length, heads, kv_heads, hd, *, dtype=torch.float16, timer=None):
    from rhinoforge_b200.ops import kernels as K
    from rhinoforge_b200.runtime.kv_cache import PagedKV
    cache = PagedKV(1, seqs, length + 16, kv_heads, hd, dtype=dtype)
    cache.reserve_all()
    cache.kv.normal_(0, 0.5)
    q = (torch.randn(seqs, heads * hd, device="cuda") * 0.5).to(dtype)
    out = torch.empty_like(q)
    kl = torch.full((seqs,), length, dtype=torch.int32, device="cuda")
    ws = K.attn_decode_scratch(seqs, heads, hd, q.device)
    fn = lambda: K.attention_decode(q, out, Hq=heads, Hkv=kv_heads, hd=hd, kv_len=kl, max_kv_len=length, k_pool=cache.kv[0, 0],
                                    v_pool=cache.kv[0, 1], page_table=cache.page_table, ws=ws)
    us = (timer or time_us)(fn)
    r = report("attn_decode", us, bytes_=2.0 * seqs * length * kv_heads * hd * 2, seqs=seqs, len=length, heads=heads,
               kv_heads=kv_heads, hd=hd)
    cache.close()
    return r


def bench_gdn(seqs, length, hk, hv, *, dk=128, dv=128, dtype=torch.float16, timer=None, chunked=False):
    from rhinoforge_b200.ops import kernels as K
    T = seqs * length
    qkv = torch.randn(T, 2 * hk * dk + hv * dv, device="cuda").to(dtype)
    ba = torch.randn(T, 2 * ((hv + 7) // 8 * 8), device="cuda").to(dtype)
    half = ba.shape[1] // 2
    state = torch.zeros(seqs, hv, dk, dv, device="cuda")
    A, dtb = torch.zeros(hv, device="cuda"), torch.zeros(hv, device="cuda")
    ql = torch.full((seqs,), length, dtype=torch.int32, device="cuda")
    qs = (torch.arange(seqs, dtype=torch.int32, device="cuda") * length).contiguous()
    if length == 1:
        fn = lambda: K.gdn_recurrent(qkv, ba[:, :half], ba[:, half:], state, A, dtb, Hk=hk, Hv=hv, Dk=dk, Dv=dv)
    else:
        fn = lambda: K.gdn_recurrent(qkv, ba[:, :half], ba[:, half:], state, A, dtb, Hk=hk, Hv=hv, Dk=dk, Dv=dv, q_start=qs, q_len=ql, chunked=chunked)
    us = timer(fn) if timer else time_us(fn, iters=10)
    return report("gdn_chunked" if chunked else "gdn_recurrent", us, flops=6.0 * T * hv * dk * dv, bytes_=2.0 * seqs * hv * dk * dv * 4, seqs=seqs, len=length,
                  hk=hk, hv=hv, us_per_token=round(us / length, 3))


def time_hot_us(fn, n: int = 50) -> float:
    """Mean in-stream time of ``n`` back-to-back launches of one closure in a CUDA graph, operands L2-resident: the regime
    of the action heads' denoise loops, where the same few MB of weights serve every step."""
    s = torch.cuda.Stream()
    s.wait_stream(torch.cuda.current_stream())
    with torch.cuda.stream(s):
        fn()
    torch.cuda.synchronize()
    g = torch.cuda.CUDAGraph()
    with torch.cuda.graph(g, stream=s):
        for _ in range(n):
            fn()
    g.replay()
    torch.cuda.synchronize()
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    e0.record()
    for _ in range(5):
        g.replay()
    e1.record()
    torch.cuda.synchronize()
    return e0.elapsed_time(e1) * 1e3 / (5 * n)


def heads() -> None:
    """The latency-bound shapes of the action heads: short attention with and without the host-side key bound (which
    selects the register-accumulator kernel), and few-row GEMMs on the kernel the router picks (set ``RF_GEMM_SMALL=0`` to
    time the streaming kernel on the same shapes) against ``torch.matmul``."""
    import math
    from rhinoforge_b200.ops import kernels as K
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device="cuda")
    for name, B, Q, KV, H, hd in (("navdp self", 4, 24, 24, 8, 64), ("navdp cross", 4, 24, 34, 8, 64), ("nextdit self", 4, 32, 32, 12, 64),
                                  ("nextdit cross", 4, 32, 260, 12, 64), ("gr00t self", 1, 41, 41, 32, 64), ("gr00t cross", 1, 41, 148, 32, 64),
                                  ("rgbd self", 1, 32, 32, 6, 64), ("50x350 hd128", 1, 50, 350, 16, 128), ("64x512 hd128", 2, 64, 512, 16, 128)):
        q = torch.randn(B * Q, H * hd, device="cuda", dtype=torch.float16) * 0.3
        k = torch.randn(B * KV, H * hd, device="cuda", dtype=torch.float16) * 0.3
        v = torch.randn(B * KV, H * hd, device="cuda", dtype=torch.float16)
        out = torch.empty_like(q)
        qs, ql, ks, kl = i32([j * Q for j in range(B)]), i32([Q] * B), i32([j * KV for j in range(B)]), i32([KV] * B)
        r = {}
        for arm, bound in (("bounded_us", KV), ("unbounded_us", 0)):
            r[arm] = round(time_hot_us(lambda: K.attention_prefill(q, out, Hq=H, Hkv=H, hd=hd, q_start=qs, q_len=ql, kv_len=kl, max_q_len=Q,
                                                                   k=k, v=v, kv_start=ks, causal=False, scale=1 / math.sqrt(hd),
                                                                   max_kv_len=bound)), 2)
        print(json.dumps({"kernel": "attention_prefill", "case": name, "seqs": B, "q": Q, "kv": KV, "heads": H, "hd": hd, **r}), flush=True)
    for M, N, Kd, dual in ((128, 384, 1536, False), (128, 1536, 384, False), (128, 1152, 384, False), (96, 384, 384, False), (24, 1152, 384, False),
                           (24, 384, 384, False), (31, 1024, 1024, False), (31, 2560, 1024, False), (31, 4096, 1024, True), (50, 2560, 1024, False),
                           (50, 4096, 1024, True), (50, 1024, 2048, False), (41, 4608, 1536, False), (41, 1536, 6144, False)):
        x = torch.randn(M, Kd, device="cuda", dtype=torch.float16)
        w = torch.randn(N * (2 if dual else 1), Kd, device="cuda", dtype=torch.float16) * 0.05
        wp = K.pack_weight(w, sections=2) if dual else K.pack_weight(w)
        out = torch.empty(M, N, device="cuda", dtype=torch.float16)
        kw = dict(act="silu_mul", dual=True) if dual else {}
        us = time_hot_us(lambda: K.gemm(x, wp, packed_shape=(w.shape[0], Kd), out=out, **kw))
        ref = torch.empty(M, w.shape[0], device="cuda", dtype=torch.float16)
        lib = time_hot_us(lambda: torch.matmul(x, w.t(), out=ref))
        print(json.dumps({"kernel": "gemm", "m": M, "n": N, "k": Kd, "dual": dual, "small_kernel": os.environ.get("RF_GEMM_SMALL", "1") != "0",
                          "us": round(us, 2), "torch_matmul_us": round(lib, 2)}), flush=True)


def sweep() -> None:
    """Split-K factors around the planner's choice for the Qwen3-8B decode GEMMs and two mid-size GEMMs."""
    for shape in ((64, 6144, 4096, False), (64, 4096, 4096, False), (64, 12288, 4096, True), (64, 4096, 12288, False),
                  (1, 4096, 4096, False), (768, 6144, 1152, False), (768, 1152, 4304, False), (968, 2048, 16384, False)):
        m, n, k, dual = shape
        for sp in (0, 1, 2, 3, 4, 6, 8):
            if sp > max(1, (k // 64) // 4):
                continue
            bench_gemm(m, n, k, dual=dual, packed=True, splits=sp)


def suite() -> None:
    """Qwen3-8B shapes: the four decode GEMMs at 64 tokens, the same at 2048 tokens, attention at both."""
    for packed in (True,):
        for m in (64, 2048):
            bench_gemm(m, 6144, 4096, packed=packed)                 # qkv
            bench_gemm(m, 4096, 4096, packed=packed)                 # o_proj
            bench_gemm(m, 12288, 4096, dual=True, packed=packed)     # gate/up + SwiGLU
            bench_gemm(m, 4096, 12288, packed=packed)                # down
    bench_gemm(64, 151936, 4096, packed=True)                        # lm_head
    bench_gemm(64, 12288, 4096, dual=True, packed=True, int8=True)
    bench_attn_decode(64, 1024, 32, 8, 128)
    bench_attn_prefill(4, 2048, 32, 8, 128)
    bench_attn_prefill(1, 968, 8, 1, 256, causal=False)              # Pi0.5 prefix
    bench_attn_prefill(3, 256, 16, 16, 128, causal=False)            # SigLIP (72 padded to 128)
    bench_gdn(1, 1, 16, 32)
    bench_gdn(1, 1024, 16, 32)


def bench_mixed(hidden, heads, *, dim=128, vdim=128, rank=512, window=1024, batch=64, prefill=(4, 2048), dtype=torch.bfloat16) -> None:
    """Kernels of a decoder with per-layer mixers (latent attention, HGRN2, fp32 residual stream), each beside the like kernel of
    the K/V and Gated-DeltaNet decoders at equal size."""
    from rhinoforge_b200.ops import kernels as K
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device="cuda")
    tag = dict(hidden=hidden, heads=heads)
    rnd = lambda *sh: torch.randn(*sh, device="cuda", dtype=dtype)
    f32 = lambda *sh: torch.randn(*sh, device="cuda")
    S, Lp = prefill
    T = S * Lp
    seq = i32([j for j in range(S) for _ in range(Lp)])
    pos_p, starts, lens = i32(list(range(Lp)) * S), i32([j * Lp for j in range(S)]), i32([Lp] * S)
    rows_p = lambda **kw: K.rows(pos_p, seq_of_row=seq, q_start=starts, q_len=lens, slot=i32(list(range(S))), **kw)
    # ---- residual stream, decode and prefill rows
    nw, mu, st = f32(hidden), torch.rand(hidden, device="cuda"), f32(max(batch, S), hidden)
    for n, r in ((batch, K.rows(i32([7] * batch))), (T, rows_p())):
        x, y, w16 = f32(n, hidden), rnd(n, hidden), rnd(hidden)
        us = time_cold_us(lambda: K.stream_norm(x, r, dtype=dtype, eps=1e-6, norm_w=nw, y=y, shift=mu, shift_state=st))
        report("stream_norm (add + norm + token shift)", us, bytes_=n * hidden * 12, rows=n, **tag)
        xx, out = rnd(n, hidden), rnd(n, hidden)
        us = time_cold_us(lambda: K.rmsnorm(xx, w16, 1e-6, residual=y, residual_out=xx, out=out))
        report("like: rmsnorm with residual", us, bytes_=n * hidden * 8, rows=n, **tag)
    # ---- latent attention, decode
    wa, wu = rnd(heads, rank, dim) / dim ** 0.5, rnd(heads, vdim, rank) / rank ** 0.5
    q = rnd(batch, heads, dim)
    us = time_cold_us(lambda: K.head_linear(q, wa))
    report("head_linear (query -> latent)", us, bytes_=2 * (wa.numel() + batch * heads * (dim + rank)), flops=2.0 * batch * wa.numel(), rows=batch, **tag)
    ol = rnd(batch, heads, rank)
    us = time_cold_us(lambda: K.head_linear(ol, wu))
    report("head_linear (latent -> value)", us, bytes_=2 * (wu.numel() + batch * heads * (vdim + rank)), flops=2.0 * batch * wu.numel(), rows=batch, **tag)
    del wa, wu
    bench_gemm(batch, rank * heads // 4, dim * 4, packed=True, dtype=dtype)
    for b in (1, batch):
        pages = (window + 15) // 16 + 1
        pool, ql = rnd(b * pages, 16, rank), rnd(b, heads, rank)
        pt = torch.randperm(b * pages, device="cuda").to(torch.int32).view(b, pages)
        r = K.rows(i32([window] * b), page_table=pt)
        us = time_cold_us(lambda: K.latent_attention(ql, pool, r, window=window, scale=0.05, max_kv=window))
        report("latent_attn decode", us, bytes_=2.0 * b * (window * rank + 2 * heads * rank), flops=4.0 * b * heads * window * rank, rows=b, window=window, **tag)
        bench_attn_decode(b, window, heads, max(1, heads // 4), 128, dtype=dtype, timer=time_cold_us)
    # ---- latent attention, prefill: gather + expansion + attention
    pages = (Lp + 15) // 16
    pool = rnd(S * pages, 16, rank)
    pt = torch.randperm(S * pages, device="cuda").to(torch.int32).view(S, pages)
    r = rows_p(page_table=pt)
    us = time_cold_us(lambda: K.latent_gather(pool, r, starts, lens, T, Lp))
    report("latent_gather", us, bytes_=4.0 * T * rank, rows=T, **tag)
    bench_gemm(T, 2 * heads * dim, rank, packed=True, dtype=dtype)
    qq, kv, oo = rnd(T, heads * dim), rnd(T, 2 * heads * dim), rnd(T, heads * dim)
    vis = sum(min(i + 1, window) for i in range(Lp)) * S
    us = time_cold_us(lambda: K.attention_prefill(qq, oo, Hq=heads, Hkv=heads, hd=dim, q_start=starts, q_len=lens, kv_len=lens, max_q_len=Lp,
                                             k=kv[:, :heads * dim], v=kv[:, heads * dim:], kv_start=starts, causal=True, window=window, scale=0.05))
    report("attention over expanded keys (windowed)", us, flops=4.0 * vis * heads * dim, rows=T, window=window, **tag)
    bench_attn_prefill(S, Lp, heads, max(1, heads // 4), 128, dtype=dtype, timer=time_cold_us)
    del qq, kv, oo, pool
    # ---- linear attention
    width = heads * (2 * dim + vdim)
    fb, lo, hw = f32(heads * dim), torch.rand(heads * dim, device="cuda"), f32(vdim)
    for b in (1, batch):
        x, state = rnd(b, width), f32(b, heads, dim, vdim)
        rr = K.rows(i32([5] * b))
        us = time_cold_us(lambda: K.hgrn2(x, fb, lo, hw, state, rr, eps=1e-6))
        report("hgrn2 decode step", us, bytes_=8.0 * state.numel() + 2.0 * b * (width + heads * vdim), rows=b, **tag)
        bench_gdn(b, 1, heads, heads, dtype=dtype, timer=time_cold_us)
    for s_, l_ in ((1, 4096), (S, Lp)):
        x, state = rnd(s_ * l_, width), f32(s_, heads, dim, vdim)
        rr = K.rows(i32(list(range(l_)) * s_), q_start=i32([j * l_ for j in range(s_)]), q_len=i32([l_] * s_))
        us = time_cold_us(lambda: K.hgrn2(x, fb, lo, hw, state, rr, eps=1e-6, chunked=True))
        report("hgrn2 prefill (16-token blocks)", us, flops=s_ * l_ * heads * (4.0 * dim * vdim + 32.0 * dim + 32.0 * vdim),
               bytes_=2.0 * s_ * l_ * (width + heads * vdim), seqs=s_, length=l_, **tag)
        bench_gdn(s_, l_, heads, heads, dtype=dtype, timer=time_cold_us, chunked=True)


def bench_routed(hidden, heads, kv, inner, experts, top, ff, *, chunk=1024, groups=8, keep=4, states=16, batch=64, prefill=(4, 2048),
                 dtype=torch.bfloat16) -> None:
    """Kernels of decoders with chunked grouped attention, selective-scan layers and routed experts, each beside the like kernel of
    the K/V and Gated-DeltaNet decoders at equal size."""
    from rhinoforge_b200.ops import kernels as K
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device="cuda")
    tag = dict(hidden=hidden)
    rnd = lambda *sh: torch.randn(*sh, device="cuda", dtype=dtype)
    f32 = lambda *sh: torch.randn(*sh, device="cuda")
    S, Lp = prefill
    T, hd = S * Lp, 128
    starts, lens = i32([j * Lp for j in range(S)]), i32([Lp] * S)
    seq, pos_p = i32([j for j in range(S) for _ in range(Lp)]), i32(list(range(Lp)) * S)
    rows_p = lambda **kw: K.rows(pos_p, seq_of_row=seq, q_start=starts, q_len=lens, slot=i32(list(range(S))), **kw)
    # ---- residual stream: the experts' rows added up
    for n, r in ((batch, K.rows(i32([7] * batch))), (T, rows_p())):
        x, yw, w16 = f32(n, hidden), f32(hidden), rnd(hidden)
        yg, slots = rnd(n * (top + 1), hidden), torch.randperm(n * (top + 1), device="cuda").to(torch.int32).view(n, top + 1)
        us = time_cold_us(lambda: K.stream_norm(x, r, dtype=dtype, eps=1e-6, y=yg, y_norm_w=yw, cast=True, y_slots=slots))
        report("stream_norm (sum of picked rows, norm of it, add)", us, bytes_=n * hidden * (10 + 2 * (top + 1)), rows=n, picks=top + 1, **tag)
        y1 = rnd(n, hidden)
        us = time_cold_us(lambda: K.stream_norm(x, r, dtype=dtype, eps=1e-6, y=y1, y_norm_w=yw, cast=True))
        report("stream_norm (norm of the output, add)", us, bytes_=n * hidden * 12, rows=n, **tag)
        xx, out = rnd(n, hidden), rnd(n, hidden)
        us = time_cold_us(lambda: K.rmsnorm(xx, w16, 1e-6, residual=y1, residual_out=xx, out=out))
        report("like: rmsnorm with residual", us, bytes_=n * hidden * 8, rows=n, **tag)
        del yg
    # ---- attention
    cos, sin = f32(4096, 32), f32(4096, 32)
    qn, qn16 = f32(hd), rnd(hd)
    for n, r_of, posn in ((batch, lambda **kw: K.rows(i32([chunk - 1] * batch), **kw), i32([chunk - 1] * batch)), (T, rows_p, pos_p)):
        per = (max(Lp, chunk) + 15) // 16
        nseq = batch if n == batch else S
        pt = torch.randperm(nseq * per, device="cuda").to(torch.int32).view(nseq, per)
        kp, vp = rnd(nseq * per, kv, 16, hd), rnd(nseq * per, kv, 16, hd)
        x, first = rnd(n, (2 * heads + 2 * kv) * hd), rnd(n, kv * hd)
        r = r_of(page_table=pt)
        us = time_cold_us(lambda: K.qkv_insert(x, r, kp, vp, heads=heads, kv_heads=kv, hd=hd, eps=1e-6, q_norm=qn, k_norm=qn, cos=cos, sin=sin,
                                               v_first=first, v_role="mix", v_lambda=0.5))
        report("qkv_insert", us, bytes_=n * ((2 * heads + 4 * kv) * hd * 2 + kv * hd * 2), rows=n, heads=heads, kv_heads=kv, **tag)
        x2 = rnd(n, (heads + 2 * kv) * hd)
        us = time_cold_us(lambda: K.qk_norm_rope_kv(x2, heads, kv, hd, pos=posn.view(-1, 1), cos=cos, sin=sin, rot_dim=64, q_norm_w=qn16, k_norm_w=qn16,
                                                    k_pool=kp, v_pool=vp, page_table=pt, seq_of_tok=None if n == batch else seq))
        report("like: qk_norm_rope_kv", us, bytes_=n * (2 * heads + 4 * kv) * hd * 2, rows=n, **tag)
        kw = dict(Hq=heads, Hkv=kv, hd=hd, scale=0.09, sink=f32(heads), gate=x[:, (heads + 2 * kv) * hd:])
        q = x[:, :heads * hd]
        if n == batch:
            for b in (1, batch):
                rb = K.rows(i32([chunk - 1] * b), page_table=pt[:b])
                us = time_cold_us(lambda: K.attention_rows(q[:b], rb, kp, vp, max_kv=chunk, chunk=chunk, **kw))
                report("attention by row (chunk, sink, gate)", us, bytes_=4.0 * b * chunk * kv * hd + 6.0 * b * heads * hd, rows=b, chunk=chunk, **tag)
                bench_attn_decode(b, chunk, heads, kv, hd, dtype=dtype, timer=time_cold_us)
        else:
            out = rnd(n, heads * hd)
            for ch in (chunk, Lp):
                vis = sum(i % ch + 1 for i in range(Lp)) * S
                us = time_cold_us(lambda: K.attention_prefill(q, out, q_start=starts, q_len=lens, kv_len=lens, max_q_len=Lp, k_pool=kp, v_pool=vp,
                                                              page_table=pt, max_kv_len=Lp, chunk=ch, **kw))
                report("attention prefill (chunk, sink, gate)", us, flops=4.0 * vis * heads * hd, rows=n, chunk=ch, **tag)
            bench_attn_prefill(S, Lp, heads, kv, hd, dtype=dtype, timer=time_cold_us)
            bench_attn_prefill(S * Lp // chunk, chunk, heads, kv, hd, dtype=dtype, timer=time_cold_us)
        del kp, vp, x, x2
    # ---- selective scan
    rank = hidden // 16
    a2, D, bias, w_dt = -f32(inner, states).abs(), f32(inner), f32(inner), rnd(inner, rank)
    cw, cb = f32(4, inner), f32(inner)
    for s_, l_ in ((1, 1), (batch, 1), (1, 4096), (S, Lp)):
        n = s_ * l_
        x, z, bc, dt = rnd(n, inner), rnd(n, inner), rnd(n, rank + 2 * states), rnd(n, inner)
        state, cst = f32(s_, inner, states), rnd(s_, 3, inner)
        rr = K.rows(i32([5] * n)) if l_ == 1 else K.rows(i32(list(range(l_)) * s_), q_start=i32([j * l_ for j in range(s_)]), q_len=i32([l_] * s_))
        us = time_cold_us(lambda: K.conv_silu(x, cw, cb, cst, rr, max_q_len=l_))
        report("conv_silu", us, bytes_=4.0 * n * inner + 12.0 * s_ * inner, seqs=s_, length=l_, channels=inner, **tag)
        cw16, cst16 = rnd(inner, 4), rnd(s_, 3, inner)
        us = time_cold_us(lambda: K.causal_conv1d(x, cw16, cst16, q_start=None if l_ == 1 else rr._keep[2], q_len=None if l_ == 1 else rr._keep[3], max_q_len=l_))
        report("like: causal_conv1d", us, bytes_=4.0 * n * inner + 12.0 * s_ * inner, seqs=s_, length=l_, channels=inner, **tag)
        if l_ == 1:
            us = time_cold_us(lambda: K.mamba1(x, z, bc, a2, D, bias, state, rr, w_dt=w_dt))
            report("mamba1 decode step (with step-size projection)", us, bytes_=8.0 * state.numel() + 6.0 * n * inner + 2.0 * w_dt.numel() + 4.0 * a2.numel(),
                   rows=n, channels=inner, states=states, **tag)
        else:
            us = time_cold_us(lambda: K.mamba1(x, z, bc, a2, D, bias, state, rr, dt=dt))
            report("mamba1 scan", us, bytes_=8.0 * n * inner + 2.0 * n * (rank + 2 * states), seqs=s_, length=l_, channels=inner, states=states,
                   exponentials_per_us=round(n * inner * states / us), **tag)
        bench_gdn(s_, l_, heads, heads, dtype=dtype, timer=time_cold_us, chunked=l_ > 1)
        del x, z, bc, dt, state
    # ---- routed experts
    router, corr = rnd(experts, hidden) / hidden ** 0.5, f32(experts) * (0.1 / experts)
    pad = (ff + 127) // 128 * 128
    up = K.pack_weight(rnd(2 * experts * pad, hidden) / hidden ** 0.5, 2)
    down = K.pack_weight(rnd(hidden, experts * pad) / ff ** 0.5)
    for n in (1, 8, batch, 256, T):
        x = rnd(n, hidden)
        small = n <= 256
        b = K.RoutedBatch(x, router, top, correction=corr, groups=groups, keep=keep, tile_rows=(16 if n * top <= 16 * experts else 32) if small else 128, scatter=small)
        us = time_cold_us(b.route)
        report("moe_router (logits, choice, plan)", us, bytes_=2.0 * (n + experts) * hidden, rows=n, experts=experts, top=top, **tag)
        w16 = rnd((experts + 7) // 8 * 8, hidden)

        def like():
            ids, w = K.moe_select(K.gemm(x, w16)[:, :experts], top, score_fn="softmax")
            K.moe_group(ids, w, experts)
        report("like: gemm + moe_select + moe_group", time_cold_us(like), bytes_=2.0 * (n + experts) * hidden, rows=n, **tag)
        b.route()
        torch.cuda.synchronize()
        used = int(b.ids.unique().numel())
        e = dict(rows=n, experts=experts, used=used, ff=ff, **tag)
        if small:
            h = K.moe_experts(b, x, up, n=ff, k=hidden, experts=experts, expert_pad=pad, dual=True)
            us = time_cold_us(lambda: K.moe_experts(b, x, up, n=ff, k=hidden, experts=experts, expert_pad=pad, dual=True))
            report("experts: gate and up", us, bytes_=4.0 * used * ff * hidden + 2.0 * n * top * ff + 2.0 * n * hidden, **e)
            us = time_cold_us(lambda: K.moe_experts(b, h, down, n=hidden, k=ff, experts=experts, expert_pad=pad, gathered=False, weighted=True))
            report("experts: down", us, bytes_=2.0 * used * ff * hidden + 2.0 * n * top * (ff + hidden), **e)
            # a dense GLU with as many weights as the experts that were used
            bench_gemm(n, used * ff // 128 * 128, hidden, dual=True, packed=True, dtype=dtype)
            bench_gemm(n, hidden, used * ff // 128 * 128, packed=True, dtype=dtype)
        else:
            us = time_cold_us(b.gather)
            report("moe_gather", us, bytes_=2.0 * n * hidden * (top + 1), **e)
            xg = b.gather()
            tiles, pairs = b.tiles[3:], n * top
            up_kw = dict(n=pad, k=hidden, bank_rows=experts * pad, bank_k=hidden, expert_rows=pad, dual=True, act="silu_mul", out=rnd(pairs, pad))
            us = time_cold_us(lambda: K.moe_grouped_gemm(xg, up, tiles, **up_kw))
            report("grouped GEMM: gate and up", us, flops=4.0 * pairs * ff * hidden, **e)
            hg, yo = up_kw["out"], rnd(pairs, hidden)
            us = time_cold_us(lambda: K.moe_grouped_gemm(hg, down, tiles, n=hidden, k=pad, bank_rows=hidden, bank_k=experts * pad, expert_k=pad,
                                                         row_scale=b.slot_w[:pairs], out=yo))
            report("grouped GEMM: down", us, flops=2.0 * pairs * ff * hidden, **e)
            bench_gemm(pairs // 4, ff * 4, hidden, dual=True, packed=True, dtype=dtype)
            bench_gemm(pairs // 4, hidden, ff * 4, packed=True, dtype=dtype)


def bench_windowed(hidden, heads, kv, dense, experts, top, ff, *, near=512, far=2048, keep=64, taps=4, batch=64, prefill=(4, 2048), vocab=32768,
                   dtype=torch.bfloat16) -> None:
    """Kernels of decoders with window attention (distance slopes and one norm over all heads; kept first tokens, convolved
    projections and gates per head) and clipped feed-forwards, each beside the like kernel of the chunked-attention decoders at
    equal size."""
    from rhinoforge_b200.ops import kernels as K
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device="cuda")
    tag = dict(hidden=hidden)
    rnd = lambda *sh: torch.randn(*sh, device="cuda", dtype=dtype)
    f32 = lambda *sh: torch.randn(*sh, device="cuda")
    S, Lp = prefill
    T, hd, clip = S * Lp, 128, dict(act="clipped_glu", limit=7.0, alpha=1.702)
    starts, lens = i32([j * Lp for j in range(S)]), i32([Lp] * S)
    seq, pos_p = i32([j for j in range(S) for _ in range(Lp)]), i32(list(range(Lp)) * S)
    rows_p = lambda **kw: K.rows(pos_p, seq_of_row=seq, q_start=starts, q_len=lens, slot=i32(list(range(S))), **kw)
    # ---- residual stream
    table, pair = rnd(vocab, hidden), rnd(4 * vocab + 1, hidden)
    for n, r in ((batch, K.rows(i32([7] * batch))), (T, rows_p())):
        x, nw, yw = f32(n, hidden), f32(hidden), f32(hidden)
        yg, slots = rnd(n * (top + 1), hidden), torch.randperm(n * (top + 1), device="cuda").to(torch.int32).view(n, top + 1)
        y1, ids, last = rnd(n, hidden), torch.randint(0, vocab, (n,), device="cuda").to(torch.int32), i32([0] * n)
        for what, y, sl, traffic in (("sum of picked rows", yg, slots, 2 * (top + 1)), ("one row", y1, None, 2)):
            us = time_cold_us(lambda: K.stream_norm(x, r, dtype=dtype, eps=1e-6, norm_w=nw, y=y, y_slots=sl, y_mult=0.5))
            report(f"stream_norm ({what}, factor, add, norm)", us, bytes_=n * hidden * (10 + traffic), rows=n, **tag)
            us = time_cold_us(lambda: K.stream_norm(x, r, dtype=dtype, eps=1e-6, y=y, y_norm_w=yw, cast=True, y_slots=sl))
            report(f"like: stream_norm ({what}, norm of it, add)", us, bytes_=n * hidden * (10 + traffic), rows=n, **tag)
        us = time_cold_us(lambda: K.stream_norm(None, r, dtype=dtype, eps=1e-6, norm_w=nw, table=table, ids=ids, pairs=(pair, last, 31, 7)))
        report("stream_norm (embedding and token pairs, norm)", us, bytes_=n * hidden * 10, rows=n, **tag)
        us = time_cold_us(lambda: K.stream_norm(None, r, dtype=dtype, eps=1e-6, table=table, ids=ids, cast=True))
        report("like: stream_norm (embedding)", us, bytes_=n * hidden * 8, rows=n, **tag)
        del yg
    del table, pair
    # ---- attention
    cos, sin = f32(4096, 32), f32(4096, 32)
    qn, cols = f32(hd), (heads + 2 * kv) * hd
    cw, slopes, ones = f32(taps, cols), torch.rand(heads, device="cuda"), torch.zeros(heads, device="cuda")
    kw = dict(Hq=heads, Hkv=kv, hd=hd, scale=0.09)
    for n, r_of in ((1, lambda **k: K.rows(i32([far - 1]), **k)), (batch, lambda **k: K.rows(i32([far - 1] * batch), **k)), (T, rows_p)):
        per, nseq = (max(Lp, far) + 15) // 16, S if n == T else n
        pt = torch.randperm(nseq * per, device="cuda").to(torch.int32).view(nseq, per)
        kp, vp = rnd(nseq * per, kv, 16, hd), rnd(nseq * per, kv, 16, hd)
        x, first, state = rnd(n, cols), rnd(n, kv * hd), rnd(nseq, taps - 1, cols)
        r, moved = r_of(page_table=pt), n * (2 * heads + 4 * kv) * hd * 2
        head = dict(heads=heads, kv_heads=kv, hd=hd, eps=1e-6)
        qa, ka = f32(heads, hd), f32(kv, hd)
        us = time_cold_us(lambda: K.qkv_insert(x, r, kp, vp, q_norm=qa, k_norm=ka, norm_all=True, **head))
        report("qkv_insert (one norm over all heads)", us, bytes_=moved, rows=n, heads=heads, kv_heads=kv, **tag)
        us = time_cold_us(lambda: K.qkv_insert(x, r, kp, vp, q_norm=qn, k_norm=qn, cos=cos, sin=sin, conv_w=cw, conv_state=state, max_q_len=1 if n != T else Lp, **head))
        report("qkv_insert (convolution, norms, rotation)", us, bytes_=moved + 4.0 * nseq * (taps - 1) * cols + 4.0 * taps * cols, rows=n, **tag)
        us = time_cold_us(lambda: K.qkv_insert(x, r, kp, vp, q_norm=qn, k_norm=qn, cos=cos, sin=sin, v_first=first, v_role="mix", v_lambda=0.5, **head))
        report("like: qkv_insert (norms, rotation, value mixing)", us, bytes_=moved + n * kv * hd * 2, rows=n, **tag)
        q, gate, gate1 = x[:, :heads * hd], rnd(n, heads * hd), rnd(n, (heads + 7) // 8 * 8)
        forms = (("window and slopes", near, dict(window=near, slopes=slopes)),
                 ("window, kept tokens, one in the denominator, gate per head", far, dict(window=far, keep_first=keep, sink=ones, gate=gate1, gate_by_head=True)),
                 ("window over the kept tokens", near, dict(window=near, keep_first=keep, sink=ones, gate=gate1, gate_by_head=True)),
                 ("like: chunk, sink, gate", near, dict(chunk=near, sink=ones, gate=gate)), ("like: chunk, sink, gate", far, dict(chunk=far, sink=ones, gate=gate)))
        out = rnd(n, heads * hd)
        for what, size, opt in forms:
            seen = lambda i: i % size + 1 if "chunk" in opt else min(i + 1, size) + (min(keep, max(i + 1 - size, 0)) if "keep_first" in opt else 0)
            if n == T:
                us = time_cold_us(lambda: K.attention_prefill(q, out, q_start=starts, q_len=lens, kv_len=lens, max_q_len=Lp, k_pool=kp, v_pool=vp,
                                                              page_table=pt, max_kv_len=Lp, **kw, **opt))
                report(f"attention prefill ({what})", us, flops=4.0 * S * sum(seen(i) for i in range(Lp)) * heads * hd, rows=n, size=size, **tag)
            else:
                us = time_cold_us(lambda: K.attention_rows(q, r, kp, vp, max_kv=far, **kw, **opt))
                report(f"attention by row ({what})", us, bytes_=4.0 * n * seen(far - 1) * kv * hd + 4.0 * n * heads * hd, rows=n, size=size, **tag)
        del kp, vp, x, gate
    # ---- feed-forward and head
    wu, wd = K.pack_weight(rnd(2 * dense, hidden) / hidden ** 0.5, 2), K.pack_weight(rnd(vocab, hidden) / hidden ** 0.5)
    for n in (1, 8, batch, T):
        x = rnd(n, hidden)
        shape = dict(flops=4.0 * n * dense * hidden, bytes_=4.0 * dense * hidden + 2.0 * n * (hidden + dense), rows=n, ff=dense, **tag)
        report("GEMM pair, clipped", time_cold_us(lambda: K.gemm(x, wu, packed_shape=(2 * dense, hidden), dual=True, **clip)), **shape)
        report("like: GEMM pair, silu", time_cold_us(lambda: K.gemm(x, wu, packed_shape=(2 * dense, hidden), dual=True, act="silu_mul")), **shape)
        if n <= 64:
            shape = dict(bytes_=2.0 * vocab * (hidden + n), rows=n, vocab=vocab, **tag)
            report("head with soft cap", time_cold_us(lambda: K.gemm(x, wd, packed_shape=(vocab, hidden), act="soft_cap", limit=30.0)), **shape)
            report("like: head", time_cold_us(lambda: K.gemm(x, wd, packed_shape=(vocab, hidden))), **shape)
    del wu, wd
    router, bias = rnd(experts + 1, hidden) / hidden ** 0.5, f32(experts) * 0.1
    pad = (ff + 127) // 128 * 128
    up = K.pack_weight(rnd(2 * experts * pad, hidden) / hidden ** 0.5, 2)
    down = K.pack_weight(rnd(hidden, experts * pad) / ff ** 0.5)
    for n in (1, 8, batch, T):
        x = rnd(n, hidden)
        small = n <= 256
        plan = dict(tile_rows=(16 if n * top <= 16 * experts else 32) if small else 128, scatter=small, shared=True)
        b = K.RoutedBatch(x, router, top, correction=bias, score_fn="chosen", shared_gate=True, **plan)
        report("moe_router (biased logits, softmax over the chosen, shared weight)", time_cold_us(b.route), bytes_=2.0 * (n + experts) * hidden, rows=n, experts=experts, top=top, **tag)
        like = K.RoutedBatch(x, router[:experts], top, correction=bias, **plan)
        report("like: moe_router (softmax, correction)", time_cold_us(like.route), bytes_=2.0 * (n + experts) * hidden, rows=n, **tag)
        b = K.RoutedBatch(x, router[:experts], top, correction=bias, score_fn="chosen", **dict(plan, shared=False)).route()
        torch.cuda.synchronize()
        used = int(b.ids.unique().numel())
        e = dict(rows=n, experts=experts, used=used, ff=ff, **tag)
        for what, opt in (("experts: gate and up, clipped", clip), ("like: experts: gate and up, silu", {})):
            if small:
                us = time_cold_us(lambda: K.moe_experts(b, x, up, n=ff, k=hidden, experts=experts, expert_pad=pad, dual=True, **opt))
                report(what, us, bytes_=4.0 * used * ff * hidden + 2.0 * n * top * ff + 2.0 * n * hidden, **e)
            else:
                xg, out = b.gather(), rnd(n * top, pad)
                opt = opt or dict(act="silu_mul")
                us = time_cold_us(lambda: K.moe_grouped_gemm(xg, up, b.tiles[3:], n=pad, k=hidden, bank_rows=experts * pad, bank_k=hidden, expert_rows=pad,
                                                             dual=True, out=out, **opt))
                report(what + " (grouped)", us, flops=4.0 * n * top * ff * hidden, **e)


def bench_stated(hidden, heads, kv, experts, identity, top, ff, *, rank=512, q_rank=1536, dim=128, turn=64, near=512, far=2048, taps=4, batch=64,
                 prefill=(4, 2048), dtype=torch.bfloat16) -> None:
    """Kernels of decoders with input convolutions, delta-rule layers, window attention with a logarithmic fall, latent attention with a
    rotated key part, and identity experts, each beside the like kernel of the other decoders at equal size."""
    from rhinoforge_b200.ops import kernels as K
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device="cuda")
    tag = dict(hidden=hidden)
    rnd = lambda *sh: torch.randn(*sh, device="cuda", dtype=dtype)
    f32 = lambda *sh: torch.randn(*sh, device="cuda")
    S, Lp = prefill
    T, hd = S * Lp, 128
    starts, lens = i32([j * Lp for j in range(S)]), i32([Lp] * S)
    seq, pos_p = i32([j for j in range(S) for _ in range(Lp)]), i32(list(range(Lp)) * S)
    rows_p = lambda **kw: K.rows(pos_p, seq_of_row=seq, q_start=starts, q_len=lens, slot=i32(list(range(S))), **kw)
    # ---- residual stream
    nw, yw, cw = f32(hidden), f32(hidden), f32(taps, hidden)
    for n, r in ((batch, K.rows(i32([7] * batch))), (T, rows_p())):
        x, own, sw = f32(n, hidden), rnd(n, hidden), f32(n)
        yg, slots = rnd(n * top, hidden), torch.randperm(n * top, device="cuda").to(torch.int32).view(n, top)
        y1, state = rnd(n, hidden), rnd(max(n, S), taps - 1, hidden)
        conv = dict(conv=(cw, state)) if n == batch else {}
        carried = 4 * (taps - 1) if n == batch else 0
        us = time_cold_us(lambda: K.stream_norm(x, r, dtype=dtype, eps=1e-6, norm_w=nw, y=yg, y_norm_w=yw, y_slots=slots, y_self=(own, sw), **conv))
        report("stream_norm (picked rows and identity, norm of it, add, norm" + (", convolution)" if conv else ")"), us,
               bytes_=n * hidden * (12 + 2 * top + carried), rows=n, **tag)
        us = time_cold_us(lambda: K.stream_norm(x, r, dtype=dtype, eps=1e-6, norm_w=nw, y=y1, y_norm_w=yw, **conv))
        report("stream_norm (norm of the output, add, norm" + (", convolution)" if conv else ")"), us, bytes_=n * hidden * (12 + carried), rows=n, **tag)
        us = time_cold_us(lambda: K.stream_norm(x, r, dtype=dtype, eps=1e-6, y=yg, y_norm_w=yw, cast=True, y_slots=slots))
        report("like: stream_norm (picked rows, norm of it, add)", us, bytes_=n * hidden * (10 + 2 * top), rows=n, **tag)
        us = time_cold_us(lambda: K.stream_norm(x, r, dtype=dtype, eps=1e-6, y=y1, y_norm_w=yw, cast=True))
        report("like: stream_norm (norm of the output, add)", us, bytes_=n * hidden * 12, rows=n, **tag)
        if n == T:
            us = time_cold_us(lambda: K.conv_silu(own, cw, None, state, r, max_q_len=Lp, add=True))
            report("input convolution", us, bytes_=4.0 * n * hidden, rows=n, **tag)
            us = time_cold_us(lambda: K.conv_silu(own, cw, nw, state, r, max_q_len=Lp))
            report("like: conv_silu", us, bytes_=4.0 * n * hidden, rows=n, **tag)
        del yg
    # ---- delta rule
    ch = heads // 2 * 2 * hd + heads * hd
    rate, dt, hw, taps_w = f32(heads).abs(), f32(heads), f32(hd), f32(taps, ch)
    for s_, l_ in ((1, 1), (batch, 1), (1, 4096), (S, Lp), (1, 15)):
        n = s_ * l_
        x, gates, z = rnd(n, ch), rnd(n, 2 * heads), rnd(n, heads * hd)
        state, ring = f32(s_, heads, hd, hd), rnd(s_, taps, ch)
        rr = K.rows(i32([5] * n)) if l_ == 1 else K.rows(i32(list(range(l_)) * s_), q_start=i32([j * l_ for j in range(s_)]), q_len=i32([l_] * s_))
        kw = dict(kv_heads=heads // 2, eps=1e-6)
        bytes_ = 8.0 * state.numel() + 2.0 * n * (ch + 2 * heads * hd)
        e = dict(seqs=s_, length=l_, heads=heads, **tag)
        if l_ > 1:
            us = time_cold_us(lambda: K.conv_silu(x, taps_w, None, ring, rr, max_q_len=l_, ring=True))
            report("short convolution", us, bytes_=4.0 * n * ch, **e)
            us = time_cold_us(lambda: K.delta_rule(x, gates, gates[:, heads:], z, rate, dt, hw, state, rr, chunked=l_ >= 16, **kw))
            report("delta rule, chunks and output norm" if l_ >= 16 else "delta rule, short portion", us, bytes_=bytes_, flops=6.0 * n * heads * hd * hd, **e)
        else:
            us = time_cold_us(lambda: K.delta_rule(x, gates, gates[:, heads:], z, rate, dt, hw, state, rr, conv=(taps_w, ring), **kw))
            report("delta rule, decode step (convolution, norm, gate)", us, bytes_=bytes_ + 2.0 * s_ * taps * ch, **e)
        bench_gdn(s_, l_, heads // 2, heads, dtype=dtype, timer=time_cold_us, chunked=l_ >= 16)
        xg, cst, c16 = rnd(n, ch), rnd(s_, 3, ch), rnd(ch, 4)
        qs, ql = (None, None) if l_ == 1 else (rr._keep[2], rr._keep[3])
        report("like: causal_conv1d", time_cold_us(lambda: K.causal_conv1d(xg, c16, cst, q_start=qs, q_len=ql, max_q_len=l_)), bytes_=4.0 * n * ch, **e)
        zz, w16 = rnd(n, heads * hd), rnd(hd)
        report("like: rmsnorm_gated", time_cold_us(lambda: K.rmsnorm_gated(z, zz, w16, heads, 1e-6)), bytes_=6.0 * n * heads * hd, **e)
    # ---- window attention
    r1, r2, slopes = torch.rand(heads, device="cuda"), torch.rand(heads, device="cuda"), torch.rand(heads, device="cuda")
    cols = (heads + 2 * kv) * hd
    qn, cos, sin = f32(hd), f32(4096, 32), f32(4096, 32)
    for n, r_of in ((1, lambda **k: K.rows(i32([far - 1]), **k)), (batch, lambda **k: K.rows(i32([far - 1] * batch), **k)), (T, rows_p)):
        per, nseq = (max(Lp, far) + 15) // 16, S if n == T else n
        pt = torch.randperm(nseq * per, device="cuda").to(torch.int32).view(nseq, per)
        kp, vp = rnd(nseq * per, kv, 16, hd), rnd(nseq * per, kv, 16, hd)
        x, r, moved = rnd(n, cols), r_of(page_table=pt), n * (2 * heads + 4 * kv) * hd * 2
        head = dict(heads=heads, kv_heads=kv, hd=hd, eps=1e-6)
        report("qkv_insert (growth)", time_cold_us(lambda: K.qkv_insert(x, r, kp, vp, growth=0.1, growth_every=64, **head)), bytes_=moved, rows=n, **tag)
        report("like: qkv_insert (norms, rotation)", time_cold_us(lambda: K.qkv_insert(x, r, kp, vp, q_norm=qn, k_norm=qn, cos=cos, sin=sin, **head)), bytes_=moved, rows=n, **tag)
        q, out = x[:, :heads * hd], rnd(n, heads * hd)
        for what, opt in (("window and logarithmic fall", dict(slopes=r1, rates=r2)), ("like: window and slopes", dict(slopes=slopes))):
            opt = dict(Hq=heads, Hkv=kv, hd=hd, scale=0.09, window=near, **opt)
            if n == T:
                us = time_cold_us(lambda: K.attention_prefill(q, out, q_start=starts, q_len=lens, kv_len=lens, max_q_len=Lp, k_pool=kp, v_pool=vp,
                                                              page_table=pt, max_kv_len=Lp, **opt))
                report(f"attention prefill ({what})", us, flops=4.0 * S * sum(min(i + 1, near) for i in range(Lp)) * heads * hd, rows=n, **tag)
            else:
                us = time_cold_us(lambda: K.attention_rows(q, r, kp, vp, max_kv=far, **opt))
                report(f"attention by row ({what})", us, bytes_=4.0 * n * near * kv * hd + 4.0 * n * heads * hd, rows=n, **tag)
        del kp, vp, x
    # ---- latent attention
    key, wide = dim + turn, rank + turn
    ct, st = f32(4096, turn // 2), f32(4096, turn // 2)
    lw, qw = f32(rank), f32(q_rank)
    wa, wu = rnd(heads, rank, dim) / dim ** 0.5, rnd(heads, hd, rank) / rank ** 0.5
    for b in (1, batch):
        pages = (far + 15) // 16
        pt = torch.randperm(b * pages, device="cuda").to(torch.int32).view(b, pages)
        r = K.rows(i32([far - 1] * b), page_table=pt)
        pool, xin = rnd(b * pages, 16, wide), rnd(b, q_rank + wide)
        us = time_cold_us(lambda: K.latent_insert(xin[:, q_rank:], lw, pool, r, 1e-6, cos=ct, sin=st, q=xin, q_norm=qw))
        report("latent_insert (latent, rotated part, query latent)", us, bytes_=4.0 * b * (wide + q_rank), rows=b, **tag)
        q = rnd(b, heads, key)
        for w_, x_, what in ((wa, q[..., :dim], "query -> latent"), (wu, rnd(b, heads, rank), "latent -> value")):
            report(f"head_linear ({what})", time_cold_us(lambda: K.head_linear(x_, w_)), bytes_=2.0 * (w_.numel() + b * heads * (w_.shape[1] + w_.shape[2])), rows=b, **tag)
        ql = rnd(b, heads, wide)
        us = time_cold_us(lambda: K.latent_attention(ql, pool, r, window=0, scale=0.05, max_kv=far, vrank=rank))
        report("latent_attn decode (rotated part)", us, bytes_=2.0 * b * (far * wide + 2 * heads * rank), flops=2.0 * b * heads * far * (wide + rank), rows=b, keys=far, **tag)
        pl, qp = rnd(b * pages, 16, rank), rnd(b, heads, rank)
        us = time_cold_us(lambda: K.latent_attention(qp, pl, r, window=0, scale=0.05, max_kv=far))
        report("like: latent_attn decode", us, bytes_=2.0 * b * (far * rank + 2 * heads * rank), flops=4.0 * b * heads * far * rank, rows=b, keys=far, **tag)
    pages = (Lp + 15) // 16
    pt = torch.randperm(S * pages, device="cuda").to(torch.int32).view(S, pages)
    pool, r, xin = rnd(S * pages, 16, wide), rows_p(page_table=pt), rnd(T, q_rank + wide)
    us = time_cold_us(lambda: K.latent_insert(xin[:, q_rank:], lw, pool, r, 1e-6, cos=ct, sin=st, q=xin, q_norm=qw))
    report("latent_insert (latent, rotated part, query latent)", us, bytes_=4.0 * T * (wide + q_rank), rows=T, **tag)
    pl, xl = rnd(S * pages, 16, rank), rnd(T, rank)
    report("like: latent_insert", time_cold_us(lambda: K.latent_insert(xl, lw, pl, r, 1e-6)), bytes_=4.0 * T * rank, rows=T, **tag)
    report("latent_gather", time_cold_us(lambda: K.latent_gather(pool, r, starts, lens, T, Lp)), bytes_=4.0 * T * wide, rows=T, **tag)
    report("like: latent_gather", time_cold_us(lambda: K.latent_gather(pl, r, starts, lens, T, Lp)), bytes_=4.0 * T * rank, rows=T, **tag)
    hk, hv = K.latent_heads(key, hd)
    q = rnd(T, heads * hk)
    qv = q.view(T, heads, hk)[..., dim:dim + turn]
    report("head_rotate", time_cold_us(lambda: K.head_rotate(qv, pos_p, ct, st)), bytes_=4.0 * T * heads * turn, rows=T, **tag)
    kv_, oo = rnd(T, heads * (hk + hv)), rnd(T, heads * hv)
    vis = S * Lp * (Lp + 1) // 2
    att = dict(Hq=heads, Hkv=heads, q_start=starts, q_len=lens, kv_len=lens, max_q_len=Lp, kv_start=starts, causal=True, scale=0.05)
    us = time_cold_us(lambda: K.attention_prefill(q, oo, hd=hk, vd=hv, k=kv_[:, :heads * hk], v=kv_[:, heads * hk:], **att))
    report("attention over expanded keys (rotated part)", us, flops=2.0 * vis * heads * (key + hd), rows=T, **tag)
    q1, kv1 = rnd(T, heads * hd), rnd(T, 2 * heads * hd)
    us = time_cold_us(lambda: K.attention_prefill(q1, oo[:, :heads * hd].contiguous(), hd=hd, k=kv1[:, :heads * hd], v=kv1[:, heads * hd:], **att))
    report("like: attention over expanded keys", us, flops=4.0 * vis * heads * hd, rows=T, **tag)
    del q, kv_, oo, q1, kv1, pool, pl, xin, xl
    # ---- experts
    routed = experts + identity
    router, bias = rnd(routed, hidden) / hidden ** 0.5, f32(routed) * (0.25 / routed)
    pad, like_ff = (ff + 127) // 128 * 128, 2 * ff // 3 // 8 * 8
    like_pad = (like_ff + 127) // 128 * 128
    up, down = K.pack_weight(rnd(experts * pad, hidden) / hidden ** 0.5), K.pack_weight(rnd(hidden, experts * pad) / ff ** 0.5)
    like_up = K.pack_weight(rnd(2 * experts * like_pad, hidden) / hidden ** 0.5, 2)
    for n in (1, 8, batch, 256, T):
        x = rnd(n, hidden)
        small = n <= 256
        plan = dict(tile_rows=(16 if n * top <= 16 * experts else 32) if small else 128, scatter=small)
        b = K.RoutedBatch(x, router, top, correction=bias, norm_topk=False, identity=identity, **plan)
        report("moe_router (identity experts)", time_cold_us(b.route), bytes_=2.0 * (n + routed) * hidden, rows=n, experts=routed, top=top, **tag)
        like = K.RoutedBatch(x, router[:experts], top, correction=bias[:experts].contiguous(), **plan)
        report("like: moe_router", time_cold_us(like.route), bytes_=2.0 * (n + experts) * hidden, rows=n, **tag)
        like.route()
        torch.cuda.synchronize()
        used = int(like.ids.unique().numel())
        e = dict(rows=n, experts=experts, used=used, ff=ff, **tag)
        if small:
            h = K.moe_experts(like, x, up, n=ff, k=hidden, experts=experts, expert_pad=pad, act="gelu_erf", stacked=True)
            us = time_cold_us(lambda: K.moe_experts(like, x, up, n=ff, k=hidden, experts=experts, expert_pad=pad, act="gelu_erf", stacked=True))
            report("experts: up, gelu", us, bytes_=2.0 * used * ff * hidden + 2.0 * n * top * ff + 2.0 * n * hidden, **e)
            us = time_cold_us(lambda: K.moe_experts(like, x, like_up, n=like_ff, k=hidden, experts=experts, expert_pad=like_pad, dual=True))
            report("like: experts: gate and up, silu", us, bytes_=4.0 * used * like_ff * hidden + 2.0 * n * top * like_ff + 2.0 * n * hidden, **e)
            us = time_cold_us(lambda: K.moe_experts(like, h, down, n=hidden, k=ff, experts=experts, expert_pad=pad, gathered=False, weighted=True))
            report("experts: down", us, bytes_=2.0 * used * ff * hidden + 2.0 * n * top * (ff + hidden), **e)
        else:
            xg, out, like_out = like.gather(), rnd(n * top, pad), rnd(n * top, like_pad)
            us = time_cold_us(lambda: K.moe_grouped_gemm(xg, up, like.tiles[3:], n=pad, k=hidden, bank_rows=experts * pad, bank_k=hidden, expert_rows=pad,
                                                         act="gelu_erf", out=out))
            report("experts: up, gelu (grouped)", us, flops=2.0 * n * top * ff * hidden, **e)
            us = time_cold_us(lambda: K.moe_grouped_gemm(xg, like_up, like.tiles[3:], n=like_pad, k=hidden, bank_rows=experts * like_pad, bank_k=hidden,
                                                         expert_rows=like_pad, dual=True, act="silu_mul", out=like_out))
            report("like: experts: gate and up, silu (grouped)", us, flops=4.0 * n * top * like_ff * hidden, **e)


def stated() -> None:
    bench_stated(2048, 16, 4, 16, 4, 2, 1536, q_rank=768)
    bench_stated(4096, 32, 8, 64, 16, 6, 2112)


def windowed() -> None:
    bench_windowed(2048, 16, 4, 8192, 16, 2, 1024)
    bench_windowed(4096, 32, 8, 16384, 64, 6, 1408)


def routed() -> None:
    bench_routed(2048, 16, 4, 4096, 16, 2, 1024, groups=4, keep=2)
    bench_routed(4096, 32, 8, 8192, 64, 6, 1408)


def mixed() -> None:
    bench_mixed(2048, 16)
    bench_mixed(4096, 32)


def main() -> int:
    ap = argparse.ArgumentParser(description=__doc__, formatter_class=argparse.RawDescriptionHelpFormatter)
    ap.add_argument("what", choices=["gemm", "attn_prefill", "attn_decode", "gdn", "suite", "sweep", "heads", "mixed", "routed", "windowed", "stated"])
    for name, d in (("m", 64), ("n", 4096), ("k", 4096), ("seqs", 4), ("len", 2048), ("heads", 32), ("kv-heads", 8),
                    ("hd", 128), ("hk", 16), ("hv", 32)):
        ap.add_argument(f"--{name}", type=int, default=d)
    ap.add_argument("--splits", type=int, default=0, help="force the split-K factor (0: planner)")
    ap.add_argument("--dual", action="store_true")
    ap.add_argument("--packed", action="store_true")
    ap.add_argument("--int8", action="store_true")
    ap.add_argument("--bidirectional", action="store_true")
    ap.add_argument("--bf16", action="store_true")
    ap.add_argument("--profile", action="store_true",
                    help="run the kernel once inside cudaProfilerStart/Stop (for ncu --profile-from-start off)")
    a = ap.parse_args()
    dt = torch.bfloat16 if a.bf16 else torch.float16
    if a.what == "gemm":
        bench_gemm(a.m, a.n, a.k, dual=a.dual, packed=a.packed, int8=a.int8, dtype=dt, profile=a.profile, splits=a.splits)
    elif a.what == "attn_prefill":
        bench_attn_prefill(a.seqs, a.len, a.heads, a.kv_heads, a.hd, causal=not a.bidirectional, dtype=dt, profile=a.profile)
    elif a.what == "attn_decode":
        bench_attn_decode(a.seqs, a.len, a.heads, a.kv_heads, a.hd, dtype=dt)
    elif a.what == "gdn":
        bench_gdn(a.seqs, a.len, a.hk, a.hv, dtype=dt)
    elif a.what == "sweep":
        sweep()
    elif a.what == "heads":
        heads()
    elif a.what == "mixed":
        mixed()
    elif a.what == "routed":
        routed()
    elif a.what == "stated":
        stated()
    elif a.what == "windowed":
        windowed()
    else:
        suite()
    return 0


if __name__ == "__main__":
    sys.exit(main())
