"""Plain, slow formulation of the Zulopel decoder for the tests: one function per mechanism, whole sequences, no cache, no
batching, loops over tokens where the definition has them.  Nothing here is shared with the product code.

Notation: rows of a matrix are tokens; ``w`` maps tensor names to tensors; everything is evaluated in the dtype of the weights
handed in (the tests pass float64 or float32)."""
import math

import torch


def rms(x, eps, weight=None):
    y = x / (x.pow(2).mean(-1, keepdim=True) + eps).sqrt()
    return y if weight is None else y * weight


def silu(z):
    return z / (1 + torch.exp(-z))


def softplus(z):
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


# ------------------------------------------------------------------------------------------------ rotary positions
def rotation_frequencies(rot, dtype=torch.float64):
    """One frequency per pair of dimensions and the factor of cos and sin.  With ``scaling``, fast rotations keep their
    frequency, slow ones are divided by the factor, and a linear ramp over the pair index lies between."""
    n, base = rot["dims"], rot["base"]
    f = torch.tensor([base ** (-2.0 * i / n) for i in range(n // 2)], dtype=dtype)
    sc = rot.get("scaling")
    if not sc:
        return f, 1.0
    pair = lambda turns: n * math.log(sc["original"] / (2 * math.pi * turns)) / (2 * math.log(base))
    lo, hi = max(math.floor(pair(sc["fast"])), 0), min(math.ceil(pair(sc["slow"])), n - 1)
    ramp = torch.tensor([min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0) for i in range(n // 2)], dtype=dtype)
    return f / sc["factor"] * ramp + f * (1 - ramp), 0.1 * math.log(sc["factor"]) + 1


def rotate(x, first, rot):
    """``x [tokens, heads, dim]`` of positions first, first + 1, ...: the halves of the first ``dims`` dimensions turn."""
    if not rot:
        return x
    f, factor = rotation_frequencies(rot, x.dtype)
    half = rot["dims"] // 2
    out = x.clone()
    for t in range(x.shape[0]):
        c, s = torch.cos((first + t) * f) * factor, torch.sin((first + t) * f) * factor
        u, v = x[t, :, :half], x[t, :, half:2 * half]
        out[t, :, :half], out[t, :, half:2 * half] = u * c - v * s, v * c + u * s
    return out


# ------------------------------------------------------------------------------------------------ attention
def sink_softmax(scores, sink):
    """Softmax weights whose denominator has one more term, ``exp(sink)``, without a value of its own."""
    top = torch.maximum(scores.max(), sink)
    e = torch.exp(scores - top)
    return e / (e.sum() + torch.exp(sink - top))


def first_visible(i, chunk):
    """First key that position ``i`` sees when positions only see their own chunk of ``chunk`` positions."""
    return i // chunk * chunk if chunk else 0


def attend(q, k, v, scale, sink, chunk):
    """``q [tokens, heads, dim]`` over ``k, v [tokens, kv_heads, ...]``; neighbouring query heads share a key/value head."""
    n, heads = q.shape[:2]
    share = heads // k.shape[1]
    out = torch.zeros(n, heads, v.shape[2], dtype=q.dtype)
    for i in range(n):
        lo = first_visible(i, chunk)
        for a in range(heads):
            g = a // share
            out[i, a] = sink_softmax((k[lo:i + 1, g] @ q[i, a]) * scale, sink[a]) @ v[lo:i + 1, g]
    return out


def mix_values(v, first, lam):
    return (1 - lam) * v + lam * first


def attention(h, w, p, m, eps, v_first):
    """Returns the mixer's output and the values of the first value-mixing layer (this layer's, when there was none yet)."""
    n, heads, kv, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms((h @ w[p + "q"].T).view(n, heads, d), eps, w[p + "q.norm"])
    k = rms((h @ w[p + "k"].T).view(n, kv, d), eps, w[p + "k.norm"])
    v = (h @ w[p + "v"].T).view(n, kv, dv)
    q, k = rotate(q, 0, m.get("rot")), rotate(k, 0, m.get("rot"))
    if m.get("v_mix"):
        if v_first is None:
            v_first = v
        else:
            v = mix_values(v, v_first, w[p + "vmix"])
    o = attend(q, k, v, m["scale"], w[p + "sink"], (m.get("mask") or {}).get("size"))
    o = o.reshape(n, heads * dv) * torch.sigmoid(h @ w[p + "g"].T)
    return o @ w[p + "o"].T, v_first


# ------------------------------------------------------------------------------------------------ selective scan
def causal_convolution(x, taps, bias):
    """Per channel; the last tap meets the current row, rows before the first are zero."""
    n, k = x.shape[0], taps.shape[1]
    padded = torch.cat((torch.zeros(k - 1, x.shape[1], dtype=x.dtype), x), 0)
    return sum(padded[j:j + n] * taps[:, j] for j in range(k)) + bias


def selective_scan(x, dt, A, B, C, D, state):
    """``S <- exp(dt A) S + dt x B``, ``y = S C + D x`` token by token; ``state [channels, states]``."""
    y = torch.zeros_like(x)
    for t in range(x.shape[0]):
        state = torch.exp(dt[t][:, None] * A) * state + (dt[t] * x[t])[:, None] * B[t][None]
        y[t] = state @ C[t] + D * x[t]
    return y, state


def mamba1(h, w, p, m):
    inner, rank, st = m["inner"], m["dt_rank"], m["state"]
    x, z = (h @ w[p + "in"].T).split((inner, inner), -1)
    x = silu(causal_convolution(x, w[p + "conv"], w[p + "conv.b"]))
    dt, B, C = (x @ w[p + "x"].T).split((rank, st, st), -1)
    dt = softplus(dt @ w[p + "dt"].T + w[p + "dt.b"])
    y, _ = selective_scan(x, dt, -torch.exp(w[p + "A_log"]), B, C, w[p + "D"], torch.zeros(inner, st, dtype=h.dtype))
    return (y * silu(z)) @ w[p + "o"].T


# ------------------------------------------------------------------------------------------------ experts
def glu(h, w, p):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def choose(scores, correction, top, groups):
    """Indices of the experts one token uses: the largest corrected scores among those of the best groups, a group counting as
    much as its best expert."""
    key = (scores + correction).tolist()
    count, keep = (groups["count"], groups["keep"]) if groups else (1, 1)
    size = len(key) // count
    best = sorted(range(count), key=lambda g: (-max(key[g * size:(g + 1) * size]), g))[:keep]
    allowed = [e for e in range(len(key)) if e // size in best]
    return sorted(allowed, key=lambda e: (-key[e], e))[:top]


def experts(h, w, p, m):
    r = m["router"]
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        s = torch.softmax(w[p + "router"] @ h[t], 0)
        picks = choose(s, w[p + "correction"], r["top"], r.get("groups"))
        total = sum(s[e] for e in picks) + 1e-20
        for e in picks:
            out[t] += s[e] / total * glu(h[t], w, f"{p}e{e}.")
    return out + glu(h, w, p + "shared.") if m.get("shared") else out


# ------------------------------------------------------------------------------------------------ model
def forward(cfg, w, tokens, taps=None, dtype=torch.float64):
    """Logits ``[tokens, vocab]`` of one sequence; ``taps`` collects the residual stream after every layer."""
    w = {k: (v if v.dtype == torch.int32 else v.to(dtype)) for k, v in w.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][tokens.long()] * (cfg.get("embedding") or {}).get("scale", 1.0)
    v_first = None
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        if layer["type"] == "attention":
            y, v_first = attention(x, w, p + "mix.", layer["mixer"], eps, v_first)
        else:
            y = mamba1(x, w, p + "mix.", layer["mixer"])
        x = x + rms(y, eps, w[p + "norm1"]) * w[p + "ls1"]
        if layer.get("mlp"):
            x = x + rms(experts(x, w, p + "mlp.", layer["mlp"]), eps, w[p + "norm2"]) * w[p + "ls2"]
        if taps is not None:
            taps.append(x.clone())
    return rms(x, eps, w["final.norm"]) @ w["head"].T
