"""Plain, slow formulation of the Vasosun decoder for the tests: one function per mechanism, whole sequences, no cache, no batching,
loops over tokens where the definition has them.  Nothing here is shared with the product code.

Notation: rows of a matrix are tokens; ``w`` maps tensor names to tensors; everything is evaluated in the dtype handed in (the tests
pass float64 or float32)."""
import math

import torch


def rms(x, eps, weight):
    """``weight`` is a vector or, for the norms around the sublayers, one number."""
    return x / (x.pow(2).mean(-1, keepdim=True) + eps).sqrt() * weight


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


def gelu(z):
    return 0.5 * z * (1 + torch.erf(z / math.sqrt(2.0)))


def softmax(s):
    e = torch.exp(s - s.max())
    return e / e.sum()


# ------------------------------------------------------------------------------------------------ embedding
def pair_row(previous, token, b):
    """Row of the pair table; a sequence's first token (no previous one) has the row behind the last bucket."""
    return b["buckets"] if previous is None else (previous * b["mul_prev"] + token * b["mul_cur"]) % b["buckets"]


def embed(tokens, w, e):
    ids = [int(t) for t in tokens]
    x = w["embed"][ids]
    if e.get("bigram"):
        x = x + w["bigram"][[pair_row(ids[i - 1] if i else None, t, e["bigram"]) for i, t in enumerate(ids)]]
    return x


# ------------------------------------------------------------------------------------------------ convolutions
def causal_convolution(x, taps):
    """Per channel; the last tap meets the current row, rows before the first are zero."""
    n, k = x.shape[0], taps.shape[1]
    y = torch.zeros_like(x)
    for back in range(min(k, n)):
        y[back:] += x[:n - back] * taps[:, k - 1 - back]
    return y


def input_convolution(h, w, name):
    return h + causal_convolution(h, w[name]) if name in w else h


# ------------------------------------------------------------------------------------------------ window attention
def query_factor(position, q_temp):
    """Growth of the queries with their position."""
    return 1.0 if not q_temp else 1.0 + q_temp["coef"] * math.log((position + 1) // q_temp["every"] + 1)


def log_bias(r1, r2, distance):
    """What a head's score loses at a distance."""
    return r1 * torch.log(1 + r2 * distance)


def heads_of(x, n):
    return x.view(x.shape[0], n, -1)


def attend(q, k, v, scale, size=None, r1=None, r2=None):
    """``q [tokens, heads, dim]`` over ``k, v [tokens, kv_heads, ...]``; neighbouring query heads share a key / value head; a position
    sees the last ``size`` positions, its own included (None: all)."""
    n, heads = q.shape[:2]
    share = heads // k.shape[1]
    out = torch.zeros(n, heads, v.shape[2], dtype=q.dtype)
    for i in range(n):
        js = torch.arange(0 if size is None else max(0, i - size + 1), i + 1)
        for a in range(heads):
            s = (k[js, a // share] @ q[i, a]) * scale
            if r1 is not None:
                s = s - log_bias(r1[a], r2[a], (i - js).to(s.dtype))
            out[i, a] = softmax(s) @ v[js, a // share]
    return out


def window_attention(h, w, p, m, eps, kept):
    q = heads_of(h @ w[p + "q"].T, m["heads"])
    q = q * torch.tensor([query_factor(i, m.get("q_temp")) for i in range(h.shape[0])], dtype=q.dtype)[:, None, None]
    k, v = heads_of(h @ w[p + "k"].T, m["kv_heads"]), heads_of(h @ w[p + "v"].T, m["kv_heads"])
    o = attend(q, k, v, m["scale"], (m.get("mask") or {}).get("size"), w[p + "r1"], w[p + "r2"])
    return o.reshape(h.shape[0], -1) @ w[p + "o"].T


# ------------------------------------------------------------------------------------------------ latent attention
def frequencies(rot):
    """Turning rate of every pair, and the factor on cosine and sine."""
    n, base, y = rot["dims"], rot["base"], rot.get("scaling")
    f = [base ** (-2.0 * i / n) for i in range(n // 2)]
    if not y:
        return f, 1.0
    where = lambda turns: n * math.log(y["original"] / (2 * math.pi * turns)) / (2 * math.log(base))
    lo, hi = max(math.floor(where(y["fast"])), 0), min(math.ceil(where(y["slow"])), n - 1)
    out = []
    for i, x in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(x / y["factor"] * ramp + x * (1 - ramp))
    return out, 0.1 * math.log(y["factor"]) + 1.0


def rotate(x, rot):
    """``x [tokens, heads, dims]``: even dimensions turn with the odd ones behind them."""
    f, amp = frequencies(rot)
    out = torch.zeros_like(x)
    for t in range(x.shape[0]):
        for i, rate in enumerate(f):
            c, s = amp * math.cos(t * rate), amp * math.sin(t * rate)
            u, v = x[t, :, 2 * i], x[t, :, 2 * i + 1]
            out[t, :, 2 * i], out[t, :, 2 * i + 1] = u * c - v * s, v * c + u * s
    return out


def latent_rows(h, w, p, m, eps):
    """What a layer caches per token: the normalised latent and the rotated key part all heads share."""
    z = h @ w[p + "dkv"].T
    return rms(z[:, :m["kv_rank"]], eps, w[p + "dkv.norm"]), rotate(z[:, None, m["kv_rank"]:], m["rot"])


def latent_attention(h, w, p, m, eps, kept):
    n = h.shape[0]
    q = heads_of(rms(h @ w[p + "dq"].T, eps, w[p + "dq.norm"]) @ w[p + "uq"].T, m["heads"])
    q = torch.cat((q[:, :, :m["dim"]], rotate(q[:, :, m["dim"]:], m["rot"])), 2)
    c, turned = kept[m["kv_from"]] if m.get("kv_from") is not None else latent_rows(h, w, p, m, eps)
    kept[int(p.split(".")[0][1:])] = (c, turned)
    k = torch.cat((heads_of(c @ w[p + "uk"].T, m["heads"]), turned.expand(n, m["heads"], -1)), 2)
    o = attend(q, k, heads_of(c @ w[p + "uv"].T, m["heads"]), m["scale"])
    return o.reshape(n, -1) @ w[p + "o"].T


# ------------------------------------------------------------------------------------------------ delta rule
def unit(x):
    return x / (x.pow(2).sum(-1, keepdim=True) + 1e-6).sqrt()


def delta_rule(q, k, v, beta, decay, state=None):
    """``q, k [tokens, heads, dim]``, ``v [tokens, heads, vdim]``, ``beta, decay [tokens, heads]`` -> outputs and the last state."""
    n, heads, dim = q.shape
    s = torch.zeros(heads, dim, v.shape[2], dtype=q.dtype) if state is None else state.clone()
    out = torch.zeros(n, heads, v.shape[2], dtype=q.dtype)
    for t in range(n):
        s = s * decay[t, :, None, None]
        u = beta[t, :, None] * (v[t] - torch.einsum("hkv,hk->hv", s, k[t]))
        s = s + k[t, :, :, None] * u[:, None, :]
        out[t] = torch.einsum("hkv,hk->hv", s, q[t])
    return out, s


def delta(h, w, p, m, eps, kept):
    q, k, v = (silu(causal_convolution(h @ w[p + x].T, w[f"{p}{x}.conv"])) for x in "qkv")
    share = m["heads"] // m["kv_heads"]
    q = (unit(heads_of(q, m["kv_heads"])) * m["dim"] ** -0.5).repeat_interleave(share, 1)
    k = unit(heads_of(k, m["kv_heads"])).repeat_interleave(share, 1)
    beta = sigmoid(h @ w[p + "b"].T)
    decay = torch.exp(-torch.exp(w[p + "A_log"]) * softplus(h @ w[p + "a"].T + w[p + "dt_bias"]))
    o, _ = delta_rule(q, k, heads_of(v, m["heads"]), beta, decay)
    o = rms(o, eps, w[p + "norm"]) * silu(heads_of(h @ w[p + "g"].T, m["heads"]))
    return o.reshape(h.shape[0], -1) @ w[p + "o"].T


# ------------------------------------------------------------------------------------------------ feed-forward
def gated_unit(h, w, p):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def expert(h, w, p):
    return gelu(h @ w[p + "up"].T) @ w[p + "down"].T


def choose(logits, correction, top):
    """The chosen entries and their weights: softmax scores over all entries, the correction only for the choice."""
    s = softmax(logits)
    c = (s + correction).tolist()
    picks = sorted(range(len(c)), key=lambda e: (-c[e], e))[:top]
    return picks, s[picks]


def experts(h, w, p, m):
    r = m["router"]
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        picks, weights = choose(w[p + "router"] @ h[t], w[p + "correction"], r["top"])
        for e, a in zip(picks, weights):
            out[t] += a * (expert(h[t], w, f"{p}e{e}.") if e < r["experts"] else h[t])
    return out


def feed_forward(h, w, p, m):
    return experts(h, w, p, m) if m["kind"] == "moe" else gated_unit(h, w, p)


# ------------------------------------------------------------------------------------------------ model
MIXERS = {"attention": window_attention, "latent_attention": latent_attention, "delta": delta}


def soft_cap(z, cap):
    return cap * torch.tanh(z / cap) if cap else z


def forward(cfg, w, tokens, taps=None, dtype=torch.float64):
    """Logits ``[tokens, vocab]`` of one sequence; ``taps`` collects the residual stream after every layer."""
    w = {k: v.to(dtype) for k, v in w.items()}
    eps = cfg["norm"]["eps"]
    x = embed(tokens, w, cfg.get("embedding") or {})
    kept = {}
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        h = input_convolution(rms(x, eps, w[p + "norm1"]), w, p + "canon1")
        x = x + rms(MIXERS[layer["type"]](h, w, p + "mix.", layer["mixer"], eps, kept), eps, w[p + "norm1b"])
        if layer.get("mlp"):
            h = input_convolution(rms(x, eps, w[p + "norm2"]), w, p + "canon2")
            x = x + rms(feed_forward(h, w, p + "mlp.", layer["mlp"]), eps, w[p + "norm2b"])
        if taps is not None:
            taps.append(x.clone())
    return soft_cap(rms(x, eps, w["final.norm"]) @ w["head"].T, cfg.get("logit_softcap"))
