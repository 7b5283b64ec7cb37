"""Plain, slow formulation of the Kuzupel decoder for the tests: one function per mechanism, whole sequences, no cache, no
batching, loops over tokens where the definition has them.  Nothing here is shared with the product code.

Notation: rows of a matrix are tokens; ``w`` maps tensor names to tensors; everything is evaluated in the dtype of the weights
handed in (the tests pass float64 or float32)."""
import torch


def rms(x, eps, weight):
    return x / (x.pow(2).mean(-1, keepdim=True) + eps).sqrt() * weight


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


# ------------------------------------------------------------------------------------------------ embedding
def bigram_row(previous, token, b):
    """Row of the pair table; a sequence's first token (no previous one) has the row behind the last bucket."""
    if previous is None:
        return b["buckets"]
    return (previous * b["mul_prev"] + token * b["mul_cur"]) % b["buckets"]


def embed(tokens, w, e):
    ids = [int(t) for t in tokens]
    x = w["embed"][ids] * e.get("scale", 1.0)
    if e.get("bigram"):
        rows = [bigram_row(ids[i - 1] if i else None, t, e["bigram"]) for i, t in enumerate(ids)]
        x = x + w["bigram"][rows]
    return x


# ------------------------------------------------------------------------------------------------ attention
def causal_convolution(x, taps):
    """Per channel; the last tap meets the current row, rows before the first are zero."""
    n, k = x.shape[0], taps.shape[1]
    y = torch.zeros_like(x)
    for t in range(n):
        for j in range(k):
            s = t - (k - 1) + j
            if s >= 0:
                y[t] += taps[:, j] * x[s]
    return y


def rotate(x, first, rot):
    """``x [tokens, heads, dim]`` of positions first, first + 1, ...: dimension i of the first ``dims`` turns with i + dims / 2."""
    if not rot:
        return x
    n = rot["dims"]
    half = n // 2
    f = torch.tensor([rot["base"] ** (-2.0 * i / n) for i in range(half)], dtype=torch.float64)
    out = x.clone()
    for t in range(x.shape[0]):
        a = (first + t) * f
        c, s = torch.cos(a).to(x.dtype), torch.sin(a).to(x.dtype)
        u, v = x[t, :, :half], x[t, :, half:n]
        out[t, :, :half], out[t, :, half:n] = u * c - v * s, v * c + u * s
    return out


def slope(head, heads):
    """How much a head's scores fall per token of distance."""
    return 2.0 ** (-8.0 * (head + 1) / heads)


def visible(i, mask):
    """Positions that position ``i`` sees: the last ``size`` ones, its own included, and the first ``keep_first``."""
    mask = mask or {}
    size, keep = mask.get("size"), mask.get("keep_first", 0)
    return [j for j in range(i + 1) if size is None or i - j < size or j < keep]


def softmax(scores, with_one):
    """Softmax weights; ``with_one`` adds exp(0) to the denominator."""
    top = scores.max()
    if with_one:
        top = torch.clamp(top, min=0.0)
    e = torch.exp(scores - top)
    return e / (e.sum() + torch.exp(-top)) if with_one else e / e.sum()


def attend(q, k, v, scale, mask, distance_bias, with_one):
    """``q [tokens, heads, dim]`` over ``k, v [tokens, kv_heads, ...]``; neighbouring query heads share a key/value head."""
    n, heads = q.shape[:2]
    share = heads // k.shape[1]
    out = torch.zeros(n, heads, v.shape[2], dtype=q.dtype)
    for i in range(n):
        js = torch.tensor(visible(i, mask))
        for a in range(heads):
            s = (k[js, a // share] @ q[i, a]) * scale
            if distance_bias:
                s = s - slope(a, heads) * (i - js).to(s.dtype)
            out[i, a] = softmax(s, with_one) @ v[js, a // share]
    return out


def heads_of(x, n):
    return x.view(x.shape[0], n, -1)


def biased_attention(h, w, p, m, eps):
    """Distance-biased attention; one norm over all query heads together, and over all key heads."""
    q = heads_of(rms(h @ w[p + "q"].T, eps, w[p + "q.norm"]), m["heads"])
    k = heads_of(rms(h @ w[p + "k"].T, eps, w[p + "k.norm"]), m["kv_heads"])
    v = heads_of(h @ w[p + "v"].T, m["kv_heads"])
    o = attend(q, k, v, m["scale"], m.get("mask"), True, False)
    return o.reshape(h.shape[0], -1) @ w[p + "o"].T


def rotary_attention(h, w, p, m, eps):
    """Convolved projections, a norm per head, rotation, the one in the denominator, a gate per head."""
    q, k, v = (causal_convolution(h @ w[p + x].T, w[f"{p}{x}.conv"]) for x in "qkv")
    q = rotate(rms(heads_of(q, m["heads"]), eps, w[p + "q.norm"]), 0, m.get("rot"))
    k = rotate(rms(heads_of(k, m["kv_heads"]), eps, w[p + "k.norm"]), 0, m.get("rot"))
    o = attend(q, k, heads_of(v, m["kv_heads"]), m["scale"], m.get("mask"), False, True)
    o = o * sigmoid(h @ w[p + "g"].T)[:, :, None]
    return o.reshape(h.shape[0], -1) @ w[p + "o"].T


# ------------------------------------------------------------------------------------------------ feed-forward
def clipped_glu(h, w, p, limit):
    g = torch.clamp(h @ w[p + "gate"].T, max=limit)
    u = torch.clamp(h @ w[p + "up"].T, min=-limit, max=limit)
    return (g * sigmoid(1.702 * g) * (u + 1)) @ w[p + "down"].T


def choose(logits, top):
    """The chosen experts and their weights: a softmax over the chosen logits alone."""
    z = logits.tolist()
    picks = sorted(range(len(z)), key=lambda e: (-z[e], e))[:top]
    chosen = logits[picks]
    e = torch.exp(chosen - chosen.max())
    return picks, e / e.sum()


def experts(h, w, p, m):
    r = m["router"]
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        picks, weights = choose(w[p + "router"] @ h[t] + w[p + "router.b"], r["top"])
        for e, a in zip(picks, weights):
            out[t] += a * clipped_glu(h[t], w, f"{p}e{e}.", m["expert"]["limit"])
    if m.get("shared"):
        out = out + sigmoid(h @ w[p + "shared.sg"].T) * clipped_glu(h, w, p + "shared.", m["shared"]["limit"])
    return out


def feed_forward(h, w, p, m):
    return experts(h, w, p, m) if m["kind"] == "moe" else clipped_glu(h, w, p, m["limit"])


# ------------------------------------------------------------------------------------------------ model
def soft_cap(z, cap):
    return cap * torch.tanh(z / cap) if cap else z


def forward(cfg, w, tokens, taps=None, dtype=torch.float64):
    """Logits ``[tokens, vocab]`` of one sequence; ``taps`` collects the residual stream after every layer."""
    w = {k: (v if v.dtype == torch.int32 else v.to(dtype)) for k, v in w.items()}
    eps, m = cfg["norm"]["eps"], cfg.get("residual_mult", 1.0)
    x = embed(tokens, w, cfg.get("embedding") or {})
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        mixer = biased_attention if layer["type"] == "attention" else rotary_attention
        x = x + m * mixer(rms(x, eps, w[p + "norm1"]), w, p + "mix.", layer["mixer"], eps)
        if layer.get("mlp"):
            x = x + m * feed_forward(rms(x, eps, w[p + "norm2"]), w, p + "mlp.", layer["mlp"])
        if taps is not None:
            taps.append(x.clone())
    return soft_cap(rms(x, eps, w["final.norm"]) @ w["head"].T, cfg.get("logit_softcap"))
