"""Plain, slow formulation of the Vabarax decoder for the tests: one function per mechanism, whole sequences, no cache,
no batching, loops over tokens where the definition has them.  Nothing here is shared with the product code.

Notation: rows of a matrix are tokens; ``w`` maps tensor names to tensors; everything is evaluated in the dtype of the
weights handed in (the tests pass float64 or float32)."""
import math

import torch


def rms(x, eps, weight=None):
    y = x / (x.pow(2).mean(-1, keepdim=True) + eps).sqrt()
    return y if weight is None else y * weight


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def token_shift(h, mu, previous=None):
    """Mix every row with the row before it; ``previous`` is the row before the first one (zeros when there is none)."""
    before = torch.zeros_like(h[:1]) if previous is None else previous[None]
    shifted = torch.cat((before, h[:-1]), 0)
    return h + (shifted - h) * mu


def latent_attention(h, w, p, m, eps):
    """Softmax attention whose keys and values are linear maps of one small latent row per token."""
    n, heads, d, dv, window = h.shape[0], m["heads"], m["dim"], m["vdim"], m.get("mask", {}).get("size", h.shape[0])
    q = (h @ w[p + "q"].T).view(n, heads, d)
    c = rms(h @ w[p + "dkv"].T, eps, w[p + "dkv.norm"])
    k = (c @ w[p + "uk"].T).view(n, heads, d)
    v = (c @ w[p + "uv"].T).view(n, heads, dv)
    out = torch.zeros(n, heads, dv, dtype=h.dtype)
    for i in range(n):
        lo = max(0, i - window + 1)
        for a in range(heads):
            s = (k[lo:i + 1, a] @ q[i, a]) * m["scale"]
            out[i, a] = torch.softmax(s, 0) @ v[lo:i + 1, a]
    return out.reshape(n, heads * dv) @ w[p + "o"].T


def gated_recurrence(q, f, v, state):
    """``S <- diag(f) S + (1 - f) v^T``, ``o = S^T q`` token by token for one head; returns the outputs and the last state."""
    out = torch.zeros_like(v)
    for t in range(v.shape[0]):
        state = f[t][:, None] * state + torch.outer(1 - f[t], v[t])
        out[t] = state.T @ q[t]
    return out, state


def hgrn2(h, w, p, m, eps):
    n, heads, d, dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    z = h @ w[p + "q"].T
    q = (z * torch.sigmoid(z)).view(n, heads, d)
    lower = w[p + "lower"]
    f = (lower + (1 - lower) * torch.sigmoid(h @ w[p + "f"].T + w[p + "f.b"])).view(n, heads, d)
    v = (h @ w[p + "v"].T).view(n, heads, dv)
    out = torch.zeros(n, heads, dv, dtype=h.dtype)
    for a in range(heads):
        o, _ = gated_recurrence(q[:, a], f[:, a], v[:, a], torch.zeros(d, dv, dtype=h.dtype))
        out[:, a] = rms(o, eps, w[p + "norm"])
    return out.reshape(n, heads * dv) @ w[p + "o"].T


def dense_mlp(h, w, p):
    return torch.relu(h @ w[p + "up"].T).pow(2) @ w[p + "down"].T


def side_input(x, ids, w, p, layer, dim, eps):
    e = w["side.embed"][ids][:, layer * dim:(layer + 1) * dim]
    y = (gelu_tanh(x @ w[p + "gate"].T) * e) @ w[p + "proj"].T
    return x + rms(y, eps, w[p + "norm"])


def forward(cfg, weights, ids, taps=None, dtype=torch.float64):
    """Logits of every position of one sequence; ``taps`` (a list) receives the residual stream after every layer."""
    w = {k: v.to(dtype) for k, v in weights.items()}
    eps, ids = cfg["norm"]["eps"], torch.as_tensor(ids, dtype=torch.long)
    x = w["embed"][ids]
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        h = token_shift(rms(x, eps, w[p + "norm1"]), w[p + "shift"])
        mixer = {"latent_attention": latent_attention, "hgrn2": hgrn2}[layer["type"]]
        x = x + mixer(h, w, p + "mix.", layer["mixer"], eps)
        if layer["mlp"] is not None:
            assert layer["mlp"]["kind"] == "dense"
            x = x + dense_mlp(rms(x, eps, w[p + "norm2"]), w, p + "mlp.")
        x = side_input(x, ids, w, p + "side.", i, cfg["token_side"]["dim"], eps)
        if taps is not None:
            taps.append(x.clone())
    return rms(x, eps, w["final.norm"]) @ w["embed"].T
