"""Plain, slow restatement of the Fasolorn equations in float64/float32 torch, one function per mechanism.

Written for the tests only: it shares no code with the product path, keeps no cache (a sequence is
always computed from its first token) and knows nothing about pages, slots, portions or batches.
"""
from __future__ import annotations

import math

import torch


def rms(x, w, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def silu(x):
    return x * torch.sigmoid(x)


def angles(T, i, dims, base, dtype):
    a = torch.arange(T, dtype=torch.float64) * float(base) ** (-2 * i / dims)
    return torch.cos(a).to(dtype), torch.sin(a).to(dtype)


def turn(x, a, b, i, dims, base, out):
    """Entries ``a`` and ``b`` of x [T, ..., n] turn together by position * base^(-2i / dims)."""
    T = x.shape[0]
    shape = (T,) + (1,) * (x.dim() - 2)
    c, s = (t.view(shape) for t in angles(T, i, dims, base, x.dtype))
    out[..., a], out[..., b] = x[..., a] * c - x[..., b] * s, x[..., b] * c + x[..., a] * s


def rotate_pairs(x, dims, base):
    """Neighbours (2i, 2i + 1) of the first ``dims`` entries are a pair."""
    out = x.clone()
    for i in range(dims // 2):
        turn(x, 2 * i, 2 * i + 1, i, dims, base, out)
    return out


def rotate_halves(x, dims, base):
    """Entry i of the first ``dims`` is paired with entry i + dims / 2."""
    out = x.clone()
    for i in range(dims // 2):
        turn(x, i, i + dims // 2, i, dims, base, out)
    return out


def visible(T, window):
    """[T, T] bool: query i sees key j (``window`` None: everything up to itself)."""
    d = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    return (d >= 0) & (d < (T if window is None else window))


def windowed_average(scores, v, window, sink=None):
    """Softmax over the visible keys of scores [T, T] (with ``sink`` one more entry that carries no value), times v [T, e]."""
    s = scores.masked_fill(~visible(scores.shape[0], window), -math.inf)
    m = s.max(-1, keepdim=True).values
    if sink is not None:
        m = torch.maximum(m, sink.expand_as(m))
    p = torch.exp(s - m)
    den = p.sum(-1, keepdim=True)
    if sink is not None:
        den = den + torch.exp(sink - m)
    return (p / den) @ v


def window_of(m):
    return m["mask"]["size"] if m.get("mask") else None


def attention(h, W, m, first_values):
    """Returns the mixer's result and the layer's own values (before mixing)."""
    T, H, G, d, e = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rotate_pairs((h @ W["q"].T).view(T, H, d), m["rot"]["dims"], m["rot"]["base"])
    k = rotate_pairs((h @ W["k"].T).view(T, G, d), m["rot"]["dims"], m["rot"]["base"])
    own = h @ W["v"].T
    v = own
    if m.get("v_mix") and first_values is not None:
        v = (1 - W["vmix"]) * own + W["vmix"] * first_values
    v = v.view(T, G, e)
    out = torch.zeros(T, H, e, dtype=h.dtype)
    for i in range(H):
        g = i // (H // G)
        out[:, i] = windowed_average(q[:, i] @ k[:, g].T * m["scale"], v[:, g], window_of(m), W["sink"][i])
    out = out.reshape(T, H * e) * torch.sigmoid(h @ W["g"].T)
    return out @ W["o"].T, own


def latent_attention(h, W, m, eps):
    T, H, n, r, e, R = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    rot = (m["rot"]["dims"], m["rot"]["base"])
    q = (h @ W["q"].T).view(T, H, n + r)
    qn, qr = q[..., :n], rotate_halves(q[..., n:], *rot)
    low = h @ W["dkv"].T
    c, kr = rms(low[:, :R], W["dkv.norm"], eps), rotate_halves(low[:, R:], *rot)
    k, v = (c @ W["uk"].T).view(T, H, n), (c @ W["uv"].T).view(T, H, e)
    out = torch.zeros(T, H, e, dtype=h.dtype)
    for i in range(H):
        out[:, i] = windowed_average((qn[:, i] @ k[:, i].T + qr[:, i] @ kr.T) * m["scale"], v[:, i], window_of(m))
    return out.reshape(T, H * e) @ W["o"].T


def swiglu(h, W):
    return (silu(h @ W["gate"].T) * (h @ W["up"].T)) @ W["down"].T


def squared_relu(h, up, down):
    return torch.relu(h @ up.T) ** 2 @ down.T


def route(z, correction, router):
    """Chosen outputs [T, top] and their weights."""
    s = torch.softmax(z, -1)
    idx = torch.topk(s + correction, router["top"], dim=-1).indices
    w = torch.gather(s, 1, idx)
    return idx, w / (w.sum(-1, keepdim=True) + 1e-20) * router["scale"]


def experts(h, W, mlp):
    r = mlp["router"]
    idx, w = route(h @ W["router"].T, W["correction"], r)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, we in zip(idx[t].tolist(), w[t]):
            one = h[t:t + 1]
            y = squared_relu(one, W[f"e{e}.up"], W[f"e{e}.down"]) if e < r["experts"] else one
            out[t] += we * y[0]
    if mlp.get("shared"):
        out = out + squared_relu(h, W["shared.up"], W["shared.down"])
    return out


def layer_tensors(W, i, part):
    p = f"l{i}.{part}."
    return {k[len(p):]: v for k, v in W.items() if k.startswith(p)}


def forward(cfg: dict, weights: dict, tokens: list[int], dtype=torch.float32, layers_out: list | None = None):
    """Logits [T, vocab] of one sequence from its first token."""
    W = {k: v.to(dtype) if v.is_floating_point() else v for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    x = W["embed"][torch.tensor(tokens)] * cfg["embedding"]["scale"]
    first = None
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        h, mix = rms(x, W[p + "norm1"], eps), layer_tensors(W, i, "mix")
        if layer["type"] == "attention":
            y, own = attention(h, mix, m, first)
            if m.get("v_mix") and first is None:
                first = own
        else:
            y = latent_attention(h, mix, m, eps)
        x = x + y
        if layer["mlp"] is not None:
            h, ff = rms(x, W[p + "norm2"], eps), layer_tensors(W, i, "mlp")
            x = x + (experts(h, ff, layer["mlp"]) if layer["mlp"]["kind"] == "moe" else swiglu(h, ff))
        if layers_out is not None:
            layers_out.append(x)
    return rms(x, W["final.norm"], eps) @ W["embed"].T
