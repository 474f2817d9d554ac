"""Plain, slow restatement of the Nodutar equations in float64/float32 torch, one function per mechanism.

Written for the tests only: it shares no code with the product path, keeps no cache (a sequence is
always computed from its first token) and knows nothing about pages, slots, portions or batches.
"""
from __future__ import annotations

import math

import torch


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_zero(x, w, eps):
    """Weight stored around zero."""
    return unit_rms(x, eps) * (1 + w)


def silu(x):
    return x * torch.sigmoid(x)


def rotate_pairs(x, dims, base, sign=1):
    """x [T, ..., n]: neighbours (2i, 2i + 1) of the first ``dims`` entries turn by sign * position * base^(-2i / dims)."""
    out, T = x.clone(), x.shape[0]
    pos = torch.arange(T, dtype=torch.float64)
    for i in range(dims // 2):
        a = sign * pos * float(base) ** (-2 * i / dims)
        shape = (T,) + (1,) * (x.dim() - 2)
        c, s = torch.cos(a).to(x.dtype).view(shape), torch.sin(a).to(x.dtype).view(shape)
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i], out[..., 2 * i + 1] = u * c - v * s, v * c + u * s
    return out


def visible(T, chunk=None):
    """[T, T] bool: query i sees key j - not after itself and, with ``chunk``, of the same chunk."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    ok = j <= i
    return ok if chunk is None else ok & (i // chunk == j // chunk)


def average(scores, v, seen):
    return torch.softmax(scores.masked_fill(~seen, -math.inf), -1) @ v


def log_distance(T, r1, r2, dtype):
    d = (torch.arange(T)[:, None] - torch.arange(T)[None, :]).clamp(min=0).to(dtype)
    return r1 * torch.log(1 + r2 * d)


def chunk_attention(h, W, m, eps):
    T, H, G, d, e = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    rot = m["rot"]
    q = unit_rms((h @ W["q"].T).view(T, H, d), eps) * W["q.norm"]
    k = unit_rms((h @ W["k"].T).view(T, G, d), eps) * W["k.norm"]
    q, k = rotate_pairs(q, rot["dims"], rot["base"]), rotate_pairs(k, rot["dims"], rot["base"])
    v = rotate_pairs((h @ W["v"].T).view(T, G, e), e, rot["base"])
    seen = visible(T, m["mask"]["size"] if m.get("mask") else None)
    out = torch.zeros(T, H, e, dtype=h.dtype)
    for i in range(H):
        g = i // (H // G)
        out[:, i] = average(q[:, i] @ k[:, g].T * m["scale"], v[:, g], seen)
    return rotate_pairs(out, e, rot["base"], -1).reshape(T, H * e) @ W["o"].T


def gated_state(h, W, m, eps):
    """The state is a moving average of the values, per head and channel at a rate of its own."""
    T, H, d, e = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q, v = silu(h @ W["q"].T).view(T, H, d), (h @ W["v"].T).view(T, H, e)
    low = W["lower"]
    f = (low + (1 - low) * torch.sigmoid(h @ W["f"].T + W["f.b"])).view(T, H, d)
    S, out = torch.zeros(H, d, e, dtype=h.dtype), []
    for t in range(T):
        S = f[t][:, :, None] * S + (1 - f[t])[:, :, None] * v[t][:, None, :]
        out.append(torch.einsum("hde,hd->he", S, q[t]))
    return (unit_rms(torch.stack(out), eps) * W["norm"]).reshape(T, H * e) @ W["o"].T


def part(W, name):
    return {k[len(name) + 1:]: v for k, v in W.items() if k.startswith(name + ".")}


def parallel(h, W, m, eps):
    return (m["left_scale"] * chunk_attention(h, part(W, "left"), m["left"], eps)
            + m["right_scale"] * gated_state(h, part(W, "right"), m["right"], eps))


def distance_attention(h, W, m, eps):
    """Values are the projected keys; scores lose the logarithm of the distance."""
    T, H, G, d = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    q, v = (h @ W["q"].T).view(T, H, d), (h @ W["k"].T).view(T, G, d)
    q, k = unit_rms(q, eps), unit_rms(v, eps)
    out = torch.zeros(T, H, d, dtype=h.dtype)
    for i in range(H):
        g = i // (H // G)
        out[:, i] = average(q[:, i] @ k[:, g].T * m["scale"] - log_distance(T, W["r1"][i], W["r2"][i], h.dtype), v[:, g], visible(T))
    return out.reshape(T, H * d) @ W["o"].T


def route(z, top):
    """Chosen experts [T, top] of logits z and their weights."""
    idx = torch.topk(z, top, dim=-1).indices
    return idx, torch.softmax(torch.gather(z, 1, idx), -1)


def experts(h, W, mlp):
    idx, w = route(h @ W["router"].T + W["router.b"], mlp["router"]["top"])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, we in zip(idx[t].tolist(), w[t]):
            x = h[t]
            out[t] += we * (W[f"e{e}.down"] @ (silu(W[f"e{e}.gate"] @ x) * (W[f"e{e}.up"] @ x)))
    return out


def run_order(cfg):
    """(layer, whether the embedding output is added ahead of it) in the order of execution."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    again = [(i, p > 0 and i == a) for p in range(loop["times"]) for i in range(a, b)]
    return [(i, False) for i in range(a)] + again + [(i, False) for i in range(b, n)]


def forward(cfg: dict, weights: dict, tokens: list[int], dtype=torch.float32, layers_out: list | None = None):
    """Logits [T, vocab] of one sequence from its first token."""
    W = {k: v.to(dtype) if v.is_floating_point() else v for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    first = x = W["embed"][torch.tensor(tokens)]
    for i, again in run_order(cfg):
        layer, p = cfg["layers"][i], f"l{i}."
        if again:
            x = x + first
        mixer = parallel if layer["type"] == "parallel" else distance_attention
        x = x + rms_zero(mixer(rms_zero(x, W[p + "norm1"], eps), part(W, p + "mix"), layer["mixer"], eps), W[p + "norm1b"], eps)
        if layer["mlp"] is not None:
            x = x + rms_zero(experts(rms_zero(x, W[p + "norm2"], eps), part(W, p + "mlp"), layer["mlp"]), W[p + "norm2b"], eps)
        if layers_out is not None:
            layers_out.append(x)
    return rms_zero(x, W["final.norm"], eps) @ W["embed"].T
