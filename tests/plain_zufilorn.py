"""Plain, slow restatement of the Zufilorn equations in float64/float32 torch, one function per mechanism.

Written for the tests only: it shares no code with the product path, keeps no cache (a sequence is
always computed from its first token, token by token in the recurrences) and knows nothing about
pages, slots, chunks or batches.
"""
from __future__ import annotations

import math

import torch


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def centred_norm(x, w, eps):
    return rms(x, eps) * (1 + w)


def silu(x):
    return x * torch.sigmoid(x)


def softplus(x):
    return torch.where(x > 30, x, torch.log1p(torch.exp(torch.clamp(x, max=30))))


def embed(W, tokens, dtype):
    idx = torch.tensor(tokens)
    return W["embed"][idx].to(dtype) + W["pos"][: len(tokens)].to(dtype)


def short_conv(x, taps):
    """x [T, C], taps [C, n]; the last tap multiplies the current row; zeros before the start."""
    T, n = x.shape[0], taps.shape[1]
    out = torch.zeros_like(x)
    for t in range(T):
        for j in range(n):
            src = t - (n - 1) + j
            if src >= 0:
                out[t] += taps[:, j] * x[src]
    return out


def delta_rule(q, k, v, g, beta):
    """q, k [T, G, d] unit vectors (q already scaled), v [T, H, e], g [T, H, d] decays, beta [T, H] -> o [T, H, e]."""
    T, H, e = v.shape
    per = H // q.shape[1]
    out = torch.zeros_like(v)
    for h in range(H):
        S = torch.zeros(q.shape[2], e, dtype=v.dtype)
        for t in range(T):
            kt, qt = k[t, h // per], q[t, h // per]
            S = g[t, h][:, None] * S
            u = beta[t, h] * (v[t, h] - S.T @ kt)
            S = S + kt[:, None] * u[None, :]
            out[t, h] = S.T @ qt
    return out


def channel_delta(h, W, m, eps):
    T = h.shape[0]
    H, G, d, e = m["heads"], m["kv_heads"], m["dim"], m["vdim"]

    def branch(name):
        return silu(short_conv(h @ W[name].T, W[name + ".conv"]))

    def unit(x):
        return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)

    q = unit(branch("q").view(T, G, d)) * d ** -0.5
    k = unit(branch("k").view(T, G, d))
    v = branch("v").view(T, H, e)
    beta = torch.sigmoid(h @ W["b"].T)
    pre = softplus((h @ W["a1"].T) @ W["a2"].T + W["dt_bias"]).view(T, H, d)
    g = torch.exp(-torch.exp(W["A_log"])[None, :, None] * pre)
    o = rms(delta_rule(q, k, v, g, beta), eps) * W["norm"]
    o = o * torch.sigmoid((h @ W["g1"].T) @ W["g2"].T).view(T, H, e)
    return o.reshape(T, H * e) @ W["o"].T


def matrix_memory(q, k, v, ig, fg):
    """q (scaled), k [T, H, d], v [T, H, e], log gates ig, fg [T, H] -> o [T, H, e]."""
    T, H, e = v.shape
    out = torch.zeros_like(v)
    for h in range(H):
        S = torch.zeros(q.shape[2], e, dtype=v.dtype)
        n = torch.zeros(q.shape[2], dtype=v.dtype)
        m = torch.zeros((), dtype=v.dtype)
        for t in range(T):
            new = torch.maximum(fg[t, h] + m, ig[t, h])
            a, b = torch.exp(fg[t, h] + m - new), torch.exp(ig[t, h] - new)
            S = a * S + b * k[t, h][:, None] * v[t, h][None, :]
            n = a * n + b * k[t, h]
            m = new
            den = torch.maximum((n @ q[t, h]).abs(), torch.exp(-m)) + 1e-6
            out[t, h] = (S.T @ q[t, h]) / den
    return out


def mlstm(h, W, m, eps):
    T = h.shape[0]
    H, d, e, cap = m["heads"], m["dim"], m["vdim"], m["gate_cap"]
    q = (h @ W["q"].T).view(T, H, d) * d ** -0.5
    k = (h @ W["k"].T).view(T, H, d)
    v = (h @ W["v"].T).view(T, H, e)
    ig = cap * torch.tanh((h @ W["i"].T + W["i.b"]) / cap)
    fg = cap * torch.tanh((h @ W["f"].T + W["f.b"]) / cap)
    fg = -softplus(-fg)
    o = rms(matrix_memory(q, k, v, ig, fg), eps).reshape(T, H * e) * W["norm"]
    return (o * torch.sigmoid(h @ W["g"].T)) @ W["o"].T


def one_map(q, k, v, scale, cap):
    """q [T, d], k [T, d], v [T, e] -> [T, e]: capped causal softmax attention."""
    s = (q @ k.T) * scale
    if cap:
        s = cap * torch.tanh(s / cap)
    T = q.shape[0]
    s = s.masked_fill(torch.ones(T, T, dtype=torch.bool).triu(1), -math.inf)
    return torch.softmax(s, -1) @ v


def temperature(T, coef, every, dtype):
    p = torch.arange(T, dtype=dtype)
    return 1 + coef * torch.log(torch.floor((p + 1) / every) + 1)


def attention(h, W, m, eps):
    T = h.shape[0]
    H, G, d, e = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (h @ W["q"].T).view(T, H, 2, d)
    k = (h @ W["k"].T).view(T, G, 2, d)
    v = (h @ W["v"].T).view(T, G, e)
    if m.get("q_temp"):
        q = q * temperature(T, m["q_temp"]["coef"], m["q_temp"]["every"], h.dtype)[:, None, None, None]
    lam = torch.exp((W["lq1"] * W["lk1"]).sum()) - torch.exp((W["lq2"] * W["lk2"]).sum()) + m["diff"]
    out = torch.zeros(T, H, e, dtype=h.dtype)
    for i in range(H):
        j = i // (H // G)
        a1 = one_map(q[:, i, 0], k[:, j, 0], v[:, j], m["scale"], m["softcap"])
        a2 = one_map(q[:, i, 1], k[:, j, 1], v[:, j], m["scale"], m["softcap"])
        out[:, i] = rms(a1 - lam * a2, eps) * (1 - m["diff"])
    out = out * torch.sigmoid(h @ W["g"].T)[:, :, None]
    return out.reshape(T, H * e) @ W["o"].T


def feed_forward(h, W):
    return (silu(h @ W["gate"].T) * (h @ W["up"].T)) @ W["down"].T


MIXERS = {"channel_delta": channel_delta, "mlstm": mlstm, "attention": attention}


def hyper(x, hc_in, hc_mix, hc_out, fn):
    """x [s, T, C]: read one mix of the streams, run the sublayer, write it back into all of them."""
    u = torch.einsum("s,stc->tc", hc_in, x)
    y = fn(u)
    return torch.einsum("su,stc->utc", hc_mix, x) + hc_out[:, None, None] * y[None]


def forward(cfg: dict, weights: dict, tokens: list[int], dtype=torch.float32, layers_out: list | None = None):
    """Logits [T, vocab] of one sequence from its first token."""
    W = {k: v.to(dtype) if v.is_floating_point() else v for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    x = embed(W, tokens, dtype)[None].repeat(cfg["streams"], 1, 1)
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        mix = {k[len(p) + 4:]: v for k, v in W.items() if k.startswith(p + "mix.")}
        mlp = {k[len(p) + 4:]: v for k, v in W.items() if k.startswith(p + "mlp.")}
        x = hyper(x, W[p + "hc1.in"], W[p + "hc1.mix"], W[p + "hc1.out"],
                  lambda u: MIXERS[layer["type"]](centred_norm(u, W[p + "norm1"], eps), mix, layer["mixer"], eps))
        if layer["mlp"] is not None:
            x = hyper(x, W[p + "hc2.in"], W[p + "hc2.mix"], W[p + "hc2.out"],
                      lambda u: feed_forward(centred_norm(u, W[p + "norm2"], eps), mlp))
        if layers_out is not None:
            layers_out.append(x.sum(0))
    return centred_norm(x.sum(0), W["final.norm"], eps) @ W["head"].T
