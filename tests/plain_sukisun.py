"""Plain, slow restatement of the Sukisun equations in float64/float32 torch, one function per mechanism.

Written for the tests only: it shares no code with the product path, keeps no cache (a sequence is
always computed from its first token, token by token in the recurrence) and knows nothing about
pages, slots, chunks or batches.
"""
from __future__ import annotations

import math

import torch


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def layer_norm(x, w, eps):
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w


def silu(x):
    return x * torch.sigmoid(x)


def softplus(x):
    return torch.where(x > 30, x, torch.log1p(torch.exp(torch.clamp(x, max=30))))


def depth_average(weights, results):
    """sum_j weights[j] * results[j]"""
    out = torch.zeros_like(results[0])
    for j in range(len(results)):
        out = out + weights[j] * results[j]
    return out


def rotate(x, dims, base):
    """x [T, ..., n]: pairs (2i, 2i + 1) of the first ``dims`` entries turn by position * base^(-2i / dims)."""
    T = x.shape[0]
    out = x.clone()
    for i in range(dims // 2):
        a = torch.arange(T, dtype=torch.float64) * base ** (-2 * i / dims)
        c, s = torch.cos(a).to(x.dtype), torch.sin(a).to(x.dtype)
        shape = (T,) + (1,) * (x.dim() - 2)
        c, s = c.view(shape), s.view(shape)
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i], out[..., 2 * i + 1] = u * c - v * s, v * c + u * s
    return out


def latents(h, W, m, eps):
    """What a layer caches: normed latent c [T, kv_rank] and the rotated key part [T, rot_dim]."""
    r = h @ W["dkv"].T
    c = rms(r[:, :m["kv_rank"]], eps) * W["dkv.norm"]
    return c, rotate(r[:, m["kv_rank"]:], m["rot"]["dims"], m["rot"]["base"])


def causal_softmax_average(scores, v):
    T = scores.shape[0]
    s = scores.masked_fill(torch.ones(T, T, dtype=torch.bool).triu(1), -math.inf)
    return torch.softmax(s, -1) @ v


def latent_attention(h, W, m, eps, cached):
    """``cached``: (c, rotated key part) of this layer or of the layer it borrows them from."""
    T = h.shape[0]
    H, n, r, e = m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    c, kr = cached
    q = ((rms(h @ W["dq"].T, eps) * W["dq.norm"]) @ W["uq"].T).view(T, H, n + r)
    qn, qr = q[..., :n], rotate(q[..., n:], m["rot"]["dims"], m["rot"]["base"])
    k = (c @ W["uk"].T).view(T, H, n)
    v = (c @ W["uv"].T).view(T, H, e)
    gate = torch.sigmoid(h @ W["g"].T)
    out = torch.zeros(T, H, e, dtype=h.dtype)
    for i in range(H):
        s = (qn[:, i] @ k[:, i].T + qr[:, i] @ kr.T) * m["scale"]
        out[:, i] = causal_softmax_average(s, v[:, i]) * gate[:, i:i + 1]
    return out.reshape(T, H * e) @ W["o"].T


def short_conv(x, taps, bias):
    """x [T, C], taps [C, n]; the last tap multiplies the current row; zeros before the start."""
    T, n = x.shape[0], taps.shape[1]
    out = torch.zeros_like(x) + bias
    for t in range(T):
        for j in range(n):
            src = t - (n - 1) + j
            if src >= 0:
                out[t] += taps[:, j] * x[src]
    return out


def state_space(x, B, C, dt, decay, D):
    """x [T, H, e], B and C [T, G, N], dt and decay [T, H], D [H] -> y [T, H, e]."""
    T, H, e = x.shape
    per = H // B.shape[1]
    y = torch.zeros_like(x)
    for h in range(H):
        S = torch.zeros(B.shape[2], e, dtype=x.dtype)
        for t in range(T):
            S = decay[t, h] * S + dt[t, h] * B[t, h // per][:, None] * x[t, h][None, :]
            y[t, h] = S.T @ C[t, h // per] + D[h] * x[t, h]
    return y


def mamba2(h, W, m, eps):
    T = h.shape[0]
    H, e, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * e
    z, xbc, dt = torch.split(h @ W["in"].T, [inner, inner + 2 * G * N, H], dim=1)
    x, B, C = torch.split(silu(short_conv(xbc, W["conv"], W["conv.b"])), [inner, G * N, G * N], dim=1)
    dt = softplus(dt + W["dt_bias"])
    y = state_space(x.reshape(T, H, e), B.reshape(T, G, N), C.reshape(T, G, N), dt, torch.exp(-torch.exp(W["A_log"]) * dt), W["D"])
    y = y.reshape(T, inner) * silu(z)
    y = rms(y.view(T, m["norm_groups"], -1), eps).reshape(T, inner) * W["norm"]
    return y @ W["o"].T


def xielu(z, act):
    p, q = act
    pos = softplus(p) * z * z + z / 2
    neg = (0.5 + softplus(q)) * (torch.expm1(torch.clamp(z, max=0)) - z) + z / 2
    return torch.where(z > 0, pos, neg)


def feed_forward(h, W):
    return xielu(h @ W["up"].T, W["act"]) @ W["down"].T


def layer_tensors(W, i, part):
    p = f"l{i}.{part}."
    return {k[len(p):]: v for k, v in W.items() if k.startswith(p)}


def forward(cfg: dict, weights: dict, tokens: list[int], dtype=torch.float32, layers_out: list | None = None):
    """Logits [T, vocab] of one sequence from its first token."""
    W = {k: v.to(dtype) if v.is_floating_point() else v for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    x = W["embed"][torch.tensor(tokens)] * cfg["embedding"]["scale"]
    results, cached = [x], {}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        h, mix = layer_norm(x, W[p + "norm1"], eps), layer_tensors(W, i, "mix")
        if layer["type"] == "mamba2":
            x = x + mamba2(h, mix, m, eps)
        else:
            src = m.get("kv_from")
            cached[i] = latents(h, mix, m, eps) if src is None else cached[src]
            x = x + latent_attention(h, mix, m, eps, cached[i])
        if layer["mlp"] is not None:
            x = x + feed_forward(layer_norm(x, W[p + "norm2"], eps), layer_tensors(W, i, "mlp"))
        results.append(x)
        x = depth_average(W[p + "dwa"], results)
        if layers_out is not None:
            layers_out.append(x)
    return layer_norm(x, W["final.norm"], eps) @ W["embed"].T
