"""Small Zufilorn configurations and random weights for the tests (their own sizes; none is a released model's)."""
from __future__ import annotations

import torch


def delta(heads=4, kv_heads=2, dim=24, vdim=40, conv=4):
    return {"type": "channel_delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}}


def mlstm(heads=3, dim=16, vdim=24, gate_cap=9.0):
    return {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": gate_cap}}


def attention(heads=6, kv_heads=3, dim=16, vdim=40, scale=0.3, softcap=12.0, diff=0.45, coef=0.25, every=48):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "softcap": softcap, "diff": diff}
    if every:
        m["q_temp"] = {"coef": coef, "every": every}
    return {"type": "attention", "mixer": m}


def config(layers, width=72, vocab=96, streams=2, ff=88, max_positions=640, eps=2e-5, no_mlp=()):
    out = [dict(l, mlp=None if i in no_mlp or ff is None else {"kind": "dense", "ff": ff}) for i, l in enumerate(layers)]
    return {"architecture": "Zufilorn", "layers": out, "max_positions": max_positions, "norm": {"eps": eps}, "streams": streams,
            "vocab": vocab, "width": width}


def weights(cfg: dict, seed: int = 0, rank: int = 8, sharp: float = 1.0) -> dict[str, torch.Tensor]:
    """bf16 weights of ordinary scale; ``sharp`` multiplies the query rows (peaky attention / strong read-outs)."""
    g = torch.Generator().manual_seed(seed)
    W, s = cfg["width"], cfg["streams"]
    out: dict[str, torch.Tensor] = {}

    def put(name, *shape, std=1.0, mean=0.0):
        out[name] = (mean + std * torch.randn(*shape, generator=g)).to(torch.bfloat16)

    def lin(name, n, k, gain=1.0):
        put(name, n, k, std=gain * k ** -0.5)

    put("embed", cfg["vocab"], W)
    put("pos", cfg["max_positions"], W, std=0.5)
    for i, l in enumerate(cfg["layers"]):
        p, m = f"l{i}.mix.", l["mixer"]
        H, d, e = m["heads"], m["dim"], m["vdim"]
        put(f"l{i}.norm1", W, std=0.2)
        if l["type"] == "channel_delta":
            G = m["kv_heads"]
            for n, w in (("q", G * d), ("k", G * d), ("v", H * e)):
                lin(p + n, w, W, sharp if n == "q" else 1.0)
                put(p + n + ".conv", w, m["conv"], std=0.6)
            lin(p + "b", H, W, 1.5)
            put(p + "A_log", H, std=0.7, mean=-0.5)
            put(p + "dt_bias", H * d, std=1.5, mean=-2.5)
            lin(p + "a1", rank, W), lin(p + "a2", H * d, rank), lin(p + "g1", rank, W), lin(p + "g2", H * e, rank)
            put(p + "norm", e, std=0.2, mean=1.0)
        elif l["type"] == "mlstm":
            lin(p + "q", H * d, W, sharp), lin(p + "k", H * d, W), lin(p + "v", H * e, W), lin(p + "g", H * e, W)
            lin(p + "i", H, W, 2.0), lin(p + "f", H, W, 2.0)
            put(p + "i.b", H, std=1.5, mean=-1.0), put(p + "f.b", H, std=1.0, mean=3.0)
            put(p + "norm", H * e, std=0.2, mean=1.0)
        else:
            G = m["kv_heads"]
            lin(p + "q", H * 2 * d, W, 2.0 * sharp), lin(p + "k", G * 2 * d, W), lin(p + "v", G * e, W), lin(p + "g", H, W)
            for n in ("lq1", "lk1", "lq2", "lk2"):
                put(p + n, d, std=0.25)
        lin(p + "o", W, H * e)
        hcs = ["hc1"]
        if l["mlp"] is not None:
            ff = l["mlp"]["ff"]
            put(f"l{i}.norm2", W, std=0.2)
            lin(f"l{i}.mlp.gate", ff, W), lin(f"l{i}.mlp.up", ff, W), lin(f"l{i}.mlp.down", W, ff)
            hcs.append("hc2")
        for hc in hcs:
            put(f"l{i}.{hc}.in", s, std=0.4, mean=0.6)
            put(f"l{i}.{hc}.out", s, std=0.4, mean=0.8)
            out[f"l{i}.{hc}.mix"] = (0.8 * torch.eye(s) + 0.2 * torch.randn(s, s, generator=g)).to(torch.bfloat16)
    put("final.norm", W, std=0.2)
    lin("head", cfg["vocab"], W, 2.0)
    return out


ALL = config([delta(), mlstm(), attention()])
