"""Small Sukisun configurations and random weights for the tests (their own sizes; none is a released model's)."""
from __future__ import annotations

import torch


def latent(heads=5, dim=24, rot_dim=16, vdim=40, kv_rank=72, q_rank=56, scale=0.2, base=3000.0, kv_from=None, rot_dims=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank, "scale": scale,
         "rot": {"base": base, "dims": rot_dim if rot_dims is None else rot_dims}}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m}


def mamba(heads=6, vdim=24, state=40, groups=2, conv=4, norm_groups=3):
    return {"type": "mamba2", "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv,
                                        "norm_groups": norm_groups}}


def config(layers, width=72, vocab=96, ff=88, scale=3.0, eps=2e-5, no_mlp=()):
    out = [dict(l, mlp=None if i in no_mlp or ff is None else {"kind": "dense", "ff": ff}) for i, l in enumerate(layers)]
    return {"architecture": "Sukisun", "embedding": {"scale": scale}, "layers": out, "norm": {"eps": eps}, "vocab": vocab, "width": width}


def weights(cfg: dict, seed: int = 0, sharp: float = 1.0) -> dict[str, torch.Tensor]:
    """bf16 weights of ordinary scale; ``sharp`` multiplies the query rows (peaky attention)."""
    g = torch.Generator().manual_seed(seed)
    W = cfg["width"]
    out: dict[str, torch.Tensor] = {}

    def put(name, *shape, std=1.0, mean=0.0):
        out[name] = (mean + std * torch.randn(*shape, generator=g)).to(torch.bfloat16)

    def lin(name, n, k, gain=1.0):
        put(name, n, k, std=gain * k ** -0.5)

    put("embed", cfg["vocab"], W, std=0.5)
    for i, l in enumerate(cfg["layers"]):
        p, m = f"l{i}.mix.", l["mixer"]
        H, e = m["heads"], m["vdim"]
        put(f"l{i}.norm1", W, std=0.2, mean=1.0)
        if l["type"] == "latent_attention":
            R, r, n = m["kv_rank"], m["rot_dim"], m["dim"]
            lin(p + "dq", m["q_rank"], W)
            put(p + "dq.norm", m["q_rank"], std=0.2, mean=1.0)
            lin(p + "uq", H * (n + r), m["q_rank"], 2.0 * sharp)
            if "kv_from" not in m:
                lin(p + "dkv", R + r, W)
                put(p + "dkv.norm", R, std=0.2, mean=1.0)
            lin(p + "uk", H * n, R), lin(p + "uv", H * e, R), lin(p + "g", H, W), lin(p + "o", W, H * e)
        else:
            G, N, inner = m["groups"], m["state"], H * e
            lin(p + "in", 2 * inner + 2 * G * N + H, W)
            put(p + "conv", inner + 2 * G * N, m["conv"], std=0.6)
            put(p + "conv.b", inner + 2 * G * N, std=0.3)
            put(p + "dt_bias", H, std=1.0, mean=-1.5)
            put(p + "A_log", H, std=0.8, mean=0.0)
            put(p + "D", H, std=0.7, mean=0.5)
            put(p + "norm", inner, std=0.2, mean=1.0)
            lin(p + "o", W, inner)
        if l["mlp"] is not None:
            ff = l["mlp"]["ff"]
            put(f"l{i}.norm2", W, std=0.2, mean=1.0)
            lin(f"l{i}.mlp.up", ff, W), lin(f"l{i}.mlp.down", W, ff)
            put(f"l{i}.mlp.act", 2, std=0.8)
        put(f"l{i}.dwa", i + 2, std=0.25, mean=0.1)
        out[f"l{i}.dwa"][-1] += 0.8
    put("final.norm", W, std=0.2, mean=1.0)
    return out


ALL = config([mamba(), latent(), mamba(4, 16, 24, 1, 3, 1), latent(3, 16, 16, 24, 72, 40, 0.3, kv_from=1)], no_mlp=(0,))
