"""Small Fasolorn configurations and random weights for the tests (their own sizes; none is a released model's)."""
from __future__ import annotations

import torch


def attention(heads=6, kv_heads=2, dim=24, vdim=40, window=50, rot=16, base=700.0, scale=0.25, v_mix=True):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "rot": {"base": base, "dims": rot},
         "mask": {"size": window} if window else None, "v_mix": v_mix}
    return {"type": "attention", "mixer": m}


def latent(heads=5, dim=24, rot_dim=16, vdim=40, kv_rank=72, window=45, base=3000.0, scale=0.2):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale, "rot": {"base": base, "dims": rot_dim},
         "mask": {"size": window} if window else None}
    return {"type": "latent_attention", "mixer": m}


def dense(ff=88):
    return {"kind": "dense", "ff": ff}


def moe(experts=7, identity=3, top=3, ff=40, shared=56, scale=1.5):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "identity": identity, "top": top, "scale": scale},
            "shared": {"ff": shared} if shared else None}


def config(layers, mlps, width=72, vocab=96, scale=2.5, eps=2e-5):
    out = [dict(l, mlp=f) for l, f in zip(layers, mlps, strict=True)]
    return {"architecture": "Fasolorn", "embedding": {"scale": scale}, "layers": out, "norm": {"eps": eps}, "vocab": vocab, "width": width}


def weights(cfg: dict, seed: int = 0) -> dict[str, torch.Tensor]:
    """bf16 weights of ordinary scale, routers with clear preferences."""
    g = torch.Generator().manual_seed(seed)
    W = cfg["width"]
    out: dict[str, torch.Tensor] = {}

    def put(name, *shape, std=1.0, mean=0.0):
        out[name] = (mean + std * torch.randn(shape, generator=g)).to(torch.bfloat16)

    def lin(name, n, k, gain=1.0):
        put(name, n, k, std=gain * k ** -0.5)

    put("embed", cfg["vocab"], W, std=0.5)
    for i, l in enumerate(cfg["layers"]):
        p, m, f = f"l{i}.mix.", l["mixer"], l["mlp"]
        H, e = m["heads"], m["vdim"]
        put(f"l{i}.norm1", W, std=0.2, mean=1.0)
        if l["type"] == "attention":
            G = m["kv_heads"]
            lin(p + "q", H * m["dim"], W, 2.0), lin(p + "k", G * m["dim"], W), lin(p + "v", G * e, W)
            if m["v_mix"]:
                put(p + "vmix", std=0.2, mean=0.45)
            put(p + "sink", H, std=1.5, mean=0.5)
            lin(p + "g", H * e, W)
        else:
            R, r = m["kv_rank"], m["rot_dim"]
            lin(p + "q", H * (m["dim"] + r), W, 2.0), lin(p + "dkv", R + r, W)
            put(p + "dkv.norm", R, std=0.2, mean=1.0)
            lin(p + "uk", H * m["dim"], R), lin(p + "uv", H * e, R)
        lin(p + "o", W, H * e)
        if f is None:
            continue
        q = f"l{i}.mlp."
        put(f"l{i}.norm2", W, std=0.2, mean=1.0)
        if f["kind"] == "dense":
            lin(q + "gate", f["ff"], W), lin(q + "up", f["ff"], W), lin(q + "down", W, f["ff"])
            continue
        r = f["router"]
        for x in range(r["experts"]):
            lin(f"{q}e{x}.up", f["expert"]["ff"], W), lin(f"{q}e{x}.down", W, f["expert"]["ff"])
        lin(q + "router", r["experts"] + r["identity"], W, 2.0)
        put(q + "correction", r["experts"] + r["identity"], std=0.1)
        if f["shared"]:
            lin(q + "shared.up", f["shared"]["ff"], W), lin(q + "shared.down", W, f["shared"]["ff"])
    put("final.norm", W, std=0.2, mean=1.0)
    return out


ALL = config([attention(), latent(), attention(4, 4, 16, 20, 33, 8, 90.0, 0.4), attention(10, 5, 20, 16, 70, 20, 5000.0, 0.3), latent(3, 16, 8, 24, 40, 64, 800.0, 0.3)],
             [dense(), moe(), moe(5, 1, 2, 24, 24, 0.7), None, moe(6, 0, 1, 32, 0, 2.5)])
