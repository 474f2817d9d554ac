"""Small Nodutar configurations and random weights for the tests (their own sizes; none is a released model's)."""
from __future__ import annotations

import torch


def parallel(heads=6, kv_heads=3, dim=24, vdim=40, chunk=50, rot=16, base=700.0, scale=0.4, mem=(3, 40, 24), ls=0.7, rs=1.6):
    left = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "rot": {"base": base, "dims": rot},
            "mask": {"size": chunk} if chunk else None}
    return {"type": "parallel", "mixer": {"left": left, "right": dict(zip(("heads", "dim", "vdim"), mem)), "left_scale": ls, "right_scale": rs}}


def attention(heads=4, kv_heads=2, dim=40, scale=0.3):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale}}


def moe(experts=7, top=3, ff=40):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def config(layers, mlps, loop=None, width=72, vocab=96, eps=3e-5):
    out = [dict(l, mlp=f) for l, f in zip(layers, mlps, strict=True)]
    return {"architecture": "Nodutar", "layers": out, "loop": dict(zip(("start", "stop", "times"), loop)) if loop else None, "norm": {"eps": eps},
            "vocab": vocab, "width": width}


def weights(cfg: dict, seed: int = 0, clear: bool = False) -> dict[str, torch.Tensor]:
    """bf16 weights of ordinary scale, forget gates from short to long memories.  ``clear``: routers read a few columns that hold the
    token's class, which no sublayer writes to, so that rounding never changes a choice (a flipped one spoils its token's row
    and, through the attention, later ones)."""
    g = torch.Generator().manual_seed(seed)
    W = cfg["width"]
    out: dict[str, torch.Tensor] = {}

    def put(name, *shape, std=1.0, mean=0.0):
        out[name] = (mean + std * torch.randn(shape, generator=g)).to(torch.bfloat16)

    def uniform(name, n, lo, hi):
        out[name] = (lo + (hi - lo) * torch.rand(n, generator=g)).to(torch.bfloat16)

    def lin(name, n, k, gain=1.0):
        put(name, n, k, std=gain * k ** -0.5)

    put("embed", cfg["vocab"], W, std=0.5)
    for i, l in enumerate(cfg["layers"]):
        p, m, f = f"l{i}.mix.", l["mixer"], l["mlp"]
        for n in ("norm1", "norm1b") + (("norm2", "norm2b") if f else ()):
            put(f"l{i}.{n}", W, std=0.2)
        if l["type"] == "parallel":
            a, r = m["left"], m["right"]
            H, G, n = a["heads"], a["kv_heads"], r["heads"] * r["dim"]
            lin(p + "left.q", H * a["dim"], W), lin(p + "left.k", G * a["dim"], W), lin(p + "left.v", G * a["vdim"], W)
            put(p + "left.q.norm", a["dim"], std=0.3, mean=1.2), put(p + "left.k.norm", a["dim"], std=0.3, mean=0.9)
            lin(p + "left.o", W, H * a["vdim"])
            lin(p + "right.q", n, W), lin(p + "right.f", n, W, 1.5)
            put(p + "right.f.b", n, std=1.5, mean=1.0), uniform(p + "right.lower", n, 0.0, 0.9)
            lin(p + "right.v", r["heads"] * r["vdim"], W)
            put(p + "right.norm", r["vdim"], std=0.3, mean=1.0)
            lin(p + "right.o", W, r["heads"] * r["vdim"])
        else:
            H, G, d = m["heads"], m["kv_heads"], m["dim"]
            lin(p + "q", H * d, W), lin(p + "k", G * d, W), lin(p + "o", W, H * d)
            uniform(p + "r1", H, 0.2, 1.2), uniform(p + "r2", H, 0.01, 0.6)
        if f is None:
            continue
        q = f"l{i}.mlp."
        for x in range(f["router"]["experts"]):
            lin(f"{q}e{x}.gate", f["expert"]["ff"], W), lin(f"{q}e{x}.up", f["expert"]["ff"], W), lin(f"{q}e{x}.down", W, f["expert"]["ff"])
        lin(q + "router", f["router"]["experts"], W, 2.0)
        put(q + "router.b", f["router"]["experts"], std=0.6)
    put("final.norm", W, std=0.2)
    if clear:
        C = min(8, W // 4)
        out["embed"][:, :C] = 0.0
        out["embed"][torch.arange(cfg["vocab"]), torch.arange(cfg["vocab"]) % C] = 5.0
        for n, t in out.items():
            if n.endswith(("norm1b", "norm2b")):
                t[:C] = -1.0
            elif n.endswith("mlp.router"):
                t.zero_()
                for c in range(C):
                    t[:, c] = torch.linspace(-2, 2, t.shape[0])[torch.randperm(t.shape[0], generator=g)]
            elif n.endswith("router.b"):
                t *= 0.1
    return out


ALL = config([attention(), parallel(), attention(6, 1, 24, 0.5), parallel(4, 4, 16, 20, 33, 8, 90.0, 0.6, (2, 24, 32), 1.4, 0.6), parallel(2, 1, 32, 16, 70, 32, 5000.0, 0.5, (5, 8, 16), 1.0, 1.0)],
             [moe(), moe(5, 2, 24), None, moe(4, 1, 32), moe(6, 6, 16)], (1, 3, 3))
