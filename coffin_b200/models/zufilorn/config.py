"""Geometry of the Zufilorn family, one entry per layer.

``config.json`` lists the layers: each names its mixer (``channel_delta``, ``mlstm`` or ``attention``), that mixer's
sizes and constants, and its feed-forward (or none).  Sizes may differ from layer to layer.  The rank of the
low-rank projections of a delta layer is not a config key; it is the shape of the tensors (``rank`` here is only what
random weights are drawn with).
"""
from __future__ import annotations

import dataclasses
import json
from pathlib import Path
from typing import Any

DELTA, MLSTM, ATTENTION = "channel_delta", "mlstm", "attention"


@dataclasses.dataclass(frozen=True)
class DeltaMixer:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int
    rank: int = 0                      # 0: the smaller of dim and 128

    @property
    def low_rank(self) -> int:
        return self.rank or min(self.dim, 128)


@dataclasses.dataclass(frozen=True)
class MLstmMixer:
    heads: int
    dim: int
    vdim: int
    gate_cap: float


@dataclasses.dataclass(frozen=True)
class AttentionMixer:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    softcap: float | None
    diff: float
    temp_coef: float = 0.0
    temp_every: int = 0                # 0: no query temperature


@dataclasses.dataclass(frozen=True)
class LayerSpec:
    kind: str
    mixer: DeltaMixer | MLstmMixer | AttentionMixer
    ff: int | None                     # width of the dense gated feed-forward, None: the layer has none


def _layer(raw: dict[str, Any], i: int) -> LayerSpec:
    kind, m = raw["type"], raw["mixer"]
    if kind == DELTA:
        mixer = DeltaMixer(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), int(m["conv"]))
    elif kind == MLSTM:
        mixer = MLstmMixer(int(m["heads"]), int(m["dim"]), int(m["vdim"]), float(m["gate_cap"]))
    elif kind == ATTENTION:
        t = m.get("q_temp") or {}
        cap = m.get("softcap")
        mixer = AttentionMixer(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), float(m["scale"]),
                               float(cap) if cap else None, float(m["diff"]), float(t.get("coef", 0.0)), int(t.get("every", 0)))
    else:
        raise ValueError(f"layer {i}: unknown mixer {kind!r}")
    mlp = raw.get("mlp")
    if mlp is not None and mlp.get("kind", "dense") != "dense":
        raise ValueError(f"layer {i}: unknown feed-forward {mlp.get('kind')!r}")
    return LayerSpec(kind, mixer, int(mlp["ff"]) if mlp is not None else None)


@dataclasses.dataclass
class ZufilornConfig:
    vocab_size: int
    hidden_size: int
    layers: tuple[LayerSpec, ...]
    streams: int
    max_positions: int
    rms_norm_eps: float = 1e-5
    architecture: str = "zufilorn"
    name: str = "zufilorn"
    is_moe = False
    mtp_num_hidden_layers = 0

    def __post_init__(self) -> None:
        self.layers = tuple(self.layers)
        self.validate()

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    @property
    def layer_types(self) -> tuple[str, ...]:
        return tuple(l.kind for l in self.layers)

    def validate(self) -> None:
        if not 1 <= self.streams <= 8:
            raise ValueError("1 to 8 residual streams are supported")
        for i, l in enumerate(self.layers):
            kv = getattr(l.mixer, "kv_heads", l.mixer.heads)
            if l.mixer.heads % kv:
                raise ValueError(f"layer {i}: heads must be a multiple of kv_heads")

    def first_layers(self, n: int) -> "ZufilornConfig":
        return dataclasses.replace(self, layers=self.layers[:n])

    # ---- (de)serialisation
    @classmethod
    def from_hf(cls, raw: dict[str, Any], name: str = "checkpoint") -> "ZufilornConfig":
        return cls(vocab_size=int(raw["vocab"]), hidden_size=int(raw["width"]),
                   layers=tuple(_layer(l, i) for i, l in enumerate(raw["layers"])), streams=int(raw["streams"]),
                   max_positions=int(raw["max_positions"]), rms_norm_eps=float(raw["norm"]["eps"]), name=name)

    @classmethod
    def from_dir(cls, model_dir: str | Path) -> "ZufilornConfig":
        p = Path(model_dir)
        return cls.from_hf(json.loads((p / "config.json").read_text()), name=p.name)

    def to_hf(self) -> dict[str, Any]:
        out = []
        for l in self.layers:
            m = {k: v for k, v in dataclasses.asdict(l.mixer).items() if k not in ("rank", "temp_coef", "temp_every")}
            if l.kind == ATTENTION and l.mixer.temp_every > 0:
                m["q_temp"] = {"coef": l.mixer.temp_coef, "every": l.mixer.temp_every}
            out.append({"type": l.kind, "mixer": m, "mlp": None if l.ff is None else {"kind": "dense", "ff": l.ff}})
        return {"architecture": "Zufilorn", "layers": out, "max_positions": self.max_positions,
                "norm": {"eps": self.rms_norm_eps}, "streams": self.streams, "vocab": self.vocab_size, "width": self.hidden_size}

    # ---- tensors
    def tensor_plan(self) -> list[tuple[str, tuple[int, ...], str]]:
        """``(name, shape, kind)`` of every tensor; ``kind`` names the distribution random weights are drawn from."""
        W, s = self.hidden_size, self.streams
        plan: list[tuple[str, tuple[int, ...], str]] = [("embed", (self.vocab_size, W), "embed"), ("pos", (self.max_positions, W), "embed")]

        def lin(name, n, k):
            plan.append((name, (n, k), "w"))
        for i, l in enumerate(self.layers):
            p, q, m = f"l{i}.", f"l{i}.mix.", l.mixer
            plan.append((p + "norm1", (W,), "norm0"))
            if l.ff is not None:
                plan.append((p + "norm2", (W,), "norm0"))
            H, d, e = m.heads, m.dim, m.vdim
            if l.kind == DELTA:
                G, r = m.kv_heads, m.low_rank
                for n, w in (("q", G * d), ("k", G * d), ("v", H * e)):
                    lin(q + n, w, W)
                    plan.append((q + n + ".conv", (w, m.conv), "conv"))
                lin(q + "b", H, W)
                plan += [(q + "A_log", (H,), "alog"), (q + "norm", (e,), "norm1"), (q + "dt_bias", (H * d,), "dt")]
                lin(q + "a1", r, W), lin(q + "a2", H * d, r), lin(q + "g1", r, W), lin(q + "g2", H * e, r)
            elif l.kind == MLSTM:
                lin(q + "q", H * d, W), lin(q + "k", H * d, W), lin(q + "v", H * e, W), lin(q + "g", H * e, W)
                plan.append((q + "norm", (H * e,), "norm1"))
                for n in ("i", "f"):
                    lin(q + n, H, W)
                    plan.append((q + n + ".b", (H,), "gate_b"))
            else:
                G = m.kv_heads
                lin(q + "q", H * 2 * d, W), lin(q + "k", G * 2 * d, W), lin(q + "v", G * e, W), lin(q + "g", H, W)
                plan += [(q + n, (d,), "lam") for n in ("lq1", "lk1", "lq2", "lk2")]
            lin(q + "o", W, H * e)
            if l.ff is not None:
                lin(p + "mlp.gate", l.ff, W), lin(p + "mlp.up", l.ff, W), lin(p + "mlp.down", W, l.ff)
            for hc in ("hc1.", "hc2.") if l.ff is not None else ("hc1.",):
                plan += [(p + hc + "in", (s,), "hc_in"), (p + hc + "out", (s,), "hc_out"), (p + hc + "mix", (s, s), "hc_mix")]
        plan.append(("final.norm", (W,), "norm0"))
        lin("head", self.vocab_size, W)
        return plan


def preset_zufilorn(name: str) -> ZufilornConfig:
    """``tiny-zufilorn``: every mixer once, odd sizes.  ``zufilorn-4b`` / ``zufilorn-1b``: layers of a real model's
    size (the widths, heads and vocabulary of the Qwen3.5 4B shape, and half of them) for throughput figures."""
    def cycle(n, H, ff, mixers):
        return tuple(LayerSpec(*mixers[i % len(mixers)], ff) for i in range(n))
    if name == "tiny-zufilorn":
        mix = ((DELTA, DeltaMixer(4, 2, 32, 24, 4, rank=16)), (MLSTM, MLstmMixer(3, 16, 40, 12.0)),
               (ATTENTION, AttentionMixer(6, 3, 16, 40, 0.25, 15.0, 0.5, 0.2, 64)))
        return ZufilornConfig(512, 192, cycle(3, 4, 256, mix), 2, 1024, name=name)
    if name in ("zufilorn-4b", "zufilorn-1b"):
        big = name == "zufilorn-4b"
        W, H, A, ff, n, voc = (2560, 32, 16, 9216, 32, 151936) if big else (1280, 16, 8, 4608, 16, 65536)
        delta = (DELTA, DeltaMixer(H, H // 2, 128, 128, 4))
        mem = (MLSTM, MLstmMixer(H // 2, 128, 256, 12.0))
        att = (ATTENTION, AttentionMixer(A, A // 4, 128, 256, 128 ** -0.5, 30.0, 0.5, 0.1, 4096))
        return ZufilornConfig(voc, W, cycle(n, H, ff, (delta, mem, delta, att)), 2, 8192, name=name)
    raise KeyError(f"unknown preset {name!r}")
