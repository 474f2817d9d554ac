"""Geometry of the Sukisun family, one entry per layer.

``config.json`` lists the layers: each names its mixer (``latent_attention`` or ``mamba2``), that mixer's sizes and
constants, and its feed-forward (or none).  Sizes may differ from layer to layer; an attention layer may name an
earlier one (``kv_from``) whose cached latents it reads instead of projecting its own.
"""
from __future__ import annotations

import dataclasses
import json
from pathlib import Path
from typing import Any

LATENT, MAMBA2 = "latent_attention", "mamba2"


@dataclasses.dataclass(frozen=True)
class LatentMixer:
    heads: int
    dim: int                           # unrotated query / key dimensions per head
    rot_dim: int                       # rotated ones; the rotated key part is shared by all heads
    vdim: int
    kv_rank: int
    q_rank: int
    scale: float
    rot_base: float
    rot_dims: int                      # how many of the rotated part turn (all of it as a rule)
    kv_from: int | None = None


@dataclasses.dataclass(frozen=True)
class Mamba2Mixer:
    heads: int
    vdim: int
    state: int
    groups: int
    conv: int
    norm_groups: int

    @property
    def inner(self) -> int:
        return self.heads * self.vdim

    @property
    def conv_width(self) -> int:
        return self.inner + 2 * self.groups * self.state


@dataclasses.dataclass(frozen=True)
class LayerSpec:
    kind: str
    mixer: LatentMixer | Mamba2Mixer
    ff: int | None                     # width of the dense xIELU feed-forward, None: the layer has none


def _layer(raw: dict[str, Any], i: int) -> LayerSpec:
    kind, m = raw["type"], raw["mixer"]
    if kind == LATENT:
        rot, src = m["rot"], m.get("kv_from")
        mixer = LatentMixer(int(m["heads"]), int(m["dim"]), int(m["rot_dim"]), int(m["vdim"]), int(m["kv_rank"]), int(m["q_rank"]),
                            float(m["scale"]), float(rot["base"]), int(rot["dims"]), int(src) if src is not None else None)
    elif kind == MAMBA2:
        mixer = Mamba2Mixer(*(int(m[k]) for k in ("heads", "vdim", "state", "groups", "conv", "norm_groups")))
    else:
        raise ValueError(f"layer {i}: unknown mixer {kind!r}")
    mlp = raw.get("mlp")
    if mlp is not None and mlp.get("kind", "dense") != "dense":
        raise ValueError(f"layer {i}: unknown feed-forward {mlp.get('kind')!r}")
    return LayerSpec(kind, mixer, int(mlp["ff"]) if mlp is not None else None)


@dataclasses.dataclass
class SukisunConfig:
    vocab_size: int
    hidden_size: int
    layers: tuple[LayerSpec, ...]
    embedding_scale: float = 1.0
    rms_norm_eps: float = 1e-5         # of every norm, the layer norms included
    architecture: str = "sukisun"
    name: str = "sukisun"
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
        for i, l in enumerate(self.layers):
            m = l.mixer
            if l.kind == MAMBA2:
                if m.heads % m.groups or m.inner % m.norm_groups:
                    raise ValueError(f"layer {i}: heads must be a multiple of groups, heads * vdim of norm_groups")
                continue
            if m.rot_dims % 2 or m.rot_dims > m.rot_dim:
                raise ValueError(f"layer {i}: rot.dims must be even and at most rot_dim")
            if m.kv_from is not None:
                src = self.layers[m.kv_from] if 0 <= m.kv_from < i else None
                s = src.mixer if src is not None and src.kind == LATENT else None
                if s is None or s.kv_from is not None:
                    raise ValueError(f"layer {i}: kv_from must name an earlier attention layer with latents of its own")
                if (s.kv_rank, s.rot_dim, s.rot_base, s.rot_dims) != (m.kv_rank, m.rot_dim, m.rot_base, m.rot_dims):
                    raise ValueError(f"layer {i}: latents of layer {m.kv_from} have another size or rotation")

    def first_layers(self, n: int) -> "SukisunConfig":
        return dataclasses.replace(self, layers=self.layers[:n])

    # ---- (de)serialisation
    @classmethod
    def from_hf(cls, raw: dict[str, Any], name: str = "checkpoint") -> "SukisunConfig":
        return cls(vocab_size=int(raw["vocab"]), hidden_size=int(raw["width"]),
                   layers=tuple(_layer(l, i) for i, l in enumerate(raw["layers"])),
                   embedding_scale=float(raw.get("embedding", {}).get("scale", 1.0)), rms_norm_eps=float(raw["norm"]["eps"]), name=name)

    @classmethod
    def from_dir(cls, model_dir: str | Path) -> "SukisunConfig":
        p = Path(model_dir)
        return cls.from_hf(json.loads((p / "config.json").read_text()), name=p.name)

    def to_hf(self) -> dict[str, Any]:
        out = []
        for l in self.layers:
            m = dataclasses.asdict(l.mixer)
            if l.kind == LATENT:
                m["rot"] = {"base": m.pop("rot_base"), "dims": m.pop("rot_dims")}
                if m["kv_from"] is None:
                    del m["kv_from"]
            out.append({"type": l.kind, "mixer": m, "mlp": None if l.ff is None else {"kind": "dense", "ff": l.ff}})
        return {"architecture": "Sukisun", "embedding": {"scale": self.embedding_scale}, "layers": out, "norm": {"eps": self.rms_norm_eps},
                "vocab": self.vocab_size, "width": self.hidden_size}

    # ---- tensors
    def tensor_plan(self) -> list[tuple[str, tuple[int, ...], str]]:
        """``(name, shape, kind)`` of every tensor; ``kind`` names the distribution random weights are drawn from."""
        W = self.hidden_size
        plan: list[tuple[str, tuple[int, ...], str]] = [("embed", (self.vocab_size, W), "embed")]

        def lin(name, n, k):
            plan.append((name, (n, k), "w"))
        for i, l in enumerate(self.layers):
            p, q, m = f"l{i}.", f"l{i}.mix.", l.mixer
            plan.append((p + "norm1", (W,), "norm1"))
            if l.kind == LATENT:
                lin(q + "dq", m.q_rank, W)
                plan.append((q + "dq.norm", (m.q_rank,), "norm1"))
                lin(q + "uq", m.heads * (m.dim + m.rot_dim), m.q_rank)
                if m.kv_from is None:
                    lin(q + "dkv", m.kv_rank + m.rot_dim, W)
                    plan.append((q + "dkv.norm", (m.kv_rank,), "norm1"))
                lin(q + "uk", m.heads * m.dim, m.kv_rank), lin(q + "uv", m.heads * m.vdim, m.kv_rank)
                lin(q + "g", m.heads, W), lin(q + "o", W, m.heads * m.vdim)
            else:
                lin(q + "in", m.inner + m.conv_width + m.heads, W)
                plan += [(q + "conv", (m.conv_width, m.conv), "conv"), (q + "conv.b", (m.conv_width,), "lam"),
                         (q + "dt_bias", (m.heads,), "dt"), (q + "A_log", (m.heads,), "alog"), (q + "D", (m.heads,), "norm1"),
                         (q + "norm", (m.inner,), "norm1")]
                lin(q + "o", W, m.inner)
            if l.ff is not None:
                plan.append((p + "norm2", (W,), "norm1"))
                lin(p + "mlp.up", l.ff, W), lin(p + "mlp.down", W, l.ff)
                plan.append((p + "mlp.act", (2,), "gate_b"))
            plan.append((p + "dwa", (i + 2,), "dwa"))
        plan.append(("final.norm", (W,), "norm1"))
        return plan


def preset_sukisun(name: str) -> SukisunConfig:
    """``tiny-sukisun``: every mechanism once, odd sizes.  ``sukisun-4b`` / ``sukisun-1b``: layers of a real model's size
    (width, depth, vocabulary and weights per layer of the Qwen3.5 4B shape, and half of its width) for throughput
    figures: three Mamba-2 layers to one of latent attention, every second attention layer on the latents before it."""
    if name == "tiny-sukisun":
        lat = lambda src=None: LayerSpec(LATENT, LatentMixer(5, 24, 16, 40, 72, 56, 0.16, 5000.0, 16, src), 160)
        mam = lambda ff=None: LayerSpec(MAMBA2, Mamba2Mixer(6, 24, 40, 2, 4, 3), ff)
        return SukisunConfig(512, 192, (mam(), lat(), mam(128), lat(1)), 4.0, name=name)
    if name in ("sukisun-4b", "sukisun-1b"):
        f, n, voc = (1, 32, 151936) if name == "sukisun-4b" else (2, 16, 65536)
        layers = []
        for i in range(n):
            if i % 4 == 3:
                mixer = LatentMixer(32 // f, 128, 64, 128, 512, 1536 // f, 192 ** -0.5, 10000.0, 64, i - 4 if i % 8 == 7 else None)
            else:
                mixer = Mamba2Mixer(80 // f, 64, 128, 1, 4, 1)
            layers.append(LayerSpec(LATENT if i % 4 == 3 else MAMBA2, mixer, 13824 // f))
        return SukisunConfig(voc, 2560 // f, tuple(layers), name=name)
    raise KeyError(f"unknown preset {name!r}")
