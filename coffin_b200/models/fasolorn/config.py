"""Geometry of the Fasolorn family, one entry per layer.

``config.json`` lists the layers: each names its mixer (``attention`` or ``latent_attention``), that mixer's sizes and
constants, and its feed-forward (dense, routed, or none).  Everything may differ from layer to layer.
"""
from __future__ import annotations

import dataclasses
import json
from pathlib import Path
from typing import Any

ATTENTION, LATENT = "attention", "latent_attention"
DENSE, ROUTED = "dense", "moe"
MAX_OUTPUTS, MAX_TOP = 512, 32         # router outputs and choices the routing kernel takes


@dataclasses.dataclass(frozen=True)
class AttentionMixer:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot_base: float
    rot_dims: int                      # leading columns of a head that turn, neighbouring pairs
    window: int                        # tokens a query sees, itself included; 0: all
    v_mix: bool                        # values take a share of the first such layer's


@dataclasses.dataclass(frozen=True)
class LatentMixer:
    heads: int
    dim: int                           # unrotated query / key dimensions per head
    rot_dim: int                       # rotated ones; the rotated key part is shared by all heads
    vdim: int
    kv_rank: int
    scale: float
    rot_base: float
    rot_dims: int                      # paired i with i + rot_dims / 2
    window: int
    q_rank = 0                         # queries are projected directly


@dataclasses.dataclass(frozen=True)
class DenseFF:
    ff: int


@dataclasses.dataclass(frozen=True)
class RoutedFF:
    ff: int                            # width of an expert
    experts: int
    identity: int                      # further router outputs that return the input
    top: int
    scale: float
    shared: int                        # width of the shared expert, 0: none


@dataclasses.dataclass(frozen=True)
class LayerSpec:
    kind: str
    mixer: AttentionMixer | LatentMixer
    ff: DenseFF | RoutedFF | None


def _window(m: dict[str, Any], i: int) -> int:
    mask = m.get("mask")
    if not mask:
        return 0
    n = int(mask["size"])
    if n < 1:
        raise ValueError(f"layer {i}: a window of {n} tokens")
    return n


def _feed_forward(raw: dict[str, Any] | None, i: int) -> DenseFF | RoutedFF | None:
    if raw is None:
        return None
    kind = raw.get("kind", DENSE)
    if kind == DENSE:
        return DenseFF(int(raw["ff"]))
    if kind != ROUTED:
        raise ValueError(f"layer {i}: unknown feed-forward {kind!r}")
    r, shared = raw["router"], raw.get("shared")
    return RoutedFF(int(raw["expert"]["ff"]), int(r["experts"]), int(r.get("identity", 0) or 0), int(r["top"]), float(r.get("scale", 1.0)),
                    int(shared["ff"]) if shared else 0)


def _layer(raw: dict[str, Any], i: int) -> LayerSpec:
    kind, m = raw["type"], raw["mixer"]
    if kind not in (ATTENTION, LATENT):
        raise ValueError(f"layer {i}: unknown mixer {kind!r}")
    rot, win = m["rot"], _window(m, i)
    if kind == ATTENTION:
        mixer = AttentionMixer(*(int(m[k]) for k in ("heads", "kv_heads", "dim", "vdim")), float(m["scale"]), float(rot["base"]), int(rot["dims"]),
                               win, bool(m.get("v_mix", False)))
    else:
        mixer = LatentMixer(*(int(m[k]) for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank")), float(m["scale"]), float(rot["base"]),
                            int(rot["dims"]), win)
    return LayerSpec(kind, mixer, _feed_forward(raw.get("mlp"), i))


@dataclasses.dataclass
class FasolornConfig:
    vocab_size: int
    hidden_size: int
    layers: tuple[LayerSpec, ...]
    embedding_scale: float = 1.0
    rms_norm_eps: float = 1e-5         # of every norm
    architecture: str = "fasolorn"
    name: str = "fasolorn"
    is_moe = False                     # routed layers are the family's own
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

    @property
    def first_mixed(self) -> int | None:
        """The layer whose values the later ``v_mix`` layers take their share of."""
        return next((i for i, l in enumerate(self.layers) if l.kind == ATTENTION and l.mixer.v_mix), None)

    def validate(self) -> None:
        first = self.first_mixed
        for i, l in enumerate(self.layers):
            m, f = l.mixer, l.ff
            room = m.dim if l.kind == ATTENTION else m.rot_dim
            if m.rot_dims % 2 or not 0 <= m.rot_dims <= room:
                raise ValueError(f"layer {i}: rot.dims must be even and at most {room}")
            if l.kind == ATTENTION:
                if m.heads % m.kv_heads:
                    raise ValueError(f"layer {i}: heads must be a multiple of kv_heads")
                if m.v_mix and m.kv_heads * m.vdim != self.layers[first].mixer.kv_heads * self.layers[first].mixer.vdim:
                    raise ValueError(f"layer {i}: values of another size than those of layer {first}, which are mixed in")
            if isinstance(f, RoutedFF):
                n = f.experts + f.identity
                if f.experts < 1 or f.identity < 0 or n > MAX_OUTPUTS or not 1 <= f.top <= min(n, MAX_TOP):
                    raise ValueError(f"layer {i}: top {f.top} of {f.experts} + {f.identity} experts")

    def first_layers(self, n: int) -> "FasolornConfig":
        return dataclasses.replace(self, layers=self.layers[:n])

    # ---- (de)serialisation
    @classmethod
    def from_hf(cls, raw: dict[str, Any], name: str = "checkpoint") -> "FasolornConfig":
        return cls(vocab_size=int(raw["vocab"]), hidden_size=int(raw["width"]),
                   layers=tuple(_layer(l, i) for i, l in enumerate(raw["layers"])),
                   embedding_scale=float(raw.get("embedding", {}).get("scale", 1.0)), rms_norm_eps=float(raw["norm"]["eps"]), name=name)

    @classmethod
    def from_dir(cls, model_dir: str | Path) -> "FasolornConfig":
        p = Path(model_dir)
        return cls.from_hf(json.loads((p / "config.json").read_text()), name=p.name)

    def to_hf(self) -> dict[str, Any]:
        out = []
        for l in self.layers:
            m = dataclasses.asdict(l.mixer)
            m["rot"] = {"base": m.pop("rot_base"), "dims": m.pop("rot_dims")}
            win = m.pop("window")
            m["mask"] = {"size": win} if win else None
            f, mlp = l.ff, None
            if isinstance(f, DenseFF):
                mlp = {"kind": DENSE, "ff": f.ff}
            elif f is not None:
                mlp = {"kind": ROUTED, "expert": {"ff": f.ff}, "router": {"experts": f.experts, "identity": f.identity, "top": f.top, "scale": f.scale},
                       "shared": {"ff": f.shared} if f.shared else None}
            out.append({"type": l.kind, "mixer": m, "mlp": mlp})
        return {"architecture": "Fasolorn", "embedding": {"scale": self.embedding_scale}, "layers": out, "norm": {"eps": self.rms_norm_eps},
                "vocab": self.vocab_size, "width": self.hidden_size}

    # ---- tensors
    def tensor_plan(self) -> list[tuple[str, tuple[int, ...], str]]:
        """``(name, shape, kind)`` of every tensor; ``kind`` names the distribution random weights are drawn from."""
        W = self.hidden_size
        plan: list[tuple[str, tuple[int, ...], str]] = [("embed", (self.vocab_size, W), "embed")]

        def lin(name, n, k):
            plan.append((name, (n, k), "w"))
        for i, l in enumerate(self.layers):
            p, q, m, f = f"l{i}.", f"l{i}.mix.", l.mixer, l.ff
            plan.append((p + "norm1", (W,), "norm1"))
            if l.kind == ATTENTION:
                lin(q + "q", m.heads * m.dim, W), lin(q + "k", m.kv_heads * m.dim, W), lin(q + "v", m.kv_heads * m.vdim, W)
                if m.v_mix:
                    plan.append((q + "vmix", (), "share"))
                plan.append((q + "sink", (m.heads,), "gate_b"))
                lin(q + "g", m.heads * m.vdim, W)
            else:
                lin(q + "q", m.heads * (m.dim + m.rot_dim), W), lin(q + "dkv", m.kv_rank + m.rot_dim, W)
                plan.append((q + "dkv.norm", (m.kv_rank,), "norm1"))
                lin(q + "uk", m.heads * m.dim, m.kv_rank), lin(q + "uv", m.heads * m.vdim, m.kv_rank)
            lin(q + "o", W, m.heads * m.vdim)
            if f is None:
                continue
            plan.append((p + "norm2", (W,), "norm1"))
            if isinstance(f, DenseFF):
                lin(p + "mlp.gate", f.ff, W), lin(p + "mlp.up", f.ff, W), lin(p + "mlp.down", W, f.ff)
                continue
            for e in range(f.experts):
                lin(f"{p}mlp.e{e}.up", f.ff, W), lin(f"{p}mlp.e{e}.down", W, f.ff)
            lin(p + "mlp.router", f.experts + f.identity, W)
            plan.append((p + "mlp.correction", (f.experts + f.identity,), "route"))
            if f.shared:
                lin(p + "mlp.shared.up", f.shared, W), lin(p + "mlp.shared.down", W, f.shared)
        plan.append(("final.norm", (W,), "norm1"))
        return plan


def preset_fasolorn(name: str) -> FasolornConfig:
    """``tiny-fasolorn``: every mechanism once, odd sizes.  ``fasolorn-4b``: layers of a real model's size, dense (width, depth,
    vocabulary and weights per layer of the Qwen3.5 4B shape), three windowed attention layers to one of latent attention.
    ``fasolorn-35b-a3b``: the same mixers with routed feed-forwards in all layers but the first (width, depth, number of experts
    and weights per expert of the Qwen3.5 35B-A3B shape)."""
    if name == "tiny-fasolorn":
        att = lambda ff, win: LayerSpec(ATTENTION, AttentionMixer(6, 2, 24, 40, 0.2, 9000.0, 16, win, True), ff)
        lat = lambda ff: LayerSpec(LATENT, LatentMixer(5, 24, 16, 40, 72, 0.16, 5000.0, 16, 50), ff)
        moe = RoutedFF(56, 12, 3, 3, 1.5, 72)
        return FasolornConfig(512, 192, (att(DenseFF(160), 70), lat(moe), att(moe, 33), lat(None)), 4.0, name=name)
    if name in ("fasolorn-4b", "fasolorn-35b-a3b"):
        big = name == "fasolorn-4b"
        n, W, kv, kv_rank = (32, 2560, 4, 512) if big else (40, 2048, 2, 512)
        layers = []
        for i in range(n):
            ff = DenseFF(9216) if big else (DenseFF(4608) if i == 0 else RoutedFF(768, 256, 32, 8, 2.0, 768))
            if i % 4 == 3:
                layers.append(LayerSpec(LATENT, LatentMixer(32, 128, 64, 128, kv_rank, 192 ** -0.5, 10000.0, 64, 4096), ff))
            else:
                layers.append(LayerSpec(ATTENTION, AttentionMixer(32, 2 * kv, 128, 128, 128 ** -0.5, 500000.0, 64, 1024, True), ff))
        return FasolornConfig(151936, W, tuple(layers), 1.0, name=name)
    raise KeyError(f"unknown preset {name!r}")
