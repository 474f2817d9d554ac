"""Geometry of the Nodutar family, one entry per layer, and the order in which layers run.

``config.json`` lists the layers: each names its mixer (``parallel`` or ``attention``), that mixer's sizes and constants, and its
routed feed-forward (or none).  Everything may differ from layer to layer.  ``loop`` names a range of layers that run several
times in a row.
"""
from __future__ import annotations

import dataclasses
import json
from pathlib import Path
from typing import Any

PARALLEL, ATTENTION = "parallel", "attention"
ROUTED = "moe"
MAX_OUTPUTS, MAX_TOP = 512, 32         # router outputs and choices the routing kernel takes


@dataclasses.dataclass(frozen=True)
class ChunkAttention:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot_base: float
    rot_dims: int                      # leading columns of a query / key head that turn, neighbouring pairs; values turn whole
    chunk: int                         # tokens that see one another, counted from position 0; 0: all


@dataclasses.dataclass(frozen=True)
class GatedState:
    heads: int
    dim: int
    vdim: int


@dataclasses.dataclass(frozen=True)
class ParallelMixer:
    left: ChunkAttention
    right: GatedState
    left_scale: float
    right_scale: float


@dataclasses.dataclass(frozen=True)
class DistanceMixer:
    heads: int
    kv_heads: int
    dim: int                           # of queries, keys and values: the values are the keys
    scale: float


@dataclasses.dataclass(frozen=True)
class RoutedFF:
    ff: int                            # width of an expert
    experts: int
    top: int


@dataclasses.dataclass(frozen=True)
class LayerSpec:
    kind: str
    mixer: ParallelMixer | DistanceMixer
    ff: RoutedFF | None


@dataclasses.dataclass(frozen=True)
class Loop:
    """Layers ``start .. stop - 1`` run ``times`` times in a row."""
    start: int
    stop: int
    times: int


def _feed_forward(raw: dict[str, Any] | None, i: int) -> RoutedFF | None:
    if raw is None:
        return None
    if raw.get("kind", ROUTED) != ROUTED:
        raise ValueError(f"layer {i}: unknown feed-forward {raw['kind']!r}")
    return RoutedFF(int(raw["expert"]["ff"]), int(raw["router"]["experts"]), int(raw["router"]["top"]))


def _layer(raw: dict[str, Any], i: int) -> LayerSpec:
    kind, m = raw["type"], raw["mixer"]
    if kind == PARALLEL:
        a, r = m["left"], m["right"]
        mask, rot = a.get("mask"), a["rot"]
        chunk = int(mask["size"]) if mask else 0
        if mask and chunk < 1:
            raise ValueError(f"layer {i}: chunks of {chunk} tokens")
        mixer = ParallelMixer(ChunkAttention(*(int(a[k]) for k in ("heads", "kv_heads", "dim", "vdim")), float(a["scale"]), float(rot["base"]),
                                             int(rot["dims"]), chunk),
                              GatedState(*(int(r[k]) for k in ("heads", "dim", "vdim"))), float(m["left_scale"]), float(m["right_scale"]))
    elif kind == ATTENTION:
        mixer = DistanceMixer(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), float(m["scale"]))
        if int(m.get("vdim", mixer.dim)) != mixer.dim:
            raise ValueError(f"layer {i}: the values are the keys, vdim must be dim")
    else:
        raise ValueError(f"layer {i}: unknown mixer {kind!r}")
    return LayerSpec(kind, mixer, _feed_forward(raw.get("mlp"), i))


@dataclasses.dataclass
class NodutarConfig:
    vocab_size: int
    hidden_size: int
    layers: tuple[LayerSpec, ...]
    loop: Loop | None = None
    rms_norm_eps: float = 1e-6         # of every norm
    architecture: str = "nodutar"
    name: str = "nodutar"
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

    def runs(self) -> list[tuple[int, int, bool]]:
        """``(layer, pass, embeddings are added ahead of it)`` in the order of execution."""
        n, p = len(self.layers), self.loop or Loop(0, 0, 0)
        order = [(i, 0, False) for i in range(p.start)]
        order += [(i, k, k > 0 and i == p.start) for k in range(p.times) for i in range(p.start, p.stop)]
        return order + [(i, 0, False) for i in range(p.stop, n)]

    def validate(self) -> None:
        p = self.loop
        if p is not None and not (0 <= p.start < p.stop <= len(self.layers) and p.times >= 1):
            raise ValueError(f"loop {p} over {len(self.layers)} layers")
        for i, l in enumerate(self.layers):
            a, f = l.mixer.left if l.kind == PARALLEL else l.mixer, l.ff
            if a.heads % a.kv_heads:
                raise ValueError(f"layer {i}: heads must be a multiple of kv_heads")
            if l.kind == PARALLEL:
                if a.rot_dims % 2 or not 0 <= a.rot_dims <= a.dim:
                    raise ValueError(f"layer {i}: rot.dims must be even and at most {a.dim}")
                if a.vdim % 2:
                    raise ValueError(f"layer {i}: values turn in pairs, vdim must be even")
            if f is not None and (f.experts < 1 or f.experts > MAX_OUTPUTS or not 1 <= f.top <= min(f.experts, MAX_TOP)):
                raise ValueError(f"layer {i}: top {f.top} of {f.experts} experts")

    def first_layers(self, n: int) -> "NodutarConfig":
        """The first ``n`` layers; a loop that reaches beyond them is left out."""
        keep = self.loop if self.loop is not None and self.loop.stop <= n else None
        return dataclasses.replace(self, layers=self.layers[:n], loop=keep)

    # ---- (de)serialisation
    @classmethod
    def from_hf(cls, raw: dict[str, Any], name: str = "checkpoint") -> "NodutarConfig":
        loop = raw.get("loop")
        return cls(vocab_size=int(raw["vocab"]), hidden_size=int(raw["width"]), layers=tuple(_layer(l, i) for i, l in enumerate(raw["layers"])),
                   loop=Loop(*(int(loop[k]) for k in ("start", "stop", "times"))) if loop else None, rms_norm_eps=float(raw["norm"]["eps"]),
                   name=name)

    @classmethod
    def from_dir(cls, model_dir: str | Path) -> "NodutarConfig":
        p = Path(model_dir)
        return cls.from_hf(json.loads((p / "config.json").read_text()), name=p.name)

    def to_hf(self) -> dict[str, Any]:
        out = []
        for l in self.layers:
            m = dataclasses.asdict(l.mixer)
            if l.kind == PARALLEL:
                a = m["left"]
                a["rot"] = {"base": a.pop("rot_base"), "dims": a.pop("rot_dims")}
                chunk = a.pop("chunk")
                a["mask"] = {"size": chunk} if chunk else None
            else:
                m["vdim"] = m["dim"]
            f = l.ff
            mlp = {"kind": ROUTED, "expert": {"ff": f.ff}, "router": {"experts": f.experts, "top": f.top}} if f is not None else None
            out.append({"type": l.kind, "mixer": m, "mlp": mlp})
        return {"architecture": "Nodutar", "layers": out, "loop": dataclasses.asdict(self.loop) if self.loop else None,
                "norm": {"eps": self.rms_norm_eps}, "vocab": self.vocab_size, "width": self.hidden_size}

    # ---- tensors
    def tensor_plan(self) -> list[tuple[str, tuple[int, ...], str]]:
        """``(name, shape, kind)`` of every tensor; ``kind`` names the distribution random weights are drawn from."""
        W = self.hidden_size
        plan: list[tuple[str, tuple[int, ...], str]] = [("embed", (self.vocab_size, W), "embed")]

        def lin(name, n, k):
            plan.append((name, (n, k), "w"))
        for i, l in enumerate(self.layers):
            p, q, m, f = f"l{i}.", f"l{i}.mix.", l.mixer, l.ff
            plan += [(p + n, (W,), "norm0") for n in (("norm1", "norm1b") if f is None else ("norm1", "norm2", "norm1b", "norm2b"))]
            if l.kind == PARALLEL:
                a, r = m.left, m.right
                lin(q + "left.q", a.heads * a.dim, W), lin(q + "left.k", a.kv_heads * a.dim, W), lin(q + "left.v", a.kv_heads * a.vdim, W)
                plan += [(q + "left.q.norm", (a.dim,), "norm1"), (q + "left.k.norm", (a.dim,), "norm1")]
                lin(q + "left.o", W, a.heads * a.vdim)
                n = r.heads * r.dim
                lin(q + "right.q", n, W), lin(q + "right.f", n, W)
                plan += [(q + "right.f.b", (n,), "gate_b"), (q + "right.lower", (n,), "share")]
                lin(q + "right.v", r.heads * r.vdim, W)
                plan.append((q + "right.norm", (r.vdim,), "norm1"))
                lin(q + "right.o", W, r.heads * r.vdim)
            else:
                lin(q + "q", m.heads * m.dim, W), lin(q + "k", m.kv_heads * m.dim, W)
                plan += [(q + "r1", (m.heads,), "share"), (q + "r2", (m.heads,), "share")]
                lin(q + "o", W, m.heads * m.dim)
            if f is None:
                continue
            for e in range(f.experts):
                lin(f"{p}mlp.e{e}.gate", f.ff, W), lin(f"{p}mlp.e{e}.up", f.ff, W), lin(f"{p}mlp.e{e}.down", W, f.ff)
            lin(p + "mlp.router", f.experts, W)
            plan.append((p + "mlp.router.b", (f.experts,), "route"))
        plan.append(("final.norm", (W,), "norm0"))
        return plan


def preset_nodutar(name: str) -> NodutarConfig:
    """``tiny-nodutar``: every mechanism once, odd sizes.  ``nodutar-35b-a3b``: layers of a real model's size (width, runs, experts and
    feed-forward weights a token streams of the Qwen3.5 35B-A3B shape), three parallel layers to one of attention, four layers
    that run twice.  ``nodutar-3b``: the same at half the width and depth, with half the experts."""
    if name == "tiny-nodutar":
        par = LayerSpec(PARALLEL, ParallelMixer(ChunkAttention(6, 3, 24, 40, 0.2, 9000.0, 16, 70), GatedState(3, 40, 24), 0.8, 1.3), RoutedFF(56, 10, 3))
        att = LayerSpec(ATTENTION, DistanceMixer(4, 2, 48, 0.15), None)
        return NodutarConfig(512, 192, (att, par, att, par), Loop(1, 3, 2), name=name)
    if name in ("nodutar-35b-a3b", "nodutar-3b"):
        f = 1 if name == "nodutar-35b-a3b" else 2
        W, runs, experts = 2048 // f, 40 // f, 256 // f
        ff = RoutedFF(512, experts, 9)
        par = LayerSpec(PARALLEL, ParallelMixer(ChunkAttention(16 // f, 4 // f, 128, 128, 128 ** -0.5, 500000.0, 64, 1280), GatedState(16 // f, 128, 128),
                                                1.0, 1.0), ff)
        att = LayerSpec(ATTENTION, DistanceMixer(32 // f, 4 // f, 128, 128 ** -0.5), ff)
        layers = tuple(att if i % 4 == 3 else par for i in range(runs - 4))
        return NodutarConfig(151936, W, layers, Loop(8, 12, 2), name=name)
    raise KeyError(f"unknown preset {name!r}")
