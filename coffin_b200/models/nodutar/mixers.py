"""The family's two mixers: weights in the layout the kernels read, pages and state of a layer run, and the calls.

A layer that runs several times has one mixer per run.  ``twin`` makes the further ones: the same weights, pages and state of
their own.
"""
from __future__ import annotations

import copy

import torch

from ...ops import kernels as K
from ...ops import mixers as X
from ..attention import SingleMapAttention
from ..rowmodel import Projection, RowBatch, pad8, padded
from .config import DistanceMixer, ParallelMixer


class _Looped(SingleMapAttention):
    def twin(self):
        other = copy.copy(self)
        other._cache()
        return other


class DistanceAttention(_Looped):
    """Normed queries against normed keys, scores less a multiple of the logarithm of the distance; the values are the keys ahead of
    their norm.  Pages hold the keys as projected, once, and a fp32 factor per key and head that stands for the norm."""

    def __init__(self, m: DistanceMixer, W: dict[str, torch.Tensor], width: int, eps: float, num_blocks: int, dtype, dev) -> None:
        self.m = m
        f32 = lambda n: W[n].to(dev, torch.float32).contiguous()
        self.proj = Projection({n: W[n] for n in ("q", "k")}, {}, width, dtype, dev)
        self.w_out = padded(W["o"], pad8(width), pad8(m.heads * m.dim), dtype, dev)
        self.distance, self.norm, self.rows, self.state = (f32("r1"), f32("r2")), (eps, None, None), num_blocks * K.BLOCK, {}
        self._cache()

    def _cache(self) -> None:
        m, w, k = self.m, self.w_out, self.proj.col["k"]
        keys = torch.zeros(self.rows, m.kv_heads, m.dim, dtype=w.dtype, device=w.device)
        factors = torch.zeros(self.rows, m.kv_heads, dtype=torch.float32, device=w.device)      # a page's rows together: [G, 64]
        self.pools = (keys, factors)
        self.core = X.AttnMaps(H=m.heads, G=m.kv_heads, maps=1, dim=m.dim, vdim=m.dim, k_col=k, v_col=k, scale=m.scale, cap=None, temp=None,
                               kpool=keys, vpool=keys, norm=self.norm, factors=factors, distance=self.distance)

    def run(self, model, b: RowBatch, h: torch.Tensor) -> torch.Tensor:
        proj, _ = model.project(self.proj, h, b)
        return self.attend(model, b, proj, model.buf("act", b.T, self.w_out.shape[1]))


class Parallel(_Looped):
    """Chunked attention (normed queries and keys, rotary positions on queries, keys and values) beside a gated matrix state.  One
    product projects for both, one takes both results back: the scales of the halves are applied to the heads in fp32."""

    def __init__(self, m: ParallelMixer, W: dict[str, torch.Tensor], width: int, eps: float, num_blocks: int, slots: int, dtype, dev) -> None:
        self.m, self.eps, self.slots, self.rows = m, eps, slots, num_blocks * K.BLOCK
        a, r = m.left, m.right
        f32 = lambda n: W[n].to(dev, torch.float32).contiguous()
        self.proj = Projection({"q": W["left.q"], "k": W["left.k"], "v": W["left.v"], "rq": W["right.q"], "rv": W["right.v"]}, {"f": W["right.f"]},
                               width, dtype, dev)
        self.right_col = pad8(a.heads * a.vdim)                   # of the gated state's heads in a result row
        self.w_out = torch.cat([padded(W["left.o"], pad8(width), self.right_col, dtype, dev),
                                padded(W["right.o"], pad8(width), pad8(r.heads * r.vdim), dtype, dev)], 1).contiguous()
        self.norm = (eps, f32("left.q.norm"), f32("left.k.norm"))
        self.gates = {"gate_b": f32("right.f.b"), "lower": f32("right.lower"), "norm_w": f32("right.norm") * m.right_scale}
        self.turns, self.value_turns = X.rope_turns(a.rot_base, a.rot_dims, dev), X.rope_turns(a.rot_base, a.vdim, dev)
        self._cache()

    def _cache(self) -> None:
        a, r, col, w = self.m.left, self.m.right, self.proj.col, self.w_out
        kpool = torch.zeros(self.rows, a.kv_heads, a.dim, dtype=w.dtype, device=w.device)
        vpool = torch.zeros(self.rows, a.kv_heads, a.vdim, dtype=w.dtype, device=w.device)
        self.pools = (kpool, vpool)
        self.state = {"S": torch.zeros(self.slots, r.heads, r.dim, r.vdim, dtype=torch.float32, device=w.device)}
        self.core = X.AttnMaps(H=a.heads, G=a.kv_heads, maps=1, dim=a.dim, vdim=a.vdim, k_col=col["k"], v_col=col["v"], scale=a.scale, cap=None,
                               temp=None, kpool=kpool, vpool=vpool, rot_dims=a.rot_dims, chunk=a.chunk, norm=self.norm, out_scale=self.m.left_scale)
        self.memory = X.Linrec(X.GATED, H=r.heads, G=r.heads, dk=r.dim, dv=r.vdim, k_col=0, v_col=col["rv"] - col["rq"], eps=self.eps,
                               state=self.state, **self.gates)

    def run(self, model, b: RowBatch, h: torch.Tensor) -> torch.Tensor:
        a, c = self.m.left, self.right_col
        proj, gates = model.project(self.proj, h, b)
        act = model.buf(f"act{c}", b.T, self.w_out.shape[1])      # padding between the halves: a workspace per layout
        cs, turns = model.angles(b, a.rot_base, a.rot_dims, self.turns), model.angles(b, a.rot_base, a.vdim, self.value_turns)
        self.attend(model, b, proj, act[:, :c], cs, turns=turns)
        model.recur(self.memory, b, proj[:, self.proj.col["rq"]:], gates, None, act[:, c:], None)
        return act
