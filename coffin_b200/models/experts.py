"""Routed feed-forward of the row-batch families: squared-relu or gated silu experts, a choice by corrected scores or by logits,
identity experts, a shared expert.

The shared expert rides with the routed ones: cut into parts of about an expert's width (exact, the activation works on single
columns), its parts are stored behind the experts and every token holds a slot for each with weight one.  So a step is
router product, routing, one product for all ups and one for all downs; the weighted sum of the slots happens in the
residual boundary that follows.

Up to ``UNIT_ROWS`` rows (and in 32-bit mode) an expert's rows go in units of 8 through a GEMV that streams every chosen
expert once; more rows are sorted by expert for the grouped tcgen05 GEMM.
"""
from __future__ import annotations

import torch

from ..ops import kernels as K
from ..ops import routed as R
from .rowmodel import RowBatch, pad8, padded


#: most parts of a shared expert; one far wider than its experts gets wider parts, and the experts zero columns
MAX_PARTS = 16


class RoutedExperts:
    def __init__(self, W: dict[str, torch.Tensor], *, experts: int, identity: int = 0, top: int, scale: float = 1.0, ff: int, shared: int = 0,
                 width: int, dtype, dev, gated: bool = False, by_logit: bool = False, correction: str = "correction") -> None:
        """``W``: ``e<i>.up`` / ``e<i>.down`` (``gated``: and ``e<i>.gate``, the activation is ``silu(gate) * up`` instead of the squared
        relu of up), ``router``, its ``correction`` under that name and, with ``shared`` > 0, ``shared.up`` / ``shared.down``
        (/ ``shared.gate``).  ``by_logit``: as ``ops.routed.Router``."""
        step = max(ff, -(-shared // MAX_PARTS))                   # columns of a part
        parts = -(-shared // step)
        self.r = R.Router(experts, identity, top, scale, parts, by_logit)
        self.gated = gated
        I, W8 = pad8(step), pad8(width)
        # gate rows of an expert come before its up rows
        self.up = torch.zeros(experts + parts, 2 * I if gated else I, W8, dtype=dtype, device=dev)
        first = (("gate", 0), ("up", I)) if gated else (("up", 0),)
        self.down = torch.zeros(experts + parts, W8, I, dtype=dtype, device=dev)
        for e in range(experts):
            for n, o in first:
                self.up[e, o:o + ff, :width] = W[f"e{e}.{n}"].to(dev, dtype)
            self.down[e, :width, :ff] = W[f"e{e}.down"].to(dev, dtype)
        for p in range(parts):
            a, b = p * step, min(shared, (p + 1) * step)
            for n, o in first:
                self.up[experts + p, o:o + b - a, :width] = W[f"shared.{n}"][a:b].to(dev, dtype)
            self.down[experts + p, :width, :b - a] = W["shared.down"][:, a:b].to(dev, dtype)
        self.router = padded(W["router"], pad8(experts + identity), W8, dtype, dev)
        self.correction = W[correction].to(dev, torch.float32).contiguous()

    def weights(self) -> list[torch.Tensor]:
        """What a step of one token streams."""
        n = self.r.slots
        return [self.router, self.up[:n], self.down[:n]]

    def run(self, model, b: RowBatch, h: torch.Tensor) -> dict:
        """Keywords of the ``residual_step`` that merges the result."""
        r, T, I, W8 = self.r, b.T, self.down.shape[2], self.up.shape[2]
        relu2, swiglu = not self.gated, self.gated
        S = T * r.slots
        logits = model.buf("route_z", T, self.router.shape[0], torch.float32)
        product = None
        if T <= 8 and not model.f32:    # few rows: the product is the routing kernel's own
            product = (self.router, h, model.buf("route_ticket", 1, 1, torch.int32))
        else:
            model.linear(self.router, h, logits)
        idx, w = model.buf("route_i", T, r.slots, torch.int32), model.buf("route_w", T, r.slots, torch.float32)
        idw = model.buf("route_id", T, 1, torch.float32)
        units = T <= R.UNIT_ROWS
        if units:
            disp = R.route_units(r, logits, self.correction, b.positions, idx, w, idw, model.buf("route_u", 1, R.meta_size(r, T), torch.int32)[0],
                                 product)
        else:
            R.route(r, logits, self.correction, b.positions, idx, w, idw)
            disp = K.moe_dispatch(idx, r.stored, R.UNIT if model.f32 else 128)
        inter, y = model.buf("route_h", S, I), model.buf("route_y", S, W8)
        if units or model.f32:
            R.unit_linear(self.up, h, inter, disp, rows=T, gather=True, relu2=relu2, swiglu=swiglu)
            R.unit_linear(self.down, inter, y, disp, rows=T, gather=False, follows=True)
        else:
            rows = h.index_select(0, disp["src_tok"])
            if swiglu:
                K.swiglu(K.gemm_grouped(rows, self.up, disp, out=model.buf("route_gu", S, 2 * I)), out=inter)
            else:
                K.gemm_grouped(rows, self.up, disp, out=inter, relu2=True)
            K.gemm_grouped(inter, self.down, disp, out=y)
        return {"experts": (y, disp["pos"], w, idw if r.identity else None, h)}
