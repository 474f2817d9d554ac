"""Entry points of the routed feed-forward: choice of experts, lists of expert units, products over them.

``route_units`` (up to ``UNIT_ROWS`` rows) routes and lists units of up to 8 rows of one expert; ``unit_linear`` streams every
listed expert once.  More rows go through ``route``, ``ops.kernels.moe_dispatch`` and the grouped GEMM.
"""
from __future__ import annotations

import dataclasses

import torch

from . import kernels as K
from ._lib import call

UNIT, UNIT_ROWS = 8, 64


@dataclasses.dataclass(frozen=True)
class Router:
    """``experts`` stored experts, then ``identity`` outputs that return the input; the ``top`` largest of score + correction are
    chosen and weigh score / (their sum + 1e-20) * ``scale``; ``always`` more stored experts take every token with weight one.
    ``by_logit``: the ``top`` largest of logit + correction are chosen and weigh their softmax over the chosen ones, times ``scale``."""
    experts: int
    identity: int
    top: int
    scale: float
    always: int = 0
    by_logit: bool = False

    @property
    def slots(self) -> int:
        return self.top + self.always

    @property
    def stored(self) -> int:
        return self.experts + self.always


def _head(r: Router, logits: torch.Tensor, correction: torch.Tensor, positions: torch.Tensor | None) -> tuple:
    assert logits.dtype == correction.dtype == torch.float32 and logits.stride(1) == 1 and logits.shape[1] >= r.experts + r.identity
    return logits, logits.stride(0), correction, positions, logits.shape[0], r.experts, r.identity, r.top, r.always, float(r.scale), int(r.by_logit)


def route(r: Router, logits, correction, positions, idx, w, idw) -> None:
    """Slots ``idx`` (int32, -1: no stored expert) and weights ``w [T, slots]``, weight ``idw [T]`` of the input itself."""
    call("routed_topk", *_head(r, logits, correction, positions), idx, w, idw)
    K._count()


def max_units(r: Router, T: int) -> int:
    """Bound of the number of units of ``T`` rows: ``sum_e ceil(n_e / 8)``."""
    S = T * r.slots
    return min(S, r.stored + S // UNIT)


def route_units(r: Router, logits, correction, positions, idx, w, idw, meta, product: tuple | None = None) -> dict:
    """``route`` for at most ``UNIT_ROWS`` rows, with the expert-sorted order and its units (layout of ``moe_dispatch``'s result) in
    ``meta`` (int32).  ``product = (router weight, h, ticket)`` (at most 8 bf16 rows; the ticket a zeroed int32): the same launch
    computes the logits first."""
    T = logits.shape[0]
    S, n = T * r.slots, max_units(r, T)
    d = {"pos": meta[:S], "src_tok": meta[S:2 * S], "count": meta[2 * S:2 * S + 1], "row0": meta[2 * S + 1:2 * S + 1 + n],
         "rows": meta[2 * S + 1 + n:2 * S + 1 + 2 * n], "expert": meta[2 * S + 1 + 2 * n:2 * S + 1 + 3 * n], "max_tiles": n}
    call("routed_units", *_head(r, logits, correction, positions), idx, w, idw, d["pos"], d["src_tok"], d["count"], d["row0"], d["rows"],
         d["expert"], n, *((product[0], product[1], product[1].stride(0), product[1].shape[1], product[2]) if product is not None
                           else (None, None, 0, 0, None)))
    K._count()
    return d


def meta_size(r: Router, T: int) -> int:
    return 2 * T * r.slots + 1 + 3 * max_units(r, T)


def unit_linear(W: torch.Tensor, x: torch.Tensor, out: torch.Tensor, disp: dict, *, rows: int, gather: bool, relu2: bool = False,
                swiglu: bool = False, follows: bool = False) -> torch.Tensor:
    """``out[r] = W[expert(r)] @ x[src(r) if gather else r]`` for the sorted rows of a unit list (at most ``rows`` of them per unit).
    ``swiglu``: ``W`` holds gate rows, then as many up rows, and ``silu(gate) * up`` leaves.  ``follows``: the launch before this
    one is ``unit_linear`` over the same list."""
    E, N, Kd = W.shape
    act = 3 if swiglu else (2 if relu2 else 0)
    N = N // 2 if swiglu else N
    assert x.stride(1) == 1 and x.shape[1] == Kd and W.is_contiguous()
    src = disp["src_tok"] if gather else None
    lists = (disp["count"], disp["row0"], disp["rows"], disp["expert"], src)
    if out.dtype == torch.float32:
        call("routed_linear_f32", W, W.stride(0), x, x.stride(0), out, out.stride(0), N, Kd, *lists, disp["max_tiles"], act)
    else:
        call("gemv_units", W, W.stride(0), x, x.stride(0), out, out.stride(0), disp["max_tiles"], min(rows, UNIT), N, Kd, act,
             *lists, int(follows))
    K._count()
    return out
