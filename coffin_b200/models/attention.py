"""Attention layers of one score map per head over the rows of a batch: which kernels run for which rows.

A mixer that derives from ``SingleMapAttention`` builds its projection, pages and core (``ops.mixers.AttnMaps``, where the variants
of the mechanism are options); ``attend`` turns projection rows into finished heads.
"""
from __future__ import annotations

import torch

from ..ops import mixers as X
from .rowmodel import Mixer, RowBatch


class SingleMapAttention(Mixer):
    core: X.AttnMaps

    def attend(self, model, b: RowBatch, proj: torch.Tensor, act: torch.Tensor, cs: torch.Tensor | None = None, *,
               gate: torch.Tensor | None = None, values: torch.Tensor | None = None, lam: float = 0.0,
               turns: torch.Tensor | None = None) -> torch.Tensor:
        """Heads of all rows into ``act``; ``cs``, ``gate``, ``values``, ``lam`` and ``turns`` as for ``AttnMaps.rows_of``."""
        core, T, P = self.core, b.T, b.pre_rows
        sub = lambda t, r0, r1: t[r0:r1] if t is not None else None

        def rows(r0: int, r1: int):
            core.rows_of(sub(cs, r0, r1), sub(gate, r0, r1), sub(values, r0, r1), lam, sub(turns, r0, r1))
            return proj[r0:r1], b.positions[r0:r1], sub(b.row_seg, r0, r1)

        def parts(n: int, nsplit: int):
            return (model.buf("part_o", n, core.H * nsplit * core.vdim, torch.float32), model.buf("part_ml", n, core.H * nsplit * 2, torch.float32))

        if not core.tc:                 # 32-bit mode, or head sizes outside the tensor-core kernels
            pr, ps, rs = rows(0, T)
            po, pm = parts(T, 1)
            core.append(pr, b.tables, ps, rs, turn_queries=True)
            core.rows(pr, b.tables, ps, rs, po, pm)
            core.finish(po, pm, None, act, ps)
            return act
        r0 = 0
        if P:
            pr, ps, rs = rows(0, P)
            prompt = proj.dtype == model.dtype                    # few rows: fp32 projections, queries like any single token
            core.append(pr, b.tables, ps, rs, turn_queries=prompt)
            if prompt:
                core.flash(pr, b.tables, b.seg_row, b.seg_pos, None, None, segs=b.n_pre, max_rows=b.max_rows, positions=ps, act=act[:P])
                r0 = P
        if r0 < T:                      # the kernel norms and turns the queries, and appends the rows' own keys and values
            pr, ps, rs = rows(r0, T)
            ns = core.decode_splits(T - r0)
            if ns == 1:
                core.decode(pr, b.tables, ps, rs, None, None, 1, act=act[r0:])
            else:
                po, pm = parts(T - r0, ns)
                core.decode(pr, b.tables, ps, rs, po, pm, ns)
                core.finish(po, pm, None, act[r0:], ps, nsplit=ns)
        return act
