"""The family's attention mixer (latent attention is ``models.latent``'s): weights in the layout the kernels read, its pages, and
the calls."""
from __future__ import annotations

import torch

from ...ops import mixers as X
from ..rowmodel import Mixer, Projection, RowBatch, pad8, padded
from .config import AttentionMixer


class WindowAttention(Mixer):
    """Grouped-query attention over a sliding window with a sink per head, rotary positions, values mixed with another layer's,
    and an output gate per element.  Pages hold turned keys and mixed values."""

    def __init__(self, m: AttentionMixer, W: dict[str, torch.Tensor], width: int, num_blocks: int, page: int, dtype, dev, lends: bool) -> None:
        self.m, self.lends = m, lends              # lends: the first layer whose values are mixed into later ones
        H, G, d, e = m.heads, m.kv_heads, m.dim, m.vdim
        self.proj = Projection({n: W[n] for n in ("q", "k", "v", "g")}, {}, width, dtype, dev)
        self.w_out = padded(W["o"], pad8(width), pad8(H * e), dtype, dev)
        self.lam = float(W["vmix"]) if m.v_mix and not lends else 0.0
        kpool = torch.zeros(num_blocks * page, G, d, dtype=dtype, device=dev)
        vpool = torch.zeros(num_blocks * page, G, e, dtype=dtype, device=dev)
        self.pools, self.state = (kpool, vpool), {}
        self.turns = X.rope_turns(m.rot_base, m.rot_dims, dev)
        self.core = X.AttnMaps(H=H, G=G, maps=1, dim=d, vdim=e, k_col=self.proj.col["k"], v_col=self.proj.col["v"], scale=m.scale, cap=None,
                               temp=None, kpool=kpool, vpool=vpool, window=m.window, rot_dims=m.rot_dims,
                               sink=W["sink"].to(dev, torch.float32).contiguous())

    def run(self, model, b: RowBatch, h: torch.Tensor) -> torch.Tensor:
        m, core, col, T, P = self.m, self.core, self.proj.col, b.T, b.pre_rows
        proj, _ = model.project(self.proj, h, b, "proj_lent" if self.lends else "proj")
        cs = model.angles(b, m.rot_base, m.rot_dims, self.turns)
        values = None
        if self.lends:
            b.cache["lent_values"] = proj[:, col["v"]:col["v"] + m.kv_heads * m.vdim]
        elif m.v_mix:
            values = b.cache["lent_values"]
        gate = proj[:, col["g"]:col["g"] + m.heads * m.vdim]
        act = model.buf("act", T, pad8(m.heads * m.vdim))

        def rows(r0: int, r1: int):
            core.rows_of(cs[r0:r1], gate[r0:r1], values[r0:r1] if values is not None else None, self.lam)
            return proj[r0:r1], b.positions[r0:r1], b.row_seg[r0:r1] if b.row_seg is not None else None

        def parts(n: int, nsplit: int):
            return (model.buf("part_o", n, m.heads * nsplit * m.vdim, torch.float32), model.buf("part_ml", n, m.heads * nsplit * 2, torch.float32))

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
        if r0 < T:                      # the kernel turns the queries, and appends the rows' own keys and values
            pr, ps, rs = rows(r0, T)
            ns = core.decode_splits(T - r0)
            if ns == 1:
                core.decode(pr, b.tables, ps, rs, None, None, 1, act=act[r0:])
            else:
                po, pm = parts(T - r0, ns)
                core.decode(pr, b.tables, ps, rs, po, pm, ns)
                core.finish(po, pm, None, act[r0:], ps, nsplit=ns)
        return act
