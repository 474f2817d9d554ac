"""The family's attention mixer (latent attention is ``models.latent``'s): weights in the layout the kernels read, its pages, and
the calls."""
from __future__ import annotations

import torch

from ...ops import mixers as X
from ..attention import SingleMapAttention
from ..rowmodel import Projection, RowBatch, pad8, padded
from .config import AttentionMixer


class WindowAttention(SingleMapAttention):
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
        m, col = self.m, self.proj.col
        proj, _ = model.project(self.proj, h, b, "proj_lent" if self.lends else "proj")
        cs = model.angles(b, m.rot_base, m.rot_dims, self.turns)
        values = None
        if self.lends:
            b.cache["lent_values"] = proj[:, col["v"]:col["v"] + m.kv_heads * m.vdim]
        elif m.v_mix:
            values = b.cache["lent_values"]
        gate = proj[:, col["g"]:col["g"] + m.heads * m.vdim]
        return self.attend(model, b, proj, model.buf("act", b.T, pad8(m.heads * m.vdim)), cs, gate=gate, values=values, lam=self.lam)
