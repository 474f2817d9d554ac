"""The Mamba-2 mixer of the family (latent attention is ``models.latent``'s): weights in the layout the kernels read, what a
sequence leaves behind, and the calls."""
from __future__ import annotations

import torch

from ...ops import mixers as X
from ..rowmodel import Mixer, Projection, RowBatch, pad8, padded
from .config import Mamba2Mixer


class Mamba2(Mixer):
    def __init__(self, m: Mamba2Mixer, W: dict[str, torch.Tensor], width: int, eps: float, slots: int, dtype, dev) -> None:
        self.m, self.eps = m, eps
        H, e, N, G, inner = m.heads, m.vdim, m.state, m.groups, m.inner
        f32 = lambda t: t.to(dev, torch.float32).contiguous()
        z, x, B, C, dt = torch.split(W["in"], [inner, inner, G * N, G * N, H])
        self.proj = Projection({"C": C, "B": B, "x": x, "z": z}, {"dt": dt}, width, dtype, dev)
        col = self.proj.col
        self.conv_width = col["z"]
        conv = torch.zeros(self.conv_width, m.conv, dtype=torch.float32, device=dev)
        bias = torch.zeros(self.conv_width, dtype=torch.float32, device=dev)
        for name, w, b in zip("xBC", torch.split(W["conv"], [inner, G * N, G * N]), torch.split(W["conv.b"], [inner, G * N, G * N])):
            conv[col[name]:col[name] + w.shape[0]] = f32(w)
            bias[col[name]:col[name] + w.shape[0]] = f32(b)
        depth = X.RING
        while depth < m.conv:
            depth *= 2
        self.state = {"S": torch.zeros(slots, H, N, e, dtype=torch.float32, device=dev),
                      "ring": torch.zeros(slots, depth, self.conv_width, dtype=dtype, device=dev)}
        self.norm_w = f32(W["norm"])
        self.w_out = padded(W["o"], pad8(width), pad8(inner), dtype, dev)
        self.core = X.Linrec(X.SSD, H=H, G=G, dk=N, dv=e, k_col=col["B"], v_col=col["x"], eps=eps, state=self.state, conv_w=conv,
                             conv_b=bias, A_log=f32(W["A_log"]), dt_bias=f32(W["dt_bias"]), D=f32(W["D"]))

    def run(self, model, b: RowBatch, h: torch.Tensor) -> torch.Tensor:
        m = self.m
        proj, gates = model.project(self.proj, h, b)
        y = model.buf("ssd_y", b.T, m.inner, torch.float32)
        model.recur(self.core, b, proj, gates, None, y, None)
        z0 = self.proj.col["z"]
        act = model.buf("act", b.T, pad8(m.inner))
        return X.gated_norm(y, proj[:, z0:z0 + m.inner], self.norm_w, act, groups=m.norm_groups, n=m.inner // m.norm_groups, eps=self.eps)
