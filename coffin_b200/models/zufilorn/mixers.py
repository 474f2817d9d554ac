"""The three mixers of the family: weights in the layout the kernels read, the layer's sequence state, and the calls.

A mixer takes the normalised rows of a batch (``RowBatch``: prompt portions first, single decoded tokens after them) and
leaves its result rows before the output projection in the shared workspace.  The batch decides the kernels: rows of a
portion go through the prompt kernels, single rows through the decode kernels, projections cover all rows at once.
"""
from __future__ import annotations

import torch

from ...ops import mixers as X
from ..rowmodel import Mixer, Projection, pad8, padded
from .config import AttentionMixer, DeltaMixer, MLstmMixer


class ChannelDelta(Mixer):
    def __init__(self, m: DeltaMixer, W: dict[str, torch.Tensor], width: int, eps: float, slots: int, dtype, dev) -> None:
        self.m = m
        H, G, d, e = m.heads, m.kv_heads, m.dim, m.vdim
        f32 = lambda t: t.to(dev, torch.float32).contiguous()
        self.proj = Projection({n: W[n] for n in ("q", "k", "v", "a1", "g1")}, {"b": W["b"]}, width, dtype, dev)
        col = self.proj.col
        self.conv_width = col["v"] + pad8(H * e)
        taps = W["q.conv"].shape[1]
        conv = torch.zeros(self.conv_width, taps, dtype=torch.float32, device=dev)
        for n in ("q", "k", "v"):
            t = W[n + ".conv"]
            conv[col[n]:col[n] + t.shape[0]] = f32(t)
        ra, rg = pad8(W["a1"].shape[0]), pad8(W["g1"].shape[0])
        self.a2 = padded(W["a2"], pad8(H * d), ra, dtype, dev)
        self.g2 = padded(W["g2"], pad8(H * e), rg, dtype, dev)
        self.ra, self.rg = ra, rg
        self.w_out = padded(W["o"], pad8(width), pad8(H * e), dtype, dev)
        depth = X.RING
        while depth < taps:
            depth *= 2
        self.state = {"S": torch.zeros(slots, H, d, e, dtype=torch.float32, device=dev),
                      "ring": torch.zeros(slots, depth, self.conv_width, dtype=dtype, device=dev)}
        self.core = X.Linrec(X.DELTA, H=H, G=G, dk=d, dv=e, k_col=col["k"], v_col=col["v"], eps=eps, state=self.state,
                             norm_w=f32(W["norm"]), conv_w=conv, A_log=f32(W["A_log"]), dt_bias=f32(W["dt_bias"]), a2=self.a2,
                             a1_col=col["a1"], g2=self.g2, g1_col=col["g1"])
        self.out_width = H * e

    def weights(self):
        return [self.proj.w, self.w_out, self.a2, self.g2]

    def run(self, model, b, h: torch.Tensor) -> torch.Tensor:
        m, col = self.m, self.proj.col
        proj, gates = model.project(self.proj, h, b)
        act = model.buf("act", b.T, pad8(self.out_width))
        dec = og = None
        if b.T > 8:                     # few rows: the step kernel multiplies the low-rank factors itself
            dec = model.buf("dec", b.T, self.a2.shape[0], torch.float32)
            og = model.buf("og", b.T, self.g2.shape[0])
            model.linear(self.a2, proj[:, col["a1"]:col["a1"] + self.ra], dec)
            model.linear(self.g2, proj[:, col["g1"]:col["g1"] + self.rg], og)
        model.recur(self.core, b, proj, gates, og, act, dec)
        return act


class MLstm(Mixer):
    def __init__(self, m: MLstmMixer, W: dict[str, torch.Tensor], width: int, eps: float, slots: int, dtype, dev) -> None:
        self.m = m
        H, d, e = m.heads, m.dim, m.vdim
        self.proj = Projection({n: W[n] for n in ("q", "k", "v", "g")}, {"i": W["i"], "f": W["f"]}, width, dtype, dev)
        col = self.proj.col
        self.w_out = padded(W["o"], pad8(width), pad8(H * e), dtype, dev)
        self.state = {"S": torch.zeros(slots, H, d, e, dtype=torch.float32, device=dev),
                      "n": torch.zeros(slots, H, d, dtype=torch.float32, device=dev),
                      "m": torch.zeros(slots, H, dtype=torch.float32, device=dev)}
        bias = torch.cat([W["i.b"], W["f.b"]]).to(dev, torch.float32).contiguous()
        self.core = X.Linrec(X.MLSTM, H=H, G=H, dk=d, dv=e, k_col=col["k"], v_col=col["v"], eps=eps, state=self.state,
                             norm_w=W["norm"].to(dev, torch.float32).contiguous(), gate_b=bias, cap=m.gate_cap)
        self.out_width = H * e

    def run(self, model, b, h: torch.Tensor) -> torch.Tensor:
        proj, gates = model.project(self.proj, h, b)
        act = model.buf("act", b.T, pad8(self.out_width))
        g0 = self.proj.col["g"]
        model.recur(self.core, b, proj, gates, proj[:, g0:g0 + self.out_width], act, None)
        return act


class DiffAttention(Mixer):
    MAPS = 2

    def __init__(self, m: AttentionMixer, W: dict[str, torch.Tensor], width: int, eps: float, num_blocks: int, page: int, dtype, dev) -> None:
        self.m, self.eps = m, eps
        H, G, d, e = m.heads, m.kv_heads, m.dim, m.vdim
        self.proj = Projection({n: W[n] for n in ("q", "k", "v")}, {"g": W["g"]}, width, dtype, dev)
        col = self.proj.col
        self.w_out = padded(W["o"], pad8(width), pad8(H * e), dtype, dev)
        lq1, lk1, lq2, lk2 = (W[n].float() for n in ("lq1", "lk1", "lq2", "lk2"))
        self.lam = float(torch.exp((lq1 * lk1).sum()) - torch.exp((lq2 * lk2).sum())) + m.diff
        kpool = torch.zeros(num_blocks * page, G * self.MAPS, d, dtype=dtype, device=dev)
        vpool = torch.zeros(num_blocks * page, G, e, dtype=dtype, device=dev)
        self.pools, self.state = (kpool, vpool), {}
        temp = (m.temp_coef, m.temp_every) if m.temp_every > 0 else None
        self.core = X.AttnMaps(H=H, G=G, maps=self.MAPS, dim=d, vdim=e, k_col=col["k"], v_col=col["v"], scale=m.scale, cap=m.softcap,
                               temp=temp, kpool=kpool, vpool=vpool)
        self.out_width = H * e

    def run(self, model, b, h: torch.Tensor) -> torch.Tensor:
        proj, gates = model.project(self.proj, h, b)
        act = model.buf("act", b.T, pad8(self.out_width))
        model.attend(self.core, b, proj, gates, act, lam=self.lam, post_scale=1.0 - self.m.diff)
        return act
