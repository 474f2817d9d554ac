"""Zufilorn on one B200.

Execution model
---------------
* The residual is ``streams`` fp32 copies ``[rows, S, W]``.  One kernel per sublayer boundary writes the previous
  sublayer's output back into all streams, reads the next sublayer's mix of them and normalises it
  (``ops.mixers.streams_step``), so the streams cross HBM once per sublayer.
* Every forward is a batch of rows (``RowBatch``): portions of prompts, then single tokens.  Projections and
  feed-forwards cover all rows in one product (tensor-core GEMV up to 8 rows, tcgen05 GEMM above); mixers run their
  prompt kernels over the portions and their decode kernels over the single rows.  A step that mixes both is one
  forward, which is what ``ModelRunner.run_batch`` and the mixed steps of the scheduler use.
* A step of single tokens only is a CUDA graph per row bucket: 7 launches per layer - streams, input projection (gates
  included, fp32), recurrence or attention (2 launches), output projection, streams, gate|up with SwiGLU, down.
* Per-sequence state lives in caller-assigned slots (recurrent matrices, normalisers, convolution rings) and in pages
  addressed through block tables (keys and values of the attention layers); the engine owns placement.
* ``dtype=torch.float32`` computes everything, products included, in 32-bit with the same step function, state and
  pages.
"""
from __future__ import annotations

import dataclasses

import torch

from ...ops import kernels as K
from ...ops import mixers as X
from ..rowmodel import RowBatch, RowModel, pad8, padded
from .config import ATTENTION, DELTA, ZufilornConfig
from .mixers import ChannelDelta, DiffAttention, MLstm


@dataclasses.dataclass
class _Layer:
    kind: str
    mixer: object
    gain1: torch.Tensor
    hc1: tuple[torch.Tensor, torch.Tensor, torch.Tensor]     # read, mix, write
    gain2: torch.Tensor | None = None
    hc2: tuple[torch.Tensor, torch.Tensor, torch.Tensor] | None = None
    w_gu: torch.Tensor | None = None
    w_down: torch.Tensor | None = None

    def ff_weights(self) -> list[torch.Tensor]:
        return [self.w_gu, self.w_down] if self.w_gu is not None else []


class ZufilornModel(RowModel):
    family = "Zufilorn"

    def __init__(self, cfg: ZufilornConfig, sd: dict[str, torch.Tensor], device: str | torch.device = "cuda", max_seq: int = 4096,
                 num_slots: int = 2, num_blocks: int | None = None, max_chunk: int = 2048, pdl: bool = True,
                 dtype: torch.dtype = torch.bfloat16, free_source: bool = False, quant: str = "none", kv_dtype: str = "bf16") -> None:
        self._setup(cfg, sd, device, min(int(max_seq), cfg.max_positions), num_slots, num_blocks, max_chunk, pdl, dtype, quant, kv_dtype,
                    free_shape=("a1", "a2", "g1", "g2"))   # the rank of the low-rank projections is the tensors' own
        c, dev = self.cfg, self.device

        def take(name: str) -> torch.Tensor:
            return sd.pop(name) if free_source else sd[name]

        f32 = lambda t: t.to(dev, torch.float32).contiguous()
        gain = lambda name: (1.0 + f32(take(name))).contiguous()
        W = c.hidden_size
        self.embed = take("embed").to(dev, dtype).contiguous()
        self.pos = take("pos").to(dev, dtype).contiguous()
        for i, spec in enumerate(c.layers):
            p = f"l{i}."
            mw = {k[len(p) + 4:]: take(k) for k in [k for k in sd if k.startswith(p + "mix.")]}
            if spec.kind == ATTENTION:
                mixer = DiffAttention(spec.mixer, mw, W, self.eps, self.num_blocks, K.BLOCK, dtype, dev)
            else:
                mixer = (ChannelDelta if spec.kind == DELTA else MLstm)(spec.mixer, mw, W, self.eps, self.num_slots, dtype, dev)
            hc = lambda q: tuple(f32(take(f"{p}{q}.{n}")) for n in ("in", "mix", "out"))
            L = _Layer(spec.kind, mixer, gain(p + "norm1"), hc("hc1"))
            if spec.ff is not None:
                L.gain2, L.hc2 = gain(p + "norm2"), hc("hc2")
                I, W8 = pad8(spec.ff), pad8(W)
                L.w_gu = torch.cat([padded(take(p + "mlp.gate"), I, W8, dtype, dev), padded(take(p + "mlp.up"), I, W8, dtype, dev)])
                L.w_down = padded(take(p + "mlp.down"), W8, I, dtype, dev)
            self.layers.append(L)
        self.final_gain = gain("final.norm")
        self.head = padded(take("head"), pad8(c.vocab_size), pad8(W), dtype, dev)

    # ------------------------------------------------------------------ sublayers
    def attend(self, core: X.AttnMaps, b: RowBatch, proj, gates, act, *, lam: float, post_scale: float) -> None:
        vh, T, P = core.H * core.maps, b.T, b.pre_rows
        fin = dict(lam=lam, post_scale=post_scale, eps=self.eps)

        def parts(rows: int, nsplit: int):
            return (self.buf("part_o", rows, vh * nsplit * core.vdim, torch.float32),
                    self.buf("part_ml", rows, vh * nsplit * 2, torch.float32))

        def sub(r0: int, r1: int):
            return proj[r0:r1], b.positions[r0:r1], b.row_seg[r0:r1] if b.row_seg is not None else None

        if not core.tc:                 # 32-bit mode, or head sizes outside the tensor-core kernels
            po, pm = parts(T, 1)
            core.append(proj, b.tables, b.positions, b.row_seg)
            core.rows(proj, b.tables, b.positions, b.row_seg, po, pm)
            core.finish(po, pm, gates, act, b.positions, **fin)
            return
        r0 = 0
        if P:
            pr, ps, rs = sub(0, P)
            core.append(pr, b.tables, ps, rs)
            if proj.dtype == self.dtype:
                po, pm = parts(P, 1)
                core.flash(pr, b.tables, b.seg_row, b.seg_pos, po, pm, segs=b.n_pre, max_rows=b.max_rows, positions=ps)
                core.finish(po, pm, gates[:P], act[:P], ps, **fin)
                r0 = P
        if r0 < T:                      # single tokens; the rows of a few short portions are queries like any other
            pr, ps, rs = sub(r0, T)
            ns = core.decode_splits(T - r0)
            po, pm = parts(T - r0, ns)
            core.decode(pr, b.tables, ps, rs, po, pm, ns)
            core.finish(po, pm, gates[r0:], act[r0:], ps, nsplit=ns, **fin)

    # ------------------------------------------------------------------ the stack
    def _stack(self, b: RowBatch) -> tuple[torch.Tensor, tuple]:
        """All layers over the rows of ``b``; returns the streams and the last sublayer's pending write-back."""
        c, T = self.cfg, b.T
        S, W = c.streams, c.hidden_size
        x = self.buf("streams", T, S * W, torch.float32).view(T, S, W)
        h = self.buf("h", T, pad8(W))
        X.streams_embed(self.embed, self.pos, b.tokens, b.positions, x)
        pend: dict = {}
        for li, L in enumerate(self.layers):
            X.streams_step(x, h, gain=L.gain1, read=L.hc1[0], eps=self.eps, **pend)
            act = L.mixer.run(self, b, h)
            y = self.linear(L.mixer.w_out, act, self.buf("y", T, L.mixer.w_out.shape[0]))
            pend = dict(y=y, mix=L.hc1[1], write=L.hc1[2])
            if L.w_gu is not None:
                X.streams_step(x, h, gain=L.gain2, read=L.hc2[0], eps=self.eps, **pend)
                pend = dict(y=self.feed_forward(L, h, T), mix=L.hc2[1], write=L.hc2[2])
            if self.layer_hook is not None:
                X.streams_step(x, None, **pend)
                pend = {}
                self.layer_hook(li, x.sum(1))
        return x, pend

    def _out_rows(self, state, rows, n, h) -> None:
        x, pend = state
        X.streams_step(x, h, gain=self.final_gain, rows=rows, store=False, eps=self.eps, **pend)
