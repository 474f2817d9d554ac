"""Fasolorn on one B200.

Execution model
---------------
* The residual is one fp32 row per token.  One kernel per sublayer boundary adds the sublayer's output - or merges the
  expert rows of a routed feed-forward - and applies the RMS norm of the next projection (``ops.mixers.residual_step``).
* Batches, workspaces, pages and the captured decode step are ``models.rowmodel``'s: a forward is a batch of rows, portions
  of prompts before single tokens, in one pass over the weights.
* Attention layers cache turned keys and mixed values, latent layers one row per token.  The values that later layers mix
  in are those of the same token, so they are rows of the same forward: the first such layer's projection stays in a
  workspace of its own until the forward ends, and nothing of it is cached.
* Windows bound the pages that kernels walk and the rows that latent layers multiply out.
* ``dtype=torch.float32`` computes everything, products included, in 32-bit with the same step function and pages.
"""
from __future__ import annotations

import dataclasses

import torch

from ...ops import kernels as K
from ...ops import mixers as X
from ..experts import RoutedExperts
from ..latent import LatentAttention
from ..rowmodel import RowBatch, RowModel, pad8, padded
from .config import ATTENTION, DenseFF, FasolornConfig
from .mixers import WindowAttention


@dataclasses.dataclass
class _Layer:
    kind: str
    mixer: object
    gain1: torch.Tensor
    gain2: torch.Tensor | None = None
    w_gu: torch.Tensor | None = None
    w_down: torch.Tensor | None = None
    routed: RoutedExperts | None = None

    def ff_weights(self) -> list[torch.Tensor]:
        return self.routed.weights() if self.routed is not None else [t for t in (self.w_gu, self.w_down) if t is not None]


class FasolornModel(RowModel):
    family = "Fasolorn"

    def __init__(self, cfg: FasolornConfig, sd: dict[str, torch.Tensor], device: str | torch.device = "cuda", max_seq: int = 4096,
                 num_slots: int = 2, num_blocks: int | None = None, max_chunk: int = 2048, pdl: bool = True,
                 dtype: torch.dtype = torch.bfloat16, free_source: bool = False, quant: str = "none", kv_dtype: str = "bf16") -> None:
        self._setup(cfg, sd, device, max_seq, num_slots, num_blocks, max_chunk, pdl, dtype, quant, kv_dtype)
        c, dev, W = self.cfg, self.device, cfg.hidden_size

        def take(name: str) -> torch.Tensor:
            return sd.pop(name) if free_source else sd[name]

        def group(prefix: str) -> dict[str, torch.Tensor]:
            return {k[len(prefix):]: take(k) for k in [k for k in sd if k.startswith(prefix)]}

        f32 = lambda name: take(name).to(dev, torch.float32).contiguous()
        for i, spec in enumerate(c.layers):
            p, f = f"l{i}.", spec.ff
            mw = group(p + "mix.")
            if spec.kind == ATTENTION:
                mixer = WindowAttention(spec.mixer, mw, W, self.num_blocks, K.BLOCK, dtype, dev, lends=i == c.first_mixed)
            else:
                mixer = LatentAttention(spec.mixer, mw, W, self.eps, self.num_blocks, K.BLOCK, dtype, dev, window=spec.mixer.window, halves=True)
            L = _Layer(spec.kind, mixer, f32(p + "norm1"))
            if f is not None:
                L.gain2 = f32(p + "norm2")
                fw = group(p + "mlp.")
                if isinstance(f, DenseFF):
                    I, W8 = pad8(f.ff), pad8(W)
                    L.w_gu = torch.cat([padded(fw["gate"], I, W8, dtype, dev), padded(fw["up"], I, W8, dtype, dev)])
                    L.w_down = padded(fw["down"], W8, I, dtype, dev)
                else:
                    L.routed = RoutedExperts(fw, experts=f.experts, identity=f.identity, top=f.top, scale=f.scale, ff=f.ff, shared=f.shared,
                                             width=W, dtype=dtype, dev=dev)
            self.layers.append(L)
        self.final_gain = f32("final.norm")
        # the table serves as the head too; padded once, rows of the table are its first columns
        self.head = padded(take("embed"), pad8(c.vocab_size), pad8(W), dtype, dev)
        self.embed = self.head[:c.vocab_size, :W] if pad8(W) == W else self.head[:c.vocab_size, :W].contiguous()

    # ------------------------------------------------------------------ the stack
    def _stack(self, b: RowBatch):
        c, T, W = self.cfg, b.T, self.cfg.hidden_size
        x = self.buf("residual", T, W, torch.float32)
        h = self.buf("h", T, pad8(W))
        X.residual_embed(self.embed, b.tokens, x, c.embedding_scale)
        pend: dict = {}
        for li, L in enumerate(self.layers):
            X.residual_step(x, h, gain=L.gain1, eps=self.eps, **pend)
            act = L.mixer.run(self, b, h)
            pend = dict(y=self.linear(L.mixer.w_out, act, self.buf("y", T, L.mixer.w_out.shape[0])))
            if L.gain2 is not None:
                X.residual_step(x, h, gain=L.gain2, eps=self.eps, **pend)
                pend = L.routed.run(self, b, h) if L.routed is not None else dict(y=self.feed_forward(L, h, T))
            if self.layer_hook is not None:
                X.residual_step(x, None, **pend)
                pend = {}
                self.layer_hook(li, x)
        return x, pend

    def _out_rows(self, state, rows, n, h) -> None:
        x, pend = state
        X.residual_step(x, h, gain=self.final_gain, rows=rows, store=False, eps=self.eps, **pend)
