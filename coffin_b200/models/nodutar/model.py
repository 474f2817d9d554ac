"""Nodutar on one B200.

Execution model
---------------
* The residual is one fp32 row per token.  One kernel per sublayer boundary takes the sublayer's output - or merges the expert
  rows of a routed feed-forward -, applies the norm behind the sublayer, adds it and leaves the row for the next projection,
  normed again (``ops.mixers.residual_step``).
* Layers run in the order of ``NodutarConfig.runs``.  A layer that runs several times is several entries of ``layers`` with the
  same weights; pages and state are an entry's own, so batches, slots, snapshots and page copies are ``models.rowmodel``'s
  unchanged.  The embeddings that come back ahead of a repeated pass are read from the table by the boundary kernel.
* The two halves of a parallel layer share the projection and the output product; neither half's result is stored apart.
* Attention layers whose values are their keys cache one row per key, read once for both products.
* ``dtype=torch.float32`` computes everything, products included, in 32-bit with the same step function, state and pages.
"""
from __future__ import annotations

import dataclasses

import torch

from ...ops import mixers as X
from ..experts import RoutedExperts
from ..rowmodel import RowBatch, RowModel, pad8, padded
from .config import PARALLEL, NodutarConfig
from .mixers import DistanceAttention, Parallel


@dataclasses.dataclass
class _Layer:
    kind: str
    mixer: object
    gain1: torch.Tensor
    post1: torch.Tensor
    gain2: torch.Tensor | None = None
    post2: torch.Tensor | None = None
    routed: RoutedExperts | None = None
    again: bool = False                # the embeddings are added ahead of this run

    def ff_weights(self) -> list[torch.Tensor]:
        return self.routed.weights() if self.routed is not None else []


class NodutarModel(RowModel):
    family = "Nodutar"

    def __init__(self, cfg: NodutarConfig, sd: dict[str, torch.Tensor], device: str | torch.device = "cuda", max_seq: int = 4096,
                 num_slots: int = 2, num_blocks: int | None = None, max_chunk: int = 2048, pdl: bool = True,
                 dtype: torch.dtype = torch.bfloat16, free_source: bool = False, quant: str = "none", kv_dtype: str = "bf16") -> None:
        self._setup(cfg, sd, device, max_seq, num_slots, num_blocks, max_chunk, pdl, dtype, quant, kv_dtype)
        c, dev, W = self.cfg, self.device, cfg.hidden_size

        def take(name: str) -> torch.Tensor:
            return sd.pop(name) if free_source else sd[name]

        def group(prefix: str) -> dict[str, torch.Tensor]:
            return {k[len(prefix):]: take(k) for k in [k for k in sd if k.startswith(prefix)]}

        gain = lambda name: (1.0 + take(name).to(dev, torch.float32)).contiguous()         # stored around zero
        built: dict[int, _Layer] = {}
        for i, _, again in c.runs():
            L = built.get(i)
            if L is None:
                L = built[i] = self._build(c.layers[i], f"l{i}.", group, gain)
            else:
                L = dataclasses.replace(L, mixer=L.mixer.twin(), again=again)
            self.layers.append(L)
        self.final_gain = gain("final.norm")
        # the table serves as the head too; padded once, rows of the table are its first columns
        self.head = padded(take("embed"), pad8(c.vocab_size), pad8(W), dtype, dev)
        self.embed = self.head[:c.vocab_size, :W] if pad8(W) == W else self.head[:c.vocab_size, :W].contiguous()

    def _build(self, spec, p: str, group, gain) -> _Layer:
        mw, W, f, dtype, dev = group(p + "mix."), self.cfg.hidden_size, spec.ff, self.dtype, self.device
        if spec.kind == PARALLEL:
            mixer = Parallel(spec.mixer, mw, W, self.eps, self.num_blocks, self.num_slots, dtype, dev)
        else:
            mixer = DistanceAttention(spec.mixer, mw, W, self.eps, self.num_blocks, dtype, dev)
        L = _Layer(spec.kind, mixer, gain(p + "norm1"), gain(p + "norm1b"))
        if f is not None:
            L.gain2, L.post2 = gain(p + "norm2"), gain(p + "norm2b")
            L.routed = RoutedExperts(group(p + "mlp."), experts=f.experts, top=f.top, ff=f.ff, width=W, dtype=dtype, dev=dev, gated=True,
                                     by_logit=True, correction="router.b")
        return L

    # ------------------------------------------------------------------ the stack
    def _stack(self, b: RowBatch):
        T, W = b.T, self.cfg.hidden_size
        x = self.buf("residual", T, W, torch.float32)
        h = self.buf("h", T, pad8(W))
        X.residual_embed(self.embed, b.tokens, x, 1.0)
        pend: dict = {}
        for li, L in enumerate(self.layers):
            X.residual_step(x, h, gain=L.gain1, eps=self.eps, again=(self.embed, b.tokens) if L.again else None, **pend)
            act = L.mixer.run(self, b, h)
            pend = dict(y=self.linear(L.mixer.w_out, act, self.buf("y", T, L.mixer.w_out.shape[0])), post=L.post1)
            if L.routed is not None:
                X.residual_step(x, h, gain=L.gain2, eps=self.eps, **pend)
                pend = dict(L.routed.run(self, b, h), post=L.post2)
            if self.layer_hook is not None:
                X.residual_step(x, None, eps=self.eps, **pend)
                pend = {}
                self.layer_hook(li, x)
        return x, pend

    def _out_rows(self, state, rows, n, h) -> None:
        x, pend = state
        X.residual_step(x, h, gain=self.final_gain, rows=rows, store=False, eps=self.eps, **pend)
