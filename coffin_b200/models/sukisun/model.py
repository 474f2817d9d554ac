"""Sukisun on one B200.

Execution model
---------------
* The residual is fp32.  Every row keeps the embedding output and all layer results side by side (``[rows, planes, W]``);
  one kernel per sublayer boundary adds the sublayer's output, takes the depth average at a layer's end and applies the
  layer norm of the next projection (``ops.mixers.depth_step``).
* Batches, workspaces, sequence state and the captured decode step are ``models.rowmodel``'s: a forward is a batch of rows,
  portions of prompts before single tokens, in one pass over the weights.
* Attention layers cache one row per token, ``[latent | rotated key part]``; a layer with ``kv_from`` reads the pages of the
  layer it names and owns none.  Recurrent matrices and convolution rings live in state slots.
* ``dtype=torch.float32`` computes everything, products included, in 32-bit with the same step function, state and pages.
"""
from __future__ import annotations

import dataclasses

import torch
import torch.nn.functional as F

from ...ops import kernels as K
from ...ops import mixers as X
from ..latent import LatentAttention
from ..rowmodel import RowBatch, RowModel, pad8, padded
from .config import LATENT, SukisunConfig
from .mixers import Mamba2


@dataclasses.dataclass
class _Layer:
    kind: str
    mixer: object
    gain1: torch.Tensor
    dwa: torch.Tensor                           # weights of the embedding output and of the results, rows of later layers behind
    plan: dict                                  # which planes the average still has to read, what it prepares
    gain2: torch.Tensor | None = None
    w_up: torch.Tensor | None = None
    w_down: torch.Tensor | None = None
    act: tuple[float, float] = (0.0, 0.0)       # coefficients of the two xIELU branches

    def ff_weights(self) -> list[torch.Tensor]:
        return [self.w_up, self.w_down] if self.w_up is not None else []


class SukisunModel(RowModel):
    family = "Sukisun"

    def __init__(self, cfg: SukisunConfig, sd: dict[str, torch.Tensor], device: str | torch.device = "cuda", max_seq: int = 4096,
                 num_slots: int = 2, num_blocks: int | None = None, max_chunk: int = 2048, pdl: bool = True,
                 dtype: torch.dtype = torch.bfloat16, free_source: bool = False, quant: str = "none", kv_dtype: str = "bf16") -> None:
        self._setup(cfg, sd, device, max_seq, num_slots, num_blocks, max_chunk, pdl, dtype, quant, kv_dtype)
        c, dev, W = self.cfg, self.device, cfg.hidden_size

        def take(name: str) -> torch.Tensor:
            return sd.pop(name) if free_source else sd[name]

        f32 = lambda name: take(name).to(dev, torch.float32).contiguous()
        n = len(c.layers)
        dwa = torch.zeros(n, n + 1, dtype=torch.float32, device=dev)       # row i: planes 0 .. i + 1
        for i, spec in enumerate(c.layers):
            p = f"l{i}."
            mw = {k[len(p) + 4:]: take(k) for k in [k for k in sd if k.startswith(p + "mix.")]}
            if spec.kind == LATENT:
                src = self.layers[spec.mixer.kv_from].mixer if spec.mixer.kv_from is not None else None
                mixer = LatentAttention(spec.mixer, mw, W, self.eps, self.num_blocks, K.BLOCK, dtype, dev, src)
                if src is not None:
                    src._lent = mixer._lent = True
            else:
                mixer = Mamba2(spec.mixer, mw, W, self.eps, self.num_slots, dtype, dev)
            dwa[i, :i + 2] = take(p + "dwa").to(dev)
            L = _Layer(spec.kind, mixer, f32(p + "norm1"), dwa[i:], X.depth_plan(i, n))
            if spec.ff is not None:
                I, W8 = pad8(spec.ff), pad8(W)
                L.gain2 = f32(p + "norm2")
                L.w_up, L.w_down = padded(take(p + "mlp.up"), I, W8, dtype, dev), padded(take(p + "mlp.down"), W8, I, dtype, dev)
                pos, neg = F.softplus(take(p + "mlp.act").double()).tolist()
                L.act = (pos, 0.5 + neg)
            self.layers.append(L)
        self.final_gain = f32("final.norm")
        # the table serves as the head too; padded once, rows of the table are its first columns
        self.head = padded(take("embed"), pad8(c.vocab_size), pad8(W), dtype, dev)
        self.embed = self.head[:c.vocab_size, :W] if pad8(W) == W else self.head[:c.vocab_size, :W].contiguous()

    # ------------------------------------------------------------------ the stack
    def _stack(self, b: RowBatch):
        c, T, W = self.cfg, b.T, self.cfg.hidden_size
        planes = len(self.layers) + 2
        x = self.buf("depth", T, planes * W, torch.float32).view(T, planes, W)
        h = self.buf("h", T, pad8(W))
        X.depth_embed(self.embed, b.tokens, x, c.embedding_scale)
        pend: dict = {}
        plane = 1
        for li, L in enumerate(self.layers):
            # the boundary before layer i works on plane i (the previous layer's result), then plane i + 1 is the running residual
            X.depth_step(x, plane, h, gain=L.gain1, eps=self.eps, **pend)
            plane = li + 1
            act = L.mixer.run(self, b, h)
            pend = dict(y=self.linear(L.mixer.w_out, act, self.buf("y", T, L.mixer.w_out.shape[0])))
            if L.w_up is not None:
                X.depth_step(x, plane, h, gain=L.gain2, eps=self.eps, **pend)
                inter = X.linear_xielu(L.w_up, h, self.buf("inter", T, L.w_up.shape[0]), *L.act)
                pend = dict(y=self.linear(L.w_down, inter, self.buf("y", T, L.w_down.shape[0])))
            pend.update(weights=L.dwa, **L.plan)
            if self.layer_hook is not None:
                X.depth_step(x, plane, None, **pend)
                pend, plane = {}, plane + 1
                self.layer_hook(li, x[:, plane])
        return x, plane, pend

    def _out_rows(self, state, rows, n, h) -> None:
        x, plane, pend = state
        X.depth_step(x, plane, h, gain=self.final_gain, rows=rows, store=False, eps=self.eps, **pend)     # nothing left to prepare
