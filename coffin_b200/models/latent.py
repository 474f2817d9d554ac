"""The latent attention mixer: weights in the layout the kernels read, its pages, and the calls.

Computed in one of two forms, chosen by the batch.  Single tokens and a few rows of portions use the absorbed form (queries
meet the cached latents themselves); longer portions multiply keys and values of every head out of the cached rows and run
the prompt kernels.  The weights carry the padding: heads are laid out at the tile sizes of the prompt kernel with zero rows,
and the product that expands keys has identity rows for the rotated part that all heads share.  They carry the rotation's
layout too: the kernels turn neighbouring pairs, and rows of a rotation that pairs halves are reordered at load (queries
and keys alike, so that scores do not change).
"""
from __future__ import annotations

import torch

from ..ops import kernels as K
from ..ops import mixers as X
from .rowmodel import Mixer, Projection, RowBatch, pad8

#: portions of at most this many rows in a batch stay in the absorbed form
ABSORB_ROWS = 24


def halves_to_pairs(t: torch.Tensor, dims: int) -> torch.Tensor:
    """Rows ``[.., n, K]`` of a rotated part whose entry i turns with entry i + dims / 2, reordered so that neighbours do."""
    o = torch.arange(t.shape[-2], device=t.device)
    o[:dims] = torch.arange(dims, device=t.device).view(2, dims // 2).t().reshape(-1)
    return t[..., o, :]


def pad16(n: int) -> int:
    return (n + 15) // 16 * 16


def head_size(n: int, sizes: tuple[int, ...]) -> int:
    """Columns of a head: the next tile size of the prompt kernel, beyond them whole 16-byte pieces."""
    return next((s for s in sizes if n <= s), pad8(n))


class LatentAttention(Mixer):
    """``m``: sizes (``heads``, ``dim``, ``rot_dim``, ``vdim``, ``kv_rank``, ``q_rank``), ``scale``, ``rot_base``, ``rot_dims``.  ``q_rank`` 0: queries are
    projected directly (weight ``q``).  Head gates where there is a weight ``g``.  ``window``: tokens a query sees, itself included
    (0: all).  ``halves``: the rotation pairs entry i with entry i + rot_dims / 2.  ``source``: the layer whose pages are read."""

    _lent = False                       # set on a layer whose latents others read

    def __init__(self, m, W: dict[str, torch.Tensor], width: int, eps: float, num_blocks: int, page: int, dtype, dev,
                 source: "LatentAttention | None" = None, *, window: int = 0, halves: bool = False) -> None:
        self.m, self.window = m, window
        H, n, r, e, R = m.heads, m.dim, m.rot_dim, m.vdim, m.kv_rank
        turn = (lambda t: halves_to_pairs(t, m.rot_dims)) if halves else (lambda t: t)
        n8 = self.r_off = pad8(n)                                 # the rotated part's column inside a head
        self.qd, self.vd = head_size(n8 + r, (64, 128, 192, 256)), head_size(e, (64, 128, 256))

        def heads(t: torch.Tensor, cols: int) -> torch.Tensor:
            """Query rows ``[H (n + r), k]`` at the padded head layout ``[H qd, cols]``."""
            out, t = torch.zeros(H, self.qd, cols, dtype=dtype, device=dev), t.to(dev, dtype).view(H, n + r, -1)
            k = t.shape[2]
            out[:, :n, :k], out[:, n8:n8 + r, :k] = t[:, :n], turn(t[:, n:])
            return out.view(H * self.qd, cols)
        f32 = lambda t: t.to(dev, torch.float32).contiguous()
        own = source is None
        parts = {"cq": W["dq"]} if m.q_rank else {"q": heads(W["q"], width)}
        if own:
            parts.update(c=W["dkv"][:R], r=turn(W["dkv"][R:]))
        self.proj = Projection(parts, {"g": W["g"]} if "g" in W else {}, width, dtype, dev)
        col = self.proj.col
        self.qr, self.cp, rp = pad8(m.q_rank), pad16(R), pad16(r)
        LW = self.cp + rp
        self.w_uq = heads(W["uq"], self.qr) if m.q_rank else None
        uk, uv = W["uk"].to(dev, dtype).view(H, n, R), W["uv"].to(dev, dtype).view(H, e, R)
        # absorbed form: q~ = uk^T q (per head [cp, n8]), o = uv c (per head [vd, cp])
        self.w_abs = torch.zeros(H, self.cp, n8, dtype=dtype, device=dev)
        self.w_abs[:, :R, :n] = uk.transpose(1, 2)
        self.w_val = torch.zeros(H, self.vd, self.cp, dtype=dtype, device=dev)
        self.w_val[:, :e, :R] = uv
        self.expandable = dtype == torch.bfloat16 and self.qd <= 256 and self.vd <= 256
        if self.expandable:                                       # keys of all heads, then values of all heads
            w = torch.zeros(H * (self.qd + self.vd), LW, dtype=dtype, device=dev)
            k = w[:H * self.qd].view(H, self.qd, LW)
            k[:, :n, :R] = uk
            k[:, n8:n8 + r, self.cp:self.cp + r] = torch.eye(r, dtype=dtype, device=dev)
            w[H * self.qd:].view(H, self.vd, LW)[:, :e, :R] = uv
            self.w_kv = w
        w_o = torch.zeros(pad8(width), H, self.vd, dtype=dtype, device=dev)
        w_o[:width, :, :e] = W["o"].to(dev, dtype).view(width, H, e)
        self.w_out = w_o.view(pad8(width), H * self.vd)
        if own:
            self.pool = torch.zeros(num_blocks * page, LW, dtype=dtype, device=dev)
            self.pools = (self.pool,)
        else:
            self.pool = source.pool
        self.state = {}
        self.turns = X.rope_turns(m.rot_base, m.rot_dims, dev)
        self.core = X.LatentAttn(H=H, q_rank=m.q_rank, kv_rank=R, rot=r, rot_dims=m.rot_dims, cp=self.cp, scale=m.scale, eps=eps,
                                 pool=self.pool, norm_q=f32(W["dq.norm"]) if m.q_rank else None, norm_c=f32(W["dkv.norm"]) if own else None,
                                 c_col=col.get("c", 0), r_col=col.get("r", 0), hq=self.qd, r_off=self.r_off, window=window)
        self.flash = None
        if self.expandable:
            z = self.w_kv                                         # pools are set per batch
            self.flash = X.AttnMaps(H=H, G=H, maps=1, dim=self.qd, vdim=self.vd, k_col=0, v_col=0, scale=m.scale, cap=None, temp=None, kpool=z,
                                    vpool=z, window=window)

    def weights(self):
        return [t for t in (self.proj.w, self.w_uq, self.w_abs, self.w_val, self.w_out) if t is not None]

    def run(self, model, b: RowBatch, h: torch.Tensor) -> torch.Tensor:
        m, T = self.m, b.T
        r0 = b.pre_rows if self.expandable and b.pre_rows > ABSORB_ROWS else 0       # rows in the expanded form
        cs = model.angles(b, m.rot_base, m.rot_dims, self.turns)
        act = model.buf("act", T, m.heads * self.vd)
        qa = model.buf("qa", T - r0, m.heads * self.core.ldk) if r0 < T else None
        if m.q_rank:
            proj, gates = model.project(self.proj, h, b)
            cq = model.buf("cq", T, self.qr)
            self.core.rows(proj, cq, b.tables, b.positions, b.row_seg, cs)
            q = model.linear(self.w_uq, cq, model.buf("q", T, m.heads * self.qd))
            if r0:
                self._rotate(q[:r0], q, self.qd, self.r_off, cs)
            if r0 < T:
                self._rotate(q[r0:], qa, self.core.ldk, self.cp, cs[r0:])
        else:
            # queries, latent and rotated key part from one product, in the activation type whatever the number of rows
            proj, gates = model.linear(self.proj.main, h, model.buf("proj", T, self.proj.n_main)), None
            self.core.rows(proj, None, b.tables, b.positions, b.row_seg, cs, split=r0, qa=qa)
            q = proj[:, :m.heads * self.qd]
        sub = lambda t, *s: t[slice(*s)] if t is not None else None
        if r0:
            self._expanded(model, b, q[:r0], sub(gates, r0), act[:r0])
        if r0 < T:
            self._absorbed(model, b, q[r0:], qa, sub(gates, r0, T), act[r0:], r0)
        return act

    def _rotate(self, q, dst, hd: int, off: int, cs) -> None:
        m = self.m
        X.rope_heads(q[:, self.r_off:], self.qd, dst[:, off:], hd, cs, half=m.rot_dims // 2, rot=m.rot_dim, H=m.heads)

    def _absorbed(self, model, b: RowBatch, q, qa, gates, act, r0: int) -> None:
        core, n, LW, H = self.core, q.shape[0], self.core.ldk, self.m.heads
        ps, rs = b.positions[r0:], b.row_seg[r0:] if b.row_seg is not None else None
        X.head_linear(self.w_abs, q, self.qd, qa, LW)
        ns = core.decode_splits(n) if core.tc else 1
        po, pm = model.buf("lat_o", n, H * ns * self.cp, torch.float32), model.buf("lat_ml", n, H * ns * 2, torch.float32)
        core.absorbed(qa, b.tables, ps, rs, po, pm, ns)
        oc = model.buf("oc", n, H * self.cp)
        core.merge(po, pm, oc, ps, ns)
        X.head_linear(self.w_val, oc, self.cp, act, self.vd, gate=gates)

    def _expanded(self, model, b: RowBatch, q, gates, act) -> None:
        m, core, fl = self.m, self.core, self.flash
        x = b.expansion(self.window)
        key = ("gathered", core.pool.data_ptr(), self.window)     # layers that share latents share the gathered rows
        g = b.cache.get(key)
        if g is None:
            g = model.buf(f"gather{core.pool.data_ptr()}" if self._lent else "gather", x["rows"], core.ldk)
            core.gather(b.tables, x["base"], x["lens"], x["skip"], g, segs=b.n_pre, max_pages=x["pages"])
            if self._lent:
                b.cache[key] = g
        kv = model.buf("kv", x["rows"], m.heads * (self.qd + self.vd))
        K.gemm(g, self.w_kv, out=kv)
        split = m.heads * self.qd
        fl.set_pools(kv[:, :split], kv[:, split:])
        fl.flash(q, x["tables"], b.seg_row, x["pos"], None, None, segs=b.n_pre, max_rows=b.max_rows, positions=b.positions, act=act, gates=gates)
