"""The two mixers of the family: weights in the layout the kernels read, what a sequence leaves behind, and the calls.

Latent attention is computed in one of two forms, chosen by the batch.  Single tokens and a few rows of portions use the
absorbed form (queries meet the cached latents themselves); longer portions multiply keys and values of every head out of
the cached rows and run the prompt kernels.  The weights carry the padding: heads are laid out at the tile sizes of the
prompt kernel with zero rows, and the product that expands keys has identity rows for the rotated part that all heads share.
"""
from __future__ import annotations

import torch

from ...ops import kernels as K
from ...ops import mixers as X
from ..rowmodel import Mixer, Projection, RowBatch, pad8, padded
from .config import LatentMixer, Mamba2Mixer

#: portions of at most this many rows in a batch stay in the absorbed form
ABSORB_ROWS = 24


def pad16(n: int) -> int:
    return (n + 15) // 16 * 16


def head_size(n: int, sizes: tuple[int, ...]) -> int:
    """Columns of a head: the next tile size of the prompt kernel, beyond them whole 16-byte pieces."""
    return next((s for s in sizes if n <= s), pad8(n))


class LatentAttention(Mixer):
    def __init__(self, m: LatentMixer, W: dict[str, torch.Tensor], width: int, eps: float, num_blocks: int, page: int, dtype, dev,
                 source: "LatentAttention | None") -> None:
        self.m = m
        H, n, r, e, R = m.heads, m.dim, m.rot_dim, m.vdim, m.kv_rank
        f32 = lambda t: t.to(dev, torch.float32).contiguous()
        own = source is None
        parts = {"cq": W["dq"]}
        if own:
            parts.update(c=W["dkv"][:R], r=W["dkv"][R:])
        self.proj = Projection(parts, {"g": W["g"]}, width, dtype, dev)
        col = self.proj.col
        self.qr, self.cp, rp = pad8(m.q_rank), pad16(R), pad16(r)
        LW = self.cp + rp
        n8 = self.r_off = pad8(n)                                 # the rotated part's column inside a head
        self.qd, self.vd = head_size(n8 + r, (64, 128, 192, 256)), head_size(e, (64, 128, 256))
        uq = torch.zeros(H, self.qd, self.qr, dtype=dtype, device=dev)
        src = W["uq"].to(dev, dtype).view(H, n + r, m.q_rank)
        uq[:, :n, :m.q_rank], uq[:, n8:n8 + r, :m.q_rank] = src[:, :n], src[:, n:]
        self.w_uq = uq.view(H * self.qd, self.qr)
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
                                 pool=self.pool, norm_q=f32(W["dq.norm"]), norm_c=f32(W["dkv.norm"]) if own else None,
                                 c_col=col.get("c", 0), r_col=col.get("r", 0))
        self.flash = None
        if self.expandable:
            z = self.w_kv                                         # pools are set per batch
            self.flash = X.AttnMaps(H=H, G=H, maps=1, dim=self.qd, vdim=self.vd, k_col=0, v_col=0, scale=m.scale, cap=None, temp=None, kpool=z,
                                    vpool=z)

    def weights(self):
        return [self.proj.w, self.w_uq, self.w_abs, self.w_val, self.w_out]

    # ---- angles of the batch, shared by the layers of one rotation
    def angles(self, model, b: RowBatch) -> torch.Tensor:
        m = self.m
        key = ("rope", m.rot_base, m.rot_dims)
        cs = b.cache.get(key)
        if cs is None:
            cs = model.buf(f"rope{m.rot_base}/{m.rot_dims}", b.T, max(2, m.rot_dims), torch.float32)
            if m.rot_dims:
                X.rope_rows(b.positions, self.turns, cs)
            b.cache[key] = cs
        return cs

    def run(self, model, b: RowBatch, h: torch.Tensor) -> torch.Tensor:
        m, T = self.m, b.T
        proj, gates = model.project(self.proj, h, b)
        cs = self.angles(model, b)
        cq = model.buf("cq", T, self.qr)
        self.core.rows(proj, cq, b.tables, b.positions, b.row_seg, cs)
        q = model.linear(self.w_uq, cq, model.buf("q", T, m.heads * self.qd))
        act = model.buf("act", T, m.heads * self.vd)
        r0 = 0
        if self.expandable and b.pre_rows > ABSORB_ROWS:
            r0 = b.pre_rows
            self._expanded(model, b, q[:r0], cs[:r0], gates[:r0], act[:r0])
        if r0 < T:
            self._absorbed(model, b, q[r0:], cs[r0:], gates[r0:], act[r0:], r0)
        return act

    def _rotate(self, q, dst, hd: int, off: int, cs) -> None:
        m = self.m
        X.rope_heads(q[:, self.r_off:], self.qd, dst[:, off:], hd, cs, half=m.rot_dims // 2, rot=m.rot_dim, H=m.heads)

    def _absorbed(self, model, b: RowBatch, q, cs, gates, act, r0: int) -> None:
        core, n, LW, H = self.core, q.shape[0], self.core.ldk, self.m.heads
        ps, rs = b.positions[r0:], b.row_seg[r0:] if b.row_seg is not None else None
        qa = model.buf("qa", n, H * LW)
        X.head_linear(self.w_abs, q, self.qd, qa, LW)
        self._rotate(q, qa, LW, self.cp, cs)
        ns = core.decode_splits(n) if core.tc else 1
        po, pm = model.buf("lat_o", n, H * ns * self.cp, torch.float32), model.buf("lat_ml", n, H * ns * 2, torch.float32)
        core.absorbed(qa, b.tables, ps, rs, po, pm, ns)
        oc = model.buf("oc", n, H * self.cp)
        core.merge(po, pm, oc, ps, ns)
        X.head_linear(self.w_val, oc, self.cp, act, self.vd, gate=gates)

    def _expanded(self, model, b: RowBatch, q, cs, gates, act) -> None:
        m, core, fl = self.m, self.core, self.flash
        base, lens, tables, rows, max_pages = b.expansion()
        g = b.cache.get(("gathered", core.pool.data_ptr()))       # layers that share latents share the gathered rows
        if g is None:
            g = model.buf(f"gather{core.pool.data_ptr()}" if self._lent else "gather", rows, core.ldk)
            core.gather(b.tables, base, lens, g, segs=b.n_pre, max_pages=max_pages)
            if self._lent:
                b.cache[("gathered", core.pool.data_ptr())] = g
        kv = model.buf("kv", rows, m.heads * (self.qd + self.vd))
        K.gemm(g, self.w_kv, out=kv)
        self._rotate(q, q, self.qd, self.r_off, cs)
        split = m.heads * self.qd
        fl.set_pools(kv[:, :split], kv[:, split:])
        fl.flash(q, tables, b.seg_row, b.seg_pos, None, None, segs=b.n_pre, max_rows=b.max_rows, positions=b.positions, act=act, gates=gates)

    _lent = False                       # set on a layer whose latents others read


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
