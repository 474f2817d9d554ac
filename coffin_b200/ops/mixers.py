"""Entry points of the kernels behind fp32 residuals, the recurrent mixers, multi-map attention and latent attention.

Like ``ops.kernels`` these are thin wrappers that launch on the current stream into caller-owned buffers.  Every
constant of a mechanism (tap count, gate cap, number of maps, score cap, query temperature, number of streams, rotary
base) is an argument, so a model family picks what it needs:

* ``streams_embed`` / ``streams_step``: a residual of several fp32 streams with static read / write / mixing weights;
* ``depth_embed`` / ``depth_step``: a residual that becomes a weighted sum of all layer results after every layer;
* ``Linrec``: recurrences with a matrix state - the per-channel gated delta rule, the mLSTM matrix memory, forget gates that
  also write (HGRN2) and the state space with scalar decays (Mamba-2); ``gated_norm``: its output gate and grouped RMS norm;
* ``AttnMaps``: paged attention with several score maps per head over the same values, capped scores, a
  position-dependent query temperature, a sliding window or chunks, sinks, rotary positions (of values too), norms of queries
  and keys, penalties by the logarithm of the distance, keys that are their own values, mixed values and gates per element;
* ``LatentAttn``: attention over cached low-rank latents with a rotated key part shared by all heads; ``rope_rows`` /
  ``rope_heads``: rotary angles of a batch and interleaved rotation of head parts;
* ``residual_embed`` / ``residual_step``: a plain fp32 residual whose boundaries also merge expert rows, norm what they add
  and repeat the embedding;
* ``gemm_f32out`` / ``gemm_f32``: projections whose result (or everything) stays fp32; ``linear_xielu``: a projection
  with xIELU in its epilogue.
"""
from __future__ import annotations

import ctypes

import torch

from . import _lib
from . import kernels as K
from ._lib import call

DELTA, MLSTM, SSD, GATED = 0, 1, 2, 3
RING = 16             # shallowest convolution ring
_P, _I64, _I32, _F = ctypes.c_void_p, ctypes.c_int64, ctypes.c_int, ctypes.c_float


def _ptr(t: torch.Tensor | None) -> int | None:
    return None if t is None else t.data_ptr()


def _is_f32(t: torch.Tensor) -> int:
    return int(t.dtype == torch.float32)


# ------------------------------------------------------------------ projections
def gemm_f32out(A: torch.Tensor, W: torch.Tensor, out: torch.Tensor) -> torch.Tensor:
    """``out[M, N] (fp32) = A[M, K] @ W[N, K]^T`` from bf16 operands on tcgen05, accumulator unrounded."""
    M, Kd = A.shape
    N = W.shape[0]
    assert out.dtype == torch.float32 and out.stride(1) == 1 and A.stride(1) == 1 and W.stride(1) == 1
    ws = tickets = None
    if M <= 128 and K.SPLITK_GEMM:
        ws, tickets = K._splitk_scratch(A.device)
    call("gemm_bf16_f32out", A, A.stride(0), W, W.stride(0), out, out.stride(0), M, N, Kd, ws,
         ws.numel() * 4 if ws is not None else 0, tickets, tickets.numel() if tickets is not None else 0, K.status_word(A.device))
    K._count()
    return out


def gemm_mixed(A: torch.Tensor, W: torch.Tensor, main: torch.Tensor, gates: torch.Tensor) -> None:
    """One product ``A @ W^T``: its first columns rounded to bf16 in ``main``, the others unrounded in ``gates`` (fp32)."""
    M, Kd = A.shape
    N, n_main = W.shape[0], main.shape[1]
    assert gates.dtype == torch.float32 and gates.shape[1] == N - n_main and main.stride(1) == gates.stride(1) == A.stride(1) == 1
    ws = tickets = None
    if M <= 128 and K.SPLITK_GEMM:
        ws, tickets = K._splitk_scratch(A.device)
    call("gemm_bf16_mixed", A, A.stride(0), W, W.stride(0), main, main.stride(0), gates, gates.stride(0), n_main, M, N, Kd, ws,
         ws.numel() * 4 if ws is not None else 0, tickets, tickets.numel() if tickets is not None else 0, K.status_word(A.device))
    K._count()


def gemm_f32(A: torch.Tensor, W: torch.Tensor, out: torch.Tensor) -> torch.Tensor:
    """True fp32 product of any shape (the 32-bit mode of a model)."""
    M, Kd = A.shape
    N = W.shape[0]
    assert A.dtype == W.dtype == out.dtype == torch.float32 and A.stride(1) == W.stride(1) == out.stride(1) == 1
    call("gemm_f32", A, A.stride(0), W, W.stride(0), out, out.stride(0), M, N, Kd)
    K._count()
    return out


def swiglu_f32(gu: torch.Tensor, out: torch.Tensor) -> torch.Tensor:
    M, two_i = gu.shape
    call("swiglu_f32", gu, gu.stride(0), out, out.stride(0), M, two_i // 2)
    K._count()
    return out


def linear_xielu(W: torch.Tensor, x: torch.Tensor, out: torch.Tensor, a: float, b: float) -> torch.Tensor:
    """``out = xielu(x @ W^T)``, ``xielu(z) = z / 2 + (a z^2 if z > 0 else b (exp(z) - 1 - z))``."""
    T, Kd = x.shape
    if out.dtype == torch.float32:
        gemm_f32(x, W, out)
        call("xielu_f32", out, out.stride(0), out, out.stride(0), T, W.shape[0], float(a), float(b))
    elif T <= 8 and T * Kd * 2 <= 160 * 1024:
        call("gemv_mma_bf16_xielu", W, x.contiguous(), out, T, W.shape[0], Kd, out.stride(0), float(a), float(b))
    else:
        ws = tickets = None
        if T <= 128 and K.SPLITK_GEMM:
            ws, tickets = K._splitk_scratch(x.device)
        call("gemm_bf16_xielu", x, x.stride(0), W, W.stride(0), out, out.stride(0), T, W.shape[0], Kd, float(a), float(b), ws,
             ws.numel() * 4 if ws is not None else 0, tickets, tickets.numel() if tickets is not None else 0, K.status_word(x.device))
    K._count(2 if out.dtype == torch.float32 else 1)
    return out


# ------------------------------------------------------------------ hyper-connected streams
def streams_embed(embed: torch.Tensor, pos: torch.Tensor | None, tokens: torch.Tensor, positions: torch.Tensor,
                  x: torch.Tensor) -> torch.Tensor:
    """Every stream of row ``t`` of ``x [T, S, W]`` (fp32) starts as ``embed[token] + pos[position]``."""
    T, S, W = x.shape
    assert x.dtype == torch.float32 and x.is_contiguous() and tokens.dtype == torch.int64 and positions.dtype == torch.int32
    call("streams_embed", embed, pos, tokens, positions, x, T, S, W, embed.shape[0], pos.shape[0] if pos is not None else 0, _is_f32(embed))
    K._count()
    return x


def streams_step(x: torch.Tensor, h: torch.Tensor | None, *, gain: torch.Tensor | None = None, read: torch.Tensor | None = None,
                 y: torch.Tensor | None = None, mix: torch.Tensor | None = None, write: torch.Tensor | None = None,
                 rows: torch.Tensor | None = None, store: bool = True, eps: float = 1e-5) -> torch.Tensor | None:
    """Boundary between two sublayers: write ``y`` back (``x_t <- sum_s mix[s, t] x_s + write[t] y``), then
    ``h = rmsnorm(sum_s read[s] x_s) * gain`` (``read`` None: plain sum).  ``rows`` picks the stream rows behind the
    rows of ``h`` (with ``store=False``)."""
    T, S, W = x.shape
    n = rows.numel() if rows is not None else (h.shape[0] if h is not None else T)
    t = h if h is not None else y
    call("streams_step", x, y, y.stride(0) if y is not None else 0, mix, write, read, gain, h, h.stride(0) if h is not None else 0,
         rows, n, S, W, float(eps), int(store), _is_f32(t))
    K._count()
    return h


# ------------------------------------------------------------------ plain residual
def residual_embed(embed: torch.Tensor, tokens: torch.Tensor, x: torch.Tensor, scale: float) -> torch.Tensor:
    """``x [T, W]`` (fp32) = ``embed[token] * scale``."""
    T, W = x.shape
    assert x.dtype == torch.float32 and x.is_contiguous() and embed.is_contiguous() and tokens.dtype == torch.int64
    call("residual_embed", embed, tokens, x, T, W, embed.shape[0], float(scale), _is_f32(embed))
    K._count()
    return x


def residual_step(x: torch.Tensor, h: torch.Tensor | None, *, gain: torch.Tensor | None = None, y: torch.Tensor | None = None,
                  experts: tuple | None = None, post: torch.Tensor | None = None, again: tuple | None = None, rows: torch.Tensor | None = None,
                  store: bool = True, eps: float = 1e-5) -> torch.Tensor | None:
    """Boundary between two sublayers: ``x [T, W] += y``, or with ``experts = (ys, pos, w, idw, hin)`` the weighted expert rows
    ``sum_j w[t, j] ys[pos[t, j]] + idw[t] hin[t]``; with ``post`` what is added is ``rmsnorm(that) * post``; with
    ``again = (table, tokens)`` the embeddings are added too; then ``h = rmsnorm(x) * gain``.  ``rows`` picks the residual rows
    behind the rows of ``h`` (with ``store=False``)."""
    T, W = x.shape
    n = rows.numel() if rows is not None else (h.shape[0] if h is not None else T)
    ys, pos, w, idw, hin = experts if experts is not None else (None,) * 5
    table, tokens = again if again is not None else (None, None)
    t = next((v for v in (h, y, ys, table) if v is not None), None)
    assert table is None or (table.is_contiguous() and table.shape[1] == W and table.dtype == t.dtype and tokens.dtype == torch.int64)
    ld = lambda v: v.stride(0) if v is not None else 0
    call("residual_step", x, y, ld(y), ys, ld(ys), pos, w, w.shape[1] if w is not None else 0, idw, hin, ld(hin), gain, h, ld(h), rows, n, W,
         float(eps), int(store), post, table, tokens, table.shape[0] if table is not None else 0, _is_f32(t) if t is not None else 0)
    K._count()
    return h


# ------------------------------------------------------------------ depth-averaged residual
def depth_embed(embed: torch.Tensor, tokens: torch.Tensor, x: torch.Tensor, scale: float) -> torch.Tensor:
    """Planes 0 (the embedding output) and 1 (the running residual of the first layer) of ``x [T, planes, W]`` (fp32)."""
    T, planes, W = x.shape
    assert x.dtype == torch.float32 and x.stride(2) == 1 and x.stride(1) == W and planes >= 2 and tokens.dtype == torch.int64
    call("depth_embed", embed, tokens, x, x.stride(0), T, W, embed.shape[0], float(scale), _is_f32(embed))
    K._count()
    return x


DEPTH_BLOCK = 8


def depth_plan(layer: int, layers: int) -> dict[str, int]:
    """``first`` / ``prep`` of a layer's end when the averages are taken in blocks of ``DEPTH_BLOCK`` layers."""
    start = layer // DEPTH_BLOCK * DEPTH_BLOCK               # the planes 0 .. start were summed up before the block
    prep = min(DEPTH_BLOCK, layers - 1 - layer) if (layer + 1) % DEPTH_BLOCK == 0 else 0
    return {"first": start + 1 if start and not prep else 0, "prep": prep}


def depth_step(x: torch.Tensor, plane: int, h: torch.Tensor | None, *, gain: torch.Tensor | None = None, y: torch.Tensor | None = None,
               weights: torch.Tensor | None = None, first: int = 0, prep: int = 0, rows: torch.Tensor | None = None, store: bool = True,
               eps: float = 1e-5, center: bool = True) -> torch.Tensor | None:
    """Boundary between two sublayers: plane ``plane`` of ``x [T, planes, W]`` += ``y``; with ``weights`` (a layer's end) the
    weighted sum of planes ``0 .. plane`` becomes plane ``plane + 1``.  Row 0 of ``weights`` is this layer's; ``prep``: the sums of
    that many following layers (the next rows) over the same planes are left where their averages will go; ``first``: planes
    below it have been summed up that way already (``depth_plan``).  Then ``h = norm(result) * gain``, layer norm
    (``center``) or RMS norm.  ``rows`` picks the rows behind the rows of ``h`` (with ``store=False``)."""
    T, planes, W = x.shape
    n = rows.numel() if rows is not None else (h.shape[0] if h is not None else T)
    t = h if h is not None else y
    assert weights is None or (weights.stride(-1) == 1 and weights.shape[-1] > plane and (not store or plane + 2 + prep <= planes))
    assert not prep or (weights.dim() == 2 and weights.shape[0] > prep)
    call("depth_step", x, x.stride(0), plane, y, y.stride(0) if y is not None else 0, weights, weights.stride(0) if weights is not None else 0, first, prep,
         gain, h, h.stride(0) if h is not None else 0, rows, n, W, float(eps), int(center), int(store), _is_f32(t) if t is not None else 0)
    K._count()
    return h


# ------------------------------------------------------------------ recurrences with a matrix state
class _LinrecStruct(ctypes.Structure):
    _fields_ = [("proj", _P), ("ldp", _I64), ("gates", _P), ("ldg", _I64), ("dec", _P), ("ldd", _I64), ("og", _P), ("ldo", _I64),
                ("act", _P), ("lda", _I64), ("seg_row", _P), ("seg_pos", _P), ("seg_slot", _P), ("conv_w", _P), ("taps", _I32),
                ("A_log", _P), ("dt_bias", _P), ("a2", _P), ("ra", _I64), ("a1_col", _I64), ("g2", _P), ("rg", _I64), ("g1_col", _I64),
                ("norm_w", _P), ("gate_b", _P), ("S", _P), ("n", _P), ("m", _P), ("ring", _P), ("ring_mask", _I32), ("ring_w", _I64),
                ("H", _I32), ("G", _I32), ("dk", _I32), ("dv", _I32), ("jc", _I32), ("k_col", _I64), ("v_col", _I64),
                ("eps", _F), ("cap", _F), ("conv_b", _P), ("D", _P), ("lower", _P)]


def linrec_supported(H: int, dk: int, dv: int) -> bool:
    return bool(_lib.call_nostream("linrec_supported", H, dk, dv))


class Linrec:
    """One recurrent layer: fixed weights, state tensors and sizes; ``step`` / ``ring`` launch on a batch of rows.

    ``state``: ``S [slots, H, dk, dv]`` and, by kind, ``ring [slots, depth, width]`` (delta: the last raw projection
    rows, indexed by position modulo depth) or ``n [slots, H, dk]`` and ``m [slots, H]`` (mLSTM), all zero at the
    start of a sequence.  Gated: the gate columns are the forget gates' pre-activations of all channels, ``gate_b`` their bias,
    ``lower`` their lower bounds; there are no keys and no output gate.  State space: keys, queries and values are B, C and x, the ring is the delta's, and the rows
    that leave are fp32 and unnormed (``gated_norm`` follows)."""

    def __init__(self, kind: int, *, H: int, G: int, dk: int, dv: int, k_col: int, v_col: int, eps: float, state: dict,
                 norm_w: torch.Tensor | None = None, conv_w: torch.Tensor | None = None, A_log=None, dt_bias=None, a2=None,
                 a1_col: int = 0, g2=None, g1_col: int = 0, gate_b=None, cap: float = 0.0, conv_b=None, D=None, lower=None) -> None:
        if kind != SSD and not linrec_supported(H, dk, dv):
            raise ValueError(f"recurrent head of {dk} x {dv} is outside the kernel's range")
        a = self.a = _LinrecStruct()
        size = _lib.call_nostream("linrec_args_size")
        assert ctypes.sizeof(a) == size, f"argument layout: {ctypes.sizeof(a)} here, {size} in the library"
        self.kind, self.state, self.conv_w = kind, state, conv_w
        self._keep = (norm_w, conv_w, A_log, dt_bias, a2, g2, gate_b, conv_b, D, lower, *state.values())
        a.conv_b, a.D, a.lower = _ptr(conv_b), _ptr(D), _ptr(lower)
        a.H, a.G, a.dk, a.dv, a.k_col, a.v_col, a.eps, a.cap = H, G, dk, dv, k_col, v_col, float(eps), float(cap)
        a.norm_w, a.conv_w, a.A_log, a.dt_bias, a.gate_b = _ptr(norm_w), _ptr(conv_w), _ptr(A_log), _ptr(dt_bias), _ptr(gate_b)
        a.taps = conv_w.shape[1] if conv_w is not None else 0
        if a2 is not None:
            a.a2, a.ra, a.a1_col, a.g2, a.rg, a.g1_col = _ptr(a2), a2.shape[1], a1_col, _ptr(g2), g2.shape[1], g1_col
        a.S, a.n, a.m, a.ring = _ptr(state["S"]), _ptr(state.get("n")), _ptr(state.get("m")), _ptr(state.get("ring"))
        ring = state.get("ring")
        if ring is not None:
            assert ring.shape[1] & (ring.shape[1] - 1) == 0, "ring depth must be a power of two"
            a.ring_mask, a.ring_w = ring.shape[1] - 1, ring.shape[2]

    def _fill(self, proj, gates, og, act, dec, seg_row, seg_pos, seg_slot) -> None:
        a = self.a
        a.proj, a.ldp, a.gates, a.ldg = proj.data_ptr(), proj.stride(0), gates.data_ptr(), gates.stride(0)
        a.og, a.ldo = _ptr(og), og.stride(0) if og is not None else 0
        a.dec, a.ldd = _ptr(dec), dec.stride(0) if dec is not None else 0
        a.act, a.lda = act.data_ptr(), act.stride(0)
        a.seg_row, a.seg_pos, a.seg_slot = _ptr(seg_row), _ptr(seg_pos), _ptr(seg_slot)

    def step(self, proj, gates, og, act, seg_pos, seg_slot, *, segs: int, seg_row=None, dec=None) -> None:
        """Token by token over ``segs`` segments (``seg_row`` None: one row each)."""
        self._fill(proj, gates, og, act, dec, seg_row, seg_pos, seg_slot)
        if self.kind == SSD:
            call("ssd_step", ctypes.byref(self.a), segs, _is_f32(proj), _is_f32(self.state["ring"]))
        else:
            call("linrec_step", ctypes.byref(self.a), self.kind, segs, _is_f32(proj), _is_f32(act))
        K._count()

    @property
    def chunked(self) -> bool:
        """Whether prompts of this head size run in chunks on the tensor cores (bf16 activations)."""
        if self.kind == SSD:
            return bool(_lib.call_nostream("ssd_chunk_ok", self.a.dk, self.a.dv))
        return bool(_lib.call_nostream("linrec_chunk_ok", self.a.dk, self.a.dv))

    def chunk_scratch(self, rows: int, segs: int) -> int:
        if self.kind == SSD:
            fn = _lib.lib().cb_ssd_chunk_scratch
            fn.restype = ctypes.c_int64
            return int(fn(*[ctypes.c_int64(v) for v in (rows, self.a.H, self.a.ring_w)]))
        fn = _lib.lib().cb_linrec_chunk_scratch
        fn.restype = ctypes.c_int64
        a = self.a
        return int(fn(*[ctypes.c_int64(v) for v in (self.kind, rows, segs, a.H, a.dk, a.dv)]))

    def chunk(self, proj, gates, og, act, seg_row, seg_pos, seg_slot, scratch, *, segs: int, max_rows: int, rows: int, dec=None) -> None:
        """The first ``segs`` segments (rows ``[0, rows)``, at most ``max_rows`` each) in chunks; ``scratch`` bytes as
        ``chunk_scratch`` says.  The convolution ring is left as it was (``ring`` afterwards)."""
        self._fill(proj, gates, og, act, dec, seg_row, seg_pos, seg_slot)
        if self.kind == SSD:
            call("ssd_chunk", ctypes.byref(self.a), segs, max_rows, rows, scratch, scratch.numel() * scratch.element_size())
            K._count(2)
            return
        call("linrec_chunk", ctypes.byref(self.a), self.kind, segs, max_rows, rows, scratch, scratch.numel() * scratch.element_size())
        K._count(4 if self.kind == MLSTM else 3)

    def ring(self, proj, seg_row, seg_pos, seg_slot, segs: int) -> None:
        """After the readers: the raw rows at the end of every segment of two or more tokens enter the ring."""
        r = self.state.get("ring")
        if r is None or segs < 1:
            return
        if proj.dtype != r.dtype:
            proj = proj.to(r.dtype)
        call("linrec_ring", proj, proj.stride(0), seg_row, seg_pos, seg_slot, segs, r, r.shape[1], r.shape[2], self.a.taps, _is_f32(r))
        K._count()


def gated_norm(y: torch.Tensor, z: torch.Tensor, weight: torch.Tensor, act: torch.Tensor, *, groups: int, n: int, eps: float) -> torch.Tensor:
    """``act = rmsnorm(y * silu(z)) * weight``, each row in ``groups`` parts of ``n`` columns with a root mean square of their own."""
    call("gated_norm", y, y.stride(0), z, z.stride(0), weight, act, act.stride(0), y.shape[0], groups, n, float(eps), _is_f32(z), _is_f32(act))
    K._count()
    return act


# ------------------------------------------------------------------ attention with several maps per head
class _AttnStruct(ctypes.Structure):
    _fields_ = [("proj", _P), ("ldp", _I64), ("k_col", _I64), ("v_col", _I64), ("kpool", _P), ("vpool", _P), ("tables", _P),
                ("ldbt", _I64), ("row_seg", _P), ("positions", _P), ("seg_row", _P), ("seg_pos", _P), ("part_o", _P), ("part_ml", _P),
                ("H", _I32), ("G", _I32), ("maps", _I32), ("dim", _I32), ("vdim", _I32), ("nsplit", _I32), ("scale", _F), ("cap", _F),
                ("temp_coef", _F), ("temp_every", _I32), ("ldk", _I64), ("ldv", _I64), ("act", _P), ("lda", _I64), ("gates", _P), ("ldg", _I64),
                ("window", _I32), ("rot_half", _I32), ("sink", _P), ("cs", _P), ("v0", _P), ("ldv0", _I64), ("v_own", _F), ("v_mix", _F),
                ("egate", _P), ("lde", _I64), ("chunk", _I32), ("norm", _I32), ("eps", _F), ("qn", _P), ("kn", _P), ("vcs", _P), ("kr", _P), ("r1", _P),
                ("r2", _P), ("oscale", _F), ("bound", _F)]


#: largest bound of scores that serves as the reference of a softmax: weights down to exp(-2 bound) stay normal numbers
MAX_BOUND = 34.0


MAX_VDIM = 512


def window_pages(window: int) -> int:
    """Most pages that hold keys of one query."""
    return (window + K.BLOCK - 2) // K.BLOCK + 1 if window > 0 else 1 << 30


class AttnMaps:
    """Attention layer constants plus its pages ``kpool [slots, G * maps, dim]``, ``vpool [slots, G, vdim]``."""

    def __init__(self, *, H: int, G: int, maps: int, dim: int, vdim: int, k_col: int, v_col: int, scale: float, cap: float | None,
                 temp: tuple[float, int] | None, kpool: torch.Tensor, vpool: torch.Tensor, finish: bool = True, window: int = 0,
                 rot_dims: int = 0, sink: torch.Tensor | None = None, chunk: int = 0, norm: tuple | None = None,
                 factors: torch.Tensor | None = None, distance: tuple | None = None, out_scale: float = 1.0) -> None:
        """``finish``: the heads will be finished by ``finish``, which bounds the value size.  ``window``: tokens a query sees,
        itself included (0: all).  ``rot_dims``: leading columns of queries and keys that turn, in neighbouring pairs, by the
        angles of ``rows_of``.  ``sink`` (fp32 ``[H * maps]``): a score without key or value in every softmax.  ``chunk``: a query
        sees the tokens of its own chunk of this size.  ``norm = (eps, q weight, k weight)``: queries and keys are RMS-normed per
        head before they turn (weights fp32 ``[dim]`` or None).  ``factors`` (fp32, a page's ``[G, 64]`` together): keys are cached as
        projected and are the values, ``vpool`` is not used, and a key's factor takes its norm's place.  ``distance = (r1, r2)``
        (fp32 ``[H]``): scores lose ``r1 ln(1 + r2 distance)``.  ``out_scale``: factor of the finished heads."""
        if (finish and vdim > MAX_VDIM) or maps not in (1, 2):
            raise ValueError(f"attention with {maps} maps and values of {vdim} is outside the kernels' range")
        a = self.a = _AttnStruct()
        size = _lib.call_nostream("attn_maps_args_size")
        assert ctypes.sizeof(a) == size, f"argument layout: {ctypes.sizeof(a)} here, {size} in the library"
        self.H, self.G, self.maps, self.dim, self.vdim = H, G, maps, dim, vdim
        a.H, a.G, a.maps, a.dim, a.vdim, a.k_col, a.v_col = H, G, maps, dim, vdim, k_col, v_col
        a.scale, a.cap = float(scale), float(cap or 0.0)
        self.set_pools(kpool, vpool)
        self._tcgen05 = scale > 0 and bool(_lib.call_nostream("attn_maps_flash_tc_ok", dim, vdim))
        a.window, a.rot_half, a.sink = int(window), rot_dims // 2, _ptr(sink)
        self.window, self.sink, self._egate = int(window), sink, None
        if temp is not None:
            a.temp_coef, a.temp_every = float(temp[0]), int(temp[1])
        qn, kn = (norm[1], norm[2]) if norm is not None else (None, None)
        r1, r2 = distance if distance is not None else (None, None)
        a.chunk, a.norm, a.eps, a.qn, a.kn = int(chunk), int(norm is not None), float(norm[0]) if norm is not None else 0.0, _ptr(qn), _ptr(kn)
        a.kr, a.r1, a.r2, a.oscale = _ptr(factors), _ptr(r1), _ptr(r2), float(out_scale)
        a.bound = self.bound = self._bound(scale, dim, norm, distance) if cap is None else 0.0
        self.chunk, self._vcs, self.out_scale, self._keep = int(chunk), None, float(out_scale), (qn, kn, r1, r2, factors)
        self.keys_only = factors is not None
        if self.keys_only and (maps != 1 or dim != vdim):
            raise ValueError("keys that are their own values: one map, one size")

    @staticmethod
    def _bound(scale: float, dim: int, norm: tuple | None, distance: tuple | None) -> float:
        """What no score exceeds (a normed head's length is at most the root of its size, times its largest weight), or 0 if nothing
        useful is known.  A margin covers the rounding of queries and keys; penalties have to take off, never add."""
        if norm is None or (distance is not None and not bool(((distance[0] >= 0) & (distance[1] >= 0)).all())):
            return 0.0
        most = lambda w: float(w.abs().max()) if w is not None else 1.0
        b = 1.02 * abs(scale) * dim * most(norm[1]) * most(norm[2])
        return b if 0.0 < b <= MAX_BOUND else 0.0

    def set_pools(self, kpool: torch.Tensor, vpool: torch.Tensor) -> None:
        """Rows of keys and values; they may be column ranges of wider rows."""
        a = self.a
        self.kpool, self.vpool = kpool, vpool
        a.kpool, a.vpool, a.ldk, a.ldv = _ptr(kpool), _ptr(vpool), kpool.stride(0), vpool.stride(0)

    def _fill(self, proj, tables, positions, row_seg, part_o=None, part_ml=None, nsplit: int = 1, seg_row=None, seg_pos=None) -> None:
        a = self.a
        a.proj, a.ldp, a.tables, a.ldbt = proj.data_ptr(), proj.stride(0), tables.data_ptr(), tables.stride(0)
        a.positions, a.row_seg, a.part_o, a.part_ml, a.nsplit = positions.data_ptr(), _ptr(row_seg), _ptr(part_o), _ptr(part_ml), nsplit
        a.seg_row, a.seg_pos = _ptr(seg_row), _ptr(seg_pos)

    def rows_of(self, cs: torch.Tensor | None = None, egate: torch.Tensor | None = None, values: torch.Tensor | None = None,
                lam: float = 0.0, turns: torch.Tensor | None = None) -> None:
        """What the rows of the next calls carry beside their projection: angles ``cs [rows, rot_dims]``, output gate
        pre-activations ``egate [rows, H * vdim]`` (one map), and ``values [rows, G * vdim]`` of another layer, of which
        ``lam`` is mixed into their own (both typed like the projection).  ``turns [rows, vdim]``: angles by which values are turned
        when they are cached and heads are turned back."""
        a = self.a
        a.vcs, self._vcs = _ptr(turns), turns
        a.cs, a.egate, a.lde = _ptr(cs), _ptr(egate), egate.stride(0) if egate is not None else 0
        a.v0, a.ldv0, a.v_own, a.v_mix = _ptr(values), values.stride(0) if values is not None else 0, 1.0 - lam, lam
        self._egate = egate

    def append(self, proj, tables, positions, row_seg=None, turn_queries: bool = False) -> None:
        """Keys (turned) and values (mixed) into the pages; ``turn_queries``: the rows' queries are turned in place."""
        self._fill(proj, tables, positions, row_seg)
        call("attn_maps_append", ctypes.byref(self.a), positions.numel(), int(turn_queries), _is_f32(proj), _is_f32(self.kpool))
        K._count()

    def rows(self, proj, tables, positions, row_seg, part_o, part_ml, nsplit: int = 1) -> None:
        """The plain kernel: one query row at a time (keys of the rows themselves appended before)."""
        self._fill(proj, tables, positions, row_seg, part_o, part_ml, nsplit)
        call("attn_maps_rows", ctypes.byref(self.a), positions.numel(), _is_f32(proj), _is_f32(self.kpool))
        K._count()

    @property
    def tc(self) -> bool:
        """Whether the tensor-core prompt kernel and the split decode kernel take this head."""
        return self.kpool.dtype == torch.bfloat16 and bool(_lib.call_nostream("attn_maps_tc_ok", self.G, self.maps, self.dim, self.vdim))

    def flash(self, proj, tables, seg_row, seg_pos, part_o, part_ml, *, segs: int, max_rows: int, positions, act=None, gates=None) -> None:
        """Portions of several tokens (bf16 projection rows; keys and values appended before): tcgen05 for head sizes of
        64 / 128 / 192 / 256 (values 64 / 128 / 256) and portions worth a 128-row tile, ``mma.sync`` otherwise.  With one map
        ``act`` takes the finished heads, times ``sigmoid(gates)`` if given, and there are no parts."""
        self._fill(proj, tables, positions, None, part_o, part_ml, 1, seg_row, seg_pos)
        a = self.a
        a.act, a.lda = _ptr(act), act.stride(0) if act is not None else 0
        a.gates, a.ldg = _ptr(gates), gates.stride(0) if gates is not None else 0
        if K.ATTN_TC and max_rows >= K.ATTN_TC_MIN_T and self._tcgen05:
            call("attn_maps_flash_tc", ctypes.byref(self.a), segs, max_rows, self.kpool.shape[0], K.status_word(proj.device))
        else:
            call("attn_maps_flash", ctypes.byref(self.a), segs, max_rows)
        K._count()

    def decode_splits(self, rows: int) -> int:
        R = self.H // self.G
        hpc = min(R, 8 // self.maps)
        resident = 296 if self.maps == 1 and max(self.dim, self.vdim) <= 128 else 148        # CTAs on the machine at once
        return max(1, min(64, window_pages(self.window), window_pages(self.chunk), resident // max(1, self.G * -(-R // hpc) * rows)))

    def decode(self, proj, tables, positions, row_seg, part_o, part_ml, nsplit: int, act=None) -> None:
        """Single tokens (their keys and values are appended by the kernel): ``nsplit`` key splits per row.  With one map and one
        split ``act`` takes the finished heads and there are no parts."""
        self._fill(proj, tables, positions, row_seg, part_o, part_ml, nsplit)
        self.a.act, self.a.lda, self.a.gates = _ptr(act), act.stride(0) if act is not None else 0, None
        call("attn_maps_decode", ctypes.byref(self.a), positions.numel(), _is_f32(proj))
        K._count()

    def finish(self, part_o, part_ml, gates, act, positions, *, nsplit: int = 1, lam: float = 0.0, post_scale: float = 1.0,
               eps: float = 1e-5) -> None:
        """Merge splits and sinks, ``o = a_0 - lam a_1`` + RMS norm (two maps), ``* post_scale * sigmoid(gate)`` per head, then per
        element (``rows_of``)."""
        eg = self._egate
        call("attn_maps_finish", part_o, part_ml, gates, gates.stride(0) if gates is not None else 0, act, act.stride(0), positions,
             positions.numel(), self.H, self.maps, self.vdim, nsplit, float(lam), post_scale * self.out_scale, float(eps), self.sink,
             eg, eg.stride(0) if eg is not None else 0, _is_f32(eg) if eg is not None else 0, self._vcs, _is_f32(act))
        K._count()


# ------------------------------------------------------------------ rotary angles
def rope_turns(base: float, dims: int, device) -> torch.Tensor:
    """fp64 ``[dims / 2]``: turns per position of pair ``i``, ``base^(-2 i / dims) / (2 pi)``."""
    i = torch.arange(dims // 2, dtype=torch.float64)
    return (torch.tensor(float(base), dtype=torch.float64) ** (-2.0 * i / dims) / (2.0 * torch.pi)).to(device)


def rope_rows(positions: torch.Tensor, turns: torch.Tensor, cs: torch.Tensor) -> torch.Tensor:
    """``cs [rows, pairs * 2]`` (fp32) = (cos, sin) of every pair at the rows' positions."""
    call("rope_rows", positions, turns, cs, positions.numel(), turns.numel())
    K._count()
    return cs


def rope_heads(src: torch.Tensor, hs: int, dst: torch.Tensor, hd: int, cs: torch.Tensor, *, half: int, rot: int, H: int) -> None:
    """Rotate ``rot`` columns of ``H`` heads, pairs ``(2i, 2i + 1)`` for the first ``half`` pairs; ``src`` / ``dst`` start at the
    first head's rotated column, heads are ``hs`` / ``hd`` columns apart; may be in place."""
    assert src.dtype == dst.dtype
    call("rope_heads", src, src.stride(0), hs, dst, dst.stride(0), hd, cs, half, rot, H, src.shape[0], _is_f32(dst))
    K._count()


# ------------------------------------------------------------------ latent attention
class _LatentStruct(ctypes.Structure):
    _fields_ = [("proj", _P), ("ldp", _I64), ("c_col", _I64), ("r_col", _I64), ("norm_q", _P), ("norm_c", _P), ("cq", _P), ("ldq", _I64),
                ("pool", _P), ("ldk", _I64), ("tables", _P), ("ldbt", _I64), ("row_seg", _P), ("positions", _P), ("cs", _P), ("half", _I32),
                ("q_rank", _I32), ("kv_rank", _I32), ("rot", _I32), ("cp", _I32), ("eps", _F), ("H", _I32), ("split", _I32), ("hq", _I64),
                ("r_off", _I64), ("qa", _P), ("ldqa", _I64)]


def head_linear(w: torch.Tensor, x: torch.Tensor, hx: int, y: torch.Tensor, hy: int, gate: torch.Tensor | None = None) -> torch.Tensor:
    """``y[t, h hy : h hy + N] = w[h] @ x[t, h hx : h hx + K]`` for ``w [H, N, K]``, times ``sigmoid(gate[t, h])`` if given."""
    H, N, Kd = w.shape
    call("head_linear", w, x, x.stride(0), hx, y, y.stride(0), hy, gate, gate.stride(0) if gate is not None else 0, x.shape[0], H, N, Kd,
         _is_f32(w))
    K._count()
    return y


class LatentAttn:
    """Latent attention of one layer: pages ``pool [slots, ldk]`` hold ``[c | rotated key part]`` (the part at column ``cp``),
    its own or those of the layer it borrows them from.  ``q_rank`` 0: the projection rows hold the queries themselves, heads of
    ``hq`` columns whose rotated part starts at ``r_off``.  ``window``: tokens a query sees, itself included (0: all)."""

    def __init__(self, *, H: int, q_rank: int, kv_rank: int, rot: int, rot_dims: int, cp: int, scale: float, eps: float, pool: torch.Tensor,
                 norm_q: torch.Tensor | None, norm_c: torch.Tensor | None, c_col: int = 0, r_col: int = 0, hq: int = 0, r_off: int = 0,
                 window: int = 0) -> None:
        a = self.a = _LatentStruct()
        size = _lib.call_nostream("latent_args_size")
        assert ctypes.sizeof(a) == size, f"argument layout: {ctypes.sizeof(a)} here, {size} in the library"
        self.H, self.cp, self.scale, self.pool, self.own, self.ldk = H, cp, float(scale), pool, norm_c is not None, pool.shape[1]
        self._keep = (norm_q, norm_c)
        a.q_rank, a.kv_rank, a.rot, a.cp, a.eps, a.half, a.c_col, a.r_col = q_rank, kv_rank, rot, cp, float(eps), rot_dims // 2, c_col, r_col
        a.norm_q, a.norm_c, a.pool, a.ldk = _ptr(norm_q), _ptr(norm_c), _ptr(pool), pool.stride(0)
        a.H, a.hq, a.r_off, self.window = H, hq, r_off, int(window)
        # the plain kernel and the merge of key splits see one key / value head whose values are the head of the key row
        self._plain = AttnMaps(H=H, G=1, maps=1, dim=self.ldk, vdim=cp, k_col=0, v_col=0, scale=scale, cap=None, temp=None, kpool=pool,
                               vpool=pool, finish=False, window=window)
        self.tc = pool.dtype == torch.bfloat16 and bool(_lib.call_nostream("latent_decode_ok", self.ldk, cp))

    def rows(self, proj, cq, tables, positions, row_seg, cs, *, split: int = 0, qa: torch.Tensor | None = None) -> None:
        """Norm the query latents into ``cq``; without them turn the rotated query parts, in place for the rows before ``split`` and
        into the absorbed queries ``qa`` of the others.  An owner also norms, rotates and appends what it caches."""
        a = self.a
        a.proj, a.ldp, a.cq, a.ldq = proj.data_ptr(), proj.stride(0), _ptr(cq), cq.stride(0) if cq is not None else 0
        a.split, a.qa, a.ldqa = split, _ptr(qa), qa.stride(0) if qa is not None else 0
        a.tables, a.ldbt, a.row_seg, a.positions, a.cs = tables.data_ptr(), tables.stride(0), _ptr(row_seg), positions.data_ptr(), _ptr(cs)
        call("latent_rows", ctypes.byref(a), positions.numel(), int(self.own), _is_f32(proj), _is_f32(self.pool))
        K._count()

    def gather(self, tables, base, lens, first, out, *, segs: int, max_pages: int) -> None:
        """Page rows of ``segs`` sequences side by side in ``out`` (segment ``s`` from row ``base[s]``, its pages from ``first[s]`` on)."""
        call("latent_gather", self.pool, self.pool.stride(0) * self.pool.element_size(), tables, tables.stride(0), base, lens, first, out, segs,
             max_pages)
        K._count()

    def _tiles(self, rows: int) -> int:
        """Groups of 16 heads per CTA of the decode kernel: two share the staged pages unless few rows leave SMs idle."""
        return 1 if self.H <= 16 or rows <= 2 else 2

    def decode_splits(self, rows: int) -> int:
        groups = -(-self.H // (16 * self._tiles(rows)))
        return max(1, min(64, window_pages(self.window), 148 // max(1, groups * rows)))

    def absorbed(self, q, tables, positions, row_seg, part_o, part_ml, nsplit: int) -> None:
        """Queries ``q [rows, H * ldk]`` against the pages: key splits for ``merge`` (one split without the tensor-core kernel)."""
        if self.tc:
            call("latent_decode", q, q.stride(0), self.pool, self.pool.stride(0), tables, tables.stride(0), row_seg, positions, part_o, part_ml,
                 positions.numel(), self.H, self.cp, nsplit, self._tiles(positions.numel()), self.window, self.scale)
            K._count()
        else:
            self._plain.rows(q, tables, positions, row_seg, part_o, part_ml, nsplit)

    def merge(self, part_o, part_ml, out, positions, nsplit: int) -> None:
        """Weighted averages of the latents, ``out [rows, H * cp]``."""
        call("latent_merge", part_o, part_ml, positions, out, out.stride(0), positions.numel(), self.H, self.cp, nsplit, _is_f32(out))
        K._count()
