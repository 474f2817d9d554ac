"""What the row-batch families share: batches of portions and single tokens, projections, workspaces, sequence state and
the captured decode step.

A family derives from ``RowModel``, builds its mixers (``Mixer`` objects: weights, state tensors, page pools) and
supplies two methods: ``_stack`` runs all layers over the rows of a ``RowBatch`` and ``_out_rows`` turns picked rows of
the result into the normalised input of the vocabulary head.  Everything a sequence leaves behind lives in the mixers:
``state`` tensors are indexed by the slot that the engine assigns, ``pools`` by the pages of its block table; the
engine owns both and uses the zero / snapshot / restore / copy hooks here.
"""
from __future__ import annotations

import dataclasses

import torch

from ..ops import kernels as K
from ..ops import mixers as X

BUCKETS = (1, 2, 4, 8, 16, 32, 64)


@dataclasses.dataclass
class RowBatch:
    """Rows of one forward.  Segments ``0 .. n_pre - 1`` are portions of several tokens, the others one token each; the
    rows of a segment are consecutive and segments are in row order."""
    T: int
    n_seg: int
    n_pre: int                      # leading segments with more than one row
    pre_rows: int                   # rows of those segments
    tokens: torch.Tensor            # int64 [T]
    positions: torch.Tensor         # int32 [T], -1: padding
    row_seg: torch.Tensor | None    # int32 [T]; None: row r is segment r
    seg_row: torch.Tensor | None    # int32 [n_seg + 1]
    seg_pos: torch.Tensor           # int32 [n_seg]
    seg_slot: torch.Tensor          # int32 [n_seg]
    tables: torch.Tensor            # int32 [n_seg, pages]
    max_rows: int = 1               # longest segment
    max_len: int = 0                # largest position + 1 (0: unknown, inside a graph)
    pre_lens: tuple = ()            # tokens of every leading segment's sequence so far, its own rows included
    pre_pos: tuple = ()             # position of every leading segment's first row
    cache: dict = dataclasses.field(default_factory=dict)     # what mixers of one forward share

    def expansion(self, window: int = 0) -> dict:
        """Whole-page rows of the leading segments side by side, from the first page that a query of the segment sees through
        ``window`` (0: all).  Per segment on the device: ``base`` (first row), ``lens``, ``skip`` (pages left out), ``pos`` (the
        segment's first position counted from the first row), ``tables`` of consecutive blocks; ``rows``: all rows, ``pages``: the
        most of a segment."""
        e = self.cache.get(("expansion", window))
        if e is None:
            skip = [max(0, p - window + 1) // K.BLOCK if window else 0 for p in self.pre_pos]
            lens = [n - s * K.BLOCK for n, s in zip(self.pre_lens, skip)]
            pages = [(n + K.BLOCK - 1) // K.BLOCK for n in lens]
            first = [sum(pages[:i]) for i in range(len(pages))]
            n, most = len(pages), max(pages)
            host = torch.zeros(4 * n + n * most, dtype=torch.int32)
            for i, (p, f) in enumerate(zip(pages, first)):
                host[i], host[n + i], host[2 * n + i], host[3 * n + i] = f * K.BLOCK, lens[i], skip[i], self.pre_pos[i] - skip[i] * K.BLOCK
                host[4 * n + i * most:4 * n + i * most + p] = torch.arange(f, f + p, dtype=torch.int32)
            if self.positions.is_cuda:
                host = host.pin_memory()
            dev = host.to(self.positions.device, non_blocking=True)
            e = self.cache[("expansion", window)] = {"base": dev[:n], "lens": dev[n:2 * n], "skip": dev[2 * n:3 * n], "pos": dev[3 * n:4 * n],
                                                     "tables": dev[4 * n:].view(n, most), "rows": sum(pages) * K.BLOCK, "pages": most}
        return e


def pad8(n: int) -> int:
    return (n + 7) // 8 * 8


class Projection:
    """Row-concatenated projections of one input.  Sections start at multiples of 8 columns (16-byte tiles); ``main``
    holds the activations, ``gate`` the columns whose result stays fp32 (gates of a recurrence, head gates)."""

    def __init__(self, parts: dict[str, torch.Tensor], gates: dict[str, torch.Tensor], width: int, dtype, device) -> None:
        self.col: dict[str, int] = {}
        rows = []

        def add(t: torch.Tensor) -> None:
            w = torch.zeros(pad8(t.shape[0]), pad8(width), dtype=dtype, device=device)
            w[:t.shape[0], :t.shape[1]] = t.to(device, dtype)
            rows.append(w)

        n = 0
        for name, t in parts.items():
            self.col[name] = n
            add(t)
            n += pad8(t.shape[0])
        self.n_main = n
        if gates:
            add(torch.cat([t.to(device, dtype) for t in gates.values()]))
        self.w = torch.cat(rows).contiguous()
        self.n = self.w.shape[0]
        self.main, self.gate = self.w[:self.n_main], self.w[self.n_main:]


class Mixer:
    #: named state tensors ``[slots, ...]`` that travel with a sequence; paged pools are separate
    state: dict[str, torch.Tensor]
    pools: tuple[torch.Tensor, ...] = ()

    def weights(self):
        return [self.proj.w, self.w_out]


def padded(t: torch.Tensor, rows: int, cols: int, dtype, dev) -> torch.Tensor:
    out = torch.zeros(rows, cols, dtype=dtype, device=dev)
    out[:t.shape[0], :t.shape[1]] = t.to(dev, dtype)
    return out


class RowModel:
    mixed_batches = True            # portions of prompts and single tokens share a forward
    family = ""

    def _setup(self, cfg, sd: dict[str, torch.Tensor], device, max_seq: int, num_slots: int, num_blocks: int | None, max_chunk: int,
               pdl: bool, dtype: torch.dtype, quant: str, kv_dtype: str, free_shape: tuple[str, ...] = ()) -> None:
        """Sizes, placement and the check of the checkpoint against the configuration's tensor plan (``free_shape``:
        last name parts of tensors whose size the configuration does not give)."""
        if quant != "none" or kv_dtype != "bf16":
            raise NotImplementedError(f"the {self.family} family has 16-bit (or fp32) weights and pages only")
        if dtype not in (torch.bfloat16, torch.float32):
            raise ValueError(f"dtype {dtype}: expected bfloat16 or float32")
        self.cfg = cfg
        self.dtype, self.f32 = dtype, dtype == torch.float32
        self.device = dev = torch.device(device)
        self.max_seq = int(max_seq)
        self.num_slots, self.max_chunk = int(num_slots), int(max_chunk)
        self.max_blocks_per_seq = (self.max_seq + K.BLOCK - 1) // K.BLOCK
        self.num_blocks = int(num_blocks) if num_blocks else self.max_blocks_per_seq * self.num_slots + 1
        self.eps = cfg.rms_norm_eps
        self.tp_world = 1
        K.status_word(dev)
        K._lib.set_pdl(pdl)
        for name, shape, _ in cfg.tensor_plan():
            if name not in sd:
                raise KeyError(f"checkpoint lacks {name}")
            if tuple(sd[name].shape) != shape and name.rpartition(".")[2] not in free_shape:
                raise ValueError(f"{name}: shape {tuple(sd[name].shape)}, config.json gives {shape}")
        self.layers: list = []
        self._bufs: dict = {}
        self._rows: dict[int, dict] = {}
        self._graphs: dict = {}
        self._step_launches: dict[int, int] = {}
        self.graph_pool = None
        self._advance = False
        self.layer_hook = None          # debugging: called as hook(layer index, residual [rows, W]) after every layer

    # ------------------------------------------------------------------ supplied by the family
    def _stack(self, b: RowBatch):
        """All layers over the rows of ``b``; whatever ``_out_rows`` needs."""
        raise NotImplementedError

    def _out_rows(self, state, rows: torch.Tensor | None, n: int, h: torch.Tensor) -> None:
        """The head's input of ``n`` rows (``rows`` None: the first n) into ``h [n, padded width]``."""
        raise NotImplementedError

    # ------------------------------------------------------------------ bookkeeping
    def weight_bytes(self) -> int:
        """Bytes of weights one decode step streams."""
        ts = [self.head]
        for L in self.layers:
            ts += L.mixer.weights() + L.ff_weights()
        return sum(t.numel() * t.element_size() for t in ts)

    def launches_per_step(self, M: int) -> int:
        return self._step_launches.get(M, 0)

    @staticmethod
    def bucket_for(n: int) -> int:
        for m in BUCKETS:
            if n <= m:
                return m
        raise ValueError(f"{n} rows exceed the largest decode bucket {BUCKETS[-1]}")

    @property
    def max_decode_rows(self) -> int:
        return BUCKETS[-1]

    def poll_status(self) -> None:
        K.poll_status()

    def check_status(self) -> None:
        K.raise_on_status()

    def sample(self, logits: torch.Tensor, temps, us) -> torch.Tensor:
        if temps is None:
            return K.argmax(logits.contiguous())
        t = torch.tensor(temps, dtype=torch.float32, device=self.device)
        u = torch.tensor(us, dtype=torch.float32, device=self.device)
        return K.sample(logits.contiguous(), t, u)

    def embed_tokens(self, tokens: torch.Tensor) -> torch.Tensor:
        return self.embed.index_select(0, tokens)

    # ------------------------------------------------------------------ sequence state
    @property
    def stateless(self) -> bool:
        """Whether a sequence leaves nothing behind but pages: any cached page prefix can be reused without a snapshot."""
        return not any(L.mixer.state for L in self.layers)

    def zero_state(self, slot: int) -> None:
        for L in self.layers:
            for t in L.mixer.state.values():
                t[slot].zero_()

    def snapshot_state(self, slot: int) -> list[torch.Tensor]:
        return [t[slot].clone() for L in self.layers for t in L.mixer.state.values()]

    def restore_state(self, slot: int, snap: list[torch.Tensor]) -> None:
        it = iter(snap)
        for L in self.layers:
            for t in L.mixer.state.values():
                t[slot].copy_(next(it))

    def copy_block(self, src: int, dst: int) -> None:
        s, d = src * K.BLOCK, dst * K.BLOCK
        for L in self.layers:
            for pool in L.mixer.pools:
                pool[d:d + K.BLOCK].copy_(pool[s:s + K.BLOCK])

    # ------------------------------------------------------------------ workspaces and products
    def buf(self, name: str, rows: int, cols: int, dtype: torch.dtype | None = None) -> torch.Tensor:
        """Scratch ``[rows, cols]``, contiguous.  Buffers of a name and width are zero when first handed out and padding
        columns are never written, so a product over the padded width adds nothing.  Sizes of the decode buckets
        have buffers of their own (fixed addresses inside CUDA graphs); larger batches share one that grows."""
        dtype = dtype or self.dtype
        small = rows if rows in BUCKETS else 0
        key = (name, cols, dtype, small)
        t = self._bufs.get(key)
        if t is None or t.shape[0] < rows:
            cap = small or max(rows, min(self.max_chunk, 256))
            t = self._bufs[key] = torch.zeros(cap, cols, dtype=dtype, device=self.device)
        return t[:rows]

    def _scratch(self, floats: int) -> torch.Tensor:
        """Untyped scratch of the chunked recurrences (grows; stream-ordered reuse)."""
        t = self._bufs.get("scratch")
        if t is None or t.numel() < floats:
            t = self._bufs["scratch"] = torch.empty(floats, dtype=torch.float32, device=self.device)
        return t

    def linear(self, W: torch.Tensor, x: torch.Tensor, out: torch.Tensor) -> torch.Tensor:
        """``out = x @ W^T``; the result type is ``out``'s."""
        T, Kd = x.shape
        if self.f32:
            return X.gemm_f32(x, W, out)
        if T <= 8 and T * Kd * 2 <= 160 * 1024:
            return K.gemv(W, x.contiguous(), out)
        if out.dtype == torch.float32:
            return X.gemm_f32out(x, W, out)
        return K.gemm(x, W, out=out)

    def project(self, P, h: torch.Tensor, b: RowBatch, name: str = "proj") -> tuple[torch.Tensor, torch.Tensor]:
        """``(main, gates)`` of an input projection, one product: fp32 for few rows (and in 32-bit mode), else the main columns
        in the activation type and the gate columns fp32.  ``name``: workspace of the rows, for rows that outlive the layer."""
        T = b.T
        if self.f32 or T <= 8:
            y = self.buf(name + "32", T, P.n, torch.float32)
            self.linear(P.w, h, y)
            return y[:, :P.n_main], y[:, P.n_main:]
        main = self.buf(name, T, P.n_main)
        if P.n == P.n_main:
            return self.linear(P.w, h, main), main[:, P.n_main:]
        gates = self.buf("gates", T, P.gate.shape[0], torch.float32)
        X.gemm_mixed(h, P.w, main, gates)
        return main, gates

    def feed_forward(self, L, h: torch.Tensor, T: int) -> torch.Tensor:
        """``w_down (silu(gate) * up)`` of a layer with ``w_gu`` (gate rows, then up rows) and ``w_down``."""
        I = L.w_down.shape[1]
        inter = self.buf("inter", T, I)
        y = self.buf("y", T, L.w_down.shape[0])
        if self.f32:
            X.swiglu_f32(X.gemm_f32(h, L.w_gu, self.buf("gu", T, 2 * I)), inter)
        elif T <= 8 and T * h.shape[1] * 2 <= 160 * 1024:
            K.gemv(L.w_gu, h, inter, swiglu=True)
        elif K.PAIR_GEMM and T >= K.PAIR_MIN_ROWS and I >= 128:
            K.gemm_swiglu(h, L.w_gu, out=inter)
        else:
            K.swiglu(K.gemm(h, L.w_gu, out=self.buf("gu", T, 2 * I)), out=inter)
        return self.linear(L.w_down, inter, y)

    def angles(self, b: RowBatch, base: float, dims: int, turns: torch.Tensor) -> torch.Tensor:
        """(cos, sin) of the batch's rows, shared by the layers of one rotation."""
        key = ("rope", base, dims)
        cs = b.cache.get(key)
        if cs is None:
            cs = self.buf(f"rope{base}/{dims}", b.T, max(2, dims), torch.float32)
            if dims:
                X.rope_rows(b.positions, turns, cs)
            b.cache[key] = cs
        return cs

    # ------------------------------------------------------------------ mixer cores
    def recur(self, core: X.Linrec, b: RowBatch, proj, gates, og, act, dec) -> None:
        n0 = 0
        if b.n_pre and proj.dtype == torch.bfloat16 and core.chunked:
            need = (core.chunk_scratch(b.pre_rows, b.n_pre) + 3) // 4
            core.chunk(proj, gates, og, act, b.seg_row, b.seg_pos, b.seg_slot, self._scratch(need), segs=b.n_pre, max_rows=b.max_rows,
                       rows=b.pre_rows, dec=dec)
            n0 = b.n_pre
        if n0 < b.n_seg:
            core.step(proj, gates, og, act, b.seg_pos[n0:], b.seg_slot[n0:], segs=b.n_seg - n0,
                      seg_row=b.seg_row[n0:] if b.seg_row is not None else None, dec=dec)
        if b.n_pre:
            core.ring(proj, b.seg_row, b.seg_pos, b.seg_slot, b.n_pre)

    def _logits(self, state, rows: torch.Tensor | None, n: int, out: torch.Tensor) -> torch.Tensor:
        """fp32 logits of ``n`` rows (``rows`` None: the first n) into ``out [n, padded vocab]``."""
        h = self.buf("h_out", n, pad8(self.cfg.hidden_size))
        self._out_rows(state, rows, n, h)
        return self.linear(self.head, h, out)

    # ------------------------------------------------------------------ batches of portions and tokens
    def _check_row(self, pos0: int, n: int, table_len: int, slot: int) -> None:
        """Everything a kernel indexes with a position or a slot is checked here, on the host."""
        end = pos0 + n
        if n < 1 or pos0 < 0 or end > self.max_seq or end > table_len * K.BLOCK or table_len > self.max_blocks_per_seq:
            raise ValueError(f"positions {pos0}..{end - 1} outside the block table ({table_len} blocks) or the {self.max_seq}-token window")
        if not 0 <= slot < self.num_slots:
            raise ValueError(f"state slot {slot} outside 0..{self.num_slots - 1}")

    def make_batch(self, items: list[tuple]) -> tuple[RowBatch, list[int], list[int]]:
        """``items[i] = (tokens, pos0, slot, block_table)``.  Returns the batch, the segment order (item index per
        segment: portions before single tokens) and the first row of every ITEM."""
        toks = [t.tolist() if isinstance(t, torch.Tensor) else list(t) for t, *_ in items]
        tabs = [t.tolist() if isinstance(t, torch.Tensor) else list(t) for *_, t in items]
        for tk, (_, pos0, slot, _t), tb in zip(toks, items, tabs):
            self._check_row(int(pos0), len(tk), len(tb), int(slot))
            if any(not 0 <= b_ < self.num_blocks for b_ in tb):
                raise ValueError("block table names a block outside the pool")
        if len({int(it[2]) for it in items}) != len(items):
            raise ValueError("two entries of a batch share a state slot")
        order = sorted(range(len(items)), key=lambda i: len(toks[i]) == 1)
        n_seg, T = len(items), sum(len(t) for t in toks)
        n_pre = sum(len(t) > 1 for t in toks)
        pages = max(len(t) for t in tabs)
        host = torch.zeros(2 * T + (n_seg + 1) + 2 * n_seg + n_seg * pages, dtype=torch.int32)
        if self.device.type == "cuda":
            host = host.pin_memory()
        positions, row_seg = host[:T], host[T:2 * T]
        o = 2 * T
        seg_row, seg_pos, seg_slot = host[o:o + n_seg + 1], host[o + n_seg + 1:o + 2 * n_seg + 1], host[o + 2 * n_seg + 1:o + 3 * n_seg + 1]
        tables = host[o + 3 * n_seg + 1:].view(n_seg, pages)
        first = [0] * len(items)
        r, flat = 0, []
        for s, i in enumerate(order):
            n, pos0 = len(toks[i]), int(items[i][1])
            first[i] = r
            positions[r:r + n] = torch.arange(pos0, pos0 + n, dtype=torch.int32)
            row_seg[r:r + n] = s
            seg_row[s], seg_pos[s], seg_slot[s] = r, pos0, int(items[i][2])
            tables[s, :len(tabs[i])] = torch.tensor(tabs[i], dtype=torch.int32)
            flat += toks[i]
            r += n
        seg_row[n_seg] = r
        tok = torch.tensor(flat, dtype=torch.int64)
        if self.device.type == "cuda":
            tok = tok.pin_memory()
        dev = host.to(self.device, non_blocking=True)
        b = RowBatch(T=T, n_seg=n_seg, n_pre=n_pre, pre_rows=T - (n_seg - n_pre), tokens=tok.to(self.device, non_blocking=True),
                     positions=dev[:T], row_seg=dev[T:2 * T], seg_row=dev[o:o + n_seg + 1], seg_pos=dev[o + n_seg + 1:o + 2 * n_seg + 1],
                     seg_slot=dev[o + 2 * n_seg + 1:o + 3 * n_seg + 1], tables=dev[o + 3 * n_seg + 1:].view(n_seg, pages),
                     pre_lens=tuple(int(items[i][1]) + len(toks[i]) for i in order[:n_pre]),
                     pre_pos=tuple(int(items[i][1]) for i in order[:n_pre]),
                     max_rows=max(len(t) for t in toks), max_len=max(int(it[1]) + len(t) for it, t in zip(items, toks)))
        return b, order, first

    @torch.no_grad()
    def forward_batch(self, items: list[tuple], want: list[list[int]]) -> torch.Tensor | None:
        """One forward over portions and single tokens of several sequences.  ``want[i]``: places among the tokens of
        item ``i`` whose logits are wanted; returns fp32 ``[wanted, vocab]`` in the order of the items (None: none)."""
        b, _order, first = self.make_batch(items)
        state = self._stack(b)
        rows = [first[i] + int(p) for i, ps in enumerate(want) for p in ps]
        if not rows:
            return None                 # the last boundary feeds nothing
        V8 = self.head.shape[0]
        out = torch.empty(len(rows), V8, dtype=torch.float32, device=self.device)
        idx = torch.tensor(rows, dtype=torch.int32).to(self.device)
        self._logits(state, idx, len(rows), out)
        return out[:, :self.cfg.vocab_size]

    @torch.no_grad()
    def prefill_group(self, items: list[tuple], want_logits: list[bool] | None = None) -> list:
        """Portions of several sequences in one forward; per item the logits ``[vocab]`` of its last token or None."""
        want_logits = list(want_logits) if want_logits is not None else [True] * len(items)
        out = self.forward_batch(items, [[int(len(it[0])) - 1] if w else [] for it, w in zip(items, want_logits)])
        rows = iter(out if out is not None else ())
        return [next(rows) if w else None for w in want_logits]

    def prefill(self, tokens, pos0: int, slot: int, block_table, embeds=None, cos_sin=None, want_logits: bool = True):
        if embeds is not None or cos_sin is not None:
            raise ValueError("this family takes token ids only")
        return self.prefill_group([(tokens, pos0, slot, block_table)], [want_logits])[0]

    # ------------------------------------------------------------------ decode
    def _row_buffers(self, M: int) -> dict:
        b = self._rows.get(M)
        if b is None:
            dev = self.device
            i32 = lambda *s: torch.zeros(*s, dtype=torch.int32, device=dev)
            pin = (lambda t: t.pin_memory()) if dev.type == "cuda" else (lambda t: t)
            b = self._rows[M] = {
                "tokens": torch.zeros(M, dtype=torch.int64, device=dev), "positions": i32(M).fill_(-1), "rope_pos": i32(M),
                "slots": i32(M).fill_(-1), "block_table": i32(M, self.max_blocks_per_seq),
                "logits8": torch.zeros(M, self.head.shape[0], dtype=torch.float32, device=dev),
                "next": torch.zeros(M, dtype=torch.int64, device=dev),
                "h_tokens": pin(torch.zeros(M, dtype=torch.int64)), "h_meta": pin(torch.zeros(2, M, dtype=torch.int32)),
                "h_bt": pin(torch.zeros(M, self.max_blocks_per_seq, dtype=torch.int32))}
            b["logits"] = b["logits8"][:, :self.cfg.vocab_size]
        return b

    def set_rows(self, M: int, tokens, positions, slots, block_tables, rope_deltas=None) -> None:
        """Stage up to ``M`` single tokens; missing rows are padding."""
        b, n = self._row_buffers(M), len(tokens)
        if n > M:
            raise ValueError(f"{n} rows do not fit bucket {M}")
        for r in range(n):
            self._check_row(positions[r], 1, len(block_tables[r]), slots[r])
        ev = b.get("h_event")
        if ev is None:
            ev = b["h_event"] = torch.cuda.Event()
        else:
            ev.synchronize()            # the pinned arrays are reused: the copies of the previous call have to have left them
        ht, hm, hb = b["h_tokens"], b["h_meta"], b["h_bt"]
        ht.zero_()
        hm.fill_(-1)
        for r in range(n):
            ht[r], hm[0, r], hm[1, r] = int(tokens[r]), int(positions[r]), int(slots[r])
            hb[r, :len(block_tables[r])] = torch.as_tensor(block_tables[r], dtype=torch.int32)
        for dst, src in (("tokens", ht), ("positions", hm[0]), ("slots", hm[1]), ("block_table", hb)):
            b[dst].copy_(src, non_blocking=True)
        ev.record()

    def _decode_body(self, M: int) -> None:
        rb = self._row_buffers(M)
        b = RowBatch(T=M, n_seg=M, n_pre=0, pre_rows=0, tokens=rb["tokens"], positions=rb["positions"], row_seg=None, seg_row=None,
                     seg_pos=rb["positions"], seg_slot=rb["slots"], tables=rb["block_table"])
        state = self._stack(b)
        self._logits(state, None, M, rb["logits8"])
        K.argmax(rb["logits"], rb["next"])
        if self._advance:
            self.advance_rows(M)

    def advance_rows(self, M: int) -> None:
        """Feed the sampled tokens back and advance the positions (no host synchronisation)."""
        b = self._row_buffers(M)
        K.call("advance_rows", b["tokens"], b["next"], b["positions"], b["rope_pos"], M)
        K._count()

    def _gkey(self, M: int, advance: bool):
        return (M, bool(advance))

    def capture(self, M: int, warmup: int = 2, advance: bool = False) -> None:
        """Capture the step of bucket ``M`` into a CUDA graph; warm-up runs on padding rows and touches no state."""
        key = self._gkey(M, advance)
        if key in self._graphs:
            return
        b = self._row_buffers(M)
        saved = {k: b[k].clone() for k in ("positions", "slots", "tokens")}
        b["positions"].fill_(-1)
        b["slots"].fill_(-1)
        self._advance = bool(advance)
        try:
            s = torch.cuda.Stream(device=self.device)
            s.wait_stream(torch.cuda.current_stream())
            with torch.cuda.stream(s), torch.no_grad():
                for _ in range(warmup):
                    self._decode_body(M)
            torch.cuda.current_stream().wait_stream(s)
            torch.cuda.synchronize()
            g = torch.cuda.CUDAGraph()
            if self.graph_pool is None:
                self.graph_pool = torch.cuda.graph_pool_handle()
            l0 = K.LAUNCHES
            with K.capture_graph(g, pool=self.graph_pool), torch.no_grad():
                self._decode_body(M)
            self._step_launches[M] = K.LAUNCHES - l0
            self._graphs[key] = g
        finally:
            self._advance = False
        for k, v in saved.items():
            b[k].copy_(v)

    @torch.no_grad()
    def decode(self, M: int, graph: bool = True, advance: bool = False) -> tuple[torch.Tensor, torch.Tensor]:
        """One token for every staged row: ``(next_tokens [M], logits [M, vocab])``, overwritten by the next step."""
        b = self._row_buffers(M)
        if graph:
            key = self._gkey(M, advance)
            if key not in self._graphs:
                self.capture(M, advance=advance)
            self._graphs[key].replay()
        else:
            self._advance = bool(advance)
            try:
                self._decode_body(M)
            finally:
                self._advance = False
        return b["next"], b["logits"]

