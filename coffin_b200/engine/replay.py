"""Replaying a trace: given token ids pushed through a model step by step, logits out, nothing sampled.

``TraceReplayer`` drives what generation drives - the engine's block manager, state slots, ``ModelRunner`` and the
model's step function - with the batches that a trace prescribes instead of the scheduler's.  A step names, per
request, its next tokens and the places among them whose logits are wanted; requests are admitted at their first
entry, may sit out steps, and give their pages and slot back when they end.
"""
from __future__ import annotations

import torch

from .config import EngineConfig
from .llm_engine import LLMEngine
from .sequence import SamplingParams, Sequence, SequenceStatus

PAGE = 64


def pool_blocks(max_tokens: int) -> int:
    """Pages for ``max_tokens`` live tokens (each request rounded up to whole pages) plus the padding page."""
    return (max_tokens + PAGE - 1) // PAGE + 1


class TraceReplayer:
    def __init__(self, model, max_live: int = 4) -> None:
        self.engine = LLMEngine(model, EngineConfig(max_seq=model.max_seq, max_num_seqs=max_live, prefix_cache=False))
        self.live: dict[str, Sequence] = {}

    def step(self, entries: list[dict], end: list[str] = ()) -> torch.Tensor | None:
        """``entries``: ``{"id", "tokens", "want"}`` dicts.  Returns fp32 logits ``[wanted, vocab]`` on the host, or None."""
        eng = self.engine
        batch = []
        for e in entries:
            toks = [int(t) for t in e["tokens"]]
            if not toks:
                raise ValueError(f"request {e['id']!r}: an entry without tokens")
            seq = self.live.get(e["id"])
            if seq is None:
                if not eng.scheduler.free_slots:
                    raise RuntimeError("no free state slot: too many live requests")
                seq = self.live[e["id"]] = eng.scheduler.admit(Sequence(toks, SamplingParams(), request_id=str(e["id"])))
                eng.runner.begin_prefill(seq)
            else:
                seq.prompt += toks
            if seq.num_tokens > eng.max_seq:
                raise ValueError(f"request {e['id']!r} exceeds the {eng.max_seq}-token window")
            if not eng.bm.ensure_blocks(seq.blocks, len(toks)):
                raise RuntimeError("the page pool is exhausted")
            batch.append((seq, toks, [int(w) for w in e.get("want", ())]))
        logits = eng.runner.run_batch(batch) if batch else None
        host = logits.float().cpu() if logits is not None else None
        if host is not None and eng.runner._check is not None:
            eng.runner._check()
        for seq, _t, _w in batch:
            if seq.status is SequenceStatus.PREFILLING:
                eng.scheduler.prefill_done(seq)
        for rid in end:
            seq = self.live.pop(rid, None)
            if seq is not None:
                eng.abort(seq, "end")
        return host
