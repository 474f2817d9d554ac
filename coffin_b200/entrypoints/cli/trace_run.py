"""Replay a trace of token ids through a model and write the logits it asks for.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N  < steps.jsonl

Standard input carries one JSON object per line:

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

Every step is one batch of the engine; for a step that wants logits ``<out>/<step>.f32`` receives them (little-endian
fp32, ``[wanted, vocab]``), and after every step ``done <step>`` is printed.  ``--max-tokens`` sizes the page pool
(live tokens, every request rounded up to whole pages); there are state slots for four live requests.
"""
from __future__ import annotations

import argparse
import json
import sys
from pathlib import Path

MAX_LIVE = 4


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description=__doc__.split("\n\n")[0])
    ap.add_argument("--model", required=True, help="directory with config.json and safetensors")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="directory for the logits")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens that live requests hold at any time")
    args = ap.parse_args(argv)
    import torch
    from ...config import load_config
    from ...engine.replay import TraceReplayer, pool_blocks
    from ...models import FLOAT32, build_model, detect_architecture, kernel_sources
    from ...ops import _lib
    from ...weights.loader import load_checkpoint
    cfg = load_config(args.model)
    arch = detect_architecture(cfg)
    if args.dtype == "float32" and arch not in FLOAT32:
        print(f"{arch}: this family computes in 16 bits only", file=sys.stderr)
        return 3
    _lib.use_sources(kernel_sources(arch))
    blocks = pool_blocks(args.max_tokens)
    window = min((blocks - 1) * 64, getattr(cfg, "max_positions", (blocks - 1) * 64))
    kw = {"dtype": torch.float32} if args.dtype == "float32" else {}
    model = build_model(cfg, load_checkpoint(args.model), device="cuda", max_seq=window, num_slots=MAX_LIVE, num_blocks=blocks,
                        vision=False, **kw)
    rep = TraceReplayer(model, MAX_LIVE)
    out = Path(args.out)
    for line in sys.stdin:
        if not line.strip():
            continue
        st = json.loads(line)
        logits = rep.step(st.get("entries", []), st.get("end", []))
        if logits is not None:
            part = out / f".{st['step']}.part"
            part.write_bytes(logits.contiguous().numpy().astype("<f4").tobytes())
            part.rename(out / f"{st['step']}.f32")
        print(f"done {st['step']}", flush=True)
    return 0


if __name__ == "__main__":
    sys.exit(main())
