"""Replaying a trace through the serving engine (the program ``bin/trace_run``): requests of known
token ids, cut into steps by the trace, run with the engine's own step function, cache and state."""
from __future__ import annotations

import argparse
import json
import os
import sys
from typing import Dict, List, Optional

import numpy as np
import torch

from ..foundation.error import ProcessingError
from ..ops.decode import PAGE
from ..ops.ragged import Entry

SLOTS = 4            # requests that are live at the same time


class TraceRunner:
    def __init__(self, engine, max_tokens: int, slots: int = SLOTS) -> None:
        self.engine = engine
        pages = max(1, (max_tokens + PAGE - 1) // PAGE)
        engine.open_slots(slots, pages * PAGE, num_pages=pages)
        self.free: List[int] = list(range(slots - 1, -1, -1))
        self.live: Dict[str, int] = {}

    def step(self, entries: List[dict], end: List[str]) -> Optional[np.ndarray]:
        """Runs one step; the wanted logits ``[wanted, vocab]`` or None."""
        batch, cache = [], self.engine.cache
        for e in entries:
            if e["id"] not in self.live:
                if not self.free:
                    raise ProcessingError.limit_exceeded("live requests", len(self.live),
                                                         len(self.live) + 1)
                self.live[e["id"]] = self.free.pop()
            slot = self.live[e["id"]]
            batch.append(Entry(slot, cache.length(slot), e["tokens"], e["want"]))
        out = self.engine.step(batch) if batch else None
        rows = None
        if out is not None:
            rows = out[:, :self.engine.cfg.vocab_size].float().cpu().numpy()
        for rid in end:
            slot = self.live.pop(rid, None)
            if slot is not None:
                cache.release(slot)
                self.free.append(slot)
        return rows


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run")
    ap.add_argument("--model", required=True)
    ap.add_argument("--dtype", choices=["bfloat16", "float32"], default="bfloat16")
    ap.add_argument("--out", required=True)
    ap.add_argument("--max-tokens", type=int, required=True)
    ap.add_argument("--device", default="cuda")
    a = ap.parse_args(argv)
    from ..models.registry import load_dir
    from .engine import make_engine
    torch.backends.cuda.matmul.allow_tf32 = False
    try:
        model = load_dir(a.model, device=a.device, dtype=getattr(torch, a.dtype))
    except ProcessingError as e:
        if a.dtype == "float32":
            print(e, file=sys.stderr)
            return 3
        raise
    runner = TraceRunner(make_engine(model, max_batch=SLOTS), a.max_tokens)
    for line in sys.stdin:
        if not line.strip():
            continue
        s = json.loads(line)
        rows = runner.step(s["entries"], s.get("end", []))
        if rows is not None:
            rows.astype("<f4").tofile(os.path.join(a.out, f"{s['step']}.f32"))
        print(f"done {s['step']}", flush=True)
    if model.device.type == "cuda":
        from ..ops._lib import check_status
        check_status(model.device)
    return 0
