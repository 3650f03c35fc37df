"""Replay of recorded steps: token ids in, logits out, nothing sampled.

Every input line is one step, ``{"step": n, "entries": [{"id": .., "tokens": [..], "want": [..]}], "end": [..]}``: each entry brings the
next tokens of a request and names the places among them whose logits are asked for; the requests in ``end`` are finished after
the step and give their row back.  Steps run on a :class:`SequencePool`, i.e. through the step functions, caches and kernels of
generation: one token of a running request goes through the (captured) decode step, anything longer is a portion.
"""
from __future__ import annotations

import json
import os
from typing import Any, Dict, Iterable, Optional

import torch

from .pool import SequencePool


class TraceRunner:
    def __init__(self, model, max_tokens: int, rows: int = 2, use_graph: Optional[bool] = None):
        self.pool = SequencePool(model, rows, max_tokens, use_graph)
        self.slot: Dict[str, int] = {}

    def entry(self, e: Dict[str, Any]) -> Optional[torch.Tensor]:
        """-> fp32 logits of the wanted places [n, V] on the host, or ``None``."""
        pool, rid = self.pool, e["id"]
        if rid not in self.slot:
            self.slot[rid] = pool.open()
        s, want = self.slot[rid], list(e.get("want") or ())
        if len(e["tokens"]) == 1 and pool.lengths[s] > 0:
            pool.last[s] = int(e["tokens"][0])
            pool.cache.device_active.zero_()
            pool.cache.device_active[s] = 1
            out = pool.decode([s])[s:s + 1]
            pool.cache.device_active.zero_()
            out = out[[0] * len(want)] if want else None
        else:
            out = pool.extend(s, e["tokens"], logits_at=want)
        return None if out is None else out.float().cpu()

    def step(self, record: Dict[str, Any]) -> Optional[torch.Tensor]:
        parts = [self.entry(e) for e in record.get("entries", ())]
        for rid in record.get("end", ()):
            if rid in self.slot:
                self.pool.close(self.slot.pop(rid))
        parts = [p for p in parts if p is not None]
        return torch.cat(parts) if parts else None


def replay(runner: TraceRunner, lines: Iterable[str], out_dir: str) -> None:
    """Writes ``out_dir/<step>.f32`` for every step in which something is wanted and prints ``done <step>`` after every step."""
    from ..ops import check_status
    for line in lines:
        if not line.strip():
            continue
        record = json.loads(line)
        logits = runner.step(record)
        if runner.pool.device.type == "cuda":
            check_status()
        if logits is not None:
            part = os.path.join(out_dir, f"{record['step']}.f32.part")
            with open(part, "wb") as f:
                f.write(logits.contiguous().numpy().astype("<f4").tobytes())
            os.replace(part, os.path.join(out_dir, f"{record['step']}.f32"))
        print(f"done {record['step']}", flush=True)
