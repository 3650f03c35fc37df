"""A pool of cache rows that sequences come to and leave one by one.

One cache of ``rows`` rows, a free list, and one decode step over all rows -- captured into a CUDA graph on a GPU.  A sequence opens a
row, is extended by portions of any size (written straight into the row through a one-row view of the cache), decodes one token at a
time together with the other rows, and closes the row again.  Rows that do not take part in a decode step come out of it unchanged.
``ContinuousBatcher`` schedules requests on such a pool; ``TraceRunner`` replays recorded steps on one.
"""
from __future__ import annotations

from typing import Dict, Optional, Sequence

import torch


from .engine import GraphDecoder, KVSlotManager


class SequencePool:
    def __init__(self, model, rows: int, max_len: int, use_graph: Optional[bool] = None):
        self.model, self.rows, self.max_len = model, rows, max_len
        p = next(model.parameters())
        self.device = p.device
        self.cache = model.make_cache(rows, max_len)
        self.slots = KVSlotManager(rows)
        self.lengths: Dict[int, int] = {}                 # open rows -> tokens they hold
        self.use_graph = (self.device.type == "cuda") if use_graph is None else use_graph
        if not self.use_graph and not getattr(model, "eager_row_decode", False):
            raise RuntimeError("decoding rows of different lengths replays a CUDA graph of the decode step: a CUDA device is required")
        self._decoder: Optional[GraphDecoder] = None
        self.last = torch.zeros(rows, dtype=torch.long, device=self.device)
        if self.use_graph:
            self.decoder()
        else:
            self.cache.enable_device_lengths()
        self.cache.device_lengths.zero_()
        self.cache.device_positions.zero_()
        self.cache.device_active.zero_()

    @torch.no_grad()
    def decoder(self) -> GraphDecoder:
        if self._decoder is None:
            self._decoder = GraphDecoder(self.model, self.cache)   # captured once; rows come and go underneath it
        return self._decoder

    # -- rows -----------------------------------------------------------------------------------------------------
    @property
    def available(self) -> int:
        return self.slots.available

    def open(self) -> int:
        slot = self.slots.alloc(1)
        if slot is None:
            raise RuntimeError(f"all {self.rows} rows of the pool are taken")
        self.lengths[int(slot[0])] = 0
        return int(slot[0])

    def close(self, slot: int) -> None:
        del self.lengths[slot]
        self.cache.set_row(slot, 0, False)
        self.slots.free(torch.tensor([slot]))

    # -- tokens ---------------------------------------------------------------------------------------------------
    @torch.no_grad()
    def extend(self, slot: int, ids: Sequence[int], logits_at: Optional[Sequence[int]] = None, active: bool = False) -> Optional[torch.Tensor]:
        """Runs the next portion of a sequence -> logits [1, V] of its last token, or [n, V] of the places ``logits_at`` of the portion
        (``None`` when that is empty).  ``active``: the row takes part in decode steps from now on."""
        ids = torch.as_tensor(ids, dtype=torch.long).flatten()
        n = self.lengths[slot]
        view = self.cache.row(slot)
        view.length = n
        at = [ids.numel() - 1] if logits_at is None else list(logits_at)
        logits = self.model(ids.to(self.device).view(1, -1), cache=view, logits_at=at or [0], return_aux_loss=False)
        self.lengths[slot] = n + ids.numel()
        self.cache.set_row(slot, self.lengths[slot], active)
        return logits[0] if at else None

    @torch.no_grad()
    def decode(self, slots: Sequence[int]) -> torch.Tensor:
        """One decode step: every row of ``slots`` feeds its token in ``last`` -> logits [rows, V] (rows outside ``slots`` are
        meaningless; a static buffer that the next step overwrites).  ``cache.device_active`` must mark exactly these rows."""
        for s in slots:
            if self.lengths[s] + 1 > self.max_len:
                raise RuntimeError(f"cache overflow: {self.lengths[s]}+1 > {self.max_len}")
        if self.use_graph:
            d = self.decoder()
            d.tokens.copy_(self.last.view(-1, 1))
            d.graph.replay()
            logits = d.logits
        else:
            logits = self.model(self.last.view(-1, 1), cache=self.cache, last_token_only=True, return_aux_loss=False)[:, -1]
            self.cache.device_advance()
        for s in slots:
            self.lengths[s] += 1
        return logits

