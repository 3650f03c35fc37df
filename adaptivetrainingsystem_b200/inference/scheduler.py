"""Continuous batching: a fixed pool of cache rows, requests of any length admitted and retired between decode steps.

The rows live in a :class:`SequencePool` (one cache of ``max_batch`` rows and one captured decode step over it).  Every call of
:meth:`ContinuousBatcher.step`

1. admits waiting requests into free rows and prefills them straight into the row (a one-row view of the pool's cache), either the
   whole prompt at once or, with ``prefill_chunk``, at most that many prompt tokens per step, so that a long prompt does not hold up the
   rows that are decoding; the first token is sampled from the logits of the prompt's last position;
2. replays the decode graph once for all rows (each row at its own length; rows that are free or still in their prompt come out
   unchanged and their output is ignored), samples one token per row in one launch;
3. retires rows that produced a stop token or their token budget and frees their slots.

The reference's own generator serves one sequence at a time and re-runs the context for every token (``Chat.py:355-465``); its
vendored serving engine keeps a slot table per batch (``colossalai/inference/kv_cache/kvcache_manager.py:11-106`` allocator,
``kv_cache/batch_infer_state.py:13-118`` per-batch lengths and start locations), which is the bookkeeping done here on rows.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Dict, List, Optional, Sequence

import torch

from .engine import GenerationEngine, SamplingParams, sample_next
from .pool import SequencePool


@dataclass
class Request:
    rid: int
    prompt: torch.Tensor                      # [Lp] token ids (host or device)
    max_new_tokens: int
    tokens: List[int] = field(default_factory=list)
    slot: int = -1
    prefilled: int = 0                        # prompt tokens the row already holds
    done: bool = False


class ContinuousBatcher:
    def __init__(self, engine: GenerationEngine, max_batch: int = 64, max_len: int = 2048, params: Optional[SamplingParams] = None,
                 prefill_chunk: Optional[int] = None):
        self.engine, self.model = engine, engine.model
        self.params = params or SamplingParams.from_mode("greedy")
        self.max_batch, self.max_len = max_batch, max_len
        self.prefill_chunk = prefill_chunk
        self.device = next(self.model.parameters()).device
        if getattr(self.model, "_ep_comm", None) is not None:
            # admission prefills one request on one rank, which the expert-parallel exchange (a collective of all ranks) cannot serve
            raise RuntimeError("continuous batching runs on one GPU (or on replicas): the model must not be expert-parallel")
        self.pool = SequencePool(self.model, max_batch, max_len)
        self.cache, self.slots = self.pool.cache, self.pool.slots
        self.history = torch.zeros(max_batch, self.params.repetition_window, dtype=torch.long, device=self.device)
        self.by_slot: Dict[int, Request] = {}          # rows that decode
        self.prefilling: List[Request] = []            # rows still in their prompt, oldest first
        self.waiting: List[Request] = []
        self.finished: Dict[int, Request] = {}
        self._next_id = 0
        self._stop = set(int(t) for t in (self.params.stop_token_ids or ()))
        self.steps = 0
        self.generator = torch.Generator(device=self.device).manual_seed(self.params.seed) if self.params.seed is not None else None

    # -- requests --------------------------------------------------------------------------------------------------
    def submit(self, prompt: Sequence[int], max_new_tokens: Optional[int] = None) -> int:
        ids = torch.as_tensor(prompt, dtype=torch.long).flatten()
        budget = int(max_new_tokens if max_new_tokens is not None else self.params.max_new_tokens)
        if ids.numel() < 1 or ids.numel() + budget > self.max_len:
            raise ValueError(f"prompt of {ids.numel()} tokens + {budget} new tokens does not fit rows of {self.max_len}")
        r = Request(self._next_id, ids, budget)
        self._next_id += 1
        self.waiting.append(r)
        return r.rid

    @property
    def pending(self) -> int:
        return len(self.waiting) + len(self.prefilling) + len(self.by_slot)

    # -- one scheduling step ---------------------------------------------------------------------------------------
    @torch.no_grad()
    def _admit(self) -> None:
        budget = self.prefill_chunk or (1 << 62)       # prompt tokens this step may still run
        while budget > 0:
            if not self.prefilling:
                if not (self.waiting and self.pool.available):
                    return
                r = self.waiting.pop(0)
                r.slot = self.pool.open()
                self.prefilling.append(r)
            r = self.prefilling[0]
            n = min(budget, r.prompt.numel() - r.prefilled)
            budget -= n
            part = r.prompt[r.prefilled:r.prefilled + n]
            r.prefilled += n
            done = r.prefilled == r.prompt.numel()
            logits = self.pool.extend(r.slot, part, active=done)
            if done:
                self.prefilling.pop(0)
                self._first_token(r, logits)

    def _first_token(self, r: Request, logits: torch.Tensor) -> None:
        slot, ids, w = r.slot, r.prompt.to(self.device), self.history.shape[1]
        n = ids.numel()
        self.history[slot].fill_(int(r.prompt[0]))     # left padding of a short prompt repeats its first token
        self.history[slot, -min(n, w):] = ids[-min(n, w):]
        first = sample_next(logits, self.params, self.history[slot:slot + 1], self.generator)
        self.pool.last[slot:slot + 1] = first
        self.history[slot] = torch.roll(self.history[slot], -1)
        self.history[slot, -1:] = first
        self.by_slot[slot] = r
        self._accept(slot, int(first))

    def _accept(self, slot: int, token: int) -> None:
        """Host-side bookkeeping of one generated token (the device-side state was updated for all rows at once)."""
        r = self.by_slot[slot]
        r.tokens.append(token)
        if token in self._stop or len(r.tokens) >= r.max_new_tokens:
            self._retire(slot)

    def _retire(self, slot: int) -> None:
        r = self.by_slot.pop(slot)
        r.done = True
        self.finished[r.rid] = r
        self.pool.close(slot)

    @torch.no_grad()
    def step(self) -> int:
        """Admit, decode one token for every live row, retire.  Returns the number of live rows that were decoded."""
        self._admit()
        live = sorted(self.by_slot)
        if not live:
            return 0
        logits = self.pool.decode(live)
        nxt_dev = sample_next(logits, self.params, self.history, self.generator)
        self.pool.last.copy_(nxt_dev)
        self.history = torch.roll(self.history, -1, dims=1)
        self.history[:, -1] = nxt_dev
        nxt = nxt_dev.tolist()                       # the one device-to-host read of the step
        for slot in live:
            self._accept(slot, int(nxt[slot]))
        self.steps += 1
        return len(live)

    def run(self, prompts: Sequence[Sequence[int]], max_new_tokens: Optional[int] = None) -> List[List[int]]:
        """Serve all prompts; returns the generated ids in the order of ``prompts``."""
        rids = [self.submit(p, max_new_tokens) for p in prompts]
        while self.pending:
            self.step()
        return [self.finished.pop(r).tokens for r in rids]
