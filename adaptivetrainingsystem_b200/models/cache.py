"""What a decoder keeps per sequence between steps.

:class:`SequenceCache` is the part every model shares: the fill level, its device-side copy for decode steps that are replayed from a
CUDA graph, and row views for schedulers that admit sequences one by one into a pool.  ``KVCache`` (``transformer.py``) holds keys and
values of every position; :class:`LayerStateCache` holds whatever its layers declare -- rings of the last tokens, recurrent states,
convolution inputs -- one entry per layer *run*, so a layer that is run several times per token has a state for each run.
"""
from __future__ import annotations

from typing import Dict, List, Optional

import torch


class SequenceCache:
    """``length`` (host) is the number of tokens every row holds during a portion of a prompt; decode steps read the device-side
    ``device_lengths`` / ``device_positions`` (int32 [batch]).  Rows whose ``device_active`` entry is 0 are computed by a replayed decode
    step but must come out of it unchanged."""

    def __init__(self, batch: int, max_len: int, device):
        self.batch, self.max_len, self.device = batch, max_len, torch.device(device)
        self.length = 0
        self.device_lengths: Optional[torch.Tensor] = None
        self.device_positions: Optional[torch.Tensor] = None
        self.device_active: Optional[torch.Tensor] = None

    def enable_device_lengths(self) -> None:
        self.device_lengths = torch.full((self.batch,), self.length, dtype=torch.int32, device=self.device)
        self.device_positions = torch.full((self.batch,), self.length, dtype=torch.int32, device=self.device)
        self.device_active = torch.ones(self.batch, dtype=torch.int32, device=self.device)

    def device_advance(self) -> None:
        """One decoded token of every active row: called inside the captured step."""
        self.device_lengths += self.device_active
        self.device_positions += self.device_active

    def set_row(self, row: int, length: int, active: bool) -> None:
        self.device_lengths[row] = length
        self.device_positions[row] = length
        self.device_active[row] = int(active)

    def advance(self, n: int) -> None:
        self.length += n

    def reset(self) -> None:
        self.length = 0

    def row(self, i: int) -> "SequenceCache":
        """Row ``i`` as an empty cache of batch 1 whose writes land in this cache."""
        raise NotImplementedError


class LayerStateCache(SequenceCache):
    """``states[r]``: named tensors ``[batch, ...]`` of layer run ``r``.  A sequence at position 0 starts from nothing whatever its row
    still holds, so a row can be handed to the next sequence without being cleared."""

    def __init__(self, batch: int, max_len: int, device, states: List[Dict[str, torch.Tensor]]):
        super().__init__(batch, max_len, device)
        self.states = states

    def row(self, i: int) -> "LayerStateCache":
        return LayerStateCache(1, self.max_len, self.device, [{k: t[i:i + 1] for k, t in s.items()} for s in self.states])
