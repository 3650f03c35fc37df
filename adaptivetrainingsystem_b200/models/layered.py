"""What decoders whose layers are listed one by one share (``vimodra.py``, ``nemipel.py``): weights from a model folder or random ones,
the layer-state cache, the step that tells the mixers where a call's tokens belong, and the output head.

A subclass builds ``mixers`` and ``mlps`` from its configuration, names its tensors (:meth:`tensor_shapes`), loads them
(:meth:`_load`) and defines the block structure (:meth:`hidden_states`).
"""
from __future__ import annotations

from typing import Callable, Dict, List, Optional, Sequence, Tuple

import torch
import torch.nn as nn

from .. import ops
from ..ops import gemm as G
from .cache import LayerStateCache
from .mixers import Step, Take
from .transformer import RotaryEmbedding


class LayeredDecoder(nn.Module):
    """Inference model; build it with :meth:`from_tensors` or :meth:`random`.  ``dtype`` bf16: tcgen05 products and bf16 activations
    around an fp32 residual; fp32: everything in true 32-bit."""

    # csrc files a program needs that only runs this model's step function
    KERNEL_SOURCES: Tuple[str, ...] = ()
    # decode steps over pool rows of different lengths work without a captured graph too
    eager_row_decode = True

    def __init__(self, config):
        super().__init__()
        self.config = config
        self._ropes: Dict[Tuple[int, float], RotaryEmbedding] = {}

    def _rope(self, dims: int, base: float) -> RotaryEmbedding:
        key = (dims, base)
        if key not in self._ropes:
            self._ropes[key] = RotaryEmbedding(dims, self.config.seq_length, base)
        return self._ropes[key]

    # -- weights ----------------------------------------------------------------------------------------------
    def tensor_shapes(self) -> Dict[str, Tuple[int, ...]]:
        """Name -> shape of every tensor of a model folder."""
        raise NotImplementedError

    def _load(self, take: Take, dtype, device) -> None:
        raise NotImplementedError

    @staticmethod
    def random_tensor(name: str, shape: Tuple[int, ...], gen: torch.Generator, device) -> torch.Tensor:
        raise NotImplementedError

    @classmethod
    def from_tensors(cls, config, get: Callable[[str], torch.Tensor], names: Sequence[str], dtype=torch.bfloat16, device="cuda"):
        """``get(name)`` for the names of :meth:`tensor_shapes`; ``names`` is what the source holds (a surplus or a gap is an error)."""
        model = cls(config)
        shapes = model.tensor_shapes()
        missing, extra = sorted(set(shapes) - set(names)), sorted(set(names) - set(shapes))
        if missing or extra:
            raise ValueError(f"the tensors do not fit the configuration: missing {missing[:5]}, unexpected {extra[:5]}")

        def take(name):
            t = get(name)
            if tuple(t.shape) != shapes[name] and not (shapes[name] == () and t.numel() == 1):
                raise ValueError(f"{name}: shape {tuple(t.shape)}, the configuration says {shapes[name]}")
            return t
        model._load(take, dtype, torch.device(device))
        return model

    @classmethod
    def random(cls, config, dtype=torch.bfloat16, device="cuda", seed: int = 0):
        model = cls(config)
        shapes = model.tensor_shapes()
        gen = torch.Generator(device=device).manual_seed(seed)
        model._load(lambda name: cls.random_tensor(name, shapes[name], gen, device), dtype, torch.device(device))
        return model

    # -- forward ----------------------------------------------------------------------------------------------
    def layer_states(self, batch: int, max_len: int, dtype, device) -> List[Dict[str, torch.Tensor]]:
        """What the cache holds for every layer run."""
        raise NotImplementedError

    def make_cache(self, batch: int, max_len: int, dtype=None, device=None) -> LayerStateCache:
        dtype, device = dtype or self.embed.dtype, device or self.embed.device
        return LayerStateCache(batch, max_len, device, self.layer_states(batch, max_len, dtype, device))

    def hidden_states(self, input_ids: torch.Tensor, cache: LayerStateCache, collect: Optional[List[torch.Tensor]] = None) -> torch.Tensor:
        """Runs the tokens [B, L] that follow what ``cache`` holds -> normed hidden states [B * L, padded width].  ``collect`` receives the
        residual stream [B, L, width] after every layer run."""
        raise NotImplementedError

    def _step(self, input_ids: torch.Tensor, cache: LayerStateCache) -> Step:
        B, L = input_ids.shape
        on_device = cache.device_lengths is not None and L == 1   # graph-replayed (or pool) decode: positions live on the device
        if not on_device and cache.length + L > cache.max_len:
            raise RuntimeError(f"cache overflow: {cache.length}+{L} > {cache.max_len}")
        for rope in self._ropes.values():
            rope.ensure(cache.max_len + 1, self.embed.device)     # a full row that sits out a decode step stands at max_len
        if on_device:
            return Step(B, 1, 0, cache.device_lengths, cache.device_active, on_device=True)
        if L == 1:
            return Step(B, 1, cache.length, torch.full((B,), cache.length, dtype=torch.int32, device=self.embed.device))
        return Step(B, L, cache.length)

    def forward(self, input_ids: torch.Tensor, attention_mask: Optional[torch.Tensor] = None, return_aux_loss: Optional[bool] = None,
                cache: Optional[LayerStateCache] = None, last_token_only: bool = False, logits_at: Optional[Sequence[int]] = None,
                collect: Optional[List[torch.Tensor]] = None) -> torch.Tensor:
        """-> fp32 logits [B, n, vocab] of all positions, of the last one, or of the positions ``logits_at``."""
        if attention_mask is not None:
            raise ValueError("sequences of a batch have equal length here: no attention mask")
        B, L = input_ids.shape
        if cache is None:
            cache = self.make_cache(B, L)
        h = self.hidden_states(input_ids, cache, collect).view(B, L, -1)
        if last_token_only:
            h = h[:, -1:]
        elif logits_at is not None:
            h = h[:, list(logits_at)]
        n = h.shape[1]
        h = h.reshape(B * n, -1)
        logits = G.gemm_nt(h, self.head, out_fp32=True) if ops._lib.use_cuda_kernels(h) else ops.linear(h, self.head).float()
        return self.finish_logits(logits).view(B, n, -1)[..., :self.config.vocab_size]

    def finish_logits(self, logits: torch.Tensor) -> torch.Tensor:
        return logits

    # -- statistics ---------------------------------------------------------------------------------------------
    def num_parameters(self, trainable_only: bool = False) -> int:
        n = 0
        for shape in self.tensor_shapes().values():
            k = 1
            for d in shape:
                k *= d
            n += k
        return 0 if trainable_only else n
