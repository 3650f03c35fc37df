"""Nemipel: a decoder whose layers are listed one by one, each with its own mixer -- lightning attention, grouped-query attention with
capped scores (optionally on another layer's keys and values), a gated delta rule with one decay per state row -- and whose norms follow
the residual sum.

    f = mixer, then feed-forward:   x <- rms(alpha x + f(x)) w_f;       logits = cap tanh(W rms(x) w / cap)

There is no norm in front of a sublayer: it reads x itself.  One launch per sublayer folds the output product, adds, normalises and
leaves both the fp32 residual and the next product's input (:func:`~..ops.postnorm.linear_postnorm`); the last one applies the
model's output norm as well.
"""
from __future__ import annotations

from typing import Callable, Dict, List, Optional, Sequence, Tuple

import torch
import torch.nn as nn

from ..config import NemipelConfig
from ..ops import postnorm as pn
from ..ops.latent import pad8
from .cache import LayerStateCache
from .layered import LayeredDecoder
from .mixers import CappedAttention, ChannelDelta, LightningAttention, SwigluMLP, padded, vector


class Nemipel(LayeredDecoder):
    KERNEL_SOURCES = ("gemm_tcgen05.cu", "postnorm.cu", "lightning.cu", "lightning_tcgen05.cu", "gqa_attention.cu", "gqa_attention_tcgen05.cu", "inference.cu",
                      "delta_rule.cu", "channel_delta.cu", "dyt.cu")

    def __init__(self, config: NemipelConfig):
        super().__init__(config)
        mixers, mlps = [], []
        for spec in config.layers:
            m, width, eps = spec.mixer, config.hidden_size, config.norm_eps
            if spec.type == "lightning":
                mixers.append(LightningAttention(m, width, eps))
            elif spec.type == "attention":
                mixers.append(CappedAttention(m, width, eps, self._rope(m["rot"]["dims"], float(m["rot"]["base"]))))
            else:
                mixers.append(ChannelDelta(m, width, eps))
            mlps.append(SwigluMLP(spec.mlp, width) if spec.mlp is not None else None)
        self.mixers = nn.ModuleList(mixers)
        self.mlps = nn.ModuleList([m if m is not None else nn.Identity() for m in mlps])
        self.eval()

    # -- weights ----------------------------------------------------------------------------------------------
    def tensor_shapes(self) -> Dict[str, Tuple[int, ...]]:
        cfg = self.config
        D = cfg.hidden_size
        out: Dict[str, Tuple[int, ...]] = {"embed": (cfg.vocab_size, D), "head": (cfg.vocab_size, D), "final.norm": (D,)}
        for i, spec in enumerate(cfg.layers):
            p = f"l{i}."
            out[p + "norm1"] = (D,)
            out.update({p + "mix." + n: s for n, s in self.mixers[i].shapes().items()})
            if spec.mlp is not None:
                out[p + "norm2"] = (D,)
                out.update({p + "mlp." + n: s for n, s in self.mlps[i].shapes().items()})
        return out

    @classmethod
    def from_tensors(cls, config: NemipelConfig, get: Callable[[str], torch.Tensor], names: Sequence[str], dtype=torch.bfloat16, device="cuda") -> "Nemipel":
        # the inner widths of the low-rank projections are sizes that only the tensors tell
        return super().from_tensors(config.with_ranks(lambda n: tuple(get(n).shape) if n in names else None), get, names, dtype, device)

    @staticmethod
    def random_tensor(name, shape, gen, device):
        leaf = name.rsplit(".", 1)[-1]
        if leaf.startswith("norm"):
            return torch.ones(shape, device=device)
        if leaf in ("A_log", "dt_bias"):
            return torch.full(shape, 0.0 if leaf == "A_log" else -2.0, device=device)
        return torch.randn(shape, generator=gen, device=device) * (1.0 if name == "embed" else shape[1] ** -0.5)

    @torch.no_grad()
    def _load(self, take, dtype, device) -> None:
        cfg = self.config
        D, Dp = cfg.hidden_size, pad8(cfg.hidden_size)
        self.register_parameter("embed", nn.Parameter(padded(take("embed"), cfg.vocab_size, Dp, dtype, device), requires_grad=False))
        self.register_parameter("head", nn.Parameter(padded(take("head"), pad8(cfg.vocab_size), Dp, dtype, device), requires_grad=False))
        self.steps: List[Tuple[pn.PostNorm, Optional[pn.PostNorm]]] = []
        for i, spec in enumerate(cfg.layers):
            self.mixers[i].load(lambda n: take(f"l{i}.mix.{n}"), dtype, device)
            if spec.mlp is not None:
                self.mlps[i].load(lambda n: take(f"l{i}.mlp.{n}"), dtype, device)
            norms = [pn.PostNorm(cfg.postln_alpha, vector(take(f"l{i}.norm{k}"), device, Dp), cfg.norm_eps, D) for k in ((1, 2) if spec.mlp is not None else (1,))]
            if i == cfg.num_layers - 1:
                norms[-1].w2 = vector(take("final.norm"), device, Dp)
            self.steps.append((norms[0], norms[1] if len(norms) > 1 else None))
        for rope in self._ropes.values():
            rope.ensure(cfg.seq_length, device)

    # -- forward ----------------------------------------------------------------------------------------------
    def layer_states(self, batch: int, max_len: int, dtype, device) -> List[Dict[str, torch.Tensor]]:
        states: List[Dict[str, torch.Tensor]] = []
        for spec, mixer in zip(self.config.layers, self.mixers):
            shared = spec.mixer.get("kv_from")   # the very tensors of that layer: one cache, appended to by its owner
            states.append(states[shared] if shared is not None else mixer.state(batch, max_len, dtype, device))
        return states

    def hidden_states(self, input_ids: torch.Tensor, cache: LayerStateCache, collect: Optional[List[torch.Tensor]] = None) -> torch.Tensor:
        B, L = input_ids.shape
        step = self._step(input_ids, cache)
        x, h = pn.embed_rows(input_ids.reshape(-1), self.embed)
        for i, (mixer, mlp) in enumerate(zip(self.mixers, self.mlps)):
            after_mixer, after_mlp = self.steps[i]
            h = pn.linear_postnorm(mixer(h, cache.states[i], step), mixer.w_o, x, after_mixer)
            if after_mlp is not None:
                h = pn.linear_postnorm(mlp(h), mlp.w_down, x, after_mlp)
            if collect is not None:
                collect.append(x[:, :self.config.hidden_size].reshape(B, L, -1).clone())
        if not step.on_device:
            cache.advance(L)
        return h

    def finish_logits(self, logits: torch.Tensor) -> torch.Tensor:
        cap = self.config.logit_softcap
        return pn.softcap_(logits, cap, self.embed.dtype != torch.float32) if cap else logits
