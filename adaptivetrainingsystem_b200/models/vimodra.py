"""Vimodra: a decoder whose layers are listed one by one, each with its own mixer, with Dynamic-Tanh norms before and after every
sublayer, layer scales, and an optional range of layers that is run several times with the same weights (every pass has its own
cache or state, and a learned vector is added to the residual before each pass).

    x <- x + ls1 * norm1b(mixer(norm1(x)));   x <- x + ls2 * norm2b(mlp(norm2(x)))

Because the norms are element-wise, everything between two products is one function of the product and the fp32 residual: a
:class:`~..ops.dyt.DytChain` per sublayer and run holds its constants (output norm times layer scale, plus the vector of a loop pass
that begins next; the input norm of whatever follows).
"""
from __future__ import annotations

from typing import Dict, List, Optional, Tuple

import torch
import torch.nn as nn

from ..config import VimodraConfig
from ..ops import dyt as dyt_ops
from ..ops.latent import pad8
from .cache import LayerStateCache
from .layered import LayeredDecoder
from .mixers import GatedDelta, GeluMLP, LatentAttention, padded, vector


class Vimodra(LayeredDecoder):
    KERNEL_SOURCES = ("gemm_tcgen05.cu", "dyt.cu", "latent_attention.cu",
                      "latent_decode.cu", "attention_window_tcgen05.cu", "delta_rule.cu")

    def __init__(self, config: VimodraConfig):
        super().__init__(config)
        mixers, mlps = [], []
        for spec in config.layers:
            m = spec.mixer
            if spec.type == "latent_attention":
                mixers.append(LatentAttention(m, config.hidden_size, config.norm_eps, self._rope(m["rot_dim"], float(m["rot"]["base"]))))
            else:
                mixers.append(GatedDelta(m, config.hidden_size, config.norm_eps))
            mlps.append(GeluMLP(spec.mlp, config.hidden_size) if spec.mlp is not None else None)
        self.mixers = nn.ModuleList(mixers)
        self.mlps = nn.ModuleList([m if m is not None else nn.Identity() for m in mlps])
        self.runs = config.runs()
        self.eval()

    # -- weights ----------------------------------------------------------------------------------------------
    def tensor_shapes(self) -> Dict[str, Tuple[int, ...]]:
        cfg = self.config
        D = cfg.hidden_size
        out: Dict[str, Tuple[int, ...]] = {"embed": (cfg.vocab_size, D), "head": (cfg.vocab_size, D)}

        def norm(name):
            out.update({name: (D,), name + ".b": (D,), name + ".alpha": ()})
        norm("final.norm")
        if cfg.loop_times:
            out["loop.step"] = (cfg.loop_times, D)
        for i, spec in enumerate(cfg.layers):
            p = f"l{i}."
            norm(p + "norm1"), norm(p + "norm1b")
            out[p + "ls1"] = (D,)
            out.update({p + "mix." + n: s for n, s in self.mixers[i].shapes().items()})
            if spec.mlp is not None:
                norm(p + "norm2"), norm(p + "norm2b")
                out[p + "ls2"] = (D,)
                out.update({p + "mlp." + n: s for n, s in self.mlps[i].shapes().items()})
        return out

    @staticmethod
    def random_tensor(name, shape, gen, device):
        leaf = name.rsplit(".", 1)[-1]
        if leaf in ("alpha", "A_log") or leaf.startswith(("ls", "norm")):
            return torch.full(shape, 0.0 if leaf == "A_log" else 0.5 if leaf == "alpha" else 1.0, device=device)
        if len(shape) < 2:
            return torch.zeros(shape, device=device)
        return torch.randn(shape, generator=gen, device=device) * (1.0 if name == "embed" else shape[1] ** -0.5)

    @torch.no_grad()
    def _load(self, take, dtype, device) -> None:
        cfg = self.config
        D, Dp = cfg.hidden_size, pad8(cfg.hidden_size)
        self.register_parameter("embed", nn.Parameter(padded(take("embed"), cfg.vocab_size, Dp, dtype, device), requires_grad=False))
        self.register_parameter("head", nn.Parameter(padded(take("head"), pad8(cfg.vocab_size), Dp, dtype, device), requires_grad=False))
        for i, spec in enumerate(cfg.layers):
            self.mixers[i].load(lambda n: take(f"l{i}.mix.{n}"), dtype, device)
            if spec.mlp is not None:
                self.mlps[i].load(lambda n: take(f"l{i}.mlp.{n}"), dtype, device)
        for rope in self._ropes.values():
            rope.ensure(cfg.seq_length, device)
        steps = vector(take("loop.step"), device).view(cfg.loop_times, D) if cfg.loop_times else None

        def norm(name):
            return vector(take(name), device, Dp), vector(take(name + ".b"), device, Dp), float(take(name + ".alpha"))

        def step_vector(run: int) -> Optional[torch.Tensor]:
            t = self.runs[run][1] if run < len(self.runs) else None
            return None if t is None else vector(steps[t], device, Dp)

        def entry(run: int):   # the norm in front of a run, or the final one
            return norm(f"l{self.runs[run][0]}.norm1") if run < len(self.runs) else norm("final.norm")

        def chain(post: str, scale: str, add: Optional[torch.Tensor], nxt) -> dyt_ops.DytChain:
            w, b, a = norm(post)
            ls = vector(take(scale), device, Dp)
            b1 = b * ls
            return dyt_ops.DytChain(w * ls, b1 if add is None else b1 + add, a, *nxt)
        self.first_add, self.first_norm = step_vector(0), entry(0)
        self.chains: List[Tuple[dyt_ops.DytChain, Optional[dyt_ops.DytChain]]] = []
        self.adds: List[Optional[torch.Tensor]] = []   # what a run's last chain adds beyond its own layer
        for r, (i, _) in enumerate(self.runs):
            add, nxt, p = step_vector(r + 1), entry(r + 1), f"l{i}."
            if cfg.layers[i].mlp is None:
                self.chains.append((chain(p + "norm1b", p + "ls1", add, nxt), None))
            else:
                self.chains.append((chain(p + "norm1b", p + "ls1", None, norm(p + "norm2")), chain(p + "norm2b", p + "ls2", add, nxt)))
            self.adds.append(add)

    # -- forward ----------------------------------------------------------------------------------------------
    def layer_states(self, batch: int, max_len: int, dtype, device) -> List[Dict[str, torch.Tensor]]:
        return [self.mixers[i].state(batch, max_len, dtype, device) for i, _ in self.runs]

    def hidden_states(self, input_ids: torch.Tensor, cache: LayerStateCache, collect: Optional[List[torch.Tensor]] = None) -> torch.Tensor:
        B, L = input_ids.shape
        step = self._step(input_ids, cache)
        x, h = dyt_ops.embed_norm(input_ids.reshape(-1), self.embed, self.first_add, *self.first_norm)
        for r, (i, _) in enumerate(self.runs):
            mixer, (after_mixer, after_mlp) = self.mixers[i], self.chains[r]
            h = dyt_ops.linear_residual(mixer(h, cache.states[r], step), mixer.w_o, None, x, after_mixer)
            if after_mlp is not None:
                mlp = self.mlps[i]
                h = dyt_ops.linear_residual(mlp(h), mlp.w_down, mlp.b_down, x, after_mlp)
            if collect is not None:
                s = x if self.adds[r] is None else x - self.adds[r]
                collect.append(s[:, :self.config.hidden_size].reshape(B, L, -1).clone())
        if not step.on_device:
            cache.advance(L)
        return h
