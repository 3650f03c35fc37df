"""Vimodra: a decoder whose layers are listed one by one, each with its own mixer, with Dynamic-Tanh norms before and after every
sublayer, layer scales, and an optional range of layers that is run several times with the same weights (every pass has its own
cache or state, and a learned vector is added to the residual before each pass).

    x <- x + ls1 * norm1b(mixer(norm1(x)));   x <- x + ls2 * norm2b(mlp(norm2(x)))

Because the norms are element-wise, everything between two products is one function of the product and the fp32 residual: a
:class:`~..ops.dyt.DytChain` per sublayer and run holds its constants (output norm times layer scale, plus the vector of a loop pass
that begins next; the input norm of whatever follows).
"""
from __future__ import annotations

from typing import Any, Callable, Dict, List, Optional, Sequence, Tuple

import torch
import torch.nn as nn

from .. import ops
from ..config import VimodraConfig
from ..ops import dyt as dyt_ops
from ..ops import gemm as G
from ..ops.latent import pad8
from .cache import LayerStateCache
from .mixers import GatedDelta, GeluMLP, LatentAttention, Step, padded, vector
from .transformer import RotaryEmbedding


class Vimodra(nn.Module):
    """Inference model; build it with :meth:`from_tensors` or :meth:`random`.  ``dtype`` bf16: tcgen05 products and bf16 activations
    around an fp32 residual; fp32: everything in true 32-bit."""

    # csrc files a program needs that only runs this model's step function
    KERNEL_SOURCES = ("gemm_tcgen05.cu", "dyt.cu", "latent_attention.cu",
                      "latent_decode.cu", "attention_window_tcgen05.cu", "delta_rule.cu")
    # decode steps over pool rows of different lengths work without a captured graph too
    eager_row_decode = True

    def __init__(self, config: VimodraConfig):
        super().__init__()
        self.config = config
        self._ropes: Dict[Tuple[int, float], RotaryEmbedding] = {}
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

    def _rope(self, dims: int, base: float) -> RotaryEmbedding:
        key = (dims, base)
        if key not in self._ropes:
            self._ropes[key] = RotaryEmbedding(dims, self.config.seq_length, base)
        return self._ropes[key]

    # -- weights ----------------------------------------------------------------------------------------------
    def tensor_shapes(self) -> Dict[str, Tuple[int, ...]]:
        """Name -> shape of every tensor of a model folder."""
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

    @classmethod
    def from_tensors(cls, config: VimodraConfig, get: Callable[[str], torch.Tensor], names: Sequence[str], dtype=torch.bfloat16, device="cuda") -> "Vimodra":
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
    def random(cls, config: VimodraConfig, dtype=torch.bfloat16, device="cuda", seed: int = 0) -> "Vimodra":
        model = cls(config)
        shapes = model.tensor_shapes()
        gen = torch.Generator(device=device).manual_seed(seed)

        def take(name):
            shape, leaf = shapes[name], name.rsplit(".", 1)[-1]
            if leaf in ("alpha", "A_log") or leaf.startswith(("ls", "norm")):
                return torch.full(shape, 0.0 if leaf == "A_log" else 0.5 if leaf == "alpha" else 1.0, device=device)
            if len(shape) < 2:
                return torch.zeros(shape, device=device)
            return torch.randn(shape, generator=gen, device=device) * (1.0 if name == "embed" else shape[1] ** -0.5)
        model._load(take, dtype, torch.device(device))
        return model

    @torch.no_grad()
    def _load(self, take: Callable[[str], torch.Tensor], dtype, device) -> None:
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
    def make_cache(self, batch: int, max_len: int, dtype=None, device=None) -> LayerStateCache:
        dtype, device = dtype or self.embed.dtype, device or self.embed.device
        return LayerStateCache(batch, max_len, device, [self.mixers[i].state(batch, max_len, dtype, device) for i, _ in self.runs])

    def hidden_states(self, input_ids: torch.Tensor, cache: LayerStateCache, collect: Optional[List[torch.Tensor]] = None) -> torch.Tensor:
        """Runs the tokens [B, L] that follow what ``cache`` holds -> normed hidden states [B * L, padded width].  ``collect`` receives the
        residual stream [B, L, width] after every layer run."""
        B, L = input_ids.shape
        on_device = cache.device_lengths is not None and L == 1   # graph-replayed (or pool) decode: positions live on the device
        if not on_device and cache.length + L > cache.max_len:
            raise RuntimeError(f"cache overflow: {cache.length}+{L} > {cache.max_len}")
        for rope in self._ropes.values():
            rope.ensure(cache.max_len, self.embed.device)
        if on_device:
            step = Step(B, 1, 0, cache.device_lengths, cache.device_active)
        elif L == 1:
            step = Step(B, 1, cache.length, torch.full((B,), cache.length, dtype=torch.int32, device=self.embed.device))
        else:
            step = Step(B, L, cache.length)
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
        if not on_device:
            cache.advance(L)
        return h

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
        return logits.view(B, n, -1)[..., :self.config.vocab_size]

    # -- statistics ---------------------------------------------------------------------------------------------
    def num_parameters(self, trainable_only: bool = False) -> int:
        n = 0
        for shape in self.tensor_shapes().values():
            k = 1
            for d in shape:
                k *= d
            n += k
        return 0 if trainable_only else n
