"""Sequence mixers and feed-forwards of models whose layers are listed one by one (``vimodra.py``, ``nemipel.py``).

A mixer turns the normed input of its sublayer into the input of its output projection; the projection itself, the output norm and
the residual add are one fused step of the block (``ops/dyt.py``, ``ops/postnorm.py``), so a mixer only exposes the projection's weight as ``w_o``.  Every
mixer declares what it keeps per sequence (:meth:`state`) and runs in two modes chosen by the :class:`Step`: a portion of L tokens at
a position known on the host, or one token per sequence at positions in device memory.

Weights are stored as the kernels read them: projections of the same input stacked into one matrix, rows and columns padded with
zeros to multiples of 8 (a padded column of an activation is zero as well).  Small vectors are fp32.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Callable, Dict, List, Optional, Tuple

import torch
import torch.nn as nn

from .. import ops
from ..ops import delta as delta_ops
from ..ops import dyt as dyt_ops
from ..ops import gemm as G
from ..ops import gqa as gqa_ops
from ..ops import latent as latent_ops
from ..ops import lightning as lightning_ops
from ..ops import postnorm as pn
from ..ops.latent import pad8

Take = Callable[[str], torch.Tensor]   # tensor name inside the layer -> tensor
Shapes = Dict[str, Tuple[int, ...]]


@dataclass
class Step:
    """Where the tokens of a call belong: ``pos0`` for portions, ``lengths`` (int32 [B], device) for single tokens."""
    B: int
    L: int
    pos0: int
    lengths: Optional[torch.Tensor] = None
    active: Optional[torch.Tensor] = None
    on_device: bool = False   # positions live on the device only (pool rows, replayed graphs): the host's fill level stays as it is


def padded(w: torch.Tensor, rows: int, cols: int, dtype, device) -> torch.Tensor:
    out = torch.zeros(rows, cols, dtype=dtype, device=device)
    out[:w.shape[0], :w.shape[1]] = w.to(device=device, dtype=dtype)
    return out


def stacked(parts: List[Tuple[torch.Tensor, int]], cols: int, dtype, device) -> torch.Tensor:
    """[(matrix, row at which it starts)] -> one matrix (its height is the padded end of the last part)."""
    last, at = parts[-1]
    out = torch.zeros(pad8(at + last.shape[0]), cols, dtype=dtype, device=device)
    for w, at in parts:
        out[at:at + w.shape[0], :w.shape[1]] = w.to(device=device, dtype=dtype)
    return out


def vector(v: torch.Tensor, device, size: int = 0) -> torch.Tensor:
    out = torch.zeros(max(size, v.numel()), dtype=torch.float32, device=device)
    out[:v.numel()] = v.reshape(-1).to(device=device, dtype=torch.float32)
    return out


class _Weights(nn.Module):
    """A module whose weights arrive from a model folder (inference only)."""

    def put(self, name: str, t: torch.Tensor) -> None:
        self.register_parameter(name, nn.Parameter(t, requires_grad=False))


class LatentAttention(_Weights):
    """Sliding-window attention whose keys and values are expanded from one normed latent per token, with an output gate."""

    def __init__(self, spec: Dict[str, Any], width: int, eps: float, rope: nn.Module):
        super().__init__()
        window = (spec.get("mask") or {}).get("size") or 1 << 30
        self.s = latent_ops.LatentShape(spec["heads"], spec["dim"], spec["rot_dim"], spec["vdim"], spec["kv_rank"], spec["q_rank"], int(window),
                                        float(spec["scale"]), eps)
        self.width = width
        self._rope = [rope]   # shared between layers: not a submodule of each

    def shapes(self) -> Shapes:
        s, D = self.s, self.width
        return {"dq": (s.q_rank, D), "dq.norm": (s.q_rank,), "uq": (s.heads * (s.dim + s.rot), s.q_rank), "dkv": (s.cw, D), "dkv.norm": (s.rank,),
                "uk": (s.heads * s.dim, s.rank), "uv": (s.heads * s.vdim, s.rank), "g": (s.heads * s.vdim, D), "o": (D, s.heads * s.vdim)}

    def load(self, take: Take, dtype, device) -> None:
        s, Dp = self.s, pad8(self.width)
        self.put("w_in", stacked([(take("dq"), 0), (take("dkv"), s.kv_col), (take("g"), s.g_col)], Dp, dtype, device))
        self.put("w_uq", padded(take("uq"), s.q_width, s.q_pad, dtype, device))
        uk, uv = take("uk"), take("uv")
        self.put("w_ukv", stacked([(uk, 0), (uv, s.v_col)], pad8(s.rank), dtype, device))
        # decoding multiplies by the value expansion the other way round: [head, rank, vdim]
        uvt = torch.zeros(s.heads, s.rank, pad8(s.vdim), dtype=dtype, device=device)
        uvt[..., :s.vdim] = uv.to(device=device, dtype=dtype).view(s.heads, s.vdim, s.rank).transpose(1, 2)
        self.put("w_uvt", uvt)
        self.w_ukt = None   # key expansion transposed per head, for the tensor-core decode kernels
        if torch.device(device).type == "cuda" and latent_ops.decode_mma_ok(s, dtype):
            self.put("w_ukt_", uk.to(device=device, dtype=dtype).view(s.heads, s.dim, s.rank).transpose(1, 2).contiguous())
            self.w_ukt = self.w_ukt_
        self.put("w_o", padded(take("o"), Dp, s.o_pad, dtype, device))
        self.put("q_norm", vector(take("dq.norm"), device))
        self.put("kv_norm", vector(take("dkv.norm"), device))

    def state(self, batch: int, max_len: int, dtype, device) -> Dict[str, torch.Tensor]:
        return {"ring": torch.zeros(batch, min(self.s.window, max_len), self.s.cwp, dtype=dtype, device=device)}

    def attend_token(self, q: torch.Tensor, ring: torch.Tensor, gate: torch.Tensor, lengths: torch.Tensor) -> torch.Tensor:
        s, rope = self.s, self._rope[0]
        return latent_ops.latent_decode(q, ring, self.w_ukv[:s.heads * s.dim], self.w_uvt, gate, s, rope.cos, rope.sin, lengths, self.w_ukt,
                                        self.w_ukv[s.v_col:])

    def forward(self, h: torch.Tensor, st: Dict[str, torch.Tensor], step: Step) -> torch.Tensor:
        s, rope, ring = self.s, self._rope[0], st["ring"]
        proj = ops.linear(h, self.w_in).view(step.B, step.L, -1)
        gate = proj.view(step.B * step.L, -1)[:, s.g_col:]
        if step.lengths is not None:
            cq, _, _ = latent_ops.latent_context(proj, s, self.q_norm, self.kv_norm, rope.cos, rope.sin, ring, lengths=step.lengths, active=step.active)
            q = ops.linear(cq, self.w_uq)
            return self.attend_token(q, ring, gate, step.lengths)
        cq, ctx, n_old = latent_ops.latent_context(proj, s, self.q_norm, self.kv_norm, rope.cos, rope.sin, ring, pos0=step.pos0)
        q = ops.linear(cq, self.w_uq)
        kv = ops.linear(ctx.view(-1, s.cwp)[:, :s.rank], self.w_ukv[:, :s.rank]).view(step.B, n_old + step.L, -1)
        latent_ops.latent_finish(q, ctx, ring, s, rope.cos, rope.sin, step.pos0, n_old, step.L)
        return latent_ops.window_attention(q, kv, ctx, gate, s, n_old)


class GatedDelta(_Weights):
    """Gated delta rule with short convolutions and a gated output norm."""

    def __init__(self, spec: Dict[str, Any], width: int, eps: float):
        super().__init__()
        self.s = delta_ops.DeltaShape(spec["heads"], spec["kv_heads"], spec["dim"], spec["vdim"], spec["conv"], eps)
        self.width = width

    def shapes(self) -> Shapes:
        s, D = self.s, self.width
        kd, vd = s.kv_heads * s.dim, s.heads * s.vdim
        return {"q": (kd, D), "q.conv": (kd, s.taps), "k": (kd, D), "k.conv": (kd, s.taps), "v": (vd, D), "v.conv": (vd, s.taps), "b": (s.heads, D),
                "A_log": (s.heads,), "norm": (s.vdim,), "a": (s.heads, D), "dt_bias": (s.heads,), "g": (vd, D), "o": (D, vd)}

    def load(self, take: Take, dtype, device) -> None:
        s, Dp = self.s, pad8(self.width)
        kd = s.kv_heads * s.dim
        self.put("w_in", stacked([(take("q"), 0), (take("k"), kd), (take("v"), 2 * kd), (take("g"), s.g_col), (take("a"), s.a_col), (take("b"), s.b_col)], Dp,
                                 dtype, device))
        self.put("w_o", padded(take("o"), Dp, s.o_pad, dtype, device))
        self.put("conv", torch.cat([take(n + ".conv") for n in "qkv"]).T.to(device=device, dtype=torch.float32).contiguous())
        self.put("neg_rate", -torch.exp(vector(take("A_log"), device)))
        self.put("dt_bias", vector(take("dt_bias"), device))
        self.put("norm", vector(take("norm"), device))

    def state(self, batch: int, max_len: int, dtype, device) -> Dict[str, torch.Tensor]:
        s = self.s
        return {"S": torch.zeros(batch, s.heads, s.dim, s.vdim, dtype=torch.float32, device=device),
                "tail": torch.zeros(batch, s.taps - 1, s.channels, dtype=dtype, device=device)}

    def forward(self, h: torch.Tensor, st: Dict[str, torch.Tensor], step: Step) -> torch.Tensor:
        s = self.s
        proj = ops.linear(h, self.w_in).view(step.B, step.L, -1)
        gate = proj.view(step.B * step.L, -1)[:, s.g_col:]
        mixed, rlen, gb = delta_ops.delta_prep(proj, s, self.conv, self.neg_rate, self.dt_bias, st["tail"], step.pos0, step.lengths, step.active)
        if step.lengths is not None:
            return delta_ops.delta_step(mixed, rlen, gb, st["S"], gate, self.norm, s, step.lengths, step.active)
        o = delta_ops.delta_scan(mixed, rlen, gb, st["S"], s, step.L, fresh=step.pos0 == 0)
        return delta_ops.delta_output(o, gate, self.norm, s)


class GeluMLP(_Weights):
    """down(gelu_tanh(up(h) + b)); the down projection and its bias belong to the block's residual step."""

    def __init__(self, spec: Dict[str, Any], width: int):
        super().__init__()
        self.ff, self.width = int(spec["ff"]), width

    def shapes(self) -> Shapes:
        return {"up": (self.ff, self.width), "up.b": (self.ff,), "down": (self.width, self.ff), "down.b": (self.width,)}

    def load(self, take: Take, dtype, device) -> None:
        Dp, fp = pad8(self.width), pad8(self.ff)
        self.put("w_up", padded(take("up"), fp, Dp, dtype, device))
        self.put("b_up", vector(take("up.b"), device, fp))
        self.put("w_down", padded(take("down"), Dp, fp, dtype, device))
        self.put("b_down", vector(take("down.b"), device, Dp))

    def forward(self, h: torch.Tensor) -> torch.Tensor:
        return dyt_ops.linear_gelu(h, self.w_up, self.b_up)


class LightningAttention(_Weights):
    """Linear attention with one constant decay per head on activated queries, keys and values; the heads are normed together and gated."""

    def __init__(self, spec: Dict[str, Any], width: int, eps: float):
        super().__init__()
        self.s = lightning_ops.LightningShape(spec["heads"], spec["dim"], spec["vdim"], tuple(float(x) for x in spec["decay"]), eps)
        self.width = width

    def shapes(self) -> Shapes:
        s, D = self.s, self.width
        kd, vd = s.heads * s.dim, s.heads * s.vdim
        return {"q": (kd, D), "k": (kd, D), "v": (vd, D), "g": (vd, D), "o": (D, vd), "norm": (vd,)}

    def load(self, take: Take, dtype, device) -> None:
        s, Dp = self.s, pad8(self.width)
        self.put("w_in", stacked([(take("q"), 0), (take("k"), s.k_col), (take("v"), s.v_col), (take("g"), s.g_col)], Dp, dtype, device))
        self.put("w_o", padded(take("o"), Dp, s.o_pad, dtype, device))
        self.put("norm", vector(take("norm"), device))
        self.put("powers", lightning_ops.decay_powers(s, device))
        self.put("decay", self.powers[:, 1].contiguous())

    def state(self, batch: int, max_len: int, dtype, device) -> Dict[str, torch.Tensor]:
        s = self.s
        return {"S": torch.zeros(batch, s.heads, s.dim, s.vdim, dtype=torch.float32, device=device)}

    def forward(self, h: torch.Tensor, st: Dict[str, torch.Tensor], step: Step) -> torch.Tensor:
        s = self.s
        proj = pn.linear_silu(h, self.w_in, s.g_col)
        if step.lengths is not None:
            o = lightning_ops.lightning_step(proj, st["S"], self.decay, s, step.lengths, step.active)
        else:
            o = lightning_ops.lightning_scan(proj, st["S"], self.powers, s, step.L, fresh=step.pos0 == 0)
        return pn.norm_gate(o, proj[:, s.g_col:], self.norm, s.eps, s.o_pad)


class CappedAttention(_Weights):
    """Causal grouped-query attention with queries and keys normed over all heads together, partial interleaved rotation, capped scores
    and one output gate per head.  With ``kv_from`` it reads the keys and values that another layer's cache holds."""

    def __init__(self, spec: Dict[str, Any], width: int, eps: float, rope: nn.Module):
        super().__init__()
        self.s = gqa_ops.GqaShape(spec["heads"], spec["kv_heads"], spec["dim"], spec["vdim"], spec["rot"]["dims"], float(spec["scale"]), float(spec.get("softcap") or 0.0),
                                  eps, own_kv=spec.get("kv_from") is None)
        self.width = width
        self._rope = [rope]   # shared between layers: not a submodule of each

    def shapes(self) -> Shapes:
        s, D = self.s, self.width
        own = {"k": (s.kv_heads * s.dim, D), "v": (s.kv_heads * s.vdim, D), "k.norm": (s.kv_heads * s.dim,)} if s.own_kv else {}
        return {"q": (s.heads * s.dim, D), "q.norm": (s.heads * s.dim,), **own, "g": (s.heads, D), "o": (D, s.heads * s.vdim)}

    def load(self, take: Take, dtype, device) -> None:
        s, Dp = self.s, pad8(self.width)
        own = [(take("k"), s.k_col), (take("v"), s.v_col)] if s.own_kv else []
        self.put("w_in", stacked([(take("q"), 0)] + own + [(take("g"), s.g_col)], Dp, dtype, device))
        self.put("w_o", padded(take("o"), Dp, s.o_pad, dtype, device))
        self.put("q_norm", vector(take("q.norm"), device))
        self.k_norm = None
        if s.own_kv:
            self.put("k_norm_", vector(take("k.norm"), device))
            self.k_norm = self.k_norm_

    def state(self, batch: int, max_len: int, dtype, device) -> Dict[str, torch.Tensor]:
        s = self.s
        return {"k": torch.zeros(batch, max_len, s.k_pad, dtype=dtype, device=device), "v": torch.zeros(batch, max_len, s.v_pad, dtype=dtype, device=device)}

    def forward(self, h: torch.Tensor, st: Dict[str, torch.Tensor], step: Step) -> torch.Tensor:
        s, rope = self.s, self._rope[0]
        proj = ops.linear(h, self.w_in).view(step.B, step.L, -1)
        gate = proj.view(step.B * step.L, -1)[:, s.g_col:]
        q = gqa_ops.gqa_prepare(proj, s, self.q_norm, self.k_norm, rope.cos, rope.sin, st["k"], st["v"], step.pos0, step.lengths, step.active)
        if step.lengths is not None:
            return gqa_ops.gqa_decode(q, st["k"], st["v"], gate, s, step.lengths)
        return gqa_ops.gqa_portion(q, st["k"], st["v"], gate, s, step.L, step.pos0)


class ChannelDelta(_Weights):
    """Gated delta rule with one decay per state row and a sigmoid output gate, both behind low-rank projections."""

    def __init__(self, spec: Dict[str, Any], width: int, eps: float):
        super().__init__()
        self.s = delta_ops.ChannelDeltaShape(spec["heads"], spec["kv_heads"], spec["dim"], spec["vdim"], spec["conv"], eps, int(spec["decay_rank"]),
                                             int(spec["gate_rank"]))
        self.width = width

    def shapes(self) -> Shapes:
        s, D = self.s, self.width
        kd, vd = s.kv_heads * s.dim, s.heads * s.vdim
        return {"q": (kd, D), "q.conv": (kd, s.taps), "k": (kd, D), "k.conv": (kd, s.taps), "v": (vd, D), "v.conv": (vd, s.taps), "b": (s.heads, D),
                "A_log": (s.heads,), "norm": (s.vdim,), "a1": (s.decay_rank, D), "a2": (s.heads * s.dim, s.decay_rank), "dt_bias": (s.heads * s.dim,),
                "g1": (s.gate_rank, D), "g2": (vd, s.gate_rank), "o": (D, vd)}

    def load(self, take: Take, dtype, device) -> None:
        s, Dp = self.s, pad8(self.width)
        kd = s.kv_heads * s.dim
        self.put("w_in", stacked([(take("q"), 0), (take("k"), kd), (take("v"), 2 * kd), (take("a1"), s.low_col), (take("g1"), s.low_col + s.g_low), (take("b"), s.b_col)],
                                 Dp, dtype, device))
        # both second products as one: [decay input | gate input] times a block-diagonal matrix
        low = torch.zeros(s.g_col + s.o_pad, s.low_width, dtype=dtype, device=device)
        low[:s.heads * s.dim, :s.decay_rank] = take("a2").to(device=device, dtype=dtype)
        low[s.g_col:s.g_col + s.heads * s.vdim, s.g_low:s.g_low + s.gate_rank] = take("g2").to(device=device, dtype=dtype)
        self.put("w_low", low)
        self.put("w_o", padded(take("o"), Dp, s.o_pad, dtype, device))
        self.put("conv", torch.cat([take(n + ".conv") for n in "qkv"]).T.to(device=device, dtype=torch.float32).contiguous())
        self.put("neg_rate", -torch.exp(vector(take("A_log"), device)))
        self.put("dt_bias", vector(take("dt_bias"), device))
        self.put("norm", vector(take("norm"), device))

    def state(self, batch: int, max_len: int, dtype, device) -> Dict[str, torch.Tensor]:
        s = self.s
        return {"S": torch.zeros(batch, s.heads, s.dim, s.vdim, dtype=torch.float32, device=device),
                "tail": torch.zeros(batch, s.taps - 1, s.channels, dtype=dtype, device=device)}

    def forward(self, h: torch.Tensor, st: Dict[str, torch.Tensor], step: Step) -> torch.Tensor:
        s = self.s
        proj = ops.linear(h, self.w_in)
        wide = ops.linear(proj[:, s.low_col:s.low_col + s.low_width], self.w_low)
        mixed, rlen, gb = delta_ops.delta_prep(proj.view(step.B, step.L, -1), s, self.conv, None, None, st["tail"], step.pos0, step.lengths, step.active)
        if step.lengths is not None:
            return delta_ops.delta_step(mixed, rlen, gb, st["S"], wide[:, s.g_col:], self.norm, s, step.lengths, step.active, wide, self.neg_rate, self.dt_bias)
        o = delta_ops.channel_delta_scan(mixed, rlen, gb, wide, self.neg_rate, self.dt_bias, st["S"], s, step.L, fresh=step.pos0 == 0)
        return delta_ops.delta_output(o, wide[:, s.g_col:], self.norm, s)


class SwigluMLP(_Weights):
    """down(silu(gate(h)) * up(h)); the down projection belongs to the block's residual step."""

    def __init__(self, spec: Dict[str, Any], width: int):
        super().__init__()
        self.ff, self.width = int(spec["ff"]), width

    def shapes(self) -> Shapes:
        return {"gate": (self.ff, self.width), "up": (self.ff, self.width), "down": (self.width, self.ff)}

    def load(self, take: Take, dtype, device) -> None:
        Dp, fp = pad8(self.width), pad8(self.ff)
        self.put("w_gate_up", torch.cat([padded(take("gate"), fp, Dp, dtype, device), padded(take("up"), fp, Dp, dtype, device)]))
        self.put("w_down", padded(take("down"), Dp, fp, dtype, device))

    def forward(self, h: torch.Tensor) -> torch.Tensor:
        return G.gemm_nt_swiglu(h, self.w_gate_up)
