"""Gated delta rule (``csrc/delta_rule.cu``, where the recurrence is written out).

``DeltaShape`` carries every size and constant.  :func:`delta_prep` (convolutions, activations, lengths, decays) feeds either
:func:`delta_scan` + :func:`delta_output` (portions of a prompt) or :func:`delta_step` (one decoded token per sequence).  The state
[B, heads, dim, vdim] is fp32 and is updated in place, as are the last inputs of the convolutions.  CPU tensors run the PyTorch
definitions below.
"""
from __future__ import annotations

import ctypes
from dataclasses import dataclass
from typing import Optional, Tuple

import torch

from . import _lib
from .latent import _call, _p, pad8

_vp, _ci, _cll, _cf = ctypes.c_void_p, ctypes.c_int, ctypes.c_longlong, ctypes.c_float
GROUP = 8  # tokens the portion kernel advances at a time


@dataclass(frozen=True)
class DeltaShape:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    taps: int
    eps: float

    # columns of the input projection [q | k | v | gate | a | b]; q, k, v are contiguous, the other parts start at multiples of 8
    @property
    def channels(self) -> int:
        return 2 * self.kv_heads * self.dim + self.heads * self.vdim

    @property
    def g_col(self) -> int:
        return pad8(self.channels)

    @property
    def o_pad(self) -> int:
        return pad8(self.heads * self.vdim)

    @property
    def a_col(self) -> int:
        return self.g_col + self.o_pad

    @property
    def b_col(self) -> int:
        return self.a_col + pad8(self.heads)

    @property
    def proj_width(self) -> int:
        return self.b_col + pad8(self.heads)


@dataclass(frozen=True)
class ChannelDeltaShape(DeltaShape):
    """One decay per state row, and a sigmoid output gate, both behind low-rank projections: the input projection is [q | k | v | decay
    input | gate input | b], and a second product expands [decay input | gate input] to [decays | gate]."""
    decay_rank: int = 8
    gate_rank: int = 8

    @property
    def low_col(self) -> int:      # of the low-rank inputs in the input projection
        return pad8(self.channels)

    @property
    def g_low(self) -> int:        # of the gate's part inside them
        return pad8(self.decay_rank)

    @property
    def low_width(self) -> int:
        return self.g_low + pad8(self.gate_rank)

    @property
    def b_col(self) -> int:
        return self.low_col + self.low_width

    @property
    def g_col(self) -> int:        # of the gate in the second product (the decays start at 0)
        return pad8(self.heads * self.dim)

    @property
    def scan_rows(self) -> int:    # state rows the portion kernel is built for
        return 64 if self.dim <= 64 else 128 if self.dim <= 128 else 256


class _Prep(ctypes.Structure):
    _fields_ = [("proj", _vp), ("ld", _cll), ("g_col", _ci), ("a_col", _ci), ("b_col", _ci), ("B", _ci), ("L", _ci), ("H", _ci), ("KH", _ci), ("dim", _ci),
                ("vdim", _ci), ("taps", _ci), ("C", _ci), ("conv", _vp), ("neg_rate", _vp), ("dt_bias", _vp), ("tail", _vp), ("tail_bs", _cll), ("pos0", _ci),
                ("lengths", _vp), ("active", _vp), ("mixed", _vp), ("ldm", _cll), ("rlen", _vp), ("gb", _vp)]


class _Scan(ctypes.Structure):
    _fields_ = [("mixed", _vp), ("ldm", _cll), ("rlen", _vp), ("gb", _vp), ("coef", _vp), ("state", _vp), ("state_bs", _cll), ("o", _vp), ("ldo", _cll), ("B", _ci),
                ("L", _ci), ("H", _ci), ("KH", _ci), ("dim", _ci), ("vdim", _ci), ("groups", _ci), ("fresh", _ci)]


class _Out(ctypes.Structure):
    _fields_ = [("o", _vp), ("ldo", _cll), ("gate", _vp), ("ldg", _cll), ("w", _vp), ("eps", _cf), ("out", _vp), ("ldout", _cll), ("rows", _cll), ("H", _ci),
                ("vdim", _ci), ("gate_sigmoid", _ci)]


class _Step(ctypes.Structure):
    _fields_ = [("mixed", _vp), ("ldm", _cll), ("rlen", _vp), ("gb", _vp), ("state", _vp), ("state_bs", _cll), ("lengths", _vp), ("active", _vp), ("gate", _vp),
                ("ldg", _cll), ("w", _vp), ("eps", _cf), ("out", _vp), ("ldout", _cll), ("B", _ci), ("H", _ci), ("KH", _ci), ("dim", _ci), ("vdim", _ci),
                ("gate_sigmoid", _ci), ("a", _vp), ("lda", _cll), ("neg_rate", _vp), ("dt_bias", _vp)]


class _Channel(ctypes.Structure):
    _fields_ = [("mixed", _vp), ("ldm", _cll), ("rlen", _vp), ("gb", _vp), ("a", _vp), ("lda", _cll), ("neg_rate", _vp), ("dt_bias", _vp), ("coef", _vp), ("state", _vp),
                ("state_bs", _cll), ("o", _vp), ("ldo", _cll), ("B", _ci), ("L", _ci), ("H", _ci), ("KH", _ci), ("dim", _ci), ("vdim", _ci), ("groups", _ci),
                ("fresh", _ci), ("DK", _ci)]


# ----------------------------------------------------------------------------------------------------------
# PyTorch definitions
# ----------------------------------------------------------------------------------------------------------
def _unit_qk(mixed: torch.Tensor, rlen: torch.Tensor, s: DeltaShape):
    rows, kd, rep = mixed.shape[0], s.kv_heads * s.dim, s.heads // s.kv_heads
    q = mixed[:, :kd].view(rows, s.kv_heads, s.dim).float() * rlen[:, :s.kv_heads, None]
    k = mixed[:, kd:2 * kd].view(rows, s.kv_heads, s.dim).float() * rlen[:, s.kv_heads:, None]
    v = mixed[:, 2 * kd:s.channels].view(rows, s.heads, s.vdim).float()
    return q.repeat_interleave(rep, 1), k.repeat_interleave(rep, 1), v


def _advance(S: torch.Tensor, q, k, v, g, beta):
    """One token of one sequence; S [H, dim, vdim] fp32, g [H] or [H, dim] -> (new S, read-out [H, vdim])."""
    S = S * (g[:, None, None] if g.dim() == 1 else g[:, :, None])
    u = beta[:, None] * (v - torch.einsum("hdv,hd->hv", S, k))
    S = S + k[:, :, None] * u[:, None, :]
    return S, torch.einsum("hdv,hd->hv", S, q)


def _norm_gate(o: torch.Tensor, gate: torch.Tensor, w: torch.Tensor, s: DeltaShape, out: torch.Tensor) -> None:
    rows = o.shape[0]
    o = o.float().view(rows, s.heads, s.vdim)
    o = o / torch.sqrt(o.pow(2).mean(-1, keepdim=True) + s.eps) * w
    act = torch.sigmoid if isinstance(s, ChannelDeltaShape) else torch.nn.functional.silu
    out[:, :s.heads * s.vdim] = (o.reshape(rows, -1) * act(gate[:, :s.heads * s.vdim].float())).to(out.dtype)


def _row_decays(a: torch.Tensor, neg_rate: torch.Tensor, dt_bias: torch.Tensor, s: ChannelDeltaShape) -> torch.Tensor:
    """a [rows, >= heads * dim] -> decays [rows, heads, dim]."""
    z = torch.nn.functional.softplus(a[:, :s.heads * s.dim].float() + dt_bias)
    return torch.exp(neg_rate[:, None] * z.view(-1, s.heads, s.dim))


# ----------------------------------------------------------------------------------------------------------
# operators
# ----------------------------------------------------------------------------------------------------------
def delta_prep(proj: torch.Tensor, s: DeltaShape, conv: torch.Tensor, neg_rate: Optional[torch.Tensor], dt_bias: Optional[torch.Tensor], tail: torch.Tensor,
               pos0: int = 0, lengths: Optional[torch.Tensor] = None, active: Optional[torch.Tensor] = None) -> Tuple[torch.Tensor, torch.Tensor, torch.Tensor]:
    """proj [B, L, proj_width]; with a :class:`ChannelDeltaShape` neg_rate and dt_bias are ``None`` and no decays are computed; conv [taps, channels] (last row: current token), neg_rate = -exp(A_log), dt_bias [H] in fp32; tail [B, taps - 1, channels] ->
    (mixed [B * L, .], reciprocal lengths [B * L, 2 kv_heads], [decay, step size] [B * L, 2 H]); the tail moves on by the portion."""
    B, L, _ = proj.shape
    H, KH, C, n = s.heads, s.kv_heads, s.channels, s.taps - 1
    if not proj.is_cuda:
        x = proj[..., :C]
        fresh = [(int(lengths[b]) if lengths is not None else pos0) == 0 for b in range(B)]
        old = torch.stack([torch.zeros_like(tail[b]) if fresh[b] else tail[b] for b in range(B)])
        full = torch.cat([old, x], dim=1)
        y = sum(full[:, j:j + L].float() * conv[j] for j in range(s.taps))
        mixed = torch.nn.functional.silu(y).to(proj.dtype).view(B * L, C)
        for b in range(B):
            if active is None or int(active[b]):
                tail[b] = full[b, L:]
        qk = mixed[:, :2 * KH * s.dim].view(B * L, 2 * KH, s.dim).float()
        rlen = 1 / torch.sqrt(qk.pow(2).sum(-1) + 1e-6)
        rlen[:, :KH] *= s.dim ** -0.5
        g = torch.zeros(B * L, H)
        if neg_rate is not None:
            g = torch.exp(neg_rate * torch.nn.functional.softplus(proj[..., s.a_col:s.a_col + H].float().reshape(B * L, H) + dt_bias))
        beta = torch.sigmoid(proj[..., s.b_col:s.b_col + H].float().reshape(B * L, H))
        return mixed, rlen, torch.cat([g, beta], dim=-1)
    assert proj.stride(2) == 1 and proj.stride(0) == L * proj.stride(1) and (n == 0 or tail.stride(1) == C)
    dev = proj.device
    mixed = torch.empty(B * L, pad8(C), dtype=proj.dtype, device=dev)
    rlen = torch.empty(B * L, 2 * KH, dtype=torch.float32, device=dev)
    gb = torch.empty(B * L, 2 * H, dtype=torch.float32, device=dev)
    _call("ats_delta_prep", _Prep(_p(proj), proj.stride(1), s.g_col, s.a_col, s.b_col, B, L, H, KH, s.dim, s.vdim, s.taps, C, _p(conv), _p(neg_rate), _p(dt_bias),
                                  _p(tail), tail.stride(0), pos0, _p(lengths), _p(active), _p(mixed), mixed.stride(0), _p(rlen), _p(gb)), proj)
    return mixed, rlen, gb


def delta_scan(mixed: torch.Tensor, rlen: torch.Tensor, gb: torch.Tensor, state: torch.Tensor, s: DeltaShape, L: int, fresh: bool) -> torch.Tensor:
    """Advances ``state`` [B, H, dim, vdim] over portions of L tokens -> read-outs [B * L, H * vdim]; ``fresh``: the state starts at zero."""
    B = state.shape[0]
    H, KH = s.heads, s.kv_heads
    if not mixed.is_cuda:
        q, k, v = _unit_qk(mixed, rlen, s)
        out = torch.empty(B * L, H * s.vdim, dtype=mixed.dtype)
        for b in range(B):
            S = torch.zeros_like(state[b]) if fresh else state[b]
            for t in range(b * L, (b + 1) * L):
                S, o = _advance(S, q[t], k[t], v[t], gb[t, :H], gb[t, H:])
                out[t] = o.reshape(-1).to(out.dtype)
            state[b] = S
        return out
    dev = mixed.device
    groups = (L + GROUP - 1) // GROUP
    coef = torch.empty(B, groups, H, 2 * GROUP * GROUP + 3 * GROUP + 8, dtype=torch.float32, device=dev)   # layout: csrc/delta_rule.cu
    o = torch.empty(B * L, H * s.vdim, dtype=mixed.dtype, device=dev)
    _call("ats_delta_scan", _Scan(_p(mixed), mixed.stride(0), _p(rlen), _p(gb), _p(coef), _p(state), state.stride(0), _p(o), o.stride(0), B, L, H, KH, s.dim, s.vdim,
                                  groups, int(fresh)), mixed)
    return o


def delta_output(o: torch.Tensor, gate: torch.Tensor, w: torch.Tensor, s: DeltaShape) -> torch.Tensor:
    """Output norm over vdim, weight, silu gate: o [rows, H * vdim], gate [rows, .] (strided view) -> [rows, o_pad]."""
    rows = o.shape[0]
    if not o.is_cuda:
        out = torch.zeros(rows, s.o_pad, dtype=o.dtype)
        _norm_gate(o, gate, w, s, out)
        return out
    out = torch.empty(rows, s.o_pad, dtype=o.dtype, device=o.device)
    _call("ats_delta_output", _Out(_p(o), o.stride(0), _p(gate), gate.stride(0), _p(w), s.eps, _p(out), out.stride(0), rows, s.heads, s.vdim,
                                    int(isinstance(s, ChannelDeltaShape))), o)
    return out


def delta_step(mixed: torch.Tensor, rlen: torch.Tensor, gb: torch.Tensor, state: torch.Tensor, gate: torch.Tensor, w: torch.Tensor, s: DeltaShape,
               lengths: torch.Tensor, active: Optional[torch.Tensor] = None, a: Optional[torch.Tensor] = None, neg_rate: Optional[torch.Tensor] = None,
               dt_bias: Optional[torch.Tensor] = None) -> torch.Tensor:
    """One token per sequence: state update, read-out, output norm and gate -> [B, o_pad].  With a :class:`ChannelDeltaShape` the decays
    come from their input ``a`` [B, >= heads * dim], neg_rate [heads] and dt_bias [heads * dim]."""
    B, H = state.shape[0], s.heads
    if not mixed.is_cuda:
        q, k, v = _unit_qk(mixed, rlen, s)
        out = torch.zeros(B, s.o_pad, dtype=mixed.dtype)
        o = torch.empty(B, H * s.vdim)
        decay = gb[:, :H] if a is None else _row_decays(a, neg_rate, dt_bias, s)
        for b in range(B):
            S = torch.zeros_like(state[b]) if int(lengths[b]) == 0 else state[b]
            S, r = _advance(S, q[b], k[b], v[b], decay[b], gb[b, H:])
            if active is None or int(active[b]):
                state[b] = S
            o[b] = r.reshape(-1)
        _norm_gate(o, gate, w, s, out)
        return out
    out = torch.empty(B, s.o_pad, dtype=mixed.dtype, device=mixed.device)
    _call("ats_delta_step", _Step(_p(mixed), mixed.stride(0), _p(rlen), _p(gb), _p(state), state.stride(0), _p(lengths), _p(active), _p(gate), gate.stride(0), _p(w),
                                  s.eps, _p(out), out.stride(0), B, H, s.kv_heads, s.dim, s.vdim, int(isinstance(s, ChannelDeltaShape)), _p(a),
                                  0 if a is None else a.stride(0), _p(neg_rate if a is not None else None), _p(dt_bias if a is not None else None)), mixed)
    return out


def channel_delta_scan(mixed: torch.Tensor, rlen: torch.Tensor, gb: torch.Tensor, a: torch.Tensor, neg_rate: torch.Tensor, dt_bias: torch.Tensor, state: torch.Tensor,
                       s: ChannelDeltaShape, L: int, fresh: bool) -> torch.Tensor:
    """:func:`delta_scan` with one decay per state row (``csrc/channel_delta.cu``): a [B * L, >= heads * dim] decay inputs."""
    B, H = state.shape[0], s.heads
    if not mixed.is_cuda:
        q, k, v = _unit_qk(mixed, rlen, s)
        g, out = _row_decays(a, neg_rate, dt_bias, s), torch.empty(B * L, H * s.vdim, dtype=mixed.dtype)
        for b in range(B):
            S = torch.zeros_like(state[b]) if fresh else state[b]
            for t in range(b * L, (b + 1) * L):
                S, o = _advance(S, q[t], k[t], v[t], g[t], gb[t, H:])
                out[t] = o.reshape(-1).to(out.dtype)
            state[b] = S
        return out
    groups, DK = (L + GROUP - 1) // GROUP, s.scan_rows
    coef = torch.empty(B, groups, H, 2 * GROUP * GROUP + (3 * GROUP + 1) * DK, dtype=torch.float32, device=mixed.device)   # layout: csrc/channel_delta.cu
    o = torch.empty(B * L, H * s.vdim, dtype=mixed.dtype, device=mixed.device)
    _call("ats_channel_delta", _Channel(_p(mixed), mixed.stride(0), _p(rlen), _p(gb), _p(a), a.stride(0), _p(neg_rate), _p(dt_bias), _p(coef), _p(state), state.stride(0),
                                        _p(o), o.stride(0), B, L, H, s.kv_heads, s.dim, s.vdim, groups, int(fresh), DK), mixed)
    return o
