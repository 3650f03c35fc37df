"""Grouped-query attention over a full key / value cache with normed queries and keys, partial interleaved rotation, capped scores and
one output gate per head (``csrc/gqa_attention.cu``, ``csrc/gqa_attention_tcgen05.cu``, ``decode_attn_mma_kernel`` of ``csrc/inference.cu``).

``GqaShape`` carries every size and constant.  :func:`gqa_prepare` norms and rotates queries and keys and appends keys and values to the
cache (queries only for a layer that reads another layer's cache); :func:`gqa_portion` attends for portions of a prompt, :func:`gqa_decode`
for one token per sequence.  CPU tensors run the PyTorch definitions below.
"""
from __future__ import annotations

import ctypes
import os
from dataclasses import dataclass
from typing import Optional

import torch

from . import _lib
from .latent import _call, _p, pad8
from .postnorm import rms

_vp, _ci, _cll, _cf = ctypes.c_void_p, ctypes.c_int, ctypes.c_longlong, ctypes.c_float
# ATS_GQA_TC=0: portions and decode steps use the general kernels for every shape (for comparison)
TENSOR_CORES = os.environ.get("ATS_GQA_TC", "1") == "1"


@dataclass(frozen=True)
class GqaShape:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    rot: int          # the first rot dimensions of a head are rotated, 2 i with 2 i + 1
    scale: float
    cap: float        # 0: scores are not capped
    eps: float
    own_kv: bool = True   # False: keys and values come from another layer's cache

    # columns of the input projection [q | k | v | gate] (no k and v without keys of its own), every part padded to a multiple of 8
    @property
    def q_pad(self) -> int:
        return pad8(self.heads * self.dim)

    @property
    def k_pad(self) -> int:
        return pad8(self.kv_heads * self.dim)

    @property
    def v_pad(self) -> int:
        return pad8(self.kv_heads * self.vdim)

    @property
    def o_pad(self) -> int:
        return pad8(self.heads * self.vdim)

    @property
    def k_col(self) -> int:
        return self.q_pad

    @property
    def v_col(self) -> int:
        return self.q_pad + self.k_pad

    @property
    def g_col(self) -> int:
        return self.q_pad + (self.k_pad + self.v_pad if self.own_kv else 0)

    @property
    def proj_width(self) -> int:
        return self.g_col + pad8(self.heads)


class _Prep(ctypes.Structure):
    _fields_ = [("proj", _vp), ("ld", _cll), ("k_col", _ci), ("v_col", _ci), ("q_w", _vp), ("k_w", _vp), ("eps", _cf), ("cos", _vp), ("sin", _vp), ("dims", _ci),
                ("q", _vp), ("ldq", _cll), ("k", _vp), ("v", _vp), ("k_bs", _cll), ("v_bs", _cll), ("ldk", _cll), ("ldv", _cll), ("B", _ci), ("L", _ci), ("H", _ci),
                ("G", _ci), ("dim", _ci), ("vdim", _ci), ("max_len", _ci), ("pos0", _ci), ("lengths", _vp), ("active", _vp)]


class _Attn(ctypes.Structure):
    _fields_ = [("q", _vp), ("ldq", _cll), ("k", _vp), ("v", _vp), ("k_bs", _cll), ("v_bs", _cll), ("ldk", _cll), ("ldv", _cll), ("gate", _vp), ("ldg", _cll),
                ("out", _vp), ("ldo", _cll), ("B", _ci), ("L", _ci), ("H", _ci), ("G", _ci), ("dim", _ci), ("vdim", _ci), ("pos0", _ci), ("max_len", _ci),
                ("scale", _cf), ("cap", _cf), ("lengths", _vp), ("chunk", _ci), ("n_chunks", _ci), ("part_o", _vp), ("part_ml", _vp)]


# ----------------------------------------------------------------------------------------------------------
# PyTorch definitions
# ----------------------------------------------------------------------------------------------------------
def _rotate_pairs(x: torch.Tensor, cos: torch.Tensor, sin: torch.Tensor, rot: int) -> torch.Tensor:
    """x [rows, heads, dim] fp32, cos / sin [rows, rot / 2]."""
    u, v, c, s = x[..., 0:rot:2], x[..., 1:rot:2], cos[:, None], sin[:, None]
    turned = torch.stack([u * c - v * s, v * c + u * s], dim=-1).flatten(-2)
    return torch.cat([turned, x[..., rot:]], dim=-1)


def _attend(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, first: int, s: GqaShape) -> torch.Tensor:
    """One sequence: q [L, H, dim] at positions first .., k [rows, G, dim], v [rows, G, vdim] -> [L, H, vdim]."""
    rep = s.heads // s.kv_heads
    sc = torch.einsum("lhd,khd->hlk", q.float(), k.float().repeat_interleave(rep, 1)) * s.scale
    if s.cap:
        sc = s.cap * torch.tanh(sc / s.cap)
    seen = torch.arange(k.shape[0])[None, :] <= torch.arange(first, first + q.shape[0])[:, None]
    return torch.einsum("hlk,khd->lhd", torch.softmax(sc.masked_fill(~seen, float("-inf")), -1), v.float().repeat_interleave(rep, 1))


def _gated(o: torch.Tensor, gate: Optional[torch.Tensor], s: GqaShape, out: torch.Tensor) -> None:
    if gate is not None:
        o = o * torch.sigmoid(gate[:, :s.heads].float())[..., None]
    out[:, :s.heads * s.vdim] = o.reshape(o.shape[0], -1).to(out.dtype)


# ----------------------------------------------------------------------------------------------------------
# operators
# ----------------------------------------------------------------------------------------------------------
def gqa_prepare(proj: torch.Tensor, s: GqaShape, q_w: torch.Tensor, k_w: Optional[torch.Tensor], cos: torch.Tensor, sin: torch.Tensor, k: torch.Tensor,
                v: torch.Tensor, pos0: int = 0, lengths: Optional[torch.Tensor] = None, active: Optional[torch.Tensor] = None) -> torch.Tensor:
    """proj [B, L, proj_width] -> normed and rotated queries [B * L, q_pad]; with ``own_kv`` the keys and values go into the cache k [B,
    max_len, k_pad], v [B, max_len, v_pad] at the tokens' positions (``pos0`` .., or ``lengths`` with L == 1)."""
    B, L, _ = proj.shape
    H, Gk, max_len = s.heads, s.kv_heads, k.shape[1]
    if not proj.is_cuda:
        p2 = proj.reshape(B * L, -1)
        pos = lengths.long() if lengths is not None else torch.arange(pos0, pos0 + L).repeat(B)

        def part(x, w, n):
            x = rms(x.float(), s.eps, x.shape[-1]) * w
            return _rotate_pairs(x.view(B * L, n, s.dim), cos[pos], sin[pos], s.rot).reshape(B * L, -1).to(proj.dtype)
        q = torch.zeros(B * L, s.q_pad, dtype=proj.dtype)
        q[:, :H * s.dim] = part(p2[:, :H * s.dim], q_w, H)
        if s.own_kv:
            kn, vn = part(p2[:, s.k_col:s.k_col + Gk * s.dim], k_w, Gk), p2[:, s.v_col:s.v_col + Gk * s.vdim]
            for i in range(B * L):
                b, at = i // L, int(pos[i])
                if at < max_len and (active is None or int(active[b])):
                    k[b, at, :Gk * s.dim], v[b, at, :Gk * s.vdim] = kn[i], vn[i]
        return q
    assert proj.stride(2) == 1 and proj.stride(0) == L * proj.stride(1) and k.stride(2) == 1 and v.stride(2) == 1
    q = torch.empty(B * L, s.q_pad, dtype=proj.dtype, device=proj.device)
    a = _Prep(_p(proj), proj.stride(1), s.k_col if s.own_kv else -1, s.v_col, _p(q_w), _p(k_w), s.eps, _p(cos), _p(sin), s.rot, _p(q), q.stride(0), _p(k), _p(v),
              k.stride(0), v.stride(0), k.stride(1), v.stride(1), B, L, H, Gk, s.dim, s.vdim, max_len, pos0, _p(lengths), _p(active))
    _call("ats_gqa_prepare", a, proj)
    return q


def portion_tc_ok(q: torch.Tensor, s: GqaShape, L: int) -> bool:
    """The tensor-core kernel covers these sizes, and the portion fills more than a few rows of its query tiles."""
    return q.dtype == torch.bfloat16 and TENSOR_CORES and L >= 16 and s.dim % 8 == 0 and s.dim <= 128 and s.vdim % 8 == 0 and s.vdim <= 128 and s.scale > 0


def gqa_portion(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, gate: Optional[torch.Tensor], s: GqaShape, L: int, pos0: int) -> torch.Tensor:
    """Queries [B * L, q_pad] at positions pos0 .. against the cache (their own keys included), gate [B * L, .] (strided view, one column per
    head) -> gated outputs [B * L, o_pad]."""
    B, max_len = k.shape[:2]
    if not q.is_cuda:
        out, n = torch.zeros(B * L, s.o_pad, dtype=q.dtype), pos0 + L
        o = torch.cat([_attend(q[b * L:(b + 1) * L, :s.heads * s.dim].view(L, s.heads, s.dim), k[b, :n, :s.kv_heads * s.dim].view(n, s.kv_heads, s.dim),
                               v[b, :n, :s.kv_heads * s.vdim].view(n, s.kv_heads, s.vdim), pos0, s) for b in range(B)])
        _gated(o, gate, s, out)
        return out
    out = torch.empty(B * L, s.o_pad, dtype=q.dtype, device=q.device)
    ldg = 0 if gate is None else gate.stride(0)
    if portion_tc_ok(q, s, L) and (B == 1 or (k.stride(0) == max_len * k.stride(1) and v.stride(0) == max_len * v.stride(1))):
        f = _lib.cuda_lib().ats_gqa_attn_tc
        f.restype, f.argtypes = _ci, [_vp, _cll, _vp, _cll, _vp, _cll, _vp, _cll, _vp, _cll] + [_ci] * 8 + [_cf, _cf, _vp, _vp]
        _lib.check(f(_p(q), q.stride(0), _p(k), k.stride(1), _p(v), v.stride(1), _p(gate), ldg, _p(out), out.stride(0), B, L, pos0, max_len, s.heads, s.kv_heads, s.dim,
                     s.vdim, s.scale, s.cap, _p(_lib.status_tensor(q.device)), _lib.stream_ptr(q.device)), "ats_gqa_attn_tc")
        return out
    a = _Attn(_p(q), q.stride(0), _p(k), _p(v), k.stride(0), v.stride(0), k.stride(1), v.stride(1), _p(gate), ldg, _p(out), out.stride(0), B, L, s.heads, s.kv_heads,
              s.dim, s.vdim, pos0, max_len, s.scale, s.cap, 0, 0, 0, 0, 0)
    _call("ats_gqa_portion", a, q)
    return out


def decode_tc_ok(q: torch.Tensor, s: GqaShape, k: torch.Tensor, v: torch.Tensor) -> bool:
    """The warp-MMA decode kernel covers these sizes."""
    from . import serving
    return (q.shape[0] * s.kv_heads <= serving.MAX_COUNTERS and q.dtype == torch.bfloat16 and TENSOR_CORES and s.dim == s.vdim and s.dim in (64, 128) and s.heads // s.kv_heads in (1, 2, 4, 8)
            and k.stride(0) == v.stride(0))


def gqa_decode(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, gate: Optional[torch.Tensor], s: GqaShape, lengths: torch.Tensor) -> torch.Tensor:
    """One query per sequence [B, q_pad] at position ``lengths`` against the cache (its own key included) -> gated outputs [B, o_pad]."""
    B, max_len = k.shape[:2]
    H, dev = s.heads, q.device
    if not q.is_cuda:
        out = torch.zeros(B, s.o_pad, dtype=q.dtype)
        o = []
        for b in range(B):
            n = min(int(lengths[b]) + 1, max_len)
            o.append(_attend(q[b:b + 1, :H * s.dim].view(1, H, s.dim), k[b, :n, :s.kv_heads * s.dim].view(n, s.kv_heads, s.dim),
                             v[b, :n, :s.kv_heads * s.vdim].view(n, s.kv_heads, s.vdim), n - 1, s))
        _gated(torch.cat(o), gate, s, out)
        return out
    out = torch.empty(B, s.o_pad, dtype=q.dtype, device=dev)
    ldg = 0 if gate is None else gate.stride(0)
    if decode_tc_ok(q, s, k, v):
        from . import serving
        serving.decode_attention_cached(q, k, v, lengths, H, s.kv_heads, s.dim, s.scale, s.cap, gate, out)
        return out
    # chunks of 64 to 256 keys, as many as fill the SMs a few times over
    chunk = 64 if B * s.kv_heads * ((max_len + 63) // 64) <= 2048 else 256
    n_chunks = (max_len + chunk - 1) // chunk
    part_o = torch.empty(B, H, n_chunks, s.vdim, dtype=torch.float32, device=dev)
    part_ml = torch.empty(B, H, n_chunks, 2, dtype=torch.float32, device=dev)
    a = _Attn(_p(q), q.stride(0), _p(k), _p(v), k.stride(0), v.stride(0), k.stride(1), v.stride(1), _p(gate), ldg, _p(out), out.stride(0), B, 1, H, s.kv_heads, s.dim,
              s.vdim, 0, max_len, s.scale, s.cap, _p(lengths), chunk, n_chunks, _p(part_o), _p(part_ml))
    _call("ats_gqa_decode", a, q)
    return out
