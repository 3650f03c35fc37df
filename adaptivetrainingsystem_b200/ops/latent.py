"""Latent attention over a sliding window (``csrc/latent_attention.cu``; the cache layout is described there).

``LatentShape`` carries every size and constant.  Portions of a prompt: :func:`latent_context` -> expansion GEMM ->
:func:`latent_finish` -> :func:`window_attention`; one decoded token per sequence: :func:`latent_context` with ``lengths`` ->
:func:`latent_decode`.  CPU tensors run the PyTorch definitions below.
"""
from __future__ import annotations

import ctypes
import os
from dataclasses import dataclass
from typing import Optional, Tuple

import torch

from . import _lib

_vp, _ci, _cll, _cf = ctypes.c_void_p, ctypes.c_int, ctypes.c_longlong, ctypes.c_float


def pad8(n: int) -> int:
    return (n + 7) // 8 * 8


# ATS_WINDOW_TC=0: portions of a prompt use the general window kernel for every shape (for comparison)
WINDOW_TC = os.environ.get("ATS_WINDOW_TC", "1") == "1"
# ATS_LATENT_DECODE_MMA=0: decode steps use the general kernels for every shape (for comparison)
DECODE_MMA = os.environ.get("ATS_LATENT_DECODE_MMA", "1") == "1"


@dataclass(frozen=True)
class LatentShape:
    heads: int
    dim: int          # unrotated query / key dimensions per head
    rot: int          # rotated ones
    vdim: int
    rank: int         # latent of keys and values
    q_rank: int       # latent of queries
    window: int       # a token sees itself and the window - 1 tokens before it
    scale: float
    eps: float

    # columns of the input projection [query latent | latent, rotated key part | gate], every part padded to a multiple of 8
    @property
    def q_pad(self) -> int:
        return pad8(self.q_rank)

    @property
    def cw(self) -> int:
        return self.rank + self.rot

    @property
    def cwp(self) -> int:
        return pad8(self.cw)

    @property
    def o_pad(self) -> int:
        return pad8(self.heads * self.vdim)

    @property
    def kv_col(self) -> int:
        return self.q_pad

    @property
    def g_col(self) -> int:
        return self.q_pad + self.cwp

    @property
    def proj_width(self) -> int:
        return self.q_pad + self.cwp + self.o_pad

    @property
    def v_col(self) -> int:   # of the expanded keys and values
        return pad8(self.heads * self.dim)

    @property
    def kv_width(self) -> int:
        return self.v_col + self.o_pad

    @property
    def q_width(self) -> int:
        return pad8(self.heads * (self.dim + self.rot))


class _Context(ctypes.Structure):
    _fields_ = [("proj", _vp), ("ld", _cll), ("q_col", _ci), ("kv_col", _ci), ("q_rank", _ci), ("q_pad", _ci), ("rank", _ci), ("rot", _ci), ("cwp", _ci),
                ("q_w", _vp), ("kv_w", _vp), ("eps", _cf), ("cos", _vp), ("sin", _vp), ("cq", _vp), ("ctx", _vp), ("ring", _vp), ("ring_bs", _cll),
                ("B", _ci), ("L", _ci), ("R", _ci), ("n_old", _ci), ("pos0", _ci), ("lengths", _vp), ("active", _vp)]


class _Finish(ctypes.Structure):
    _fields_ = [("q", _vp), ("ldq", _cll), ("H", _ci), ("dim", _ci), ("rot", _ci), ("cos", _vp), ("sin", _vp), ("ctx", _vp), ("ring", _vp), ("ring_bs", _cll),
                ("cwp", _ci), ("B", _ci), ("L", _ci), ("R", _ci), ("n_old", _ci), ("pos0", _ci)]


class _Window(ctypes.Structure):
    _fields_ = [("q", _vp), ("ldq", _cll), ("kv", _vp), ("ldkv", _cll), ("v_col", _ci), ("kr", _vp), ("ldkr", _cll), ("gate", _vp), ("ldg", _cll), ("out", _vp),
                ("ldo", _cll), ("B", _ci), ("L", _ci), ("n_old", _ci), ("H", _ci), ("dim", _ci), ("rot", _ci), ("vdim", _ci), ("window", _ci), ("scale", _cf)]


class _Absorb(ctypes.Structure):
    _fields_ = [("q", _vp), ("ldq", _cll), ("wk", _vp), ("ldw", _cll), ("cos", _vp), ("sin", _vp), ("lengths", _vp), ("qa", _vp), ("B", _ci), ("H", _ci),
                ("dim", _ci), ("rot", _ci), ("rank", _ci), ("cwp", _ci)]


class _Decode(ctypes.Structure):
    _fields_ = [("qa", _vp), ("ring", _vp), ("ring_bs", _cll), ("lengths", _vp), ("B", _ci), ("H", _ci), ("R", _ci), ("rank", _ci), ("cw", _ci), ("cwp", _ci),
                ("chunk", _ci), ("n_chunks", _ci), ("scale", _cf), ("part_o", _vp), ("part_ml", _vp)]


class _Expand(ctypes.Structure):
    _fields_ = [("part_o", _vp), ("part_ml", _vp), ("wv", _vp), ("ldv", _ci), ("gate", _vp), ("ldg", _cll), ("out", _vp), ("ldo", _cll), ("B", _ci), ("H", _ci),
                ("rank", _ci), ("vdim", _ci), ("n_chunks", _ci)]


def _call(name: str, args: ctypes.Structure, like: torch.Tensor) -> None:
    f = getattr(_lib.cuda_lib(), name)
    f.restype, f.argtypes = _ci, [_vp, _ci, _vp]
    _lib.check(f(ctypes.byref(args), int(like.dtype == torch.float32), _lib.stream_ptr(like.device)), name)


def _p(t: Optional[torch.Tensor]) -> int:
    return 0 if t is None else t.data_ptr()


# ----------------------------------------------------------------------------------------------------------
# PyTorch definitions
# ----------------------------------------------------------------------------------------------------------
def _rms(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    x = x.float()
    return x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps) * w


def _rotate(x: torch.Tensor, cos: torch.Tensor, sin: torch.Tensor) -> torch.Tensor:
    """x [..., rot] with cos / sin broadcastable to [..., rot / 2]."""
    u, v = x.float().chunk(2, dim=-1)
    return torch.cat([u * cos - v * sin, v * cos + u * sin], dim=-1)


# ----------------------------------------------------------------------------------------------------------
# operators
# ----------------------------------------------------------------------------------------------------------
def latent_context(proj: torch.Tensor, s: LatentShape, q_w: torch.Tensor, kv_w: torch.Tensor, cos: torch.Tensor, sin: torch.Tensor, ring: torch.Tensor,
                   pos0: int = 0, lengths: Optional[torch.Tensor] = None, active: Optional[torch.Tensor] = None,
                   ) -> Tuple[torch.Tensor, Optional[torch.Tensor], int]:
    """proj [B, L, proj_width] -> (normed query latents [B * L, q_pad], context [B, n_old + L, cwp], n_old).

    The context holds the window before ``pos0`` (from the ring [B, R, cwp]) followed by the portion's own entries.  With
    ``lengths`` (L == 1, int32 [B]) the new entries go straight into the ring instead and there is no context."""
    B, L, ld = proj.shape
    R = ring.shape[1]
    n_old = 0 if lengths is not None else min(pos0, s.window - 1)
    if not proj.is_cuda:
        cq = torch.zeros(B, L, s.q_pad, dtype=proj.dtype)
        cq[..., :s.q_rank] = _rms(proj[..., :s.q_rank], q_w, s.eps).to(proj.dtype)
        pos = lengths.view(B, 1).long() if lengths is not None else torch.arange(pos0, pos0 + L).expand(B, L)
        new = torch.zeros(B, L, s.cwp, dtype=proj.dtype)
        new[..., :s.rank] = _rms(proj[..., s.kv_col:s.kv_col + s.rank], kv_w, s.eps).to(proj.dtype)
        new[..., s.rank:s.cw] = _rotate(proj[..., s.kv_col + s.rank:s.kv_col + s.cw], cos[pos], sin[pos]).to(proj.dtype)
        if lengths is not None:
            for b in range(B):
                if active is None or int(active[b]):
                    ring[b, int(lengths[b]) % R] = new[b, 0]
            return cq.view(B, s.q_pad), None, 0
        old = ring[:, [(pos0 - n_old + j) % R for j in range(n_old)]]
        return cq.view(B * L, s.q_pad), torch.cat([old, new], dim=1), n_old
    assert proj.stride(2) == 1 and proj.stride(0) == L * proj.stride(1) and ring.stride(2) == 1 and ring.stride(1) == s.cwp
    cq = torch.empty(B * L, s.q_pad, dtype=proj.dtype, device=proj.device)
    ctx = None if lengths is not None else torch.empty(B, n_old + L, s.cwp, dtype=proj.dtype, device=proj.device)
    a = _Context(_p(proj), proj.stride(1), 0, s.kv_col, s.q_rank, s.q_pad, s.rank, s.rot, s.cwp, _p(q_w), _p(kv_w), s.eps, _p(cos), _p(sin), _p(cq), _p(ctx),
                 _p(ring), ring.stride(0), B, L, R, n_old, pos0, _p(lengths), _p(active))
    _call("ats_latent_context", a, proj)
    return cq, ctx, n_old


def latent_finish(q: torch.Tensor, ctx: torch.Tensor, ring: torch.Tensor, s: LatentShape, cos: torch.Tensor, sin: torch.Tensor, pos0: int, n_old: int,
                  L: int) -> None:
    """Rotates the query heads of q [B * L, q_width] in place and stores the portion's last entries in the ring."""
    B, R = ring.shape[:2]
    if not q.is_cuda:
        dq = s.dim + s.rot
        qv = q[:, :s.heads * dq].view(B, L, s.heads, dq)
        pos = torch.arange(pos0, pos0 + L)
        qv[..., s.dim:] = _rotate(qv[..., s.dim:], cos[pos].unsqueeze(1), sin[pos].unsqueeze(1)).to(q.dtype)
        for t in range(max(0, L - R), L):
            ring[:, (pos0 + t) % R] = ctx[:, n_old + t]
        return
    a = _Finish(_p(q), q.stride(0), s.heads, s.dim, s.rot, _p(cos), _p(sin), _p(ctx), _p(ring), ring.stride(0), s.cwp, B, L, R, n_old, pos0)
    _call("ats_latent_finish", a, q)


def window_tc_ok(q: torch.Tensor, s: LatentShape, L: int) -> bool:
    """The tensor-core kernel covers these sizes, and the portion is long enough to fill more than a few rows of its query tiles."""
    return (q.dtype == torch.bfloat16 and WINDOW_TC and L >= 16 and s.dim in (64, 128) and s.rot % 8 == 0 and 8 <= s.rot <= 64 and s.vdim in (64, 128)
            and s.rank % 8 == 0 and s.scale > 0)


def window_attention(q: torch.Tensor, kv: torch.Tensor, ctx: torch.Tensor, gate: Optional[torch.Tensor], s: LatentShape, n_old: int) -> torch.Tensor:
    """q [B * L, q_width] (rotated), kv [B, n_old + L, kv_width], ctx [B, n_old + L, cwp] (its rotated key part is shared by the heads),
    gate [B * L, .] (strided view, heads x vdim) -> sigmoid-gated attention output [B * L, o_pad]."""
    B, rows = kv.shape[:2]
    L = rows - n_old
    H, dq = s.heads, s.dim + s.rot
    if not q.is_cuda:
        qf = q[:, :H * dq].view(B, L, H, dq).float()
        k = kv[..., :H * s.dim].reshape(B, rows, H, s.dim).float()
        v = kv[..., s.v_col:s.v_col + H * s.vdim].reshape(B, rows, H, s.vdim).float()
        kr = ctx[..., s.rank:s.cw].float()
        sc = (torch.einsum("blhd,bkhd->bhlk", qf[..., :s.dim], k) + torch.einsum("blhd,bkd->bhlk", qf[..., s.dim:], kr)) * s.scale
        d = (torch.arange(L) + n_old)[:, None] - torch.arange(rows)[None, :]
        sc = sc.masked_fill((d < 0) | (d >= s.window), float("-inf"))
        o = torch.einsum("bhlk,bkhd->blhd", torch.softmax(sc, -1), v).reshape(B * L, H * s.vdim)
        if gate is not None:
            o = o * torch.sigmoid(gate[:, :H * s.vdim].float())
        out = torch.zeros(B * L, s.o_pad, dtype=q.dtype)
        out[:, :H * s.vdim] = o.to(q.dtype)
        return out
    out = torch.empty(B * L, s.o_pad, dtype=q.dtype, device=q.device)
    kr = ctx[..., s.rank:]
    if window_tc_ok(q, s, L):
        f = _lib.cuda_lib().ats_window_attn_tc
        f.restype, f.argtypes = _ci, [_vp, _cll, _vp, _cll, _ci, _vp, _cll, _vp, _cll, _vp, _cll] + [_ci] * 8 + [_cf, _vp, _vp]
        _lib.check(f(_p(q), q.stride(0), _p(kv), kv.stride(1), s.v_col, _p(kr), ctx.stride(1), _p(gate), 0 if gate is None else gate.stride(0), _p(out), out.stride(0),
                     B, L, n_old, H, s.dim, s.rot, s.vdim, s.window, s.scale, _p(_lib.status_tensor(q.device)), _lib.stream_ptr(q.device)), "ats_window_attn_tc")
        return out
    a = _Window(_p(q), q.stride(0), _p(kv), kv.stride(1), s.v_col, _p(kr), ctx.stride(1), _p(gate), 0 if gate is None else gate.stride(0), _p(out), out.stride(0),
                B, L, n_old, H, s.dim, s.rot, s.vdim, s.window, s.scale)
    _call("ats_window_attn", a, q)
    return out


def decode_mma_ok(s: LatentShape, dtype: torch.dtype) -> bool:
    """The tensor-core decode kernels cover these sizes (the model then keeps the key expansion transposed per head)."""
    return (dtype == torch.bfloat16 and DECODE_MMA and s.rank in (128, 256, 384, 512) and s.dim % 32 == 0 and s.dim <= 512 and s.rot % 32 == 0 and 32 <= s.rot <= 128
            and s.vdim % 8 == 0)


def latent_decode(q: torch.Tensor, ring: torch.Tensor, w_uk: torch.Tensor, w_uv_t: torch.Tensor, gate: Optional[torch.Tensor], s: LatentShape,
                  cos: torch.Tensor, sin: torch.Tensor, lengths: torch.Tensor, w_ukt: Optional[torch.Tensor] = None,
                  w_uv: Optional[torch.Tensor] = None) -> torch.Tensor:
    """One query token per sequence against its ring (which already holds the token's own entry).  q [B, q_width] not yet rotated;
    w_uk [H * dim, >= rank], w_uv_t [H, rank, >= vdim] -> gated output [B, o_pad].  With w_ukt [H, rank, dim] and w_uv
    [H * vdim, >= rank] (shapes of :func:`decode_mma_ok`) everything runs on tensor cores."""
    B, R = ring.shape[:2]
    H, dq = s.heads, s.dim + s.rot
    if not q.is_cuda:
        out = torch.zeros(B, s.o_pad, dtype=q.dtype)
        for b in range(B):
            pos = int(lengths[b])
            qb = q[b, :H * dq].view(H, dq).float()
            qa = torch.einsum("hd,hdr->hr", qb[:, :s.dim], w_uk[:, :s.rank].view(H, s.dim, s.rank).float())
            qr = _rotate(qb[:, s.dim:], cos[pos], sin[pos])
            c = ring[b, :min(pos + 1, R)].float()
            sc = (qa @ c[:, :s.rank].T + qr @ c[:, s.rank:s.cw].T) * s.scale
            o = torch.einsum("hr,hrv->hv", torch.softmax(sc, -1) @ c[:, :s.rank], w_uv_t[..., :s.vdim].float()).reshape(-1)
            if gate is not None:
                o = o * torch.sigmoid(gate[b, :H * s.vdim].float())
            out[b, :H * s.vdim] = o.to(q.dtype)
        return out
    dev = q.device
    if w_ukt is not None and w_uv is not None and R <= 64 * 4096:
        # as many chunks per sequence as fit one wave of CTAs (two per SM for up to 16 heads, else one with 32 heads), of whole 64-row
        # pieces, at most 64
        slots, ctas = (296, B) if H <= 16 else (148, B * ((H + 31) // 32))
        n_chunks = max(1, min(64, (R + 63) // 64, slots // ctas))
        chunk = ((R + n_chunks - 1) // n_chunks + 63) // 64 * 64
        n_chunks = (R + chunk - 1) // chunk
        qa = torch.empty(B, H, s.rank, dtype=q.dtype, device=dev)
        part_o = torch.empty(B, H, n_chunks, s.rank, dtype=torch.float32, device=dev)
        part_ml = torch.empty(B, H, n_chunks, 2, dtype=torch.float32, device=dev)
        out = torch.empty(B, s.o_pad, dtype=q.dtype, device=dev)
        f = _lib.cuda_lib().ats_latent_decode_mma
        f.restype, f.argtypes = _ci, [_vp, _cll, _vp, _vp, _ci, _vp, _cll, _vp, _vp, _vp, _vp, _cll, _vp, _vp, _vp, _vp, _cll] + [_ci] * 10 + [_cf, _vp]
        _lib.check(f(_p(q), q.stride(0), _p(w_ukt), _p(w_uv), w_uv.stride(0), _p(ring), ring.stride(0), _p(lengths), _p(cos), _p(sin), _p(gate),
                     0 if gate is None else gate.stride(0), _p(qa), _p(part_o), _p(part_ml), _p(out), out.stride(0), B, H, s.dim, s.rot, s.rank, s.vdim, s.cwp, R,
                     chunk, n_chunks, s.scale, _lib.stream_ptr(dev)), "ats_latent_decode_mma")
        return out
    qa = torch.empty(B, H, s.cwp, dtype=q.dtype, device=dev)
    _call("ats_latent_absorb", _Absorb(_p(q), q.stride(0), _p(w_uk), w_uk.stride(0), _p(cos), _p(sin), _p(lengths), _p(qa), B, H, s.dim, s.rot, s.rank, s.cwp), q)
    chunk = 64
    n_chunks = (R + chunk - 1) // chunk
    part_o = torch.empty(B, H, n_chunks, s.rank, dtype=torch.float32, device=dev)
    part_ml = torch.empty(B, H, n_chunks, 2, dtype=torch.float32, device=dev)
    _call("ats_latent_decode", _Decode(_p(qa), _p(ring), ring.stride(0), _p(lengths), B, H, R, s.rank, s.cw, s.cwp, chunk, n_chunks, s.scale, _p(part_o),
                                       _p(part_ml)), q)
    out = torch.empty(B, s.o_pad, dtype=q.dtype, device=dev)
    _call("ats_latent_expand", _Expand(_p(part_o), _p(part_ml), _p(w_uv_t), w_uv_t.stride(1), _p(gate), 0 if gate is None else gate.stride(0), _p(out), out.stride(0),
                                       B, H, s.rank, s.vdim, n_chunks), q)
    return out
