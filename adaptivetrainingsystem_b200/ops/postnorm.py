"""Steps of blocks whose norm follows the residual sum (``csrc/postnorm.cu``), and the small row-wise steps that go with them.

    x <- rms(alpha x + y) w,     rms(z) = z / sqrt(mean(z^2) + eps)

The residual ``x`` is fp32 whatever the element type of the products; padded columns of a row are zero and do not count in the mean.
CPU tensors run the PyTorch definitions.
"""
from __future__ import annotations

import ctypes
from dataclasses import dataclass
from typing import Optional, Tuple

import torch

from . import _lib
from . import dyt as _dyt
from . import gemm as G

_vp, _ci, _cll, _cf = ctypes.c_void_p, ctypes.c_int, ctypes.c_longlong, ctypes.c_float


class _PostNorm(ctypes.Structure):
    _fields_ = [("y", _vp), ("splits", _ci), ("split_stride", _cll), ("x", _vp), ("alpha", _cf), ("w", _vp), ("w2", _vp), ("eps", _cf), ("h", _vp), ("rows", _cll),
                ("N", _ci), ("width", _ci)]


class _NormGate(ctypes.Structure):
    _fields_ = [("o", _vp), ("ldo", _cll), ("gate", _vp), ("ldg", _cll), ("w", _vp), ("eps", _cf), ("out", _vp), ("ldout", _cll), ("rows", _cll), ("width", _ci),
                ("vec", _ci)]


_sig = False


def _fns():
    global _sig
    lib = _lib.cuda_lib()
    if not _sig:
        for name, args in (("ats_embed_rows", [_vp, _vp, _ci, _ci, _vp, _vp, _cll, _ci, _vp]), ("ats_fold_postnorm", [_vp, _ci, _vp]),
                           ("ats_norm_gate", [_vp, _ci, _vp]), ("ats_fold_silu", [_vp, _ci, _cll, _vp, _ci, _cll, _ci, _ci, _vp]),
                           ("ats_softcap", [_vp, _cll, _cf, _ci, _vp])):
            f = getattr(lib, name)
            f.restype, f.argtypes = _ci, args
        _sig = True
    return lib


@dataclass
class PostNorm:
    """Constants of one residual step: norm weight ``w`` (fp32, zero in padded columns); ``w2``: weight of a second norm whose result is
    returned instead of ``x`` (the model's last norm)."""
    alpha: float
    w: torch.Tensor
    eps: float
    width: int
    w2: Optional[torch.Tensor] = None


def rms(x: torch.Tensor, eps: float, width: int) -> torch.Tensor:
    """``x / sqrt(mean(x^2) + eps)`` over the first ``width`` columns (the others are zero)."""
    return x / torch.sqrt(x.pow(2).sum(-1, keepdim=True) / width + eps)


def embed_rows(ids: torch.Tensor, table: torch.Tensor) -> Tuple[torch.Tensor, torch.Tensor]:
    """ids [T] -> (residual x [T, N] fp32 = table[ids], h [T, N] = the same in the table's dtype)."""
    V, N = table.shape
    if not table.is_cuda:
        h = table[ids.clamp(0, V - 1)]
        return h.float().clone(), h
    ids = ids.to(torch.int64).contiguous()
    T = ids.numel()
    x = torch.empty(T, N, dtype=torch.float32, device=table.device)
    fp32 = table.dtype == torch.float32
    h = x if fp32 else torch.empty(T, N, dtype=table.dtype, device=table.device)
    _lib.check(_fns().ats_embed_rows(_lib.ptr(ids), _lib.ptr(table), int(fp32), V, _lib.ptr(x), _lib.ptr(None if fp32 else h), T, N, _lib.stream_ptr(table.device)),
               "ats_embed_rows")
    return x, h


def linear_postnorm(a: torch.Tensor, w: torch.Tensor, x: torch.Tensor, c: PostNorm) -> torch.Tensor:
    """The residual step after ``y = a @ w^T``: updates ``x`` [T, N] (fp32) in place, returns the next input [T, N] in a's dtype (``x``
    itself in fp32 without a second norm: use it before the next step)."""
    T, N = x.shape
    if not a.is_cuda:
        x.copy_(rms(c.alpha * x + torch.nn.functional.linear(a.float(), w.float()), c.eps, c.width) * c.w)
        return (x if c.w2 is None else rms(x, c.eps, c.width) * c.w2).to(a.dtype)
    part = _dyt._product_f32(a, w)
    fp32 = a.dtype == torch.float32
    h = x if fp32 and c.w2 is None else torch.empty(T, N, dtype=a.dtype, device=a.device)
    args = _PostNorm(part.data_ptr(), part.shape[0], T * N, x.data_ptr(), c.alpha, c.w.data_ptr(), 0 if c.w2 is None else c.w2.data_ptr(), c.eps,
                     0 if h is x else h.data_ptr(), T, N, c.width)
    _lib.check(_fns().ats_fold_postnorm(ctypes.byref(args), int(fp32), _lib.stream_ptr(a.device)), "ats_fold_postnorm")
    return h


def linear_silu(a: torch.Tensor, w: torch.Tensor, act_cols: int) -> torch.Tensor:
    """``a @ w^T`` in a's dtype with silu on the first ``act_cols`` columns (a multiple of 8)."""
    T, N = a.shape[0], w.shape[0]
    if not a.is_cuda:
        y = torch.nn.functional.linear(a.float(), w.float())
        y[:, :act_cols] = torch.nn.functional.silu(y[:, :act_cols])
        return y.to(a.dtype)
    out = torch.empty(T, N, dtype=a.dtype, device=a.device)
    if _dyt._fused(a, w):
        a = G._check2d(a)
        _lib.check(_dyt._fns().ats_gemm_bf16_block(_lib.ptr(a), a.stride(0), _lib.ptr(w), w.stride(0), _lib.ptr(out), out.stride(0), T, N, a.shape[1], None, None, 0,
                                                   None, None, 0.0, None, None, 0.0, act_cols, _lib.ptr(_lib.status_tensor(a.device)), 0,
                                                   _lib.stream_ptr(a.device)), "ats_gemm_bf16_block")
        return out
    part = _dyt._product_f32(a, w)
    _lib.check(_fns().ats_fold_silu(_lib.ptr(part), part.shape[0], T * N, _lib.ptr(out), int(out.dtype == torch.float32), T, N, act_cols, _lib.stream_ptr(a.device)),
               "ats_fold_silu")
    return out


def norm_gate(o: torch.Tensor, gate: torch.Tensor, w: torch.Tensor, eps: float, out_width: int) -> torch.Tensor:
    """``rms(o) w sigmoid(gate)`` over whole rows: o [rows, >= n], gate [rows, >= n] (strided views), w [n] -> [rows, out_width]."""
    rows, n = o.shape[0], w.numel()
    if not o.is_cuda:
        out = torch.zeros(rows, out_width, dtype=o.dtype)
        out[:, :n] = (rms(o[:, :n].float(), eps, n) * w * torch.sigmoid(gate[:, :n].float())).to(o.dtype)
        return out
    out = torch.empty(rows, out_width, dtype=o.dtype, device=o.device)
    vec = n % 8 == 0 and (o.stride(0) | gate.stride(0) | out_width) % 8 == 0 and (o.data_ptr() | gate.data_ptr() | out.data_ptr() | w.data_ptr()) % 16 == 0
    args = _NormGate(o.data_ptr(), o.stride(0), gate.data_ptr(), gate.stride(0), w.data_ptr(), eps, out.data_ptr(), out_width, rows, n, int(vec))
    _lib.check(_fns().ats_norm_gate(ctypes.byref(args), int(o.dtype == torch.float32), _lib.stream_ptr(o.device)), "ats_norm_gate")
    return out


def softcap_(z: torch.Tensor, cap: float, fast: bool) -> torch.Tensor:
    """``z <- cap tanh(z / cap)`` in place (fp32, contiguous, whole rows of a multiple of 4)."""
    if not z.is_cuda:
        return z.div_(cap).tanh_().mul_(cap)
    _lib.check(_fns().ats_softcap(_lib.ptr(z), z.numel(), cap, int(fast), _lib.stream_ptr(z.device)), "ats_softcap")
    return z
