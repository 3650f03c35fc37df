"""Lightning attention: linear attention with one constant decay per head (``csrc/lightning.cu``, ``csrc/lightning_tcgen05.cu``, where
the recurrence is written out).

q, k and v lie activated in one projection buffer; the state [B, heads, dim, vdim] is fp32 and is updated in place.  CPU tensors run the
PyTorch definitions below.
"""
from __future__ import annotations

import ctypes
import os
from dataclasses import dataclass
from typing import Optional, Tuple

import torch

from . import _lib
from .latent import _call, _p, pad8

_vp, _ci, _cll = ctypes.c_void_p, ctypes.c_int, ctypes.c_longlong
CHUNK = 128  # tokens the tensor-core kernel advances at a time
# ATS_LIGHTNING_TC=0: portions use the general kernel for every shape (for comparison)
TENSOR_CORES = os.environ.get("ATS_LIGHTNING_TC", "1") == "1"


@dataclass(frozen=True)
class LightningShape:
    heads: int
    dim: int
    vdim: int
    decay: Tuple[float, ...]
    eps: float

    # columns of the input projection [q | k | v | gate], every part padded to a multiple of 8
    @property
    def k_col(self) -> int:
        return pad8(self.heads * self.dim)

    @property
    def v_col(self) -> int:
        return 2 * self.k_col

    @property
    def g_col(self) -> int:
        return self.v_col + self.o_pad

    @property
    def o_pad(self) -> int:
        return pad8(self.heads * self.vdim)

    @property
    def proj_width(self) -> int:
        return self.g_col + self.o_pad


def decay_powers(s: LightningShape, device) -> torch.Tensor:
    """[heads, CHUNK + 1] decay^n, rounded once from fp64."""
    n = torch.arange(CHUNK + 1, dtype=torch.float64)
    return (torch.tensor(s.decay, dtype=torch.float64)[:, None] ** n).float().contiguous().to(device)


class _Args(ctypes.Structure):
    _fields_ = [("qkv", _vp), ("ld", _cll), ("q_col", _ci), ("k_col", _ci), ("v_col", _ci), ("decay", _vp), ("state", _vp), ("state_bs", _cll), ("o", _vp), ("ldo", _cll),
                ("B", _ci), ("L", _ci), ("H", _ci), ("dim", _ci), ("vdim", _ci), ("fresh", _ci), ("lengths", _vp), ("active", _vp)]


def _heads(proj: torch.Tensor, s: LightningShape):
    rows = proj.shape[0]

    def part(at, d):
        return proj[:, at:at + s.heads * d].view(rows, s.heads, d).float()
    return part(0, s.dim), part(s.k_col, s.dim), part(s.v_col, s.vdim)


def tensor_cores_ok(proj: torch.Tensor, s: LightningShape, L: int) -> bool:
    """The tensor-core kernel covers these sizes, and the portion fills more than a few rows of its chunks."""
    return TENSOR_CORES and proj.dtype == torch.bfloat16 and L >= 32 and s.dim % 8 == 0 and s.dim <= 128 and s.vdim % 8 == 0


def lightning_scan(proj: torch.Tensor, state: torch.Tensor, powers: torch.Tensor, s: LightningShape, L: int, fresh: bool) -> torch.Tensor:
    """Advances ``state`` over portions of L tokens: proj [B * L, proj_width] -> read-outs [B * L, o_pad]; ``fresh``: from zero."""
    B, dev = state.shape[0], proj.device
    if not proj.is_cuda:
        q, k, v = _heads(proj, s)
        out = torch.zeros(B * L, s.o_pad, dtype=proj.dtype)
        for b in range(B):
            S = torch.zeros_like(state[b]) if fresh else state[b].clone()
            for t in range(b * L, (b + 1) * L):
                S = powers[:, 1, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
                out[t, :s.heads * s.vdim] = torch.einsum("hdv,hd->hv", S, q[t]).reshape(-1).to(out.dtype)
            state[b] = S
        return out
    o = torch.empty(B * L, s.o_pad, dtype=proj.dtype, device=dev)
    if tensor_cores_ok(proj, s, L):
        f = _lib.cuda_lib().ats_lightning_tc
        f.restype, f.argtypes = _ci, [_vp, _cll, _ci, _ci, _ci, _vp, _vp, _cll, _vp, _cll] + [_ci] * 6 + [_vp, _vp]
        _lib.check(f(_p(proj), proj.stride(0), 0, s.k_col, s.v_col, _p(powers), _p(state), state.stride(0), _p(o), o.stride(0), B, L, s.heads, s.dim, s.vdim, int(fresh),
                     _p(_lib.status_tensor(dev)), _lib.stream_ptr(dev)), "ats_lightning_tc")
        return o
    decay = powers[:, 1].contiguous()
    _call("ats_lightning_scan", _Args(_p(proj), proj.stride(0), 0, s.k_col, s.v_col, _p(decay), _p(state), state.stride(0), _p(o), o.stride(0), B, L, s.heads, s.dim,
                                      s.vdim, int(fresh), 0, 0), proj)
    return o


def lightning_step(proj: torch.Tensor, state: torch.Tensor, decay: torch.Tensor, s: LightningShape, lengths: torch.Tensor,
                   active: Optional[torch.Tensor] = None) -> torch.Tensor:
    """One token per sequence: proj [B, proj_width], decay [heads] -> read-outs [B, o_pad]."""
    B = state.shape[0]
    if not proj.is_cuda:
        q, k, v = _heads(proj, s)
        out = torch.zeros(B, s.o_pad, dtype=proj.dtype)
        for b in range(B):
            S = torch.zeros_like(state[b]) if int(lengths[b]) == 0 else state[b]
            S = decay[:, None, None] * S + k[b][:, :, None] * v[b][:, None, :]
            if active is None or int(active[b]):
                state[b] = S
            out[b, :s.heads * s.vdim] = torch.einsum("hdv,hd->hv", S, q[b]).reshape(-1).to(out.dtype)
        return out
    o = torch.empty(B, s.o_pad, dtype=proj.dtype, device=proj.device)
    _call("ats_lightning_step", _Args(_p(proj), proj.stride(0), 0, s.k_col, s.v_col, _p(decay), _p(state), state.stride(0), _p(o), o.stride(0), B, 1, s.heads, s.dim,
                                      s.vdim, 0, _p(lengths), _p(active)), proj)
    return o
