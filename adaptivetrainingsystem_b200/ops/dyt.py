"""Element-wise block steps for models whose norm is Dynamic Tanh (``csrc/dyt.cu`` and the GEMM epilogues of ``csrc/gemm_tcgen05.cu``).

``dyt(x) = tanh(alpha * x) * w + b`` has no reduction, so the chain between two products of a block -- output norm, layer scale,
residual add, next input norm -- is one element-wise function of the product and the residual:

    x <- x + tanh(a1 * (y + bias)) * w1 + b1         (output norm times layer scale; b1 may also carry a vector added to x)
    h <- tanh(a2 * x) * w2 + b2

The residual ``x`` is fp32 whatever the element type of the products.  CPU tensors run the PyTorch definitions.
"""
from __future__ import annotations

import ctypes
import os
from dataclasses import dataclass
from typing import Optional, Tuple

import torch

from . import _lib
from . import gemm as G

_vp, _ci, _cll, _cf = ctypes.c_void_p, ctypes.c_int, ctypes.c_longlong, ctypes.c_float
_sig = False


def _fns():
    global _sig
    lib = _lib.cuda_lib()
    if not _sig:
        for name, args in (("ats_fold_dyt", [_vp, _ci, _cll, _vp, _vp, _vp, _vp, _cf, _vp, _vp, _cf, _vp, _ci, _cll, _ci, _vp]),
                           ("ats_fold_gelu", [_vp, _ci, _cll, _vp, _vp, _ci, _cll, _ci, _vp]),
                           ("ats_gemm_bf16_block", [_vp, _cll, _vp, _cll, _vp, _ci, _ci, _ci, _ci, _vp, _vp, _ci, _vp, _vp, _cf, _vp, _vp, _cf, _ci, _vp, _ci, _vp]),
                           ("ats_embed_dyt", [_vp, _vp, _ci, _ci, _vp, _vp, _vp, _vp, _cf, _vp, _cll, _ci, _vp])):
            f = getattr(lib, name)
            f.restype, f.argtypes = _ci, args
        _sig = True
    return lib


@dataclass
class DytChain:
    """Constants of one residual step, all fp32 ``[N]`` (see the module text)."""
    w1: torch.Tensor
    b1: torch.Tensor
    a1: float
    w2: torch.Tensor
    b2: torch.Tensor
    a2: float


def gelu_tanh(z: torch.Tensor) -> torch.Tensor:
    return torch.nn.functional.gelu(z, approximate="tanh")


def embed_norm(ids: torch.Tensor, table: torch.Tensor, add: Optional[torch.Tensor], w2: torch.Tensor, b2: torch.Tensor, a2: float,
               ) -> Tuple[torch.Tensor, torch.Tensor]:
    """ids [T] -> (residual x [T, N] fp32 = table[ids] (+ add), h [T, N] = dyt(x) in the table's dtype)."""
    V, N = table.shape
    if not table.is_cuda:
        x = table[ids.clamp(0, V - 1)].float()
        if add is not None:
            x = x + add
        return x, (torch.tanh(a2 * x) * w2 + b2).to(table.dtype)
    ids = ids.to(torch.int64).contiguous()
    T = ids.numel()
    x = torch.empty(T, N, dtype=torch.float32, device=table.device)
    h = torch.empty(T, N, dtype=table.dtype, device=table.device)
    _lib.check(_fns().ats_embed_dyt(_lib.ptr(ids), _lib.ptr(table), int(table.dtype == torch.float32), V, _lib.ptr(add), _lib.ptr(x), _lib.ptr(w2),
                                    _lib.ptr(b2), a2, _lib.ptr(h), T, N, _lib.stream_ptr(table.device)), "ats_embed_dyt")
    return x, h


def _product_f32(a: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """a [T, K] @ w [N, K]^T as fp32 blocks [splits, T, N] whose sum is the product (decode-sized bf16 products split the reduction)."""
    T, K = a.shape
    N = w.shape[0]
    if a.dtype == torch.float32:
        return torch.nn.functional.linear(a, w).view(1, T, N)
    splits = G._skinny_splits(T, N, K) if G.SPLIT_K_SKINNY else 1
    part = torch.empty(splits, T, N, dtype=torch.float32, device=a.device)
    kp = K // splits
    a = G._check2d(a)
    G._raw(a, T, K, a.stride(0), 0, w, N, K, w.stride(0), 0, part, N, None, 0, None, 0, T, N, kp, epilogue=G.EPI_F32, groups=splits, a_gs_k=kp if splits > 1 else 0,
           b_gs_k=kp if splits > 1 else 0, d_gs=T * N if splits > 1 else 0)
    return part


# bf16 products whose reduction is not split over the SMs do the element-wise step in their epilogue; ATS_BLOCK_EPILOGUE=0 runs it as a
# launch of its own instead (for comparison)
FUSED_EPILOGUE = os.environ.get("ATS_BLOCK_EPILOGUE", "1") == "1"


def _fused(a: torch.Tensor, w: torch.Tensor) -> bool:
    return FUSED_EPILOGUE and a.dtype == torch.bfloat16 and (not G.SPLIT_K_SKINNY or G._skinny_splits(a.shape[0], w.shape[0], a.shape[1]) == 1)


def _block_gemm(a: torch.Tensor, w: torch.Tensor, out: torch.Tensor, bias: Optional[torch.Tensor], x: Optional[torch.Tensor], c: Optional[DytChain]) -> None:
    a = G._check2d(a)
    (T, K), N = a.shape, w.shape[0]
    w1, b1, a1, w2, b2, a2 = (c.w1, c.b1, c.a1, c.w2, c.b2, c.a2) if c is not None else (None, None, 0.0, None, None, 0.0)
    _lib.check(_fns().ats_gemm_bf16_block(_lib.ptr(a), a.stride(0), _lib.ptr(w), w.stride(0), _lib.ptr(out), out.stride(0), T, N, K, _lib.ptr(bias), _lib.ptr(x),
                                          0 if x is None else x.stride(0), _lib.ptr(w1), _lib.ptr(b1), a1, _lib.ptr(w2), _lib.ptr(b2), a2, -1,
                                          _lib.ptr(_lib.status_tensor(a.device)), 0, _lib.stream_ptr(a.device)), "ats_gemm_bf16_block")


def linear_residual(a: torch.Tensor, w: torch.Tensor, bias: Optional[torch.Tensor], x: torch.Tensor, c: DytChain) -> torch.Tensor:
    """The residual step after ``y = a @ w^T``: updates ``x`` [T, N] (fp32) in place, returns ``h`` [T, N] in a's dtype."""
    T, N = x.shape
    if not a.is_cuda:
        y = torch.nn.functional.linear(a.float(), w.float())
        if bias is not None:
            y = y + bias
        x += torch.tanh(c.a1 * y) * c.w1 + c.b1
        return (torch.tanh(c.a2 * x) * c.w2 + c.b2).to(a.dtype)
    h = torch.empty(T, N, dtype=a.dtype, device=a.device)
    if _fused(a, w):
        _block_gemm(a, w, h, bias, x, c)
        return h
    part = _product_f32(a, w)
    _lib.check(_fns().ats_fold_dyt(_lib.ptr(part), part.shape[0], T * N, _lib.ptr(bias), _lib.ptr(x), _lib.ptr(c.w1), _lib.ptr(c.b1), c.a1, _lib.ptr(c.w2),
                                   _lib.ptr(c.b2), c.a2, _lib.ptr(h), int(h.dtype == torch.float32), T, N, _lib.stream_ptr(a.device)), "ats_fold_dyt")
    return h


def linear_gelu(a: torch.Tensor, w: torch.Tensor, bias: Optional[torch.Tensor]) -> torch.Tensor:
    """gelu_tanh(a @ w^T + bias) in a's dtype."""
    T, N = a.shape[0], w.shape[0]
    if not a.is_cuda:
        return gelu_tanh(torch.nn.functional.linear(a.float(), w.float(), bias)).to(a.dtype)
    out = torch.empty(T, N, dtype=a.dtype, device=a.device)
    if _fused(a, w):
        _block_gemm(a, w, out, bias, None, None)
        return out
    part = _product_f32(a, w)
    _lib.check(_fns().ats_fold_gelu(_lib.ptr(part), part.shape[0], T * N, _lib.ptr(bias), _lib.ptr(out), int(out.dtype == torch.float32), T, N,
                                    _lib.stream_ptr(a.device)), "ats_fold_gelu")
    return out
