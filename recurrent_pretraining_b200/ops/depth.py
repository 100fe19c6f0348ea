"""Ops of residual streams with norms over groups of columns on the sublayer outputs and weighted sums over depth: CUDA tensors run
the kernels of ``csrc/depth.cu``, CPU tensors the plain statements of ``reference``.  A CUDA tensor never takes the plain path.

Conventions as in ``ops/latent.py``."""
from __future__ import annotations

import ctypes as C
from dataclasses import dataclass
from typing import Optional

import torch

from . import reference as ref
from .latent import F32, _f32, pad8
from .memory import RowSum


class _Depth(C.Structure):
    _fields_ = [(n, C.c_int) for n in ("E", "groups", "ld_a", "ld_h", "clear", "nzero")] + [("eps", C.c_float)] + \
               [(n, C.c_void_p) for n in ("w", "bias", "x0", "x", "zero")] + [("n_past", C.c_int), ("keep", C.c_int), ("past_pitch", C.c_size_t)] + \
               [(n, C.c_void_p) for n in ("past", "dwa")] + [(n, C.c_int) for n in ("top", "ld_mix", "ld_shared")] + \
               [(n, C.c_void_p) for n in ("slot", "weight", "mix_h", "shared")]


_fns = None


def _k():
    global _fns
    if _fns is None:
        from types import SimpleNamespace

        from . import cuda as K

        vp, i, f = C.c_void_p, C.c_int, C.c_float
        _fns = SimpleNamespace(K=K, norm=K._sig("b200_depth_norm", [vp, vp, C.POINTER(_Depth)] + [i] * 3 + [vp]),
                               rows=K._sig("b200_group_norm_rows", [vp] * 4 + [i] * 4 + [f, i, vp]))
    return _fns


@dataclass
class DepthStream:
    """fp32 residual stream ``x`` [T, E] with the results it averages over: ``past[j]`` (0: the embedding output, j + 1: layer j).
    ``x`` is ``past[0]`` until the first sublayer's output is added."""

    past: torch.Tensor
    x: torch.Tensor
    out: torch.Tensor

    @classmethod
    def begin(cls, past: torch.Tensor) -> "DepthStream":
        """``past``: [layers, T, E], the embedding output in the first place."""
        return cls(past, past[0], torch.empty_like(past[0]))


def depth_norm_(s: DepthStream, a, w: torch.Tensor, groups: int, eps: float, dtype: torch.dtype, bias=None, clear: bool = False,
                zero: Optional[torch.Tensor] = None, weights: Optional[torch.Tensor] = None) -> torch.Tensor:
    """s.x += norm(a + bias) * w; returns the operand copy of s.x.  ``weights`` [j + 2]: the end of layer j; the result is kept (while a later
    layer reads it) and s.x replaced by the weighted sum of all results.  ``a`` may be a ``RowSum``; ``clear`` / ``zero`` as in
    ``memory.sandwich_norm_``."""
    T, E = s.out.shape
    n = 0 if weights is None else weights.numel() - 1
    keep = n and n < s.past.shape[0]
    if not s.out.is_cuda:
        a = a.sum() if isinstance(a, RowSum) else a
        x = s.x + ref.group_rms(a.float() if bias is None else a.float() + bias, groups, eps) * w
        if keep:
            s.past[n] = x
        if n:
            x = weights[n] * x + torch.einsum("j,jte->te", weights[:n], s.past[:n])
        s.out.copy_(x)
        s.x = s.out
        return s.out.to(dtype)
    k = _k()
    p = k.K._ptr
    assert a.shape == (T, E) and s.past.is_contiguous() and (zero is None or zero.is_contiguous())
    h = torch.empty(T, pad8(E), dtype=dtype, device=s.out.device)[:, :E]
    many = {}
    if isinstance(a, RowSum):
        assert a.h.dtype == dtype and a.rows.dtype == F32 and (a.shared is None or a.shared.dtype == F32) and a.weight.is_contiguous() and a.slot.is_contiguous()
        many = dict(top=a.weight.shape[1] - 1, ld_mix=a.h.stride(0), ld_shared=0 if a.shared is None else a.shared.stride(0), slot=p(a.slot),
                    weight=p(a.weight), mix_h=p(a.h), shared=p(a.shared))
        a = a.rows
    d = _Depth(E, groups, a.stride(0), h.stride(0), int(clear), 0 if zero is None else zero.numel() // T, eps, w.data_ptr(), p(bias), s.x.data_ptr(),
               s.out.data_ptr(), p(zero), n, int(bool(keep)), T * E, s.past.data_ptr(), p(weights), **many)
    k.K._check(k.norm(a.data_ptr(), h.data_ptr(), C.byref(d), T, _f32(a), int(dtype == F32), k.K._stream()), "depth_norm")
    s.x = s.out
    return h


def group_norm_rows(x: torch.Tensor, idx: Optional[torch.Tensor], w: torch.Tensor, groups: int, eps: float, dtype: torch.dtype) -> torch.Tensor:
    """norm(x[idx]) * w in ``dtype`` (all rows when ``idx`` is None)."""
    if not x.is_cuda:
        return (ref.group_rms(x if idx is None else x[idx.long()], groups, eps) * w).to(dtype)
    k = _k()
    n, E = (x.shape[0] if idx is None else idx.numel()), x.shape[1]
    y = torch.empty(n, pad8(E), dtype=dtype, device=x.device)[:, :E]
    k.K._check(k.rows(x.data_ptr(), k.K._ptr(idx), w.data_ptr(), y.data_ptr(), y.stride(0), n, E, groups, eps, int(dtype == F32), k.K._stream()),
               "group_norm_rows")
    return y
