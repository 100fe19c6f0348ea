"""Bindings of the tensor-core kernels of delta memories over packed prompts (``csrc/delta_chunk.cu``, read-outs in
``csrc/memory_chunk.cu``)."""
from __future__ import annotations

import ctypes as C
from functools import lru_cache

import torch

from . import cuda as K
from .latent import BF16, F32, pad8
from .memory_kernels import CHUNK, _Chunks, chunk_tables

_vp, _i, _f = C.c_void_p, C.c_int, C.c_float


class _DeltaChunks(C.Structure):
    _fields_ = [(n, _i) for n in ("H", "G", "dim", "vdim", "vpad", "pk", "pv", "ldv", "ba_t", "ba_h", "ld_u")] + \
               [(n, _vp) for n in ("chunks", "seqs", "ba", "a_log", "dt_bias", "u0", "w_hi", "w_lo", "prefix", "fk", "u", "s_hi", "s_lo", "state", "err")]


_ok = K._sig("b200_delta_chunk_supported", [_i, _i])
_chunks = K._sig("b200_delta_chunks", [_vp, _vp, _i, C.POINTER(_DeltaChunks)] + [_i] * 4 + [_vp, _vp])
_out = K._sig("b200_delta_out", [_vp] * 3 + [C.POINTER(_Chunks)] + [_i] * 3 + [_vp, _vp])


@lru_cache(None)
def supported(L) -> bool:
    """Sizes of the tensor-core kernels; the token-by-token recurrence runs otherwise."""
    return bool(_ok(L.dim, L.vdim))


def delta_prompt(L, w, act, inp, ba, state, step, out):
    """The three launches of a packed step, as a callable taking a mask of the parts to run (1: single chunks, 2: recurrence, 4: read-outs)."""
    chunks, seqs = chunk_tables(step)
    n, S, H, dev, T = chunks.shape[0], seqs.shape[0], L.heads, act.device, act.shape[0]
    vpad = (L.vdim + 15) // 16 * 16
    u0 = torch.empty(n * H, CHUNK, vpad, dtype=F32, device=dev)
    w_hl = torch.empty(2, n * H, CHUNK, L.dim, dtype=BF16, device=dev)
    s_hl = torch.empty(2, n * H, vpad, L.dim, dtype=BF16, device=dev)
    row = torch.empty(2, n * H, CHUNK, dtype=F32, device=dev)
    u = torch.empty(T, pad8(H * L.vdim), dtype=BF16, device=dev)
    q, k, v, gate = act[:, L.off_q:], act[:, L.off_k:], act[:, L.off_v:], inp[:, L.off_g:]
    d = _DeltaChunks(H, L.kv_heads, L.dim, L.vdim, 0, 0, 0, L.ldv, ba.stride(0), ba.stride(1), u.stride(0), chunks.data_ptr(), seqs.data_ptr(), ba.data_ptr(),
                     w.a_log.data_ptr(), w.dt_bias.data_ptr(), u0.data_ptr(), w_hl[0].data_ptr(), w_hl[1].data_ptr(), row[0].data_ptr(), row[1].data_ptr(),
                     u.data_ptr(), s_hl[0].data_ptr(), s_hl[1].data_ptr(), state.data_ptr(), 0)
    o = _Chunks(H=H, dim=L.dim, vdim=L.vdim, ldv=L.ldv, ld_in=act.stride(0), ld_out=out.stride(0), qscale=L.dim ** -0.5, eps=w.eps, chunks=chunks.data_ptr(),
                seqs=seqs.data_ptr(), s_hi=s_hl[0].data_ptr(), s_lo=s_hl[1].data_ptr(), group=H // L.kv_heads, ld_g=inp.stride(0), prefix=row[0].data_ptr(),
                fk=row[1].data_ptr(), gate_out=gate.data_ptr(), norm_w=w.norm.data_ptr(), out=out.data_ptr())
    keep = (chunks, seqs, u0, w_hl, s_hl, row, u, act, inp, ba, state, w)      # alive as long as the callable

    def run(parts: int = 7):
        assert keep
        err = K.err_word(dev).data_ptr()
        if parts & 3:
            K._check(_chunks(k.data_ptr(), v.data_ptr(), act.stride(0), C.byref(d), T, n, S, parts & 3, K._stream(), err), "delta_chunks")
        if parts & 4:
            K._check(_out(q.data_ptr(), k.data_ptr(), u.data_ptr(), C.byref(o), u.stride(0), T, n, K._stream(), err), "delta_out")
        return out

    return run
