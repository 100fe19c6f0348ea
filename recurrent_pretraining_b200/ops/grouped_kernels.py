"""Bindings of the tensor-core kernels of grouped-query attention over a step's key stream (``csrc/latent_attention.cu``) and over
ring caches (``csrc/gqa_decode.cu``)."""
from __future__ import annotations

import ctypes as C
from functools import lru_cache

import torch

from . import cuda as K
from .latent import F32
from .latent_attention import tile_table
from .memory_kernels import _dec_ok, _dec_per_sm, _GqaDecode

_vp, _i, _f = C.c_void_p, C.c_int, C.c_float
_attn_ok = K._sig("b200_capped_attention_supported", [_i, _i])
_attn = K._sig("b200_capped_attention", [_vp] * 6 + [_i] * 12 + [_f, _f, _f, _vp, _vp])
_dec = K._sig("b200_ring_decode", [_vp, C.POINTER(_GqaDecode), _i, _i, _vp])


@lru_cache(None)
def prompt_supported(L, a) -> bool:
    """Sizes (and sign of the score factor) that the tensor-core kernel takes; the generic kernel runs otherwise."""
    return bool(_attn_ok(L.dim, L.vdim)) and a.scale > 0


def stream_attention(L, a, inp, stream, layout, window: int, sink, out) -> None:
    cache = layout.__dict__.setdefault("tiles", {})
    if window not in cache:
        cache[window] = torch.tensor(tile_table(layout, window), dtype=torch.int32).to(inp.device)
    tiles = cache[window]
    K._check(_attn(inp.data_ptr(), stream.data_ptr(), stream[:, L.kv_v:].data_ptr(), out.data_ptr(), tiles.data_ptr(), K._ptr(sink),
                   tiles.shape[0], inp.shape[0], stream.shape[0], L.heads, L.kv_heads, L.dim, L.vdim, inp.stride(0), L.ld_kv, out.stride(0),
                   min(window, 2**30), a.keep, a.scale, a.softcap or 0.0, a.score_bound or 0.0, K._stream(), K.err_word(inp.device).data_ptr()), "capped_attention")


@lru_cache(None)
def decode_supported(L) -> bool:
    return bool(_dec_ok(L.dim, L.vdim))


@lru_cache(None)
def decode_slots(L) -> int:
    """CTAs of the decode kernel that the machine holds at a time."""
    return 148 * int(_dec_per_sm(L.dim, L.vdim))


def decode_attention(L, a, inp, tr, cache, sink, first_out, pos, row, part_o, part_ml, out) -> None:
    """Appends the new token's key and value; with one split the heads' outputs to ``out``, otherwise the unnormalised partials and
    (max, sum) of every key split."""
    splits, p = part_o.shape[2], K._ptr
    cos, sin = tr.rope if tr.rope is not None else (None, None)
    s = _GqaDecode(L.heads, L.kv_heads, L.dim, L.vdim, inp.stride(0), L.off_k, L.off_v, L.ld_kv, L.kv_v, cache.shape[1], splits, scale=a.scale,
                   pos=pos.data_ptr(), row=row.data_ptr(), cache=cache.data_ptr(), part_o=part_o.data_ptr(), part_ml=part_ml.data_ptr(), size=a.size,
                   chunked=int(a.chunked), rot=tr.rot, ld_first=0 if tr.first is None else tr.first.stride(0),
                   ld_fout=0 if first_out is None else first_out.stride(0), ld_out=out.stride(0), eps=tr.eps, softcap=a.softcap or 0.0,
                   q_norm=p(tr.q_norm), k_norm=p(tr.k_norm), cosT=p(cos), sinT=p(sin), lam=p(tr.lam), first=p(tr.first), first_out=p(first_out),
                   sink=p(sink), out=out.data_ptr() if splits == 1 else 0, in_bias=p(tr.bias), keep=tr.keep, head_norm=int(tr.head_norm),
                   bound=a.score_bound or 0.0)
    K._check(_dec(inp.data_ptr(), C.byref(s), inp.shape[0], int(inp.dtype == F32), K._stream()), "ring_decode")
