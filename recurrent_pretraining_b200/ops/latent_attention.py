"""Bindings of the tensor-core kernels of windowed latent attention: over a packed step's key stream
(``csrc/latent_attention.cu``) and, for decode steps, over the ring cache (``csrc/latent_decode.cu``)."""
from __future__ import annotations

import ctypes as C
from functools import lru_cache

import torch

from . import cuda as K

_vp, _i, _f = C.c_void_p, C.c_int, C.c_float
_supported = K._sig("b200_latent_attention_supported", [_i, _i, _i])
_attn = K._sig("b200_latent_attention", [_vp] * 7 + [_i] * 13 + [_f, _vp, _vp])
_decode_group = K._sig("b200_latent_decode_group", [_i, _i, _i])
_decode = K._sig("b200_latent_decode", [_vp] * 6 + [_i] * 8 + [_f, _vp, _vp])

TILE = 256   # queries per CTA


@lru_cache(None)
def supported(L) -> bool:
    """Sizes the tensor-core kernel takes (multiples of eight that fit its shared and tensor memory); any other size runs
    the generic window-attention kernel."""
    return bool(_supported(L.dim, L.rot, L.vdim))


def tile_table(layout, window: int) -> list:
    """(first query token, queries, stream index of the first query, first key) per CTA, most visible keys first."""
    tiles = [(t0 + i, min(TILE, n - i), k0 + h + i, k0) for t0, n, k0, h in layout.seqs for i in range(0, n, TILE)]
    return sorted(tiles, key=lambda t: -(t[1] + min(t[2] - t[3], window)))


def stream_attention(L, inp, kv, stream, layout, window: int, scale: float, out) -> None:
    cache = layout.__dict__.setdefault("tiles", {})
    if window not in cache:
        cache[window] = torch.tensor(tile_table(layout, window), dtype=torch.int32).to(inp.device)
    tiles = cache[window]
    gate = inp[:, L.off_g:]
    K._check(_attn(inp.data_ptr(), kv.data_ptr(), stream[:, L.rank_pad:].data_ptr(), kv[:, L.off_v:].data_ptr(), gate.data_ptr(),
                   out.data_ptr(), tiles.data_ptr(), tiles.shape[0], inp.shape[0], kv.shape[0], L.heads, L.dim, L.rot, L.vdim,
                   inp.stride(0), kv.stride(0), stream.stride(0), inp.stride(0), out.stride(0), min(window, 2**30), scale, K._stream(),
                   K.err_word(inp.device).data_ptr()), "latent_attention")


@lru_cache(None)
def decode_group(heads: int, rank: int, ld_lat: int) -> int:
    """Heads per CTA of the decode kernel; 0: sizes it does not take (the generic kernel runs)."""
    return int(_decode_group(heads, rank, ld_lat))


def decode_supported(L, cap: int) -> bool:
    return cap % 128 == 0 and decode_group(L.heads, L.rank, L.ld_lat) > 0


def ring_attention(L, qlat, cache, pos, row, part_o, part_ml, window: int, splits: int, scale: float) -> None:
    """Unnormalised partials [B, H, splits, rank] and (max, sum) of the newest token of every row against its ring."""
    assert qlat.is_contiguous() and cache.is_contiguous() and cache.shape[2] == L.ld_lat
    K._check(_decode(qlat.data_ptr(), cache.data_ptr(), pos.data_ptr(), row.data_ptr(), part_o.data_ptr(), part_ml.data_ptr(),
                     qlat.shape[0], L.heads, L.rank, L.ld_lat, cache.shape[0], cache.shape[1], window, splits, scale, K._stream(),
                     K.err_word(qlat.device).data_ptr()), "latent_decode")
