"""Ops of grouped-query attention layers whose keys live in a ring per sequence (chunked or windowed, capped scores, optional
sink): CUDA tensors run the kernels of ``csrc/grouped.cu``, ``csrc/latent.cu`` and the tensor-core kernels bound in
``ops/grouped_kernels.py``, CPU tensors the plain statements of ``reference``.  A CUDA tensor never takes the plain path.

Conventions as in ``ops/latent.py``."""
from __future__ import annotations

import ctypes as C
from dataclasses import dataclass, field
from functools import lru_cache
from typing import Optional

import torch

from . import latent as base
from . import reference as ref
from .latent import BF16, F32, _f32, pad8
from .memory import _offsets


@dataclass(frozen=True)
class GroupedLayout:
    """Columns of a projection row [q | k | v] and of a key / value row [k | v]."""

    heads: int
    kv_heads: int
    dim: int
    vdim: int
    width_in: int = field(init=False)

    def __post_init__(self):
        put = lambda k, v: object.__setattr__(self, k, v)  # noqa: E731
        put("width_in", _offsets(put, q=self.heads * self.dim, k=self.kv_heads * self.dim, v=self.kv_heads * self.vdim))
        put("kv_v", self.off_v - self.off_k)
        put("ld_kv", self.width_in - self.off_k)

    @property
    def v_width(self) -> int:
        return self.kv_heads * self.vdim


class _QkvRow(C.Structure):
    _fields_ = [(n, C.c_int) for n in ("ld_in", "off_k", "off_v", "H", "G", "dim", "vdim", "rot", "ld_q", "ld_kv", "kv_v", "cap", "ld_first", "ld_fout")] + \
               [("eps", C.c_float)] + [(n, C.c_void_p) for n in ("q_norm", "k_norm", "cosT", "sinT", "lam", "pos", "row", "sidx", "end")] + [("keep", C.c_int), ("bias", C.c_void_p)]


_fns = None


def _k():
    global _fns
    if _fns is None:
        from types import SimpleNamespace

        from . import cuda as K

        vp, i = C.c_void_p, C.c_int
        _fns = SimpleNamespace(K=K, prep=K._sig("b200_qkv_prep", [vp] * 6 + [C.POINTER(_QkvRow)] + [i] * 4 + [vp]),
                               heads=K._sig("b200_qkv_heads", [vp] * 4 + [C.POINTER(_QkvRow)] + [i] * 3 + [vp]),
                               merge=K._sig("b200_attention_merge", [vp] * 4 + [i] * 6 + [vp]))
    return _fns


@dataclass
class QkvTransform:
    """What happens to a projection row before it is used: norms over all of q and of k (``q_norm``, ``k_norm`` or None), rotation
    (``rope``: cos and sin tables of ``rot`` dimensions, or None), mixing of values (``lam`` and ``first``, or None).  ``head_norm``: every head
    of q and k, once rotated, and of v is normed without weights.  ``bias``: of the raw rows of a decode step (already added in prompts).
    ``keep``: first positions that the ring keeps."""

    q_norm: Optional[torch.Tensor]
    k_norm: Optional[torch.Tensor]
    eps: float
    rot: int = 0
    rope: Optional[tuple] = None
    lam: Optional[torch.Tensor] = None
    first: Optional[torch.Tensor] = None
    head_norm: bool = False
    bias: Optional[torch.Tensor] = None
    keep: int = 0


def ring_slots(p: torch.Tensor, cap: int, keep: int) -> torch.Tensor:
    """Ring slots of positions; the first ``keep`` have theirs for good."""
    return torch.where(p < cap, p, keep + (p - keep) % max(1, cap - keep))


def _row_struct(L: GroupedLayout, inp, tr: QkvTransform, ld_q: int, cap: int, first_out, pos, row, sidx=None, end=None) -> _QkvRow:
    p = _k().K._ptr
    cos, sin = tr.rope if tr.rope is not None else (None, None)
    return _QkvRow(inp.stride(0), L.off_k, L.off_v, L.heads, L.kv_heads, L.dim, L.vdim, tr.rot, ld_q, L.ld_kv, L.kv_v, cap,
                   0 if tr.first is None else tr.first.stride(0), 0 if first_out is None else first_out.stride(0), tr.eps, p(tr.q_norm), p(tr.k_norm),
                   p(cos), p(sin), p(tr.lam), p(pos), p(row), p(sidx), p(end), tr.keep, 0)


def _plain_rows(L: GroupedLayout, inp, tr: QkvTransform, pos):
    """q [T, H, dim], kv row [T, ld_kv] and unmixed values [T, v_width] of projection rows, fp32."""
    x, T = inp.float(), inp.shape[0]
    if tr.bias is not None:
        x = x + tr.bias
    q, k, v = x[:, :L.heads * L.dim], x[:, L.off_k:L.off_k + L.kv_heads * L.dim], x[:, L.off_v:L.off_v + L.v_width]
    if tr.q_norm is not None:
        q, k = ref.rms(q, tr.eps) * tr.q_norm, ref.rms(k, tr.eps) * tr.k_norm
    q, k = q.unflatten(1, (L.heads, L.dim)), k.unflatten(1, (L.kv_heads, L.dim))
    if tr.rope is not None:
        cos, sin = (t[pos.long()][:, None] for t in tr.rope)
        q, k = (torch.cat([ref.rotate_halves(t[..., :tr.rot], cos, sin), t[..., tr.rot:]], dim=-1) for t in (q, k))
    if tr.head_norm:
        q, k, v = ref.rms(q, tr.eps), ref.rms(k, tr.eps), ref.rms(v.unflatten(1, (L.kv_heads, L.vdim)), tr.eps).flatten(1)
    mixed = v if tr.lam is None else (1 - tr.lam) * v + tr.lam * tr.first.float()
    kv = torch.zeros(T, L.ld_kv)
    kv[:, :L.kv_heads * L.dim] = k.flatten(1)
    kv[:, L.kv_v:L.kv_v + L.v_width] = mixed
    return q, kv, v


def qkv_prep_(L: GroupedLayout, inp: torch.Tensor, tr: QkvTransform, step, sidx, cache: Optional[torch.Tensor], stream: torch.Tensor) -> None:
    """Prompt form: the q parts of the projection rows ``inp`` in place, keys and (mixed) values to ``stream`` and (each sequence's
    newest ``cap``) to the ring ``cache`` [rows, cap, ld_kv]."""
    if not inp.is_cuda:
        q, kv, _ = _plain_rows(L, inp, tr, step.pos)
        inp[:, :L.heads * L.dim] = q.flatten(1).to(inp.dtype)
        stream[sidx.long()] = kv.to(stream.dtype)
        if cache is not None:
            cap = cache.shape[1]
            keep = (step.pos < tr.keep) | (step.pos >= step.end - (cap - tr.keep))
            cache[step.row[keep].long(), ring_slots(step.pos[keep].long(), cap, tr.keep)] = kv[keep].to(cache.dtype)
        return
    k = _k()
    p = k.K._ptr
    s = _row_struct(L, inp, tr, inp.stride(0), 1 if cache is None else cache.shape[1], None, step.pos, step.row, sidx, step.end)
    if tr.head_norm:
        k.K._check(k.heads(inp.data_ptr(), inp.data_ptr(), p(cache), stream.data_ptr(), C.byref(s), inp.shape[0], _f32(inp), _f32(inp), k.K._stream()),
                   "qkv_heads")
        return
    k.K._check(k.prep(inp.data_ptr(), inp.data_ptr(), p(tr.first), 0, p(cache), stream.data_ptr(), C.byref(s), inp.shape[0], _f32(inp), _f32(inp),
                      _f32(inp), k.K._stream()), "qkv_prep")


def _attn_struct(L: GroupedLayout, a, q_stride: int, **kw) -> base._WindowAttn:
    return base._WindowAttn(L.heads, L.dim, 0, L.vdim, kw.pop("window"), kw.pop("splits", 1), a.scale, q_stride, L.dim, L.ld_kv, L.dim, 0, L.ld_kv,
                            L.vdim, group=L.heads // L.kv_heads, gate_mult=1.0, softcap=a.softcap or 0.0, **kw)


def _kv_heads(L: GroupedLayout, kv: torch.Tensor):
    return kv[..., :L.kv_heads * L.dim].unflatten(-1, (L.kv_heads, L.dim)), kv[..., L.kv_v:L.kv_v + L.v_width].unflatten(-1, (L.kv_heads, L.vdim))


def stream_attention(L: GroupedLayout, a, inp: torch.Tensor, stream: torch.Tensor, layout, sink: Optional[torch.Tensor]) -> torch.Tensor:
    """Attention of a packed step's queries (in ``inp``) over its key stream [K, ld_kv] -> [T, heads * vdim].  ``a``: the layer's
    ``GroupedAttentionSpec``; the layout's ``kbase`` bounds the keys of a chunk."""
    T, window = inp.shape[0], min(2**30, 2**30 if a.chunked else a.size)
    if not inp.is_cuda:
        k, v = _kv_heads(L, stream)
        j, s = torch.arange(stream.shape[0])[None], layout.sidx.long()[:, None]
        first = layout.kbase.long()[:, None]
        vis = (j <= s) & (j >= first) & ((j > s - window) | (j < first + a.keep))
        q = inp[:, :L.heads * L.dim].unflatten(1, (L.heads, L.dim))
        return ref.capped_attention(q, k, v, vis, a.scale, a.softcap, sink).flatten(1).to(inp.dtype)
    W = L.heads * L.vdim
    out = torch.empty(T, pad8(W), dtype=inp.dtype, device=inp.device)[:, :W]
    if inp.dtype == BF16:
        from . import grouped_kernels as GK

        if GK.prompt_supported(L, a):
            GK.stream_attention(L, a, inp, stream, layout, window, sink, out)
            return out
    k = base._k()
    s = _attn_struct(L, a, inp.stride(0), window=window, sidx=layout.sidx.data_ptr(), kbase=layout.kbase.data_ptr(), out_ld=out.stride(0),
                     sink=k.K._ptr(sink), keep=a.keep)
    k.K._check(k.attn(inp.data_ptr(), stream.data_ptr(), 0, stream[:, L.kv_v:].data_ptr(), 0, out.data_ptr(), C.byref(s), T, _f32(inp),
                      k.K._stream()), "window_attention")
    return out


@lru_cache(None)
def decode_splits(L: GroupedLayout, B: int, keys: int, tensor_cores: bool) -> int:
    """Key splits of the decode attention over up to ``keys`` keys: the fewest waves of CTAs, each costing its keys and a fixed part
    worth about 256 more."""
    ctas, slots = B * L.heads, 8 * 148                     # generic kernel: a small CTA per head
    if tensor_cores:
        from . import grouped_kernels as GK

        if GK.decode_supported(L):
            ctas, slots = B * L.kv_heads * -(-(L.heads // L.kv_heads) // 16), GK.decode_slots(L)
    return min(range(1, min(32, keys // 64 + 1) + 1), key=lambda s: -(-ctas * s // slots) * (keys / s + 256))


def ring_attention(L: GroupedLayout, a, inp: torch.Tensor, tr: QkvTransform, cache: torch.Tensor, sink: Optional[torch.Tensor],
                   first_out: Optional[torch.Tensor], pos, row, splits: int, dtype: torch.dtype) -> torch.Tensor:
    """Decode form: transform the newest token's projection row, append its key and value to the ring, attend to the visible
    positions -> [B, heads * vdim].  ``first_out`` [B, v_width] fp32 receives the unmixed values."""
    B, cap, W = inp.shape[0], cache.shape[1], L.heads * L.vdim
    if not inp.is_cuda:
        q, kv, v = _plain_rows(L, inp, tr, pos)
        if first_out is not None:
            first_out.copy_(v)
        p, r = pos.long(), row.long()
        cache[r, ring_slots(p, cap, a.keep)] = kv.to(cache.dtype)
        n = min(a.size, cap)
        back = torch.arange(n + a.keep)[None]                        # key = position p - back, then the kept positions in front of the window
        key = torch.where(back < n, p[:, None] - back, back - n)
        see = torch.where(back < n, back <= (p % a.size if a.chunked else p)[:, None], key <= (p - n)[:, None])
        k, v = _kv_heads(L, cache[r[:, None], ring_slots(torch.minimum(key.clamp(min=0), p[:, None]), cap, a.keep)])
        return ref.capped_attention(q.to(dtype), k, v, see, a.scale, a.softcap, sink).flatten(1).to(dtype)
    out = torch.empty(B, pad8(W), dtype=dtype, device=inp.device)[:, :W]
    attend, merge = ring_attention_pieces(L, a, inp, tr, cache, sink, first_out, pos, row, splits, out)
    attend()
    merge()
    return out


def ring_attention_pieces(L: GroupedLayout, a, inp, tr: QkvTransform, cache, sink, first_out, pos, row, splits: int, out):
    """The parts of ``ring_attention`` on a GPU as callables."""
    k, B, dtype, cap = _k(), inp.shape[0], out.dtype, cache.shape[1]
    p = k.K._ptr
    part_o = torch.empty(B, L.heads, splits, pad8(L.vdim), dtype=F32, device=inp.device)
    part_ml = torch.empty(B, L.heads, splits, 2, dtype=F32, device=inp.device)

    fused = False
    if dtype == BF16:
        from . import grouped_kernels as GK

        fused = GK.decode_supported(L)

    def attend():
        if fused:
            GK.decode_attention(L, a, inp, tr, cache, sink, first_out, pos, row, part_o, part_ml, out)
            return
        q = torch.empty(B, pad8(L.heads * L.dim), dtype=dtype, device=inp.device)
        s = _row_struct(L, inp, tr, q.stride(0), cap, first_out, pos, row)
        if tr.head_norm:
            s.bias = p(tr.bias)
            k.K._check(k.heads(inp.data_ptr(), q.data_ptr(), cache.data_ptr(), 0, C.byref(s), B, _f32(inp), int(dtype == F32), k.K._stream()), "qkv_heads")
        else:
            k.K._check(k.prep(inp.data_ptr(), q.data_ptr(), p(tr.first), p(first_out), cache.data_ptr(), 0, C.byref(s), B, _f32(inp), int(dtype == F32), 1,
                              k.K._stream()), "qkv_prep")
        w = base._k()
        s = _attn_struct(L, a, q.stride(0), window=min(a.size, cap), splits=splits, pos=pos.data_ptr(), row=row.data_ptr(), cap=cap,
                         part_o=part_o.data_ptr(), part_ml=part_ml.data_ptr(), chunk=a.size if a.chunked else 0, keep=a.keep)
        k.K._check(w.attn(q.data_ptr(), cache.data_ptr(), 0, cache[:, :, L.kv_v:].data_ptr(), 0, 0, C.byref(s), B, int(dtype == F32), k.K._stream()),
                   "window_attention")

    def merge():
        if fused and splits == 1:
            return                                             # done by the attention itself
        k.K._check(k.merge(part_o.data_ptr(), part_ml.data_ptr(), p(sink), out.data_ptr(), out.stride(0), B, L.heads, L.vdim, splits, _f32(out),
                           k.K._stream()), "attention_merge")

    return attend, merge
