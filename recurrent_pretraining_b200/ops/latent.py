"""Ops of the layered decoder models (``models/layered.py``): CUDA tensors run the kernels of ``csrc/latent.cu``,
``csrc/latent_attention.cu`` and the GEMM family, CPU tensors the plain statements of ``reference``.  A CUDA tensor never
takes the plain path.

Conventions.  ``T`` tokens of a packed step (or the ``B`` rows of a decode step).  The residual stream is fp32; matrix
operands are in the model's storage dtype, bf16 or fp32 (fp32 operands run a true fp32 product).  Row pitches are padded
to multiples of eight elements, so every matrix can be described to the copy engine whatever its sizes."""
from __future__ import annotations

import ctypes as C
from dataclasses import dataclass, field
from typing import Optional

import torch

from . import reference as ref

BF16, F32 = torch.bfloat16, torch.float32


def pad8(n: int) -> int:
    return (n + 7) // 8 * 8


def pad16(n: int) -> int:
    return (n + 15) // 16 * 16


@dataclass(frozen=True)
class LatentLayout:
    """Column layout of a latent-attention layer's projection row, key/value row and latent row."""

    heads: int
    dim: int
    rot: int
    vdim: int
    rank: int
    own: bool
    off_g: int = field(init=False)
    off_d: int = field(init=False)
    width_in: int = field(init=False)      # [q | gate | latent]
    off_v: int = field(init=False)
    width_kv: int = field(init=False)      # [unrotated keys | values]
    rank_pad: int = field(init=False)
    ld_lat: int = field(init=False)        # [latent | rotated key part]
    ld_o: int = field(init=False)

    def __post_init__(self):
        put = lambda k, v: object.__setattr__(self, k, v)  # noqa: E731
        put("off_g", pad8(self.heads * (self.dim + self.rot)))
        put("off_d", self.off_g + pad8(self.heads * self.vdim))
        put("width_in", self.off_d + (pad8(self.rank + self.rot) if self.own else 0))
        put("off_v", pad8(self.heads * self.dim))
        put("width_kv", self.off_v + pad8(self.heads * self.vdim))
        put("rank_pad", pad16(self.rank))
        put("ld_lat", pad16(self.rank) + pad16(self.rot))
        put("ld_o", pad8(self.heads * self.vdim))


class _LatentRow(C.Structure):
    _fields_ = [(n, C.c_int) for n in ("ld_in", "off_g", "off_d", "H", "dim", "rot", "rank", "vdim", "rank_pad", "ld_lat", "cap",
                                       "own")] + [("eps", C.c_float)] + \
               [(n, C.c_void_p) for n in ("norm_w", "cosT", "sinT", "pos", "row")]


class _WindowAttn(C.Structure):
    _fields_ = [(n, C.c_int) for n in ("H", "d1", "d2", "vdim", "window", "splits")] + [("scale", C.c_float)] + \
               [(n, C.c_int) for n in ("q_stride", "q_head", "k1_stride", "k1_head", "k2_stride", "v_stride", "v_head")] + \
               [(n, C.c_void_p) for n in ("sidx", "kbase", "pos", "row")] + [("cap", C.c_int)] + \
               [(n, C.c_int) for n in ("gate_ld", "out_ld")] + [(n, C.c_void_p) for n in ("part_o", "part_ml")] + \
               [("group", C.c_int), ("bias", C.c_void_p), ("bias_len", C.c_int), ("temp_every", C.c_int), ("temp_coef", C.c_float),
                ("head_gate", C.c_int), ("gate_mult", C.c_float), ("softcap", C.c_float), ("chunk", C.c_int), ("sink", C.c_void_p),
                ("keep", C.c_int)]


_fns = None


def _k():
    """The kernel bindings (importing them loads the native library)."""
    global _fns
    if _fns is None:
        from types import SimpleNamespace

        from . import cuda as K

        vp, i, f, ll = C.c_void_p, C.c_int, C.c_float, C.c_longlong
        row, att = C.POINTER(_LatentRow), C.POINTER(_WindowAttn)
        _fns = SimpleNamespace(
            K=K,
            embed=K._sig("b200_embed_resid", [vp] * 4 + [i] * 4 + [f, ll, i, vp, vp]),
            prep=K._sig("b200_latent_prep", [vp, row] + [vp] * 4 + [i, i, vp]),
            absorb=K._sig("b200_latent_absorb", [vp, row, vp, i, vp, vp, i, i, i, vp]),
            gather=K._sig("b200_gather_rows", [vp] * 4 + [i, i, vp]),
            attn=K._sig("b200_window_attention", [vp] * 6 + [att, i, i, vp]),
            expand=K._sig("b200_latent_expand", [vp, vp, i, vp, i, vp, i, vp] + [i] * 7 + [vp]),
            resid=K._sig("b200_rms_residual", [vp] + [i] * 3 + [vp] * 4 + [i] * 3 + [f, f, vp, i, i, vp]),
            norm_rows=K._sig("b200_rmsnorm_rows", [vp] * 4 + [i] * 3 + [f, f, f, i, vp]),
            bias_act=K._sig("b200_bias_act", [vp] + [i] * 3 + [vp, vp] + [i] * 5 + [vp]),
            sgemm=K._sig("b200_sgemm_nt", [vp] * 4 + [i] * 9 + [vp] * 3),
        )
    return _fns


def _f32(t) -> int:
    return int(t.dtype == F32)


_ACT = {None: 0, "relu2": 1, "silu": 2}


# ------------------------------------------------------------------------------------------
# matrix products
# ------------------------------------------------------------------------------------------
def _pitched(y: torch.Tensor, ld: int) -> torch.Tensor:
    """``y`` with a row pitch of at least ``ld`` elements."""
    if ld <= y.shape[1]:
        return y
    out = torch.zeros(y.shape[0], ld, dtype=y.dtype)
    out[:, :y.shape[1]] = y
    return out[:, :y.shape[1]]


def linear(x: torch.Tensor, w: torch.Tensor, bias: Optional[torch.Tensor] = None, act: Optional[str] = None,
           out_f32: bool = False, ld_out: int = 0, act_cols: tuple = (0, 0)) -> torch.Tensor:
    """act(x w^T + bias) for x [M, K] and w [N, K] of one storage dtype (rows may be pitched); result [M, N] in that dtype,
    or fp32 with ``out_f32`` (no bias then).  ``act`` "silu" applies to the columns ``act_cols`` (multiples of eight).  bf16: tcgen05 GEMM with the bias and the activation in its epilogue.
    fp32: true fp32 product."""
    M, Kd = x.shape
    N = w.shape[0]
    assert x.dtype == w.dtype and w.shape[1] == Kd and not (out_f32 and (bias is not None or act))
    if not x.is_cuda:
        y = ref.linear_act(x, w, bias, act, act_cols)
        return _pitched(y.float() if out_f32 else y, ld_out)
    k = _k()
    out = torch.empty(M, max(ld_out, pad8(N)), dtype=F32 if out_f32 else x.dtype, device=x.device)[:, :N]
    if x.dtype == F32:
        k.K._check(k.sgemm(x.data_ptr(), w.data_ptr(), k.K._ptr(bias), out.data_ptr(), M, N, Kd, x.stride(0), w.stride(0),
                           out.stride(0), _ACT[act], act_cols[0], act_cols[1], 0, 0, k.K._stream()), "sgemm_nt")
        return out
    if out_f32:
        return k.K.gemm(x, w, out=out, out_mode=k.K.OUT_F32)
    if bias is None and act is None:
        return k.K.gemm(x, w, out=out)
    return k.K.gemm(x, w, out=out, out_mode=k.K.OUT_BF16_BIAS_ACT, bias=bias, act=_ACT[act], act_cols=act_cols)


def bias_act(a: torch.Tensor, bias: Optional[torch.Tensor], act: Optional[str], dtype: torch.dtype, clear: bool = False) -> torch.Tensor:
    """act(a + bias) in ``dtype``; ``clear`` hands a stream-K accumulator back zeroed."""
    M, N = a.shape
    if not a.is_cuda:
        y = a.float() if bias is None else a.float() + bias
        return (ref.relu2(y) if act == "relu2" else y).to(dtype)
    k = _k()
    y = torch.empty(M, pad8(N), dtype=dtype, device=a.device)[:, :N]
    k.K._check(k.bias_act(a.data_ptr(), a.stride(0), _f32(a), int(clear), k.K._ptr(bias), y.data_ptr(), y.stride(0), M, N, _ACT[act],
                          int(dtype == F32), k.K._stream()), "bias_act")
    return y


# ------------------------------------------------------------------------------------------
# residual stream
# ------------------------------------------------------------------------------------------
def embed(tok: torch.Tensor, table: torch.Tensor, scale: float = 1.0, copy: bool = True, out: Optional[torch.Tensor] = None):
    """(fp32 residual [T, E] = scale * table row, operand copy [T, E] or None) of token ids [T]; ``out``: contiguous storage for the first."""
    T, E = tok.numel(), table.shape[1]
    if not tok.is_cuda:
        x = table[tok].float() * scale
        if out is not None:
            x = out.copy_(x)
        return x, x.to(table.dtype) if copy else None
    k = _k()
    assert tok.dtype == torch.int64 and tok.is_contiguous()
    x = torch.empty(T, E, dtype=F32, device=tok.device) if out is None else out
    xb = torch.empty(T, pad8(E), dtype=table.dtype, device=tok.device)[:, :E] if copy else None
    k.K._check(k.embed(tok.data_ptr(), table.data_ptr(), x.data_ptr(), k.K._ptr(xb), T, E, table.stride(0), xb.stride(0) if copy else 0,
                       scale, table.shape[0], _f32(table), k.K.err_word(tok.device).data_ptr(), k.K._stream()), "embed_resid")
    return x, xb


def rms_residual_(x: torch.Tensor, a: torch.Tensor, bias, w: torch.Tensor, eps: float, mult: float, dtype: torch.dtype,
                  clear: bool = False, zero: Optional[torch.Tensor] = None) -> torch.Tensor:
    """x += mult * rmsnorm(a + bias) * w in place; returns the operand copy of x.  ``clear`` / ``zero``: accumulators that are
    handed back zeroed (a itself / a second one with the same number of rows)."""
    T, E = x.shape
    if not x.is_cuda:
        x.copy_(ref.rms_residual(x, a, bias, w, eps, mult))
        return x.to(dtype)
    k = _k()
    assert x.is_contiguous() and a.shape == (T, E) and w.dtype == F32 and (zero is None or zero.is_contiguous())
    xb = torch.empty(T, pad8(E), dtype=dtype, device=x.device)[:, :E]
    nz = 0 if zero is None else zero.numel() // T
    k.K._check(k.resid(a.data_ptr(), a.stride(0), _f32(a), int(clear), k.K._ptr(bias), w.data_ptr(), x.data_ptr(), xb.data_ptr(),
                       xb.stride(0), T, E, eps, mult, k.K._ptr(zero), nz, int(dtype == F32), k.K._stream()), "rms_residual")
    return xb


def rmsnorm_rows(x: torch.Tensor, idx: Optional[torch.Tensor], w: torch.Tensor, eps: float, dtype: torch.dtype, w_add: float = 0.0,
                 mult: float = 1.0) -> torch.Tensor:
    """mult * rmsnorm(x[idx]) * (w + w_add) in ``dtype`` (all rows when ``idx`` is None)."""
    if not x.is_cuda:
        rows = x if idx is None else x[idx.long()]
        return (ref.rms(rows, eps) * (w + w_add) * mult).to(dtype)
    k = _k()
    n, E = (x.shape[0] if idx is None else idx.numel()), x.shape[1]
    assert idx is None or (idx.dtype == torch.int32 and idx.is_cuda)
    y = torch.empty(n, pad8(E), dtype=dtype, device=x.device)[:, :E]
    k.K._check(k.norm_rows(x.data_ptr(), k.K._ptr(idx), w.data_ptr(), y.data_ptr(), y.stride(0), n, E, eps, w_add, mult,
                           int(dtype == F32), k.K._stream()), "rmsnorm_rows")
    return y


# ------------------------------------------------------------------------------------------
# latents
# ------------------------------------------------------------------------------------------
def gather_rows(src: torch.Tensor, src_idx: torch.Tensor, dst: torch.Tensor, dst_idx: torch.Tensor) -> None:
    """dst[dst_idx] = src[src_idx] for row-contiguous matrices."""
    if not src.is_cuda:
        dst[dst_idx.long()] = src[src_idx.long()]
        return
    k = _k()
    assert src.is_contiguous() and dst.is_contiguous() and src.shape[1] == dst.shape[1] and src.dtype == dst.dtype
    k.K._check(k.gather(src.data_ptr(), src_idx.data_ptr(), dst.data_ptr(), dst_idx.data_ptr(), src_idx.numel(),
                        src.shape[1] * src.element_size(), k.K._stream()), "gather_rows")


def _row_struct(L: LatentLayout, inp, norm_w, eps, rope, pos, row, cap) -> _LatentRow:
    cos, sin = rope
    return _LatentRow(inp.stride(0), L.off_g, L.off_d, L.heads, L.dim, L.rot, L.rank, L.vdim, L.rank_pad, L.ld_lat, cap, int(L.own),
                      eps, 0 if norm_w is None else norm_w.data_ptr(), cos.data_ptr(), sin.data_ptr(), pos.data_ptr(),
                      0 if row is None else row.data_ptr())


def _latent_rows(L: LatentLayout, inp, norm_w, eps, cos, sin) -> torch.Tensor:
    """Plain form of the latent row [c | 0 | rotated key part | 0]."""
    d = inp[:, L.off_d:].float()
    out = torch.zeros(inp.shape[0], L.ld_lat)
    out[:, :L.rank] = ref.rms(d[:, :L.rank], eps) * norm_w
    out[:, L.rank_pad:L.rank_pad + L.rot] = ref.rotate_pairs(d[:, L.rank:L.rank + L.rot], cos, sin)
    return out


def latent_prep_(L: LatentLayout, inp: torch.Tensor, norm_w, eps: float, rope, step, sidx, cache, stream) -> None:
    """Rotate the q parts of the projection rows ``inp`` [T, width_in] in place; for a layer with latents of its own append
    the latent rows to ``stream`` and (each sequence's newest ``cap``) to the ring ``cache`` [rows, cap, ld_lat]."""
    T = inp.shape[0]
    cap = cache.shape[1] if cache is not None else 1
    if not inp.is_cuda:
        cos, sin = rope[0][step.pos.long()], rope[1][step.pos.long()]
        q = inp[:, :L.heads * (L.dim + L.rot)].unflatten(1, (L.heads, L.dim + L.rot))
        q[..., L.dim:] = ref.rotate_pairs(q[..., L.dim:], cos[:, None], sin[:, None]).to(inp.dtype)
        if L.own:
            lat = _latent_rows(L, inp, norm_w, eps, cos, sin).to(inp.dtype)
            stream[sidx.long()] = lat
            if cache is None:
                return
            keep = step.pos >= step.end - cap
            cache[step.row[keep].long(), step.pos[keep].long() % cap] = lat[keep]
        return
    k = _k()
    s = _row_struct(L, inp, norm_w, eps, rope, step.pos, step.row, cap)
    own = L.own
    k.K._check(k.prep(inp.data_ptr(), C.byref(s), sidx.data_ptr() if own else 0, step.end.data_ptr() if own else 0,
                      k.K._ptr(cache), stream.data_ptr() if own else 0, T, _f32(inp), k.K._stream()), "latent_prep")


def stream_attention(L: LatentLayout, inp: torch.Tensor, kv: torch.Tensor, stream: torch.Tensor, layout, window: int,
                     scale: float) -> torch.Tensor:
    """Gated attention of the step's queries over its key stream -> [T, heads * vdim].  ``inp``: projection rows (q rotated),
    ``kv``: [K, width_kv] up-projected keys and values, ``stream``: [K, ld_lat] latent rows (the rotated key part)."""
    T, hd = inp.shape[0], L.dim + L.rot
    kr = stream[:, L.rank_pad:]
    if not inp.is_cuda:
        q = inp[:, :L.heads * hd].unflatten(1, (L.heads, hd))
        kn = kv[:, :L.heads * L.dim].unflatten(1, (L.heads, L.dim))
        v = kv[:, L.off_v:L.off_v + L.heads * L.vdim].unflatten(1, (L.heads, L.vdim))
        key = torch.cat([kn, kr[:, None, :L.rot].expand(-1, L.heads, -1)], dim=-1)
        j = torch.arange(kv.shape[0])[None]
        s = layout.sidx.long()[:, None]
        vis = (j <= s) & (j > s - window) & (j >= layout.kbase.long()[:, None])
        o = ref.window_attention(q, key, v, vis, scale).flatten(1)
        return (o * torch.sigmoid(inp[:, L.off_g:L.off_g + o.shape[1]].float())).to(inp.dtype)
    k = _k()
    gate = inp[:, L.off_g:]
    out = torch.empty(T, L.ld_o, dtype=inp.dtype, device=inp.device)[:, :L.heads * L.vdim]
    if inp.dtype == BF16:
        from . import latent_attention as A

        if A.supported(L):
            A.stream_attention(L, inp, kv, stream, layout, window, scale, out)
            return out
    a = _WindowAttn(L.heads, L.dim, L.rot, L.vdim, window, 1, scale, inp.stride(0), hd, kv.stride(0), L.dim, stream.stride(0),
                    kv.stride(0), L.vdim, layout.sidx.data_ptr(), layout.kbase.data_ptr(), 0, 0, 0, inp.stride(0), out.stride(0), 0, 0, 1,
                    gate_mult=1.0)
    k.K._check(k.attn(inp.data_ptr(), kv.data_ptr(), kr.data_ptr(), kv[:, L.off_v:].data_ptr(), gate.data_ptr(), out.data_ptr(),
                      C.byref(a), T, _f32(inp), k.K._stream()), "window_attention")
    return out


def ring_attention(L: LatentLayout, inp: torch.Tensor, w_kv: torch.Tensor, norm_w, eps: float, rope, pos, row, cache: torch.Tensor,
                   window: int, scale: float, splits: int, dtype: torch.dtype) -> torch.Tensor:
    """Decode step of a latent-attention layer: append the latents of the newest token of every row (own layers), carry q
    through the key up-projection, attend to the cached latents of the last ``window`` positions, up-project the weighted
    latents to values and gate -> [B, heads * vdim]."""
    B, hd, cap = inp.shape[0], L.dim + L.rot, cache.shape[1]
    assert cap >= window or not bool(inp.is_cuda), "ring shorter than the window"
    if not inp.is_cuda:
        w_uk, w_uv = w_kv[:L.heads * L.dim, :L.rank], w_kv[L.off_v:L.off_v + L.heads * L.vdim, :L.rank]
        p, r = pos.long(), row.long()
        cos, sin = rope[0][p], rope[1][p]
        if L.own:
            cache[r, p % cap] = _latent_rows(L, inp, norm_w, eps, cos, sin).to(dtype)
        q = inp[:, :L.heads * hd].float().unflatten(1, (L.heads, hd))
        qa = torch.einsum("bhd,hdr->bhr", q[..., :L.dim], w_uk.float().unflatten(0, (L.heads, L.dim)))
        ql = torch.zeros(B, L.heads, L.ld_lat)
        ql[..., :L.rank] = qa
        ql[..., L.rank_pad:L.rank_pad + L.rot] = ref.rotate_pairs(q[..., L.dim:], cos[:, None], sin[:, None])
        back = torch.arange(window)[None]                       # key = position p - back
        keys = cache[r[:, None], (p[:, None] - back) % cap]
        lat = keys[:, :, None].expand(-1, -1, L.heads, -1)
        o = ref.window_attention(ql.to(dtype), lat, lat[..., :L.rank], back <= p[:, None], scale)
        o = torch.einsum("bhr,hvr->bhv", o, w_uv.float().unflatten(0, (L.heads, L.vdim))).flatten(1)
        return (o * torch.sigmoid(inp[:, L.off_g:L.off_g + o.shape[1]].float())).to(dtype)
    absorb, attend, expand = ring_attention_pieces(L, inp, w_kv, norm_w, eps, rope, pos, row, cache, window, scale, splits, dtype)
    absorb()
    attend()
    return expand()


def ring_attention_pieces(L: LatentLayout, inp, w_kv, norm_w, eps: float, rope, pos, row, cache, window: int, scale: float, splits: int,
                          dtype):
    """The three launches of ``ring_attention`` on a GPU as callables (the last returns the result)."""
    k = _k()
    B, dev, cap, f32 = inp.shape[0], inp.device, cache.shape[1], int(dtype == F32)
    w_uk, w_uv = w_kv[:L.heads * L.dim], w_kv[L.off_v:L.off_v + L.heads * L.vdim]
    qlat = torch.empty(B, L.heads, L.ld_lat, dtype=dtype, device=dev)
    part_o = torch.empty(B, L.heads, splits, pad8(L.rank), dtype=F32, device=dev)
    part_ml = torch.empty(B, L.heads, splits, 2, dtype=F32, device=dev)
    out = torch.empty(B, L.ld_o, dtype=dtype, device=dev)[:, :L.heads * L.vdim]
    gate = inp[:, L.off_g:]

    def absorb():
        s = _row_struct(L, inp, norm_w, eps, rope, pos, row, cap)
        k.K._check(k.absorb(inp.data_ptr(), C.byref(s), w_uk.data_ptr(), w_kv.stride(0), cache.data_ptr(), qlat.data_ptr(), B, _f32(inp),
                            f32, k.K._stream()), "latent_absorb")

    def attend():
        if dtype == BF16:
            from . import latent_attention as A

            if A.decode_supported(L, cap):
                A.ring_attention(L, qlat, cache, pos, row, part_o, part_ml, window, splits, scale)
                return
        a = _WindowAttn(L.heads, L.ld_lat, 0, L.rank, window, splits, scale, L.heads * L.ld_lat, L.ld_lat, L.ld_lat, 0, 0, L.ld_lat, 0,
                        0, 0, pos.data_ptr(), row.data_ptr(), cap, 0, 0, part_o.data_ptr(), part_ml.data_ptr(), 1)
        k.K._check(k.attn(qlat.data_ptr(), cache.data_ptr(), 0, cache.data_ptr(), 0, 0, C.byref(a), B, f32, k.K._stream()),
                   "window_attention")

    def expand():
        k.K._check(k.expand(part_o.data_ptr(), part_ml.data_ptr(), splits, w_uv.data_ptr(), w_kv.stride(0), gate.data_ptr(), inp.stride(0),
                            out.data_ptr(), out.stride(0), B, L.heads, L.rank, L.vdim, _f32(inp), f32, k.K._stream()), "latent_expand")
        return out

    return absorb, attend, expand
