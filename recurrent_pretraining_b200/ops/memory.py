"""Ops of the layered decoder models that mix distance-biased attention with recurrent matrix memories: CUDA tensors run the
kernels of ``csrc/memory.cu``, ``csrc/latent.cu`` and the tensor-core kernels bound in ``ops/memory_kernels.py``, CPU tensors the
plain statements of ``reference``.  A CUDA tensor never takes the plain path.

Conventions as in ``ops/latent.py``.  A projection row is "raw" when it is the accumulator of a decode step's product:
biases and activations are then applied by the kernels that read it."""
from __future__ import annotations

import ctypes as C
from dataclasses import dataclass, field
from functools import lru_cache
from typing import Optional

import torch

from . import latent as base
from . import reference as ref
from .latent import BF16, F32, _f32, linear, pad8


def pad4(n: int) -> int:
    return (n + 3) // 4 * 4


def _offsets(put, **widths) -> int:
    """Set ``off_<name>`` of consecutive column blocks padded to eight; returns the total."""
    at = 0
    for name, w in widths.items():
        put("off_" + name, at)
        at += pad8(w)
    return at


@dataclass(frozen=True)
class ParallelLayout:
    """Columns of a parallel layer's projection row [q | k | v | head gates | memory q | k | v | gate], cache row [k | v] and
    output-projection input [heads | memory heads]."""

    heads: int
    kv_heads: int
    dim: int
    vdim: int
    r_heads: int
    r_dim: int
    r_vdim: int
    width_in: int = field(init=False)

    def __post_init__(self):
        put = lambda k, v: object.__setattr__(self, k, v)  # noqa: E731
        hd, hv = self.r_heads * self.r_dim, self.r_heads * self.r_vdim
        put("width_in", _offsets(put, q=self.heads * self.dim, k=self.kv_heads * self.dim, v=self.kv_heads * self.vdim, lg=self.heads,
                                 rq=hd, rk=hd, rv=hv, rg=hv))
        put("kv_v", self.off_v - self.off_k)                       # values inside a cache row
        put("ld_kv", self.off_lg - self.off_k)
        put("off_r", pad8(self.heads * self.vdim))                 # memory part of the output-projection input
        put("width_o", self.off_r + hv)
        put("ldv", pad4(self.r_vdim))

    @property
    def act_cols(self) -> tuple:
        """Columns whose projections go through silu."""
        return self.off_rq, self.off_rg


@dataclass(frozen=True)
class MemoryLayout:
    """Columns of a gated memory's projection row [q | k | v | gate]."""

    heads: int
    dim: int
    vdim: int
    width_in: int = field(init=False)

    def __post_init__(self):
        put = lambda k, v: object.__setattr__(self, k, v)  # noqa: E731
        hd, hv = self.heads * self.dim, self.heads * self.vdim
        put("width_in", _offsets(put, q=hd, k=hd, v=hv, g=hv))
        put("ldv", pad4(self.vdim))


class _Sandwich(C.Structure):
    _fields_ = [(n, C.c_int) for n in ("E", "ld_a", "ld_h", "clear", "nzero")] + [(n, C.c_float) for n in ("eps", "bias_mult", "out_mult")] + \
               [(n, C.c_void_p) for n in ("bias", "w1", "b1", "step", "w2", "b2", "x", "zero")] + \
               [(n, C.c_int) for n in ("top", "ld_mix", "ld_shared")] + [(n, C.c_void_p) for n in ("slot", "weight", "mix_h", "shared")]


class _Memory(C.Structure):
    _fields_ = [(n, C.c_int) for n in ("H", "dim", "vdim", "ldv", "ld_in", "off_q", "off_k", "off_v", "off_g", "ld_out", "E", "ld_h", "ld_w", "gate_t", "gate_h",
                                       "silu", "stage")] + [(n, C.c_float) for n in ("qscale", "cap", "eps")] + \
               [(n, C.c_void_p) for n in ("seqs", "pos", "row", "decay", "gates", "gate_bias", "state", "stab", "norm_w", "out32")]


class _Merge(C.Structure):
    _fields_ = [(n, C.c_int) for n in ("H", "vdim", "splits", "HR", "rvdim", "ld_in", "off_lg", "off_rg", "ld_mem", "ld_out", "off_r")] + \
               [(n, C.c_float) for n in ("left_scale", "right_scale", "eps")] + [(n, C.c_void_p) for n in ("part_o", "part_ml", "norm_w")]


_fns = None


def _k():
    global _fns
    if _fns is None:
        from types import SimpleNamespace

        from . import cuda as K

        vp, i, f = C.c_void_p, C.c_int, C.c_float
        _fns = SimpleNamespace(
            K=K,
            sandwich=K._sig("b200_sandwich_norm", [vp, vp, C.POINTER(_Sandwich), i, i, i, i, vp]),
            rows=K._sig("b200_layernorm_rows", [vp] * 5 + [i] * 3 + [f, i, vp]),
            glu=K._sig("b200_glu", [vp] + [i] * 3 + [vp] + [i] * 5 + [vp]),
            append=K._sig("b200_kv_append", [vp, i, vp, vp] + [i] * 3 + [vp, vp] + [i] * 3 + [vp]),
            scan=K._sig("b200_memory_scan", [vp] * 4 + [C.POINTER(_Memory)] + [i] * 3 + [vp]),
            merge=K._sig("b200_memory_merge", [vp] * 3 + [C.POINTER(_Merge)] + [i] * 4 + [vp]),
        )
    return _fns


# ------------------------------------------------------------------------------------------
# layer norms, feed-forward
# ------------------------------------------------------------------------------------------
def _norm(x, w, b, eps: float) -> torch.Tensor:
    """Plain form: layer norm, or without ``b`` the RMS norm with weights 1 + w."""
    return ref.rms(x, eps) * (1 + w) if b is None else ref.layer_norm(x, w, b, eps)


@dataclass
class RowSum:
    """A sublayer output that is still a sum: row t is sum_k weight[t, k] rows[slot[t, k]] (h[t] where the slot is negative)
    + weight[t, top] shared[t].  ``rows`` and ``shared`` (or None) have one dtype (fp32 where the norm kernel forms the sum), ``h`` is in operand precision."""

    rows: torch.Tensor
    slot: torch.Tensor
    weight: torch.Tensor
    h: torch.Tensor
    shared: Optional[torch.Tensor] = None

    @property
    def shape(self):
        return self.h.shape

    def sum(self) -> torch.Tensor:
        """Plain form."""
        pick = self.slot.long()
        y = torch.where((pick < 0)[..., None], self.h[:, None].float(), self.rows[pick.clamp(min=0)].float())
        out = (self.weight[:, :-1, None] * y).sum(1)
        return out if self.shared is None else out + self.weight[:, -1:] * self.shared.float()


def sandwich_norm_(x: torch.Tensor, a, post, step, pre, eps: float, dtype: torch.dtype, bias=None,
                   bias_mult: float = 1.0, clear: bool = False, zero: Optional[torch.Tensor] = None,
                   out_mult: float = 1.0) -> Optional[torch.Tensor]:
    """x += norm(a + bias_mult * bias) [+ step] in place, then out_mult * norm(x) in ``dtype`` (None without ``pre``).  ``post``
    and ``pre`` are (weight, bias) of layer norms, or (weight, None) of RMS norms whose weights are stored around zero; ``a``
    may be None (only ``step`` is added then) or, with RMS norms, a ``RowSum``.  ``clear`` / ``zero``: accumulators that are handed back zeroed (a itself / a
    second one with the same number of rows)."""
    T, E = x.shape
    if not x.is_cuda:
        if a is not None:
            a = a.sum() if isinstance(a, RowSum) else a
            s = a.float() if bias is None else a.float() + bias_mult * bias
            x += _norm(s, *post, eps)
        if step is not None:
            x += step
        return None if pre is None else (_norm(x, *pre, eps) * out_mult).to(dtype)
    k = _k()
    assert x.is_contiguous() and (a is None or a.shape == (T, E)) and (zero is None or zero.is_contiguous())
    h = None if pre is None else torch.empty(T, pad8(E), dtype=dtype, device=x.device)[:, :E]
    p = k.K._ptr
    w1, b1 = post if a is not None else (None, None)
    w2, b2 = pre if pre is not None else (None, None)
    many = {}
    if isinstance(a, RowSum):
        assert a.h.dtype == dtype and a.rows.dtype == F32 and (a.shared is None or a.shared.dtype == a.rows.dtype) and a.weight.is_contiguous() and a.slot.is_contiguous()
        many = dict(top=a.weight.shape[1] - 1, ld_mix=a.h.stride(0), ld_shared=0 if a.shared is None else a.shared.stride(0), slot=p(a.slot),
                    weight=p(a.weight), mix_h=p(a.h), shared=p(a.shared))
        a = a.rows
    s = _Sandwich(E, 0 if a is None else a.stride(0), 0 if h is None else h.stride(0), int(clear), 0 if zero is None else zero.numel() // T,
                  eps, bias_mult, out_mult, p(bias), p(w1), p(b1), p(step), p(w2), p(b2), x.data_ptr(), p(zero), **many)
    f32, rms = int(dtype == F32), int(b1 is None and b2 is None)
    k.K._check(k.sandwich(p(a), p(h), C.byref(s), T, f32 if a is None else _f32(a), f32, rms, k.K._stream()), "sandwich_norm")
    return h


def norm_rows(x: torch.Tensor, idx: Optional[torch.Tensor], w, b, eps: float, dtype: torch.dtype, mult: float = 1.0) -> torch.Tensor:
    """mult * norm(x[idx]) in ``dtype`` (all rows when ``idx`` is None); the norm as in ``sandwich_norm_``."""
    if b is None:
        return base.rmsnorm_rows(x, idx, w, eps, dtype, 1.0, mult)
    assert mult == 1.0
    if not x.is_cuda:
        return ref.layer_norm(x if idx is None else x[idx.long()], w, b, eps).to(dtype)
    k = _k()
    n, E = (x.shape[0] if idx is None else idx.numel()), x.shape[1]
    y = torch.empty(n, pad8(E), dtype=dtype, device=x.device)[:, :E]
    k.K._check(k.rows(x.data_ptr(), k.K._ptr(idx), w.data_ptr(), b.data_ptr(), y.data_ptr(), y.stride(0), n, E, eps, int(dtype == F32),
                      k.K._stream()), "layernorm_rows")
    return y


def glu(a: torch.Tensor, n: int, act: str, dtype: torch.dtype, clear: bool = False) -> torch.Tensor:
    """act(a[:, :n]) * a[:, n:2n] in ``dtype``, act "gelu" (tanh form) or "silu"; ``clear`` hands a stream-K accumulator back
    zeroed."""
    M = a.shape[0]
    if not a.is_cuda:
        g = a[:, :n].float()
        g = torch.nn.functional.silu(g) if act == "silu" else torch.nn.functional.gelu(g, approximate="tanh")
        return (g * a[:, n:2 * n].float()).to(dtype)
    k = _k()
    y = torch.empty(M, pad8(n), dtype=dtype, device=a.device)[:, :n]
    k.K._check(k.glu(a.data_ptr(), a.stride(0), _f32(a), int(clear), y.data_ptr(), y.stride(0), M, n, int(act == "silu"), int(dtype == F32),
                     k.K._stream()), "glu")
    return y


def glu_linear(x: torch.Tensor, w: torch.Tensor, n: int, act: str) -> torch.Tensor:
    """act(x Wg^T) * (x Wu^T) for ``w`` [2n, K] = [Wg; Wu]; bf16: gated in the epilogue of the product."""
    if not x.is_cuda or x.dtype == F32:
        return glu(linear(x, w), n, act, x.dtype)
    k = _k()
    out = torch.empty(x.shape[0], pad8(n), dtype=x.dtype, device=x.device)[:, :n]
    return k.K.gemm(x, w, out=out, out_mode=k.K.OUT_SWIGLU, act=0 if act == "silu" else 3)


# ------------------------------------------------------------------------------------------
# attention
# ------------------------------------------------------------------------------------------
@dataclass
class BiasTable:
    """Distance bias of one layer in the form the kernels read: ``values`` [heads, distances], the last of which holds for every
    farther distance; ``ids`` the bucket of each distance."""

    values: torch.Tensor
    ids: torch.Tensor
    _padded: Optional[torch.Tensor] = None

    def padded(self) -> torch.Tensor:
        """The form of the tensor-core kernels (log2 units, repeated at both ends)."""
        if self._padded is None:
            from .memory_kernels import padded_bias

            self._padded = padded_bias(self.values)
        return self._padded

    @classmethod
    def build(cls, rel: torch.Tensor, buckets: list) -> "BiasTable":
        ids = torch.tensor(buckets, dtype=torch.int64)
        return cls(rel.float()[ids.to(rel.device)].T.contiguous(), ids.to(torch.int32).to(rel.device))


def kv_append(L: ParallelLayout, inp: torch.Tensor, bias, cache: torch.Tensor, pos, row) -> None:
    """Keys and values of the projection rows -> cache [rows, max_len, ld_kv] (``bias``: of the raw row, else None)."""
    kv = inp[:, L.off_k:L.off_k + L.ld_kv]
    b = None if bias is None else bias[L.off_k:L.off_k + L.ld_kv]
    if not inp.is_cuda:
        cache[row.long(), pos.long()] = (kv.float() if b is None else kv.float() + b).to(cache.dtype)
        return
    k = _k()
    k.K._check(k.append(kv.data_ptr(), inp.stride(0), k.K._ptr(b), cache.data_ptr(), L.ld_kv, L.ld_kv, cache.shape[1], pos.data_ptr(),
                        row.data_ptr(), inp.shape[0], _f32(inp), _f32(cache), k.K._stream()), "kv_append")


def _plain_attention(L, spec, q, cache_row, table, pos):
    """Attention [T, H, vdim] of one sequence on the CPU."""
    n = int(pos[-1]) + 1
    k = cache_row[:n, :L.kv_heads * L.dim].unflatten(1, (L.kv_heads, L.dim))
    v = cache_row[:n, L.kv_v:L.kv_v + L.kv_heads * L.vdim].unflatten(1, (L.kv_heads, L.vdim))
    t = torch.tensor([spec.q_temp.at(int(p)) if spec.q_temp else 1.0 for p in pos])
    return ref.biased_attention(q.unflatten(1, (L.heads, L.dim)), k, v, table.values, pos.long(), t * spec.scale)


def _attn_struct(L, spec, table, q_stride: int, window: int, splits: int = 1, **kw) -> base._WindowAttn:
    t = spec.q_temp
    return base._WindowAttn(L.heads, L.dim, 0, L.vdim, window, splits, spec.scale, q_stride, L.dim, L.ld_kv, L.dim, 0, L.ld_kv, L.vdim,
                            group=L.heads // L.kv_heads, bias=table.values.data_ptr(), bias_len=table.values.shape[1],
                            temp_every=0 if t is None else t.every, temp_coef=0.0 if t is None else t.coef, head_gate=1, **kw)


def prompt_attention(L: ParallelLayout, spec, inp: torch.Tensor, cache: torch.Tensor, table: BiasTable, step, mult: float, out: torch.Tensor) -> None:
    """Gated attention of a packed step's queries over the cached keys of their sequences (the step's own are appended
    already): out[:, :heads * vdim] = mult * sigmoid(gate) * attention."""
    T = inp.shape[0]
    if not inp.is_cuda:
        for t0, n, row, start in step.sequences():
            o = _plain_attention(L, spec, inp[t0:t0 + n, :L.heads * L.dim], cache[row], table, step.pos[t0:t0 + n])
            g = torch.sigmoid(inp[t0:t0 + n, L.off_lg:L.off_lg + L.heads].float()) * mult
            out[t0:t0 + n, :L.heads * L.vdim] = (o * g[:, :, None]).flatten(1).to(out.dtype)
        return
    if inp.dtype == BF16:
        from . import memory_kernels as MK

        if MK.prompt_supported(L, spec):
            MK.prompt_attention(L, spec, inp, cache, table, step, mult, out)
            return
    k, cap = base._k(), cache.shape[1]
    kbase = step.row * cap                        # key index of position 0
    sidx = kbase + step.pos
    a = _attn_struct(L, spec, table, inp.stride(0), cap, sidx=sidx.data_ptr(), kbase=kbase.data_ptr(), gate_ld=inp.stride(0),
                     out_ld=out.stride(0), gate_mult=mult)
    k.K._check(k.attn(inp.data_ptr(), cache.data_ptr(), 0, cache[:, :, L.kv_v:].data_ptr(), inp[:, L.off_lg:].data_ptr(), out.data_ptr(),
                      C.byref(a), T, _f32(inp), k.K._stream()), "window_attention")


# ------------------------------------------------------------------------------------------
# memories
# ------------------------------------------------------------------------------------------
def gate_projections(h: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """h w^T in fp32 for a few rows of w; the result may be strided.  bf16: the product streams h through the narrow-batch GEMM
    (w takes the batch's place), whose split of the contraction fills the machine where a tiled product would run on T / 128
    CTAs."""
    T, n = h.shape[0], w.shape[0]
    if h.is_cuda and h.dtype == BF16 and n <= 64 and 256 <= T <= 128 * 147 and h.shape[1] >= 512:
        from ..engine.base import skinny_linear

        work = torch.zeros(n * T, dtype=F32, device=h.device)
        out = skinny_linear(w, h, work, keep_f32=True)
        if out.dtype == F32:
            return out.T
    return linear(h, w, out_f32=True)


def _heads(inp, at: int, H: int, n: int) -> torch.Tensor:
    return inp[:, at:at + H * n].float().unflatten(1, (H, n))


def _rms_gate(o: torch.Tensor, eps: float, w, gate) -> torch.Tensor:
    return ref.rms(o, eps) * w * torch.sigmoid(gate.float())


def decay_memory_prompt(L: ParallelLayout, inp: torch.Tensor, decay: torch.Tensor, log2_decay: torch.Tensor, state: torch.Tensor,
                        step) -> torch.Tensor:
    """Memory outputs [T, r_heads * r_vdim] of a packed step (activated projections); the sequences' states are carried on."""
    T, H = inp.shape[0], L.r_heads
    if not inp.is_cuda:
        out = torch.empty(T, H * L.r_vdim)
        for t0, n, row, start in step.sequences():
            x, s = inp[t0:t0 + n], state[row][..., :L.r_vdim]
            if start == 0:
                s.zero_()
            out[t0:t0 + n] = ref.memory_scan(_heads(x, L.off_rq, H, L.r_dim), _heads(x, L.off_rk, H, L.r_dim),
                                             _heads(x, L.off_rv, H, L.r_vdim), s, decay).flatten(1)
        return out
    if inp.dtype == BF16:
        from . import memory_kernels as MK

        if MK.chunk_supported(L.r_dim, L.r_vdim, False):
            return MK.decay_memory(L, inp, log2_decay, state, step)()
    return _decay_scan(L, inp, decay, state, step.seq_table, None, None, len(step.portions), 0)


def _decay_scan(L, inp, decay, state, seqs, pos, row, n: int, raw: int, out=None) -> torch.Tensor:
    k = _k()
    p = k.K._ptr
    if out is None:
        out = torch.empty(inp.shape[0], pad8(L.r_heads * L.r_vdim), dtype=F32, device=inp.device)[:, :L.r_heads * L.r_vdim]
    m = _Memory(L.r_heads, L.r_dim, L.r_vdim, L.ldv, inp.stride(0), L.off_rq, L.off_rk, L.off_rv, 0, out.stride(0), 0, 0, 0, 0, 0, raw, 0, 1.0, 1.0, 0.0,
                p(seqs), p(pos), p(row), decay.data_ptr(), 0, 0, state.data_ptr(), 0, 0, out.data_ptr())
    k.K._check(k.scan(inp.data_ptr(), 0, 0, 0, C.byref(m), n, _f32(inp), 0, k.K._stream()), "memory_scan")
    return out


def memory_norm(L: ParallelLayout, inp: torch.Tensor, mem: torch.Tensor, norm_w: torch.Tensor, eps: float, mult: float, out: torch.Tensor,
                attn=None, left_scale: float = 1.0) -> None:
    """out[:, off_r:] = mult * rms(all memory heads) * norm_w * sigmoid(gate); ``attn`` = (partials, maxima and sums) of a decode
    step's attention: merged, gated and stored in out[:, :heads * vdim] as well."""
    W = L.r_heads * L.r_vdim
    if not inp.is_cuda:
        out[:, L.off_r:L.off_r + W] = (mult * _rms_gate(mem, eps, norm_w, inp[:, L.off_rg:L.off_rg + W])).to(out.dtype)
        return
    k = _k()
    po, ml = attn if attn is not None else (None, None)
    a = _Merge(L.heads if attn is not None else 0, L.vdim, ml.shape[2] if attn is not None else 0, L.r_heads, L.r_vdim, inp.stride(0), L.off_lg,
               L.off_rg, mem.stride(0), out.stride(0), L.off_r, left_scale, mult, eps, k.K._ptr(po), k.K._ptr(ml), norm_w.data_ptr())
    k.K._check(k.merge(inp.data_ptr(), mem.data_ptr(), out.data_ptr(), C.byref(a), inp.shape[0], _f32(inp), _f32(mem), _f32(out), k.K._stream()),
               "memory_merge")


@lru_cache(None)
def decode_splits(L: ParallelLayout, B: int, max_len: int, tensor_cores: bool) -> int:
    """Key splits of the decode attention for ``B`` rows: the fewest waves of CTAs, each costing its keys and a fixed part worth
    about 256 more."""
    ctas, slots = B * L.heads, 8 * 148                     # generic kernel: a small CTA per head
    if tensor_cores:
        from . import memory_kernels as MK

        if MK.decode_supported(L):
            ctas, slots = B * L.kv_heads * -(-(L.heads // L.kv_heads) // 16), MK.decode_slots(L)
    return min(range(1, min(32, max_len // 64 + 1) + 1), key=lambda s: -(-ctas * s // slots) * (max_len / s + 256))


def parallel_output(L: ParallelLayout, T: int, dtype, device) -> torch.Tensor:
    """Buffer for the input of the output projection; columns between the halves are zero."""
    make = torch.zeros if L.off_r != L.heads * L.vdim else torch.empty
    return make(T, pad8(L.width_o), dtype=dtype, device=device)[:, :L.width_o]


def parallel_decode(L: ParallelLayout, spec, inp: torch.Tensor, bias: torch.Tensor, cache, state, table: BiasTable, decay, norm_w, eps: float,
                    pos, row, splits: int, dtype: torch.dtype) -> torch.Tensor:
    """Both halves of a parallel layer for one token per row: raw projection rows -> input of the output projection."""
    a, B = spec.left, inp.shape[0]
    out = parallel_output(L, B, dtype, inp.device)
    if not inp.is_cuda:
        x = inp.float() + bias
        lo, hi = L.act_cols
        x[:, lo:hi] = torch.nn.functional.silu(x[:, lo:hi])
        kv_append(L, x, None, cache, pos, row)
        for b in range(B):
            r, p = int(row[b]), pos[b:b + 1]
            o = _plain_attention(L, a, x[b:b + 1, :L.heads * L.dim], cache[r], table, p)
            g = torch.sigmoid(x[b:b + 1, L.off_lg:L.off_lg + L.heads]) * spec.left_scale
            out[b, :L.heads * L.vdim] = (o * g[:, :, None]).flatten().to(dtype)
        mem = decay_memory_prompt(L, x, decay, None, state, _Rows(pos, row))
        memory_norm(L, x, mem, norm_w, eps, spec.right_scale, out)
        return out
    po = torch.empty(B, L.heads, splits, pad8(L.vdim), dtype=F32, device=inp.device)
    ml = torch.empty(B, L.heads, splits, 2, dtype=F32, device=inp.device)
    attend, scan, merge = parallel_decode_pieces(L, spec, inp, bias, cache, state, table, decay, norm_w, eps, pos, row, po, ml, out)
    from ..engine.base import PDL

    # the two halves are independent branches of a graph, unless programmatic launch ties every kernel to its one predecessor
    if torch.cuda.is_current_stream_capturing() and not PDL:
        main, side = torch.cuda.current_stream(), _side_stream(inp.device)
        side.wait_stream(main)
        with torch.cuda.stream(side):
            mem = scan()
        attend()
        main.wait_stream(side)
        merge(mem)
    else:
        attend()
        merge(scan())
    return out


@lru_cache(None)
def _side_stream(device) -> "torch.cuda.Stream":
    return torch.cuda.Stream(device)


def parallel_decode_pieces(L, spec, inp, bias, cache, state, table, decay, norm_w, eps, pos, row, po, ml, out):
    """The launches of ``parallel_decode`` on a GPU as callables."""
    a, B, cap = spec.left, inp.shape[0], cache.shape[1]
    dtype, splits = out.dtype, po.shape[2]

    def attend():
        if dtype == BF16:
            from . import memory_kernels as MK

            if MK.decode_supported(L):
                MK.decode_attention(L, a, inp, bias, cache, table, pos, row, po, ml)
                return
        kv_append(L, inp, bias, cache, pos, row)
        q = (inp[:, :L.heads * L.dim].float() + bias[:L.heads * L.dim]).to(dtype)
        k = base._k()
        s = _attn_struct(L, a, table, q.stride(0), cap, splits, pos=pos.data_ptr(), row=row.data_ptr(), cap=cap, part_o=po.data_ptr(),
                         part_ml=ml.data_ptr(), gate_mult=1.0)
        k.K._check(k.attn(q.data_ptr(), cache.data_ptr(), 0, cache[:, :, L.kv_v:].data_ptr(), 0, 0, C.byref(s), B, int(dtype == F32), k.K._stream()),
                   "window_attention")

    mem = torch.empty(B, pad8(L.r_heads * L.r_vdim), dtype=F32, device=inp.device)[:, :L.r_heads * L.r_vdim]

    def scan():
        return _decay_scan(L, inp, decay, state, None, pos, row, B, 1, mem)

    def merge(mem):
        memory_norm(L, inp, mem, norm_w, eps, spec.right_scale, out, (po, ml), spec.left_scale)

    return attend, scan, merge


class _Rows:
    """One token per row in the form of a packed step."""

    def __init__(self, pos, row):
        self.pos, self.row = pos, row

    def sequences(self) -> list:
        return [(b, 1, int(r), int(p)) for b, (p, r) in enumerate(zip(self.pos, self.row))]


def gated_memory(L: MemoryLayout, inp: torch.Tensor, gates, gate_bias: torch.Tensor, cap: float, state, stab, norm_w, eps: float, dtype,
                 step=None, rows=None, h=None, w_gate=None) -> torch.Tensor:
    """Gated matrix memory with its head norms and output gate -> [T, heads * vdim].  ``step``: a packed step with the raw fp32
    gate projections ``gates`` [T, 2 heads]; ``rows`` = (pos, row): one token per row, the projections are formed from the
    input ``h`` and ``w_gate``."""
    T, H = inp.shape[0], L.heads
    hv, qscale = H * L.vdim, L.dim ** -0.5
    if not inp.is_cuda:
        gates = linear(h, w_gate) if gates is None else gates
        li, lf = ref.log_gates(gates, gate_bias, cap)
        out = torch.zeros(T, pad8(hv), dtype=dtype)[:, :hv]
        for t0, n, row, start in (step if step is not None else _Rows(*rows)).sequences():
            x, s, e = inp[t0:t0 + n], state[row][..., :L.vdim], stab[row]
            if start == 0:
                s.zero_()
                e.zero_()
            o = ref.gated_memory_scan(_heads(x, L.off_q, H, L.dim) * qscale, _heads(x, L.off_k, H, L.dim), _heads(x, L.off_v, H, L.vdim),
                                      li[t0:t0 + n], lf[t0:t0 + n], s, e[:, :L.dim], e[:, L.dim])
            o = ref.rms(o, eps).flatten(1) * norm_w * torch.sigmoid(x[:, L.off_g:L.off_g + hv].float())
            out[t0:t0 + n] = o.to(dtype)
        return out
    if step is not None and inp.dtype == BF16:
        from . import memory_kernels as MK

        if MK.chunk_supported(L.dim, L.vdim, True):
            return MK.gated_memory(L, inp, gates, gate_bias, cap, state, stab, norm_w, eps, step)()
    k = _k()
    p = k.K._ptr
    out = torch.empty(T, pad8(hv), dtype=dtype, device=inp.device)[:, :hv]
    pos, row = rows if rows is not None else (None, None)
    m = _Memory(H, L.dim, L.vdim, L.ldv, inp.stride(0), L.off_q, L.off_k, L.off_v, L.off_g, out.stride(0), 0 if h is None else h.shape[1],
                0 if h is None else h.stride(0), 0 if w_gate is None else w_gate.stride(0), 0 if gates is None else gates.stride(0),
                0 if gates is None else gates.stride(1), 0, 0, qscale, cap, eps,
                step.seq_table.data_ptr() if step is not None else 0, p(pos), p(row), 0, p(gates), gate_bias.data_ptr(), state.data_ptr(),
                stab.data_ptr(), norm_w.data_ptr(), 0)
    k.K._check(k.scan(inp.data_ptr(), p(h), p(w_gate), out.data_ptr(), C.byref(m), len(step.portions) if step is not None else T, _f32(inp),
                      int(dtype == F32), k.K._stream()), "memory_scan")
    return out
