"""Ops of matrix memories with the gated delta rule behind short convolutions: CUDA tensors run the kernels of ``csrc/delta.cu`` and the
tensor-core kernels bound in ``ops/delta_kernels.py``, CPU tensors the plain statements of ``reference``.  A CUDA tensor never takes the
plain path.

Conventions as in ``ops/latent.py``.  The inputs of a convolution that a sequence still needs lie in a ring [rows, taps, channels], that
of position p in slot p % taps; a step at position 0 starts from nothing, so a row that is used again needs no clearing."""
from __future__ import annotations

import ctypes as C
from dataclasses import dataclass, field

import torch

from . import reference as ref
from .latent import BF16, F32, _f32, pad8
from .memory import _heads, _offsets, _Rows, pad4


@dataclass(frozen=True)
class DeltaLayout:
    """Columns of a projection row [q | k | v | output gate | step sizes, decays]; the first three are the convolution's channels."""

    heads: int
    kv_heads: int
    dim: int
    vdim: int
    width_in: int = field(init=False)

    def __post_init__(self):
        put = lambda k, v: object.__setattr__(self, k, v)  # noqa: E731
        qk, v = self.kv_heads * self.dim, self.heads * self.vdim
        put("width_in", _offsets(put, q=qk, k=qk, v=v, g=v, ba=2 * self.heads))
        put("channels", self.off_g)
        put("ldv", pad4(self.vdim))


@dataclass
class DeltaWeights:
    """``conv`` [taps, channels], ``a_log`` and ``dt_bias`` [heads], ``norm`` [vdim]; fp32."""

    conv: torch.Tensor
    a_log: torch.Tensor
    dt_bias: torch.Tensor
    norm: torch.Tensor
    eps: float


class _Conv(C.Structure):
    _fields_ = [(n, C.c_int) for n in ("ch", "taps", "ld_in", "ld_out")] + [(n, C.c_void_p) for n in ("w", "chunks", "seqs")]


class _Delta(C.Structure):
    _fields_ = [(n, C.c_int) for n in ("H", "G", "dim", "vdim", "ldv", "ld_in", "off_q", "off_k", "off_v", "ld_g", "off_g", "off_ba", "ba_t", "ba_h", "ld_out",
                                       "ch", "taps")] + [("qscale", C.c_float), ("eps", C.c_float)] + \
               [(n, C.c_void_p) for n in ("seqs", "pos", "row", "ba", "a_log", "dt_bias", "norm_w", "conv_w", "state")]


_fns = None


def _k():
    global _fns
    if _fns is None:
        from types import SimpleNamespace

        from . import cuda as K

        vp, i = C.c_void_p, C.c_int
        _fns = SimpleNamespace(K=K, conv=K._sig("b200_short_conv", [vp] * 3 + [C.POINTER(_Conv), i, i, vp]),
                               scan=K._sig("b200_delta_scan", [vp] * 4 + [C.POINTER(_Delta)] + [i] * 4 + [vp]))
    return _fns


# ------------------------------------------------------------------------------------------
# plain forms
# ------------------------------------------------------------------------------------------
def _plain_conv(L: DeltaLayout, x: torch.Tensor, w: torch.Tensor, ring: torch.Tensor, seqs) -> torch.Tensor:
    """silu(convolution) of projection rows x, fp32; the rings are carried on."""
    taps, ch = w.shape
    out = torch.empty(x.shape[0], ch)
    for t0, n, row, start in seqs:
        back = torch.arange(start - taps + 1, start)                       # positions in front of the portion
        front = torch.where((back >= 0)[:, None], ring[row, back % taps].float(), 0.0)
        rows = x[t0:t0 + n, :ch]
        full = torch.cat([front, rows.float()])
        out[t0:t0 + n] = torch.nn.functional.silu(sum(w[j] * full[j:j + n] for j in range(taps)))
        m = min(taps, n)
        ring[row, torch.arange(start + n - m, start + n) % taps] = rows[n - m:].to(ring.dtype)
    return out


def _plain(L: DeltaLayout, w: DeltaWeights, act, z, ba, state, seqs, dtype) -> torch.Tensor:
    H, G, T = L.heads, L.kv_heads, act.shape[0]
    q, k = (ref.unit(_heads(act, at, G, L.dim), 1e-6).repeat_interleave(H // G, dim=1) for at in (L.off_q, L.off_k))
    v, gate = _heads(act, L.off_v, H, L.vdim), _heads(z, L.off_g, H, L.vdim)
    beta = torch.sigmoid(ba[:, :H].float())
    log_g = -torch.exp(w.a_log) * torch.nn.functional.softplus(ba[:, H:2 * H].float() + w.dt_bias, threshold=100.0)
    out = torch.zeros(T, pad8(H * L.vdim), dtype=dtype)[:, :H * L.vdim]
    for t0, n, row, start in seqs:
        s = state[row][..., :L.vdim]
        if start == 0:
            s.zero_()
        e = slice(t0, t0 + n)
        o = ref.delta_scan(q[e] * L.dim ** -0.5, k[e], v[e], beta[e], log_g[e], s)
        out[e] = (ref.rms(o, w.eps) * w.norm * torch.nn.functional.silu(gate[e])).flatten(1).to(dtype)
    return out


# ------------------------------------------------------------------------------------------
# prompts
# ------------------------------------------------------------------------------------------
def short_conv(L: DeltaLayout, inp: torch.Tensor, w: torch.Tensor, ring: torch.Tensor, step) -> torch.Tensor:
    """Activated channels [T, channels] of a packed step's projection rows; the sequences' rings are carried on."""
    if not inp.is_cuda:
        return _plain_conv(L, inp, w, ring, step.sequences()).to(inp.dtype)
    from .memory_kernels import chunk_tables

    k = _k()
    chunks, seqs = chunk_tables(step)
    out = torch.empty(inp.shape[0], L.channels, dtype=inp.dtype, device=inp.device)
    c = _Conv(L.channels, w.shape[0], inp.stride(0), out.stride(0), w.data_ptr(), chunks.data_ptr(), seqs.data_ptr())
    assert ring.is_contiguous() and ring.dtype == inp.dtype and w.is_contiguous()
    k.K._check(k.conv(inp.data_ptr(), out.data_ptr(), ring.data_ptr(), C.byref(c), chunks.shape[0], _f32(inp), k.K._stream()), "short_conv")
    return out


def _struct(L: DeltaLayout, w: DeltaWeights, rows, z, out, state, seqs=None, pos=None, row=None, ba=None) -> _Delta:
    p = _k().K._ptr
    return _Delta(L.heads, L.kv_heads, L.dim, L.vdim, L.ldv, rows.stride(0), L.off_q, L.off_k, L.off_v, z.stride(0), L.off_g, L.off_ba,
                  0 if ba is None else ba.stride(0), 0 if ba is None else ba.stride(1), out.stride(0), L.channels, w.conv.shape[0], L.dim ** -0.5, w.eps,
                  p(seqs), p(pos), p(row), p(ba), w.a_log.data_ptr(), w.dt_bias.data_ptr(), w.norm.data_ptr(), w.conv.data_ptr(), state.data_ptr())


def delta_prompt(L: DeltaLayout, w: DeltaWeights, act: torch.Tensor, inp: torch.Tensor, ba: torch.Tensor, state: torch.Tensor, step) -> torch.Tensor:
    """Normed and gated read-outs [T, heads * vdim] of a packed step: activated channels ``act``, projection rows ``inp`` (the output gate)
    and fp32 projections ``ba`` [T, 2 heads] of step sizes and decays; the sequences' states are carried on."""
    if not inp.is_cuda:
        return _plain(L, w, act, inp, ba, state, step.sequences(), inp.dtype)
    W = L.heads * L.vdim
    out = torch.empty(inp.shape[0], pad8(W), dtype=inp.dtype, device=inp.device)[:, :W]
    if inp.dtype == BF16:
        from . import delta_kernels as DK

        if DK.supported(L):
            return DK.delta_prompt(L, w, act, inp, ba, state, step, out)()
    k = _k()
    m = _struct(L, w, act, inp, out, state, seqs=step.seq_table, ba=ba)
    k.K._check(k.scan(act.data_ptr(), inp.data_ptr(), 0, out.data_ptr(), C.byref(m), len(step.portions), 0, _f32(inp), _f32(inp), k.K._stream()),
               "delta_scan")
    return out


# ------------------------------------------------------------------------------------------
# decode steps
# ------------------------------------------------------------------------------------------
def delta_decode(L: DeltaLayout, w: DeltaWeights, inp: torch.Tensor, ring: torch.Tensor, state: torch.Tensor, pos, row, dtype: torch.dtype) -> torch.Tensor:
    """One token per row, from its projection row to the input of the output projection."""
    B, W = inp.shape[0], L.heads * L.vdim
    if not inp.is_cuda:
        seqs = _Rows(pos, row).sequences()
        act = _plain_conv(L, inp, w.conv, ring, seqs)
        return _plain(L, w, act, inp, inp[:, L.off_ba:], state, seqs, dtype)
    k = _k()
    out = torch.empty(B, pad8(W), dtype=dtype, device=inp.device)[:, :W]
    m = _struct(L, w, inp, inp, out, state, pos=pos, row=row)
    k.K._check(k.scan(inp.data_ptr(), inp.data_ptr(), ring.data_ptr(), out.data_ptr(), C.byref(m), B, 1, _f32(inp), int(dtype == F32), k.K._stream()),
               "delta_scan")
    return out
