"""Bindings of the tensor-core kernels of attention with a distance bias (prompts: ``csrc/latent_attention.cu``, decode steps:
``csrc/gqa_decode.cu``) and of chunked matrix memories (``csrc/memory_chunk.cu``)."""
from __future__ import annotations

import ctypes as C
from functools import lru_cache

import torch

from . import cuda as K
from .latent import BF16, F32, pad8

_vp, _i, _f = C.c_void_p, C.c_int, C.c_float


class _GqaDecode(C.Structure):
    _fields_ = [(n, _i) for n in ("H", "G", "dim", "vdim", "ld_in", "off_k", "off_v", "ld_kv", "kv_v", "cap", "splits", "bias_len", "ld_bias",
                                  "bias_lead", "temp_every")] + [(n, _f) for n in ("temp_coef", "scale")] + \
               [(n, _vp) for n in ("in_bias", "bias", "pos", "row", "cache", "part_o", "part_ml")] + \
               [(n, _i) for n in ("size", "chunked", "rot", "ld_first", "ld_fout", "ld_out")] + [(n, _f) for n in ("eps", "softcap")] + \
               [(n, _vp) for n in ("q_norm", "k_norm", "cosT", "sinT", "lam", "first", "first_out", "sink", "out")] + \
               [("keep", _i), ("head_norm", _i), ("bound", _f)]


class _Chunks(C.Structure):
    _fields_ = [(n, _i) for n in ("H", "dim", "vdim", "dimp", "vpad", "vrows", "pk", "pv", "ldv", "ld_in", "ld_out", "gate_t", "gate_h")] + \
               [(n, _f) for n in ("qscale", "cap", "eps")] + \
               [(n, _vp) for n in ("chunks", "seqs", "log2_decay", "gates", "gate_bias", "u", "stat", "s_hi", "s_lo", "n_before", "m_before", "m_init")] + [("group", _i), ("ld_g", _i)] + \
               [(n, _vp) for n in ("prefix", "fk", "state", "stab", "gate_out", "norm_w", "out", "err")]


_attn_ok = K._sig("b200_biased_attention_supported", [_i, _i])
_attn_pad = K._sig("b200_biased_attention_pad", [_i])
_attn = K._sig("b200_biased_attention", [_vp] * 8 + [_i] * 14 + [_f, _f, _f, _vp, _vp])
_dec_ok = K._sig("b200_gqa_decode_supported", [_i, _i])
_dec_per_sm = K._sig("b200_gqa_decode_per_sm", [_i, _i])
_dec = K._sig("b200_gqa_decode", [_vp, C.POINTER(_GqaDecode), _i, _i, _vp])
_chunk_ok = K._sig("b200_memory_chunk_supported", [_i, _i, _i])
_chunk = K._sig("b200_memory_chunks", [_vp] * 3 + [C.POINTER(_Chunks)] + [_i] * 4 + [_vp, _vp])

TILE = 256       # queries per CTA of the prompt attention
CHUNK = 128      # tokens per chunk of a memory
LOG2E = 1.4426950408889634


# ------------------------------------------------------------------------------------------
# attention
# ------------------------------------------------------------------------------------------
@lru_cache(None)
def prompt_supported(L, spec) -> bool:
    """Sizes (and signs of the score factors) that the tensor-core kernel takes; the generic kernel runs otherwise."""
    return bool(_attn_ok(L.dim, L.vdim)) and spec.scale > 0 and (spec.q_temp is None or spec.q_temp.coef >= 0)


@lru_cache(None)
def decode_supported(L) -> bool:
    return bool(_dec_ok(L.dim, L.vdim))


@lru_cache(None)
def decode_slots(L) -> int:
    """CTAs of the decode kernel that the machine holds at a time."""
    return 148 * int(_dec_per_sm(L.dim, L.vdim))


def padded_bias(values: torch.Tensor) -> torch.Tensor:
    """[heads, distances] -> log2 units with repeated values in front and behind, as far as the kernels' accesses reach."""
    lead, tail = _attn_pad(0), _attn_pad(1)
    v = values * LOG2E
    return torch.cat([v[:, :1].expand(-1, lead), v, v[:, -1:].expand(-1, tail)], dim=1).contiguous()


def tile_table(step, cap: int) -> torch.Tensor:
    """(first query token, queries, key index of the first query, key index of position 0) per CTA, most visible keys first."""
    tiles = step.derived.get(("tiles", cap))
    if tiles is None:
        t = [(t0 + i, min(TILE, n - i), row * cap + start + i, row * cap) for t0, n, row, start in step.sequences() for i in range(0, n, TILE)]
        t.sort(key=lambda x: -(x[1] + x[2] - x[3]))
        tiles = step.derived["tiles", cap] = torch.tensor(t, dtype=torch.int32).to(step.device)
    return tiles


def prompt_attention(L, spec, inp, cache, table, step, mult: float, out) -> None:
    tiles, t = tile_table(step, cache.shape[1]), spec.q_temp
    bias = table.padded()
    K._check(_attn(inp.data_ptr(), cache.data_ptr(), cache[:, :, L.kv_v:].data_ptr(), inp[:, L.off_lg:].data_ptr(), out.data_ptr(),
                   tiles.data_ptr(), bias.data_ptr(), table.ids.data_ptr(), tiles.shape[0], inp.shape[0], cache.shape[0] * cache.shape[1],
                   L.heads, L.kv_heads, L.dim, L.vdim, inp.stride(0), L.ld_kv, inp.stride(0), out.stride(0), table.ids.numel(), bias.shape[1],
                   0 if t is None else t.every, 0.0 if t is None else t.coef, spec.scale, mult, K._stream(), K.err_word(inp.device).data_ptr()),
             "biased_attention")


def decode_attention(L, spec, inp, in_bias, cache, table, pos, row, part_o, part_ml) -> None:
    """Appends the new token's key and value and leaves the unnormalised partials and (max, sum) of every key split."""
    bias, t = table.padded(), spec.q_temp
    p = _GqaDecode(L.heads, L.kv_heads, L.dim, L.vdim, inp.stride(0), L.off_k, L.off_v, L.ld_kv, L.kv_v, cache.shape[1], part_o.shape[2],
                   table.ids.numel(), bias.shape[1], _attn_pad(0), 0 if t is None else t.every, 0.0 if t is None else t.coef, spec.scale,
                   in_bias.data_ptr(), bias.data_ptr(), pos.data_ptr(), row.data_ptr(), cache.data_ptr(), part_o.data_ptr(), part_ml.data_ptr())
    K._check(_dec(inp.data_ptr(), C.byref(p), inp.shape[0], int(inp.dtype == F32), K._stream()), "gqa_decode")


# ------------------------------------------------------------------------------------------
# memories
# ------------------------------------------------------------------------------------------
@lru_cache(None)
def chunk_supported(dim: int, vdim: int, gated: bool) -> bool:
    return bool(_chunk_ok(dim, vdim, int(gated)))


def chunk_tables(step) -> tuple:
    """Per chunk (first token, tokens, sequence, where its sequence's state comes from: cache row, -1 nowhere, -2 not its first
    chunk) and per sequence (first chunk, chunks, cache row, first position)."""
    if "chunks" not in step.derived:
        chunks, seqs = [], []
        for s, (t0, n, row, start) in enumerate(step.sequences()):
            seqs.append((len(chunks), (n + CHUNK - 1) // CHUNK, row, start))
            chunks += [(t0 + i, min(CHUNK, n - i), s, -2 if i else row if start else -1) for i in range(0, n, CHUNK)]
        step.derived["chunks"] = tuple(torch.tensor(x, dtype=torch.int32).to(step.device) for x in (chunks, seqs))
    return step.derived["chunks"]


def _chunked(step, q, k, v, H: int, dim: int, vdim: int, ldv: int, out, state, qscale=1.0, decay=None, gates=None, gate_bias=None, cap=1.0,
             stab=None, gate_out=None, norm_w=None, eps=0.0):
    """The three launches of a chunked memory, as a callable taking a mask of the parts to run."""
    chunks, seqs = chunk_tables(step)
    n, S, dev, gated = chunks.shape[0], seqs.shape[0], q.device, gates is not None
    vpad = (vdim + 15) // 16 * 16
    u = torch.empty(n * H, vpad + (16 if gated else 0), dim, dtype=F32, device=dev)
    hi, lo = (torch.empty(n * H, vpad, dim, dtype=BF16, device=dev) for _ in range(2))
    nb = torch.empty(n * H, dim, dtype=F32, device=dev) if gated else None
    scal = torch.empty(3 * n * H + S * H, dtype=F32, device=dev)
    stat, m_before, m_init = scal[:2 * n * H], scal[2 * n * H:3 * n * H], scal[3 * n * H:]
    p = K._ptr
    c = _Chunks(H, dim, vdim, 0, 0, 0, 0, 0, ldv, q.stride(0), out.stride(0), 0 if gates is None else gates.stride(0), 0 if gates is None else gates.stride(1),
                qscale, cap, eps,
                chunks.data_ptr(), seqs.data_ptr(), p(decay), p(gates), p(gate_bias), u.data_ptr(), stat.data_ptr(), hi.data_ptr(), lo.data_ptr(),
                p(nb), m_before.data_ptr(), m_init.data_ptr(), state=state.data_ptr(), stab=p(stab), gate_out=p(gate_out), norm_w=p(norm_w), out=out.data_ptr())
    keep = (u, hi, lo, nb, scal, q, decay, gates, gate_bias, state, stab, gate_out, norm_w)      # alive as long as the callable

    def run(parts: int = 7):
        assert keep
        K._check(_chunk(q.data_ptr(), k.data_ptr(), v.data_ptr(), C.byref(c), q.shape[0], n, S, parts, K._stream(), K.err_word(dev).data_ptr()),
                 "memory_chunks")
        return out

    return run


def decay_memory(L, inp, log2_decay, state, step):
    """[T, r_heads * r_vdim] bf16 outputs of a packed step; see ``memory.decay_memory_prompt``."""
    W = L.r_heads * L.r_vdim
    out = torch.empty(inp.shape[0], pad8(W), dtype=BF16, device=inp.device)[:, :W]
    return _chunked(step, inp[:, L.off_rq:], inp[:, L.off_rk:], inp[:, L.off_rv:], L.r_heads, L.r_dim, L.r_vdim, L.ldv, out, state,
                    decay=log2_decay)


def gated_memory(L, inp, gates, gate_bias, cap: float, state, stab, norm_w, eps: float, step):
    """[T, heads * vdim] bf16 outputs of a packed step; see ``memory.gated_memory``."""
    W = L.heads * L.vdim
    out = torch.empty(inp.shape[0], pad8(W), dtype=BF16, device=inp.device)[:, :W]
    return _chunked(step, inp[:, L.off_q:], inp[:, L.off_k:], inp[:, L.off_v:], L.heads, L.dim, L.vdim, L.ldv, out, state, L.dim ** -0.5,
                    None, gates, gate_bias, cap, stab, inp[:, L.off_g:], norm_w, eps)
