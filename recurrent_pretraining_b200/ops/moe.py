"""Ops of mixture-of-experts feed-forwards: CUDA tensors run the kernels of ``csrc/moe.cu`` and grouped matrix products
(``csrc/gemm_tcgen05*.cu``; fp32: ``csrc/latent.cu``), CPU tensors the plain statements of ``reference``.  A CUDA tensor never takes
the plain path.  Nothing of the routing comes back to the host, so every form can be recorded in a graph.

Conventions as in ``ops/latent.py``.  ``MoeWeights`` holds the experts' matrices one below the other."""
from __future__ import annotations

import ctypes as C
from dataclasses import dataclass
from typing import Optional

import torch

from . import latent as base
from . import reference as ref
from .latent import BF16, F32, _f32, pad8
from .memory import RowSum, glu

ROWS = 64            # widest batch of the decode form


@dataclass
class MoeWeights:
    """``router`` [outputs (+ 1 with a shared expert: its gate), E], ``correction`` [outputs] or None, ``up`` [experts * ff, E] (gated experts:
    [experts * 2 ff, E], gate and up rows of an expert in turn), ``down`` [experts * E, ff], ``up_s`` [shared, E], ``down_s`` [E, shared] or None."""

    spec: object
    router: torch.Tensor
    correction: Optional[torch.Tensor]
    up: torch.Tensor
    down: torch.Tensor
    up_s: Optional[torch.Tensor]
    down_s: Optional[torch.Tensor]


class _Route(C.Structure):
    _fields_ = [(n, C.c_int) for n in ("experts", "outputs", "top", "ld_z", "gate", "sigmoid", "normalize", "groups", "keep")] + [(n, C.c_void_p) for n in ("correction", "idx", "weight")]


class _RouteRows(C.Structure):
    _fields_ = [(n, C.c_void_p) for n in ("slot", "active", "first", "row", "n_active")]


class _ExpertRows(C.Structure):
    _fields_ = [(n, C.c_int) for n in ("N", "K", "ld_w", "Ns", "Ks", "ld_ws", "ld_x", "ld_y", "ld_xs", "ld_ys", "B", "act")] + \
               [(n, C.c_void_p) for n in ("w", "ws", "x", "xs")] + [("gather", C.c_int)] + \
               [(n, C.c_void_p) for n in ("y", "ys", "active", "first", "row", "n_active")]


_fns = None


def _k():
    global _fns
    if _fns is None:
        from types import SimpleNamespace

        from . import cuda as K

        vp, i = C.c_void_p, C.c_int
        _fns = SimpleNamespace(
            K=K, max_outputs=int(K._sig("b200_moe_max_outputs", [])()), sgemm_rows=int(K._sig("b200_sgemm_tile_rows", [])()),
            logits=K._sig("b200_moe_router_logits", [vp, i, vp, i, vp] + [i] * 5 + [vp]),
            route=K._sig("b200_moe_route", [vp, C.POINTER(_Route), vp, vp, i, vp]),
            plan=K._sig("b200_moe_plan", [vp, i, i, vp, vp, vp, vp]),
            dispatch=K._sig("b200_moe_dispatch", [vp, i, vp, i, i] + [vp] * 4 + [i] * 3 + [vp]),
            route_rows=K._sig("b200_moe_route_rows", [vp, C.POINTER(_Route), C.POINTER(_RouteRows), i, vp]),
            rows=K._sig("b200_moe_rows", [C.POINTER(_ExpertRows), i, i, i, vp]),
            combine=K._sig("b200_moe_combine", [vp, i] * 3 + [vp, vp, vp] + [i] * 5 + [vp]),
            gemm=K._sig("b200_gemm_grouped", [vp] * 3 + [i] * 7 + [vp, vp] + [i] * 3 + [vp, vp]))
    return _fns


def router_logits(h: torch.Tensor, router: torch.Tensor) -> torch.Tensor:
    """h router^T in fp32 (possibly strided)."""
    if not h.is_cuda:
        return torch.nn.functional.linear(h.float(), router.float())
    B, R = h.shape[0], router.shape[0]
    if B > ROWS:
        from .memory import gate_projections

        z = gate_projections(h, router)
        return z if z.stride(1) == 1 else z.contiguous()
    k = _k()
    z = torch.empty(B, R, dtype=F32, device=h.device)
    if h.dtype == BF16:
        e = _ExpertRows(Ns=R, Ks=h.shape[1], ld_ws=router.stride(0), ld_xs=h.stride(0), ld_ys=R, B=B, ws=router.data_ptr(), xs=h.data_ptr(),
                        ys=z.data_ptr())
        k.K._check(k.rows(C.byref(e), 0, 1, 1, k.K._stream()), "moe_rows")
        return z
    k.K._check(k.logits(h.data_ptr(), h.stride(0), router.data_ptr(), router.stride(0), z.data_ptr(), R, B, R, h.shape[1], _f32(h), k.K._stream()),
               "moe_router_logits")
    return z


def _route_struct(w: MoeWeights, z, idx, weight) -> _Route:
    s = w.spec
    return _Route(s.experts, s.outputs, s.top, z.stride(0), int(w.up_s is not None), int(s.scores == "sigmoid"), int(s.normalized), s.group_count,
                  s.group_keep, _k().K._ptr(w.correction), idx.data_ptr(), weight.data_ptr())


@dataclass
class Slots:
    """Where the chosen experts' rows of a packed step lie: ``idx`` and ``slot`` [T, top] (slot -1: identity expert), ``weight``
    [T, top + 1] (the last one: gate of the shared expert), ``offset`` [experts], ``tile_expert`` of the first ``n_tiles`` tiles of
    ``rows`` slots each; ``size``: slots."""

    idx: torch.Tensor
    slot: torch.Tensor
    weight: torch.Tensor
    rank: torch.Tensor
    offset: torch.Tensor
    tile_expert: torch.Tensor
    n_tiles: torch.Tensor
    rows: int
    size: int


def plan(w: MoeWeights, z: torch.Tensor, rows: int) -> Slots:
    """Choose the experts of every token and lay out their slots in whole tiles of ``rows``."""
    k, s = _k(), w.spec
    T, dev = z.shape[0], z.device
    n = T * s.top
    tiles = n // rows + min(s.experts, n)                            # most tiles there can be
    i32 = torch.empty(3 * n + s.experts + tiles + 1, dtype=torch.int32, device=dev)
    idx, slot, rank = (i32[j * n:(j + 1) * n].view(T, s.top) for j in range(3))
    offset, tile_expert, n_tiles = i32[3 * n:3 * n + s.experts], i32[3 * n + s.experts:-1], i32[-1:]
    count = torch.zeros(s.experts, dtype=torch.int32, device=dev)
    weight = torch.empty(T, s.top + 1, dtype=F32, device=dev)
    r = _route_struct(w, z, idx, weight)
    k.K._check(k.route(z.data_ptr(), C.byref(r), count.data_ptr(), rank.data_ptr(), T, k.K._stream()), "moe_route")
    k.K._check(k.plan(count.data_ptr(), s.experts, rows, offset.data_ptr(), tile_expert.data_ptr(), n_tiles.data_ptr(), k.K._stream()), "moe_plan")
    return Slots(idx, slot, weight, rank, offset, tile_expert, n_tiles, rows, tiles * rows)


def dispatch(w: MoeWeights, h: torch.Tensor, p: Slots) -> torch.Tensor:
    """Rows of h [T, E] in their experts' slots [size, E]; rows of padding slots are not initialised."""
    k, s = _k(), w.spec
    T, E = h.shape
    xs = torch.empty(p.size, pad8(E), dtype=h.dtype, device=h.device)[:, :E]
    es = h.element_size()
    assert h.stride(0) >= pad8(E)
    k.K._check(k.dispatch(h.data_ptr(), h.stride(0) * es, xs.data_ptr(), xs.stride(0) * es, pad8(E) * es, p.idx.data_ptr(), p.rank.data_ptr(),
                          p.offset.data_ptr(), p.slot.data_ptr(), s.experts, s.top, T, k.K._stream()), "moe_dispatch")
    return xs


def grouped_linear(x: torch.Tensor, w: torch.Tensor, N: int, p: Slots, act: Optional[str] = None) -> torch.Tensor:
    """Slots x [size, K] times their experts' rows of w [experts * N, K] -> act(..) [size, N]; ``act`` "relu2", or "silu": w holds [gate; up]
    rows [experts * 2 N, K] and the result is silu(gate) * up."""
    k = _k()
    M, Kd = x.shape
    out = torch.empty(M, pad8(N), dtype=x.dtype, device=x.device)[:, :N]
    if x.dtype == F32:
        if act == "silu":
            return glu(grouped_linear(x, w, 2 * N, p), N, "silu", F32)
        k.K._check(base._k().sgemm(x.data_ptr(), w.data_ptr(), 0, out.data_ptr(), M, N, Kd, x.stride(0), w.stride(0), out.stride(0), int(act == "relu2"), 0, 0,
                                   p.tile_expert.data_ptr(), p.n_tiles.data_ptr(), k.K._stream()), "sgemm_nt")
        return out
    bn = 256 if p.rows == 256 or (N > 128 and act != "silu") else 128
    k.K._check(k.gemm(x.data_ptr(), w.data_ptr(), out.data_ptr(), M, N, Kd, x.stride(0), w.stride(0), out.stride(0),
                      w.shape[0] // (2 * N if act == "silu" else N), p.tile_expert.data_ptr(), p.n_tiles.data_ptr(), p.rows, bn, _GROUPED_ACT[act], k.K._stream(), k.K.err_word(x.device).data_ptr()),
               "b200_gemm_grouped")
    return out


_GROUPED_ACT = {None: 0, "relu2": 1, "silu": 4}


def tile_rows(spec, T: int, dtype: torch.dtype) -> int:
    """Slots per tile: whole tiles of the pair kernel when the experts are busy enough to fill them."""
    if dtype == F32:
        return _k().sgemm_rows
    return 256 if T * spec.top >= 192 * spec.outputs else 128


def combine(s: RowSum) -> torch.Tensor:
    """The sum, in the common dtype of its parts."""
    if not s.h.is_cuda:
        return s.sum().to(s.h.dtype)
    k, (T, E), y, ys = _k(), s.h.shape, s.rows, s.shared
    assert y.dtype == s.h.dtype and (ys is None or ys.dtype == y.dtype)
    out = torch.empty(T, pad8(E), dtype=y.dtype, device=y.device)[:, :E]
    k.K._check(k.combine(s.h.data_ptr(), s.h.stride(0), y.data_ptr(), y.stride(0), k.K._ptr(ys), 0 if ys is None else ys.stride(0), s.slot.data_ptr(),
                         s.weight.data_ptr(), out.data_ptr(), out.stride(0), T, E, s.slot.shape[1], _f32(y), k.K._stream()), "moe_combine")
    return out


def _plain(w: MoeWeights, h: torch.Tensor) -> torch.Tensor:
    s, E = w.spec, h.shape[1]
    z = router_logits(h, w.router)
    idx, weight = ref.route_grouped(z, s.top, s.group_count, s.group_keep) if s.grouped else ref.route(z[:, :s.outputs], w.correction, s.top)

    def hidden(x, e):
        if s.gated:
            return glu(base.linear(x, w.up[2 * e * s.ff:2 * (e + 1) * s.ff]), s.ff, "silu", x.dtype)
        return ref.linear_act(x, w.up[e * s.ff:(e + 1) * s.ff], None, "relu2")

    out = torch.zeros(h.shape)
    for e in range(s.outputs):
        t, k = (idx == e).nonzero(as_tuple=True)
        if not len(t):
            continue
        y = h[t].float() if e >= s.experts else \
            ref.linear_act(hidden(h[t], e), w.down[e * E:(e + 1) * E]).float()
        out.index_add_(0, t, weight[t, k][:, None] * y)
    if w.up_s is not None:
        ys = ref.linear_act(ref.linear_act(h, w.up_s, None, "relu2"), w.down_s).float()
        out += torch.sigmoid(z[:, s.outputs:]) * ys
    return out.to(h.dtype)


def mixture(w: MoeWeights, h: torch.Tensor) -> torch.Tensor:
    """Mixture of experts of any number of rows h [T, E]."""
    if not h.is_cuda:
        return _plain(w, h)
    s, E = w.spec, h.shape[1]
    p = plan(w, router_logits(h, w.router), tile_rows(s, h.shape[0], h.dtype))
    a = grouped_linear(dispatch(w, h, p), w.up, s.ff, p, s.act)
    y = grouped_linear(a, w.down, E, p)
    ys = None if w.up_s is None else base.linear(base.linear(h, w.up_s, None, "relu2"), w.down_s)
    return combine(RowSum(y, p.slot, p.weight, h, ys))


def mixture_rows(w: MoeWeights, h: torch.Tensor):
    """The same for the few bf16 rows of a decode step, as a stream of the chosen experts' weights; on a GPU the experts' fp32 rows,
    to be summed where they are read."""
    if not h.is_cuda or h.dtype == F32 or h.shape[0] > ROWS:
        return mixture(w, h)
    parts = mixture_rows_pieces(w, h)
    for f in parts[:-1]:
        f()
    return parts[-1]


def mixture_rows_pieces(w: MoeWeights, h: torch.Tensor):
    """The launches of ``mixture_rows`` as callables, and its result."""
    k, s = _k(), w.spec
    B, E = h.shape
    dev, n = h.device, B * s.top
    i32 = torch.empty(3 * n + 2 * s.outputs + 2, dtype=torch.int32, device=dev)
    idx, slot, row = (i32[j * n:(j + 1) * n] for j in range(3))
    active, first, n_active = i32[3 * n:3 * n + s.outputs], i32[3 * n + s.outputs:-1], i32[-1:]
    weight = torch.empty(B, s.top + 1, dtype=F32, device=dev)
    shared = w.up_s is not None
    a = torch.empty(n, pad8(s.ff), dtype=BF16, device=dev)
    y = torch.empty(n, pad8(E), dtype=F32, device=dev)
    fs = s.shared or 0
    a_s = torch.empty(B, pad8(fs), dtype=BF16, device=dev) if shared else None
    ys = torch.empty(B, pad8(E), dtype=F32, device=dev)[:, :E] if shared else None
    p = k.K._ptr
    lists = (active.data_ptr(), first.data_ptr(), row.data_ptr(), n_active.data_ptr())
    most = min(s.experts, n)
    ld = lambda t: 0 if t is None else t.stride(0)  # noqa: E731
    keep = [i32, h]

    def logits():
        keep.append(router_logits(h, w.router))

    def route():
        z = keep[2]
        r, o = _route_struct(w, z, idx, weight), _RouteRows(slot.data_ptr(), *lists)
        k.K._check(k.route_rows(z.data_ptr(), C.byref(r), C.byref(o), B, k.K._stream()), "moe_route_rows")

    def up():
        e = _ExpertRows(s.ff, E, w.up.stride(0), fs, E, ld(w.up_s), h.stride(0), a.stride(0), h.stride(0), ld(a_s), B, 2 if s.gated else 1, w.up.data_ptr(), p(w.up_s),
                        h.data_ptr(), h.data_ptr(), 1, a.data_ptr(), p(a_s), *lists)
        k.K._check(k.rows(C.byref(e), most, 0, 0, k.K._stream()), "moe_rows")

    def down():
        e = _ExpertRows(E, s.ff, w.down.stride(0), E if shared else 0, fs, ld(w.down_s), a.stride(0), y.stride(0), ld(a_s), ld(ys), B, 0,
                        w.down.data_ptr(), p(w.down_s), a.data_ptr(), p(a_s), 0, y.data_ptr(), p(ys), *lists)
        k.K._check(k.rows(C.byref(e), most, 1, 0, k.K._stream()), "moe_rows")

    return logits, route, up, down, RowSum(y[:, :E], slot.view(B, s.top), weight, h, ys)
