"""What the decode engines share: weight-streaming matrix products with a persistent accumulator, CUDA-graph replay and
programmatic dependent launch."""
from __future__ import annotations

import ctypes as C
import os
from functools import lru_cache
from types import SimpleNamespace

import torch

BF16 = torch.bfloat16
PDL = os.environ.get("B200_DECODE_PDL", "0") == "1"  # measured within noise of off (23.1-23.5 vs 23.5 ms per token): off
SKINNY_ROWS = 64   # widest batch of the weight-streaming GEMM


@lru_cache(None)
def _lib() -> SimpleNamespace:
    """Kernel bindings; loaded on first use, so that an engine on CPU tensors needs no native library."""
    from ..ops import cuda as K

    vp, i = C.c_void_p, C.c_int
    return SimpleNamespace(K=K, set_pdl=K._sig("b200_set_pdl", [i]),
                           skinny=K._sig("b200_gemm_skinny", [vp] * 4 + [i] * 7 + [vp, vp]),
                           cast_zero=K._sig("b200_cast_zero", [vp, vp, C.c_longlong, vp]))


def skinny_linear(x: torch.Tensor, w: torch.Tensor, work: torch.Tensor | None, keep_f32: bool = False,
                  ld_out: int = 0) -> torch.Tensor:
    """x [B, K] bf16 -> [B, N] through the skinny weight-streaming GEMM (B <= 64).  Narrow outputs are accumulated over K
    splits in the persistent fp32 ``work`` buffer (kept zero between uses by its consumers); ``keep_f32`` hands that
    buffer to a fused consumer, otherwise it is converted (and cleared) here."""
    lib = _lib()
    K = lib.K
    Bt, Kd = x.shape
    N = w.shape[0]
    out = torch.empty(Bt, max(N, ld_out), dtype=BF16, device=x.device)[:, :N]
    work = work[: Bt * N].view(Bt, N) if work is not None and Bt * N <= work.numel() else None
    rc = lib.skinny(x.data_ptr(), w.data_ptr(), out.data_ptr(), K._ptr(work), Bt, N, Kd, x.stride(0), w.stride(0),
                 out.stride(0), 0, K._stream(), K.err_word(x.device).data_ptr())
    K._launches += 1
    if rc < 0:
        raise RuntimeError(f"b200_gemm_skinny failed with code {rc}")
    if rc == 1:
        if keep_f32:
            return work
        assert out.stride(0) == N
        K._check(lib.cast_zero(work.data_ptr(), out.data_ptr(), Bt * N, K._stream()), "cast_zero")
    return out


class GraphRunner:
    """Replays functions as CUDA graphs (attribute ``use_graphs``; ``_graphs`` maps a key to (graph, output))."""

    use_graphs = True

    def _run(self, key, fn, once: bool = False):
        """Replay ``fn`` as a CUDA graph.  Before the first replay it is executed eagerly as a warm-up and recorded; ``fn`` must
        be idempotent then (read inputs, write separate outputs).  With ``once`` every call takes effect exactly once (``fn``
        updates state): the first call returns the eager execution's result and replays nothing."""
        if not self.use_graphs:
            return self._with_pdl(fn)
        g = self._graphs.get(key)
        if g is None:
            first = self._with_pdl(fn)
            torch.cuda.synchronize()
            graph = torch.cuda.CUDAGraph()
            with torch.cuda.graph(graph):
                out = self._with_pdl(fn)
            g = self._graphs[key] = (graph, out)
            if once:
                return first
        g[0].replay()
        return g[1]

    def _pdl_on(self) -> bool:
        return PDL

    def _with_pdl(self, fn):
        """Run ``fn`` with programmatic dependent launch on for the decode kernels: each kernel's prologue overlaps the
        tail of its predecessor (the attribute is recorded into a graph at capture time)."""
        if not self._pdl_on():
            return fn()
        set_pdl = _lib().set_pdl
        old = set_pdl(1)
        try:
            return fn()
        finally:
            set_pdl(old)
