"""Sublayers of the layered decoder models: mixers and feed-forwards, each in a prompt form (``stream`` / ``forward``, on a
``PackedStep``) and a decode form (one token per row).

Weights are stored as they are executed: projections that read the same input are one matrix, row pitches are padded to
eight elements.  ``checkpoint_tensors`` names the views that make up a checkpoint."""
from __future__ import annotations

import math
from dataclasses import dataclass, field
from typing import Callable, Optional

import torch
import torch.nn as nn

from ..ops import delta as delta_ops
from ..ops import grouped as grp_ops
from ..ops import latent as ops
from ..ops import memory as mem_ops
from ..ops import moe as moe_ops
from ..ops.delta import DeltaLayout, DeltaWeights
from ..ops.grouped import GroupedLayout, QkvTransform, ring_slots
from ..ops.latent import LatentLayout, pad8
from ..ops.memory import BiasTable, MemoryLayout, ParallelLayout
from .layered_config import (ChunkAttentionSpec, DeltaMemorySpec, DenseMLPSpec, GatedMemorySpec, GroupedAttentionSpec, KeptWindowAttentionSpec,
                             LatentAttentionSpec, LayeredConfig, LayerRun, MixtureSpec, ParallelSpec, RotarySpec, WindowAttentionSpec)


def weight(rows: int, cols: int, dtype, device) -> nn.Parameter:
    """[rows, cols] matrix with a zero-filled row pitch that is a multiple of eight."""
    return nn.Parameter(torch.zeros(rows, pad8(cols), dtype=dtype, device=device), requires_grad=False)


def vector(n: int, device) -> nn.Parameter:
    return nn.Parameter(torch.zeros(n, dtype=torch.float32, device=device), requires_grad=False)


def rope_tables(rot: RotarySpec, length: int, device) -> tuple:
    """cos / sin [length, dims / 2] of the spec's (interpolated) frequencies, times its magnitude.  The angles are formed in
    double precision and stored as fp32."""
    ang = torch.outer(torch.arange(length, dtype=torch.float64), torch.tensor(rot.frequencies(), dtype=torch.float64))
    return tuple((f(ang) * rot.magnitude).float().contiguous().to(device) for f in (torch.cos, torch.sin))


# ------------------------------------------------------------------------------------------
# one packed step
# ------------------------------------------------------------------------------------------
@dataclass
class StreamLayout:
    """Where the keys of a packed step lie: per sequence first the cached positions its portion can still see, then the portion
    itself."""

    sidx: torch.Tensor        # [T] stream index of every token
    kbase: torch.Tensor       # [T] stream index of the first key of its sequence (of its chunk)
    seqs: list                # (first token, tokens, first key, keys in front of the first token) per sequence (per chunk of one)
    total: int
    history: list             # (row, first position, count, first key) of the stretches of history


class PackedStep:
    """Token ids and positions of a batch of prompt portions; ``portions`` are (row, first position, token ids)."""

    def __init__(self, portions: list, device):
        self.device, self.portions = torch.device(device), [(r, s, len(t)) for r, s, t in portions]
        tok, pos, row, end = [], [], [], []
        for r, s, t in portions:
            n = len(t)
            tok.extend(t)
            pos.extend(range(s, s + n))
            row.extend([r] * n)
            end.extend([s + n] * n)
        self.tok = torch.tensor(tok, dtype=torch.int64).to(self.device)
        meta = torch.tensor([pos, row, end], dtype=torch.int32).to(self.device)
        self.pos, self.row, self.end = meta[0], meta[1], meta[2]
        self.T = len(tok)
        self._layouts: dict = {}
        self._seq_table = None
        self.derived: dict = {}           # tables that kernels derive from the portions

    def sequences(self) -> list:
        """(first token, tokens, cache row, first position) per portion."""
        out, t0 = [], 0
        for r, s, n in self.portions:
            out.append((t0, n, r, s))
            t0 += n
        return out

    @property
    def seq_table(self) -> torch.Tensor:
        """``sequences`` as int32 [portions, 4] on the device."""
        if self._seq_table is None:
            self._seq_table = torch.tensor(self.sequences(), dtype=torch.int32).to(self.device)
        return self._seq_table

    def layout(self, history: int, keep: int = 0) -> StreamLayout:
        """Layout with up to ``keep`` + ``history`` cached positions in front of every portion: the first ``keep`` of the sequence
        and the newest ones.  A distance in the stream that does not reach into the kept positions is a distance in the sequence."""
        if all(s == 0 for _, s, _ in self.portions):
            history = keep = 0
        if (history, keep) not in self._layouts:
            seqs, sidx, kbase, hist = [], [], [], []
            t0 = k0 = 0
            for r, s, n in self.portions:
                h = min(s, history + keep)
                first = min(h, keep)
                seqs.append((t0, n, k0, h))
                sidx.extend(range(k0 + h, k0 + h + n))
                kbase.extend([k0] * n)
                if first:
                    hist.append((r, 0, first, k0))
                if h > first:
                    hist.append((r, s - (h - first), h - first, k0 + first))
                t0, k0 = t0 + n, k0 + h + n
            idx = torch.tensor([sidx, kbase], dtype=torch.int32).to(self.device)
            self._layouts[history, keep] = StreamLayout(idx[0], idx[1], seqs, k0, hist)
        return self._layouts[history, keep]

    def chunk_layout(self, size: int) -> StreamLayout:
        """Layout for attention inside chunks of ``size`` positions: the history of a portion is what its first chunk already
        holds; every chunk counts as a sequence of its own."""
        key = ("chunk", size)
        if key not in self._layouts:
            seqs, sidx, kbase, hist = [], [], [], []
            t0 = k0 = 0
            for r, s, n in self.portions:
                h = s % size
                sidx.extend(range(k0 + h, k0 + h + n))
                if h:
                    hist.append((r, s - h, h, k0))
                at, key0, front = 0, k0, h
                while at < n:                                  # the part of one chunk at a time
                    m = min(size - front, n - at)
                    seqs.append((t0 + at, m, key0, front))
                    kbase.extend([key0] * m)
                    at, key0, front = at + m, key0 + front + m, 0
                t0, k0 = t0 + n, k0 + h + n
            idx = torch.tensor([sidx, kbase], dtype=torch.int32).to(self.device)
            self._layouts[key] = StreamLayout(idx[0], idx[1], seqs, k0, hist)
        return self._layouts[key]


@dataclass
class StepContext:
    """What the sublayers of a packed step share."""

    config: LayeredConfig
    step: PackedStep
    cache: Optional[object]
    rope: dict = field(default_factory=dict)       # rotary spec -> (cos, sin)
    windows: dict = field(default_factory=dict)    # latent source layer -> widest window
    streams: dict = field(default_factory=dict)    # latent source layer -> latent rows of the step
    first_values: Optional[torch.Tensor] = None    # values that later layers mix into theirs


@dataclass
class DecodeContext:
    """What the sublayers of a decode step share; ``dense(x, w, which)`` is the engine's narrow-batch product, ``splits(mixer, B)``
    its number of key splits."""

    config: LayeredConfig
    pos: torch.Tensor
    row: torch.Tensor
    cache: object
    dense: Callable
    splits: Callable
    first_values: Optional[torch.Tensor] = None    # values that later layers mix into theirs


def gather_history(layout: StreamLayout, cache: torch.Tensor, stream: torch.Tensor, keep: int = 0) -> None:
    """Copy the cached rows in front of every portion from the ring ``cache`` [rows, cap, ld] into the stream."""
    if not layout.history:
        return
    cap = cache.shape[1]
    src = [row * cap + ring_slots(torch.arange(p0, p0 + n), cap, keep) for row, p0, n, _ in layout.history]
    dst = [torch.arange(k0, k0 + n) for _, _, n, k0 in layout.history]
    idx = torch.stack([torch.cat(src), torch.cat(dst)]).to(torch.int32).to(cache.device)
    ops.gather_rows(cache.view(-1, cache.shape[2]), idx[0], stream, idx[1])


# ------------------------------------------------------------------------------------------
# sublayers
# ------------------------------------------------------------------------------------------
class LatentAttention(nn.Module):
    """Windowed attention over per-token latents with gated heads; see ``LatentAttentionSpec``."""

    out_bias, out_bias_mult = None, 1.0

    def __init__(self, spec: LatentAttentionSpec, width: int, eps: float, dtype, device):
        super().__init__()
        a = spec
        self.spec, self.width, self.eps, self.dtype = spec, width, eps, dtype
        L = self.layout = LatentLayout(a.heads, a.dim, a.rot_dim, a.vdim, a.kv_rank, a.kv_from is None)
        self.w_in = weight(L.width_in, width, dtype, device)
        self.w_kv = weight(L.width_kv, a.kv_rank, dtype, device)
        self.w_o = weight(width, a.heads * a.vdim, dtype, device)
        self.latent_norm = vector(a.kv_rank, device) if L.own else None

    def checkpoint_tensors(self) -> dict:
        a, L, E = self.spec, self.layout, self.width
        out = {"q": self.w_in[:a.heads * (a.dim + a.rot_dim), :E], "g": self.w_in[L.off_g:L.off_g + a.heads * a.vdim, :E],
               "uk": self.w_kv[:a.heads * a.dim, :a.kv_rank], "uv": self.w_kv[L.off_v:L.off_v + a.heads * a.vdim, :a.kv_rank],
               "o": self.w_o[:, :a.heads * a.vdim]}
        if L.own:
            out["dkv"] = self.w_in[L.off_d:L.off_d + a.kv_rank + a.rot_dim, :E]
            out["dkv.norm"] = self.latent_norm
        return out

    def project_stream(self, xb, step: PackedStep, cache, stream, lay: StreamLayout, rope):
        """The portion's projection rows (q rotated); appends the latents of an own layer to ``stream`` and the ring."""
        inp = ops.linear(xb, self.w_in[:, :self.width])
        if self.layout.own and cache is not None:
            gather_history(lay, cache, stream)     # before the ring slots of the oldest positions are written again
        ops.latent_prep_(self.layout, inp, self.latent_norm, self.eps, rope, step, lay.sidx, cache if self.layout.own else None,
                         stream)
        return inp

    def stream(self, xb, run: LayerRun, ctx: "StepContext"):
        a, src, step = self.spec, ctx.config.kv_source(run.layer), ctx.step
        cache, lay = None if ctx.cache is None else ctx.cache.data[src], step.layout(ctx.windows[src] - 1)
        if src == run.layer:
            ctx.streams[src] = torch.empty(lay.total, self.layout.ld_lat, dtype=self.dtype, device=xb.device)
        stream = ctx.streams[src]
        inp = self.project_stream(xb, step, cache, stream, lay, ctx.rope[a.rot])
        kv = ops.linear(stream[:, :a.kv_rank], self.w_kv[:, :a.kv_rank])
        o = ops.stream_attention(self.layout, inp, kv, stream, lay, a.window, a.scale)
        return ops.linear(o, self.w_o[:, :a.heads * a.vdim])

    def decode_splits(self, B: int, max_len: int, tensor_cores: bool) -> int:
        """Key splits of the decode attention: enough CTAs to fill the machine, at least 128 keys each."""
        groups, fill = self.spec.heads, 4 * 148          # generic kernel: a small CTA per head
        if tensor_cores:
            from ..ops import latent_attention as A

            n = A.decode_group(self.spec.heads, self.spec.kv_rank, self.layout.ld_lat)
            if n:                                         # tensor-core kernel: one CTA per SM, n heads each
                groups, fill = -(-self.spec.heads // n), 148
        tiles = min(self.spec.window, max_len) // 128 + 1
        return max(1, min(tiles, 32, fill // max(1, B * groups)))

    def decode(self, xb, run: LayerRun, ctx: "DecodeContext"):
        """One token per row.  Returns the sublayer output, whether it is an accumulator that the next kernel clears, and
        the projection's accumulator or None."""
        a, dense = self.spec, ctx.dense
        cache = ctx.cache.data[ctx.config.kv_source(run.layer)]
        inp, acc = dense(xb, self.w_in[:, :self.width], 0)
        o = ops.ring_attention(self.layout, inp, self.w_kv, self.latent_norm, self.eps, ctx.cache.rope[a.rot], ctx.pos, ctx.row, cache,
                               min(a.window, cache.shape[1]), a.scale, ctx.splits(self, xb.shape[0]), self.dtype)
        out, clear = dense(o, self.w_o[:, :a.heads * a.vdim], 1)
        return out, clear, inp if acc else None


class DenseMLP(nn.Module):
    """down(relu(up x)^2) with biases; the bias of the down projection is added by the norm that follows."""

    act = "relu2"
    wide = 1           # multiples of ``ff`` that its widest product has
    out_bias_mult = 1.0

    def __init__(self, spec: DenseMLPSpec, width: int, dtype, device):
        super().__init__()
        self.spec, self.width, self.dtype = spec, width, dtype
        self.w_up, self.b_up = weight(spec.ff, width, dtype, device), vector(spec.ff, device)
        self.w_down, self.b_down = weight(width, spec.ff, dtype, device), vector(width, device)

    @property
    def out_bias(self):
        return self.b_down

    def checkpoint_tensors(self) -> dict:
        return {"up": self.w_up[:, :self.width], "up.b": self.b_up, "down": self.w_down[:, :self.spec.ff], "down.b": self.b_down}

    def forward(self, xb):
        return ops.linear(ops.linear(xb, self.w_up[:, :self.width], self.b_up, self.act), self.w_down[:, :self.spec.ff])

    def decode(self, xb, dense):
        h, clear = dense(xb, self.w_up[:, :self.width], 1)
        h = ops.bias_act(h, self.b_up, self.act, self.dtype, clear)
        return dense(h, self.w_down[:, :self.spec.ff], 1)


class ParallelMixer(nn.Module):
    """Distance-biased attention and a decaying memory side by side on the same input (``ParallelSpec``).  One projection feeds
    both; the two output projections are one product over the concatenated halves, whose fixed weights are applied where the
    halves are gated (so the stored weights stay as they are)."""

    def __init__(self, spec: ParallelSpec, width: int, eps: float, dtype, device):
        super().__init__()
        a, r = spec.left, spec.right
        if a.bias_rows is None:
            raise ValueError("the height of the distance-bias table is not known: load a checkpoint or set bias_rows")
        self.spec, self.width, self.eps, self.dtype = spec, width, eps, dtype
        L = self.layout = ParallelLayout(a.heads, a.kv_heads, a.dim, a.vdim, r.heads, r.dim, r.vdim)
        self.w_in, self.b_in = weight(L.width_in, width, dtype, device), vector(L.width_in, device)
        self.w_o, self.out_bias = weight(width, L.width_o, dtype, device), vector(width, device)
        self.out_bias_mult = spec.left_scale
        self.rel = nn.Parameter(torch.zeros(a.bias_rows, a.heads, dtype=torch.float32, device=device), requires_grad=False)
        self.norm = vector(r.heads * r.vdim, device)
        self.register_buffer("decay", torch.tensor(r.decay, dtype=torch.float32).to(device), persistent=False)
        logs = [math.log2(x) if x > 0 else -1000.0 for x in r.decay]        # finite: 2^-1000 is zero in fp32
        self.register_buffer("log2_decay", torch.tensor(logs, dtype=torch.float32).to(device), persistent=False)
        self.table = None

    def checkpoint_tensors(self) -> dict:
        a, r, L, E = self.spec.left, self.spec.right, self.layout, self.width
        out = {}
        for name, at, n in (("q", L.off_q, a.heads * a.dim), ("k", L.off_k, a.kv_heads * a.dim), ("v", L.off_v, a.kv_heads * a.vdim)):
            out["left." + name], out["left." + name + ".b"] = self.w_in[at:at + n, :E], self.b_in[at:at + n]
        out.update({"left.g": self.w_in[L.off_lg:L.off_lg + a.heads, :E], "left.rel": self.rel, "left.o": self.w_o[:, :a.heads * a.vdim],
                    "left.o.b": self.out_bias})
        hd, hv = r.heads * r.dim, r.heads * r.vdim
        for name, at, n in (("q", L.off_rq, hd), ("k", L.off_rk, hd), ("v", L.off_rv, hv), ("g", L.off_rg, hv)):
            out["right." + name] = self.w_in[at:at + n, :E]
        out.update({"right.o": self.w_o[:, L.off_r:L.off_r + hv], "right.norm": self.norm})
        return out

    def weights_changed(self) -> None:
        """Derive what the kernels read instead of the stored tensors."""
        self.table = BiasTable.build(self.rel, self.spec.left.buckets())

    def cache_shapes(self, max_len: int) -> dict:
        r, L = self.spec.right, self.layout
        return {"kv": ((max_len, L.ld_kv), self.dtype), "state": ((r.heads, r.dim, L.ldv), torch.float32)}

    def stream(self, h, run: LayerRun, ctx: StepContext):
        L, spec, step = self.layout, self.spec, ctx.step
        kv, state = ctx.cache.data[run.index, "kv"], ctx.cache.data[run.index, "state"]
        inp = ops.linear(h, self.w_in[:, :self.width], self.b_in, "silu", act_cols=L.act_cols)
        mem_ops.kv_append(L, inp, None, kv, step.pos, step.row)
        o = mem_ops.parallel_output(L, h.shape[0], self.dtype, h.device)
        mem_ops.prompt_attention(L, spec.left, inp, kv, self.table, step, spec.left_scale, o)
        m = mem_ops.decay_memory_prompt(L, inp, self.decay, self.log2_decay, state, step)
        mem_ops.memory_norm(L, inp, m, self.norm, self.eps, spec.right_scale, o)
        return ops.linear(o, self.w_o[:, :L.width_o])

    def decode_splits(self, B: int, max_len: int, tensor_cores: bool) -> int:
        return mem_ops.decode_splits(self.layout, B, max_len, tensor_cores)

    def decode(self, h, run: LayerRun, ctx: DecodeContext):
        L = self.layout
        inp, acc = ctx.dense(h, self.w_in[:, :self.width], 0)
        o = mem_ops.parallel_decode(L, self.spec, inp, self.b_in, ctx.cache.data[run.index, "kv"], ctx.cache.data[run.index, "state"],
                                    self.table, self.decay, self.norm, self.eps, ctx.pos, ctx.row, ctx.splits(self, h.shape[0]), self.dtype)
        out, clear = ctx.dense(o, self.w_o[:, :L.width_o], 1)
        return out, clear, inp if acc else None


class GatedMemory(nn.Module):
    """Gated matrix memory (``GatedMemorySpec``).  The gates' projections are a product of their own with fp32 results."""

    out_bias, out_bias_mult = None, 1.0

    def __init__(self, spec: GatedMemorySpec, width: int, eps: float, dtype, device):
        super().__init__()
        self.spec, self.width, self.eps, self.dtype = spec, width, eps, dtype
        L = self.layout = MemoryLayout(spec.heads, spec.dim, spec.vdim)
        self.w_in = weight(L.width_in, width, dtype, device)
        self.w_gate, self.b_gate = weight(2 * spec.heads, width, dtype, device), vector(2 * spec.heads, device)
        self.w_o, self.norm = weight(width, spec.heads * spec.vdim, dtype, device), vector(spec.heads * spec.vdim, device)

    def checkpoint_tensors(self) -> dict:
        a, L, E = self.spec, self.layout, self.width
        hd, hv = a.heads * a.dim, a.heads * a.vdim
        out = {name: self.w_in[at:at + n, :E] for name, at, n in (("q", L.off_q, hd), ("k", L.off_k, hd), ("v", L.off_v, hv), ("g", L.off_g, hv))}
        for name, at in (("i", 0), ("f", a.heads)):
            out[name], out[name + ".b"] = self.w_gate[at:at + a.heads, :E], self.b_gate[at:at + a.heads]
        out.update({"o": self.w_o[:, :hv], "norm": self.norm})
        return out

    def cache_shapes(self, max_len: int) -> dict:
        a = self.spec
        return {"state": ((a.heads, a.dim, self.layout.ldv), torch.float32), "norm": ((a.heads, a.dim + 1), torch.float32)}

    def stream(self, h, run: LayerRun, ctx: StepContext):
        a, data = self.spec, ctx.cache.data
        inp = ops.linear(h, self.w_in[:, :self.width])
        gates = mem_ops.gate_projections(h, self.w_gate[:, :self.width])
        o = mem_ops.gated_memory(self.layout, inp, gates, self.b_gate, a.gate_cap, data[run.index, "state"], data[run.index, "norm"], self.norm,
                                 self.eps, self.dtype, step=ctx.step)
        return ops.linear(o, self.w_o[:, :a.heads * a.vdim])

    def decode(self, h, run: LayerRun, ctx: DecodeContext):
        a, data = self.spec, ctx.cache.data
        inp, acc = ctx.dense(h, self.w_in[:, :self.width], 0)
        o = mem_ops.gated_memory(self.layout, inp, None, self.b_gate, a.gate_cap, data[run.index, "state"], data[run.index, "norm"], self.norm,
                                 self.eps, self.dtype, rows=(ctx.pos, ctx.row), h=h, w_gate=self.w_gate[:, :self.width])
        out, clear = ctx.dense(o, self.w_o[:, :a.heads * a.vdim], 1)
        return out, clear, inp if acc else None


class DeltaMemory(nn.Module):
    """Matrix memories with the gated delta rule (``DeltaMemorySpec``).  Step sizes and decays have a product of their own with fp32 results
    in prompts."""

    out_bias, out_bias_mult = None, 1.0

    def __init__(self, spec: DeltaMemorySpec, width: int, eps: float, dtype, device):
        super().__init__()
        self.spec, self.width, self.eps, self.dtype = spec, width, eps, dtype
        L = self.layout = DeltaLayout(spec.heads, spec.kv_heads, spec.dim, spec.vdim)
        self.w_in, self.w_o = weight(L.width_in, width, dtype, device), weight(width, spec.heads * spec.vdim, dtype, device)
        self.conv = nn.Parameter(torch.zeros(spec.conv, L.channels, dtype=torch.float32, device=device), requires_grad=False)
        self.a_log, self.dt_bias, self.norm = vector(spec.heads, device), vector(spec.heads, device), vector(spec.vdim, device)

    def checkpoint_tensors(self) -> dict:
        a, L, E = self.spec, self.layout, self.width
        qk, hv = a.kv_heads * a.dim, a.heads * a.vdim
        out = {}
        for name, at, n in (("q", L.off_q, qk), ("k", L.off_k, qk), ("v", L.off_v, hv)):
            out[name], out[name + ".conv"] = self.w_in[at:at + n, :E], self.conv[:, at:at + n].T
        for name, at, n in (("g", L.off_g, hv), ("b", L.off_ba, a.heads), ("a", L.off_ba + a.heads, a.heads)):
            out[name] = self.w_in[at:at + n, :E]
        out.update({"A_log": self.a_log, "dt_bias": self.dt_bias, "norm": self.norm, "o": self.w_o[:, :hv]})
        return out

    @property
    def weights(self) -> DeltaWeights:
        return DeltaWeights(self.conv, self.a_log, self.dt_bias, self.norm, self.eps)

    def cache_shapes(self, max_len: int) -> dict:
        a, L = self.spec, self.layout
        return {"conv": ((a.conv, L.channels), self.dtype), "state": ((a.heads, a.dim, L.ldv), torch.float32)}

    def stream(self, h, run: LayerRun, ctx: StepContext):
        a, L, E, data = self.spec, self.layout, self.width, ctx.cache.data
        inp = ops.linear(h, self.w_in[:L.off_ba, :E])
        ba = mem_ops.gate_projections(h, self.w_in[L.off_ba:L.off_ba + 2 * a.heads, :E])
        act = delta_ops.short_conv(L, inp, self.conv, data[run.index, "conv"], ctx.step)
        o = delta_ops.delta_prompt(L, self.weights, act, inp, ba, data[run.index, "state"], ctx.step)
        return ops.linear(o, self.w_o[:, :a.heads * a.vdim])

    def decode(self, h, run: LayerRun, ctx: DecodeContext):
        a, L, data = self.spec, self.layout, ctx.cache.data
        inp, acc = ctx.dense(h, self.w_in[:, :self.width], 0)
        o = delta_ops.delta_decode(L, self.weights, inp, data[run.index, "conv"], data[run.index, "state"], ctx.pos, ctx.row, self.dtype)
        out, clear = ctx.dense(o, self.w_o[:, :a.heads * a.vdim], 1)
        return out, clear, inp if acc else None


class GroupedAttention(nn.Module):
    """Grouped-query attention over a ring of keys and values (``GroupedAttentionSpec``): inside chunks or under a window, which may
    keep a sequence's first tokens."""

    out_bias, out_bias_mult = None, 1.0

    def __init__(self, spec: GroupedAttentionSpec, width: int, eps: float, dtype, device):
        super().__init__()
        a = spec
        self.spec, self.width, self.eps, self.dtype = spec, width, eps, dtype
        L = self.layout = GroupedLayout(a.heads, a.kv_heads, a.dim, a.vdim)
        self.w_in = weight(L.width_in, width, dtype, device)
        self.b_in = vector(L.width_in, device) if a.biased else None
        self.w_o = weight(width, a.heads * a.vdim, dtype, device)
        self.q_norm, self.k_norm = (vector(n * a.dim, device) if a.qk_norm else None for n in (a.heads, a.kv_heads))
        self.sink = vector(a.heads, device) if a.sink else None
        self.vmix = nn.Parameter(torch.zeros((), dtype=torch.float32, device=device), requires_grad=False) if a.v_mix else None

    def checkpoint_tensors(self) -> dict:
        a, L, E = self.spec, self.layout, self.width
        out = {}
        for name, at, n in (("q", L.off_q, a.heads * a.dim), ("k", L.off_k, a.kv_heads * a.dim), ("v", L.off_v, L.v_width)):
            out[name] = self.w_in[at:at + n, :E]
            if a.biased:
                out[name + ".b"] = self.b_in[at:at + n]
        out["o"] = self.w_o[:, :a.heads * a.vdim]
        out.update({k: v for k, v in (("q.norm", self.q_norm), ("k.norm", self.k_norm), ("sink", self.sink), ("vmix", self.vmix)) if v is not None})
        return out

    @property
    def unused_tensors(self) -> tuple:
        """Checkpoint tensors that may stand beside the others without a use."""
        return () if self.spec.v_mix or not self.spec.capped else ("vmix",)

    def cache_shapes(self, max_len: int) -> dict:
        return {"kv": ((min(self.spec.slots, max_len), self.layout.ld_kv), self.dtype)}

    def _transform(self, role: Optional[str], rope: dict, first, raw: bool = False) -> QkvTransform:
        """``raw``: of a decode step's accumulators."""
        rot = self.spec.rot
        mix = role == "mix"
        return QkvTransform(self.q_norm, self.k_norm, self.eps, 0 if rot is None else rot.dims, None if rot is None else rope[rot],
                            self.vmix if mix else None, first if mix else None, self.spec.head_norm, self.b_in if raw else None, self.spec.keep)

    def stream(self, h, run: LayerRun, ctx: StepContext):
        a, L, step, role = self.spec, self.layout, ctx.step, ctx.config.mixes_values(run.layer)
        cache = ctx.cache.data[run.index, "kv"]
        lay = step.chunk_layout(a.size) if a.chunked else step.layout(a.size - 1, a.keep)
        inp = ops.linear(h, self.w_in[:, :self.width], self.b_in)
        kv = torch.empty(lay.total, L.ld_kv, dtype=self.dtype, device=h.device)
        gather_history(lay, cache, kv, a.keep)     # before the ring slots of the oldest positions are written again
        grp_ops.qkv_prep_(L, inp, self._transform(role, ctx.rope, ctx.first_values), step, lay.sidx, cache, kv)
        if role == "first":
            ctx.first_values = inp[:, L.off_v:L.off_v + L.v_width]
        o = grp_ops.stream_attention(L, a, inp, kv, lay, self.sink)
        return ops.linear(o, self.w_o[:, :a.heads * a.vdim])

    def decode_splits(self, B: int, max_len: int, tensor_cores: bool) -> int:
        return grp_ops.decode_splits(self.layout, B, min(self.spec.slots, max_len), tensor_cores)

    def decode(self, h, run: LayerRun, ctx: DecodeContext):
        a, L, role = self.spec, self.layout, ctx.config.mixes_values(run.layer)
        inp, acc = ctx.dense(h, self.w_in[:, :self.width], 0)
        tr = self._transform(role, ctx.cache.rope, ctx.first_values, raw=True)
        first = torch.empty(h.shape[0], pad8(L.v_width), dtype=torch.float32, device=h.device)[:, :L.v_width] if role == "first" else None
        o = grp_ops.ring_attention(L, a, inp, tr, ctx.cache.data[run.index, "kv"], self.sink, first, ctx.pos, ctx.row, ctx.splits(self, h.shape[0]),
                                   self.dtype)
        if first is not None:
            ctx.first_values = first
        out, clear = ctx.dense(o, self.w_o[:, :a.heads * a.vdim], 1)
        return out, clear, inp if acc else None


class GatedMLP(nn.Module):
    """down(act(gate x) * (up x)), no biases; ``act``: "gelu" (tanh form) or "silu"."""

    act = "gelu"
    wide = 2
    out_bias, out_bias_mult = None, 1.0

    def __init__(self, spec: DenseMLPSpec, width: int, dtype, device):
        super().__init__()
        self.spec, self.width, self.dtype = spec, width, dtype
        self.w_gu, self.w_down = weight(2 * spec.ff, width, dtype, device), weight(width, spec.ff, dtype, device)

    def checkpoint_tensors(self) -> dict:
        f, E = self.spec.ff, self.width
        return {"gate": self.w_gu[:f, :E], "up": self.w_gu[f:, :E], "down": self.w_down[:, :f]}

    def forward(self, h):
        return ops.linear(mem_ops.glu_linear(h, self.w_gu[:, :self.width], self.spec.ff, self.act), self.w_down[:, :self.spec.ff])

    def decode(self, h, dense):
        a, clear = dense(h, self.w_gu[:, :self.width], 1)
        return dense(mem_ops.glu(a, self.spec.ff, self.act, self.dtype, clear), self.w_down[:, :self.spec.ff], 1)


class SiluMLP(GatedMLP):
    act = "silu"


class MixtureMLP(nn.Module):
    """Mixture of experts (``MixtureSpec``): squared-ReLU or gated ones, identity experts, a gated shared expert.  The experts' matrices lie
    one below the other (gated: gate and up rows of an expert in turn); the shared expert's gate is one more row of the router."""

    wide = 0
    out_bias, out_bias_mult = None, 1.0

    def __init__(self, spec: MixtureSpec, width: int, dtype, device):
        super().__init__()
        s = spec
        self.spec, self.width, self.dtype = spec, width, dtype
        self.w_router = weight(s.outputs + (s.shared is not None), width, dtype, device)
        self.correction = vector(s.outputs, device) if s.corrected else None
        self.w_up, self.w_down = weight(s.experts * s.ff * (2 if s.gated else 1), width, dtype, device), weight(s.experts * width, s.ff, dtype, device)
        if s.shared is not None:
            self.s_up, self.s_down = weight(s.shared, width, dtype, device), weight(width, s.shared, dtype, device)

    def checkpoint_tensors(self) -> dict:
        s, E = self.spec, self.width
        out = {"router": self.w_router[:s.outputs, :E]}
        if s.corrected:
            out["correction"] = self.correction
        names = ("gate", "up") if s.gated else ("up",)
        for e in range(s.experts):
            for k, name in enumerate(names):
                at = (e * len(names) + k) * s.ff
                out[f"e{e}.{name}"] = self.w_up[at:at + s.ff, :E]
            out[f"e{e}.down"] = self.w_down[e * E:(e + 1) * E, :s.ff]
        if s.shared is not None:
            out.update({"shared.sg": self.w_router[s.outputs:, :E], "shared.up": self.s_up[:, :E], "shared.down": self.s_down[:, :s.shared]})
        return out

    @property
    def weights(self) -> moe_ops.MoeWeights:
        s, E = self.spec, self.width
        up, down = (None, None) if s.shared is None else (self.s_up[:, :E], self.s_down[:, :s.shared])
        return moe_ops.MoeWeights(s, self.w_router[:, :E], self.correction, self.w_up[:, :E], self.w_down[:, :s.ff], up, down)

    def forward(self, h):
        return moe_ops.mixture(self.weights, h)

    def decode(self, h, dense):
        return moe_ops.mixture_rows(self.weights, h), False


MIXERS = {LatentAttentionSpec: LatentAttention, ParallelSpec: ParallelMixer, GatedMemorySpec: GatedMemory, DeltaMemorySpec: DeltaMemory,
          ChunkAttentionSpec: GroupedAttention, WindowAttentionSpec: GroupedAttention, KeptWindowAttentionSpec: GroupedAttention}
MLPS = {"relu2": DenseMLP, "geglu": GatedMLP, "swiglu": SiluMLP, "moe": MixtureMLP}
