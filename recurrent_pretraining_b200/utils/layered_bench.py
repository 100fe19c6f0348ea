"""Prefill and decode throughput of the layered decoder models beside the recurrent model at equal size, and the time of
every kernel of a layer against its roofline.

``python -m recurrent_pretraining_b200.utils.layered_bench [--shapes gasovik-1b,fatudra-1b,...] [--ops-only]``.
Random weights.  Model runs: CUDA events around whole prefill / decode calls of the two engines (graph-replayed decode).
Kernels: CUDA events around single calls on the shapes of one layer, L2 flushed in between, median.  The comparison
model is the depth-recurrent model run for one recurrence: as many layers of the same width, head count and value
size, with a feed-forward that gives the same number of parameters per layer (of a mixture of experts: those that a token
meets)."""
from __future__ import annotations

import argparse
import json
import os
from dataclasses import replace

import torch

ROOT = os.path.dirname(os.path.dirname(os.path.dirname(os.path.abspath(__file__))))


def peaks() -> tuple:
    """(bytes/s, FLOP/s) measured on this machine type: copy bandwidth and bf16 GEMM rate."""
    try:
        p = json.load(open(os.path.join(ROOT, "MEASURED_PEAKS.json")))
        return p["hbm_gbs"] * 1e9, p["bf16_tflops"] * 1e12
    except Exception:
        return 6.65e12, 1.59e15


class Timer:
    def __init__(self):
        self.flush = torch.empty(256 << 20, dtype=torch.uint8, device="cuda")
        self.rows: list = []

    def op(self, name: str, fn, nbytes: float, flops: float, iters: int = 12) -> None:
        bw, fl = peaks()
        for _ in range(3):
            fn()
        times = []
        for _ in range(iters):
            self.flush.zero_()
            a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            a.record()
            fn()
            b.record()
            torch.cuda.synchronize()
            times.append(a.elapsed_time(b) * 1e3)
        us = sorted(times)[len(times) // 2]
        floor = max(nbytes / bw, flops / fl) * 1e6
        self.rows.append({"op": name, "us": round(us, 2), "roofline_us": round(floor, 2), "fraction": round(floor / us, 3),
                          "bound": "memory" if nbytes / bw > flops / fl else "tensor"})

    def take(self) -> list:
        rows, self.rows = self.rows, []
        return rows


def time_calls(fn, iters: int = 5) -> float:
    """Milliseconds per call."""
    fn()
    torch.cuda.synchronize()
    a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    a.record()
    for _ in range(iters):
        fn()
    b.record()
    torch.cuda.synchronize()
    return a.elapsed_time(b) / iters


def closest_model(cfg):
    """The recurrent model, one recurrence deep, with the layer count, width, heads and per-layer parameters of ``cfg``."""
    from ..models.hf import RavenForCausalLM
    from ..models.hf_config import RavenConfig

    n, E = len(cfg.layers), cfg.width
    a = next(layer.mixer for layer in cfg.layers if layer.type != "delta")         # attention heads
    a = getattr(a, "left", a)
    per_layer = (cfg.active_param_count() - 2 * cfg.vocab * E) / n
    ff = max(256, int((per_layer - 4 * E * E) / (3 * E)) // 64 * 64)
    core = max(1, n // 2)
    pre = (n - core) // 2
    rc = RavenConfig(n_embd=E, n_heads=a.heads, n_layers=n, block_size=16384, vocab_size=cfg.vocab, intermediate_size=ff,
                     n_layers_in_prelude=max(1, pre), n_layers_in_recurrent_block=core, n_layers_in_coda=n - core - pre,
                     mean_recurrence=1)
    torch.manual_seed(0)
    with torch.device("cuda"):
        return RavenForCausalLM(rc).to(torch.bfloat16).eval()


# ------------------------------------------------------------------------------------------
# single kernels
# ------------------------------------------------------------------------------------------
def visible_pairs(seqs, window: int) -> float:
    return float(sum(sum(min(i + 1, window) for i in range(n)) for n in seqs))


def layer_ops_prefill(model, seqs: list, t: Timer) -> list:
    """Kernels of one layer (with its own latents) of a packed step of fresh prompts ``seqs``."""
    from ..models.layered import PackedStep
    from ..ops import latent as ops

    cfg = model.config
    layer = model.layers[0]
    mix, a, L, E = layer.mix, layer.mix.spec, layer.mix.layout, cfg.width
    T = sum(seqs)
    cache = model.new_cache(len(seqs), max(seqs))
    step = PackedStep([(r, 0, [1] * n) for r, n in enumerate(seqs)], "cuda")
    lay = step.layout(cfg.latent_windows()[0] - 1)
    x = torch.randn(T, E, device="cuda")
    xb = x.bfloat16()
    stream = torch.empty(T, L.ld_lat, dtype=torch.bfloat16, device="cuda")
    inp = ops.linear(xb, mix.w_in[:, :E])
    rope = cache.rope[a.rot]
    ops.latent_prep_(L, inp, mix.latent_norm, mix.eps, rope, step, lay.sidx, cache.data[0], stream)
    kv = ops.linear(stream[:, :a.kv_rank], mix.w_kv[:, :a.kv_rank])
    o = ops.stream_attention(L, inp, kv, stream, lay, a.window, a.scale)
    out = ops.linear(o, mix.w_o[:, :a.heads * a.vdim])

    def gemm(name, fn, M, N, K):
        t.op(name, fn, 2.0 * (M * N + M * K + N * K), 2.0 * M * N * K)

    gemm("q|gate|latent projection", lambda: ops.linear(xb, mix.w_in[:, :E]), T, L.width_in, E)
    t.op("latent_prep", lambda: ops.latent_prep_(L, inp, mix.latent_norm, mix.eps, rope, step, lay.sidx, cache.data[0], stream),
         2.0 * T * (2 * a.heads * a.rot_dim + 3 * L.ld_lat), 0)
    gemm("key|value up-projection", lambda: ops.linear(stream[:, :a.kv_rank], mix.w_kv[:, :a.kv_rank]), T, L.width_kv, a.kv_rank)
    t.op("latent_attention", lambda: ops.stream_attention(L, inp, kv, stream, lay, a.window, a.scale),
         2.0 * T * (a.heads * (a.dim + a.rot_dim + 2 * a.vdim) + L.width_kv + a.rot_dim),
         2.0 * visible_pairs(seqs, a.window) * a.heads * (a.dim + a.rot_dim + a.vdim))
    gemm("output projection", lambda: ops.linear(o, mix.w_o[:, :a.heads * a.vdim]), T, E, a.heads * a.vdim)
    t.op("rms_residual", lambda: ops.rms_residual_(x, out, None, layer.norms["norm1"], 1e-6, 1e-6, torch.bfloat16), T * E * 12.0, 0)
    if layer.mlp is not None:
        ff = layer.mlp.spec.ff
        h = ops.linear(xb, layer.mlp.w_up[:, :E], layer.mlp.b_up, "relu2")
        gemm("up projection + bias + relu^2", lambda: ops.linear(xb, layer.mlp.w_up[:, :E], layer.mlp.b_up, "relu2"), T, ff, E)
        gemm("down projection", lambda: ops.linear(h, layer.mlp.w_down[:, :ff]), T, E, ff)
    return t.take()


def layer_ops_decode(model, B: int, context: int, t: Timer) -> list:
    from ..engine.layered import LayeredEngine
    from ..ops import latent as ops

    cfg = model.config
    layer = model.layers[0]
    mix, a, L, E = layer.mix, layer.mix.spec, layer.mix.layout, cfg.width
    eng = LayeredEngine(model, B, context + 1, use_graphs=False)
    cache = eng.cache
    for d in cache.data.values():
        d.normal_()
    pos = torch.full((B,), context, dtype=torch.int32, device="cuda")
    row = torch.arange(B, dtype=torch.int32, device="cuda")
    x = torch.randn(B, E, device="cuda")
    xb = x.bfloat16()
    inp, _ = eng._dense(xb, mix.w_in[:, :E], 0)
    inp = inp.clone()
    work = torch.zeros(B, max(E, layer.mlp.spec.ff), dtype=torch.float32, device="cuda")
    pieces = ops.ring_attention_pieces(L, inp, mix.w_kv, mix.latent_norm, mix.eps, cache.rope[a.rot], pos, row, cache.data[0],
                                       min(a.window, cache.data[0].shape[1]), a.scale, eng._splits(mix, B), torch.bfloat16)

    def skinny(name, xin, w):
        N, K = w.shape
        t.op(name, lambda: eng._dense(xin, w, 1), 2.0 * (N * K + B * K + B * N), 2.0 * B * N * K)

    skinny("q|gate|latent projection", xb, mix.w_in[:, :E])
    keys = min(a.window, context + 1)
    absorb, attend, expand = pieces
    t.op("latent_absorb", absorb, 2.0 * (a.heads * a.dim * a.kv_rank + B * (a.heads * (a.dim + a.rot_dim) * 2 + a.heads * L.ld_lat)),
         2.0 * B * a.heads * a.dim * a.kv_rank)
    t.op("latent decode attention", attend, 2.0 * B * (keys * L.ld_lat + a.heads * (L.ld_lat + a.kv_rank)),
         2.0 * B * a.heads * keys * (L.ld_lat + a.kv_rank))
    t.op("latent_expand", expand, 2.0 * (a.heads * a.vdim * a.kv_rank + B * a.heads * (a.kv_rank * 2 + 2 * a.vdim)),
         2.0 * B * a.heads * a.vdim * a.kv_rank)
    o = torch.randn(B, a.heads * a.vdim, device="cuda").bfloat16()
    skinny("output projection", o, mix.w_o[:, :a.heads * a.vdim])
    acc = work[:, :E]
    t.op("rms_residual", lambda: ops.rms_residual_(x, acc, None, layer.norms["norm1"], 1e-6, 1e-6, torch.bfloat16), B * E * 14.0, 0)
    if layer.mlp is not None:
        ff = layer.mlp.spec.ff
        skinny("up projection", xb, layer.mlp.w_up[:, :E])
        t.op("bias + relu^2", lambda: ops.bias_act(work[:, :ff], layer.mlp.b_up, "relu2", torch.bfloat16), B * ff * 6.0, 0)
        skinny("down projection", torch.randn(B, ff, device="cuda").bfloat16(), layer.mlp.w_down[:, :ff])
    return t.take()


def hybrid_ops_prefill(model, seqs: list, t: Timer) -> list:
    """Kernels of a parallel layer, of a gated memory layer and of a feed-forward of a packed step of fresh prompts ``seqs``."""
    from ..models.layered import PackedStep
    from ..ops import latent as ops
    from ..ops import memory as M
    from ..ops import memory_kernels as MK

    cfg, E, T = model.config, model.config.width, sum(seqs)
    kinds = {layer.type: i for i, layer in reversed(list(enumerate(cfg.layers)))}
    cache = model.new_cache(len(seqs), max(seqs))
    step = PackedStep([(r, 0, [1] * n) for r, n in enumerate(seqs)], "cuda")
    x = torch.randn(T, E, device="cuda")
    h = torch.randn(T, E, device="cuda").bfloat16()

    def gemm(name, fn, M_, N, K):
        t.op(name, fn, 2.0 * (M_ * N + M_ * K + N * K), 2.0 * M_ * N * K)

    i = kinds["parallel"]
    mix = model.layers[i].mix
    L, a, r = mix.layout, mix.spec.left, mix.spec.right
    kv, state = cache.data[i, "kv"], cache.data[i, "state"]
    project = lambda: ops.linear(h, mix.w_in[:, :E], mix.b_in, "silu", act_cols=L.act_cols)  # noqa: E731
    inp = project()
    o = M.parallel_output(L, T, torch.bfloat16, h.device)
    gemm("parallel: input projection + bias + silu", project, T, L.width_in, E)
    t.op("parallel: kv_append", lambda: M.kv_append(L, inp, None, kv, step.pos, step.row), 4.0 * T * L.ld_kv, 0)
    t.op("parallel: attention (bias, head gate)", lambda: M.prompt_attention(L, a, inp, kv, mix.table, step, 0.7, o),
         2.0 * T * (a.heads * (a.dim + a.vdim) + L.ld_kv), 2.0 * visible_pairs(seqs, max(seqs)) * a.heads * (a.dim + a.vdim))
    mem = M.decay_memory_prompt(L, inp, mix.decay, mix.log2_decay, state, step)
    run = MK.decay_memory(L, inp, mix.log2_decay, state, step)
    nbytes = 2.0 * T * r.heads * (2 * r.dim + 2 * r.vdim)
    t.op("parallel: memory (3 kernels)", run, nbytes, 4.0 * T * r.heads * r.dim * r.vdim)
    for part, name in ((1, "chunk states"), (2, "recurrence"), (4, "outputs")):
        t.op("  memory: " + name, lambda part=part: run(part), nbytes, 0)
    t.op("parallel: memory norm + gate", lambda: M.memory_norm(L, inp, mem, mix.norm, 1e-6, 0.7, o), 6.0 * T * r.heads * r.vdim, 0)
    gemm("parallel: output projection", lambda: ops.linear(o, mix.w_o[:, :L.width_o]), T, E, L.width_o)
    norms = model.layers[i].norms
    out = ops.linear(o, mix.w_o[:, :L.width_o])
    t.op("sandwich_norm", lambda: M.sandwich_norm_(x, out, norms["norm1b"].pair, None, norms["norm2"].pair, 1e-6, torch.bfloat16), T * E * 12.0, 0)
    i = kinds["mlstm"]
    mix = model.layers[i].mix
    L, a = mix.layout, mix.spec
    state, stab = cache.data[i, "state"], cache.data[i, "norm"]
    inp, gates = ops.linear(h, mix.w_in[:, :E]), M.gate_projections(h, mix.w_gate[:, :E])
    gemm("gated memory: input projection", lambda: ops.linear(h, mix.w_in[:, :E]), T, L.width_in, E)
    gemm("gated memory: gate projection (fp32)", lambda: M.gate_projections(h, mix.w_gate[:, :E]), T, 2 * a.heads, E)
    run = MK.gated_memory(L, inp, gates, mix.b_gate, a.gate_cap, state, stab, mix.norm, 1e-6, step)
    nbytes = 2.0 * T * a.heads * (2 * a.dim + 3 * a.vdim)
    t.op("gated memory: memory (3 kernels)", run, nbytes, 4.0 * T * a.heads * a.dim * a.vdim)
    for part, name in ((1, "chunk states"), (2, "recurrence"), (4, "outputs + norm + gate")):
        t.op("  memory: " + name, lambda part=part: run(part), nbytes, 0)
    mlp = model.layers[i].mlp
    ff = mlp.spec.ff
    g = M.glu_linear(h, mlp.w_gu[:, :E], ff, "gelu")
    gemm("gate-up projection + geglu", lambda: M.glu_linear(h, mlp.w_gu[:, :E], ff, "gelu"), T, 2 * ff, E)
    gemm("down projection", lambda: ops.linear(g, mlp.w_down[:, :ff]), T, E, ff)
    return t.take()


def hybrid_ops_decode(model, B: int, context: int, t: Timer) -> list:
    from ..engine.layered import LayeredEngine
    from ..ops import memory as M

    cfg, E = model.config, model.config.width
    kinds = {layer.type: i for i, layer in reversed(list(enumerate(cfg.layers)))}
    eng = LayeredEngine(model, B, context + 1, use_graphs=False)
    cache = eng.cache
    for key, d in cache.data.items():
        d.normal_(std=0.1)
    pos = torch.full((B,), context, dtype=torch.int32, device="cuda")
    row = torch.arange(B, dtype=torch.int32, device="cuda")
    x = torch.randn(B, E, device="cuda")
    h = x.bfloat16()
    work = torch.zeros(B, max(E, 2 * cfg.layers[0].mlp.ff), dtype=torch.float32, device="cuda")

    def skinny(name, xin, w):
        N, K = w.shape
        t.op(name, lambda: eng._dense(xin, w, 1 if N * B <= eng._work[1].numel() else 0), 2.0 * (N * K + B * K + B * N), 2.0 * B * N * K)

    i = kinds["parallel"]
    mix = model.layers[i].mix
    L, a, r = mix.layout, mix.spec.left, mix.spec.right
    skinny("parallel: input projection", h, mix.w_in[:, :E])
    inp = torch.randn(B, L.width_in, device="cuda")
    splits = mix.decode_splits(B, context + 1, True)
    po = torch.empty(B, L.heads, splits, M.pad8(L.vdim), dtype=torch.float32, device="cuda")
    ml = torch.empty(B, L.heads, splits, 2, dtype=torch.float32, device="cuda")
    o = M.parallel_output(L, B, torch.bfloat16, h.device)
    attend, scan, merge = M.parallel_decode_pieces(L, mix.spec, inp, mix.b_in, cache.data[i, "kv"], cache.data[i, "state"], mix.table, mix.decay,
                                                   mix.norm, 1e-6, pos, row, po, ml, o)
    t.op("parallel: decode attention", attend, 2.0 * B * ((context + 1) * L.ld_kv + a.heads * (a.dim + a.vdim)),
         2.0 * B * a.heads * context * (a.dim + a.vdim))
    t.op("parallel: memory update", scan, 8.0 * B * r.heads * r.dim * r.vdim, 0)
    mem = scan()
    t.op("parallel: merge, norm, gates", lambda: merge(mem), B * (4.0 * splits * a.heads * a.vdim + 2.0 * L.width_o + 8.0 * r.heads * r.vdim), 0)
    skinny("parallel: output projection", o, mix.w_o[:, :L.width_o])
    norms = model.layers[i].norms
    acc = work[:, :E]
    t.op("sandwich_norm", lambda: M.sandwich_norm_(x, acc, norms["norm1b"].pair, None, norms["norm2"].pair, 1e-6, torch.bfloat16), B * E * 14.0, 0)
    i = kinds["mlstm"]
    mix = model.layers[i].mix
    L, a = mix.layout, mix.spec
    skinny("gated memory: input projection", h, mix.w_in[:, :E])
    inp = torch.randn(B, L.width_in, device="cuda")
    t.op("gated memory: update, norm, gates", lambda: M.gated_memory(L, inp, None, mix.b_gate, a.gate_cap, cache.data[i, "state"], cache.data[i, "norm"],
                                                                     mix.norm, 1e-6, torch.bfloat16, rows=(pos, row), h=h, w_gate=mix.w_gate[:, :E]),
         8.0 * B * a.heads * a.dim * (a.vdim + 1) + 4.0 * a.heads * E, 0)
    mlp = model.layers[i].mlp
    ff = mlp.spec.ff
    skinny("gate-up projection", h, mlp.w_gu[:, :E])
    t.op("geglu", lambda: M.glu(work[:, :2 * ff], ff, "gelu", torch.bfloat16), B * ff * 10.0, 0)
    skinny("down projection", torch.randn(B, ff, device="cuda").bfloat16(), mlp.w_down[:, :ff])
    return t.take()


def routed_ops_prefill(model, seqs: list, t: Timer) -> list:
    """Kernels of a chunked and a windowed layer and of a mixture of experts of a packed step of fresh prompts ``seqs``."""
    from ..models.layered import PackedStep
    from ..ops import grouped as G
    from ..ops import latent as ops
    from ..ops import memory as M
    from ..ops import moe as X

    cfg, E, T = model.config, model.config.width, sum(seqs)
    cache = model.new_cache(len(seqs), max(seqs))
    step = PackedStep([(r, 0, [1] * n) for r, n in enumerate(seqs)], "cuda")
    x = torch.randn(T, E, device="cuda")
    h = torch.randn(T, E, device="cuda").bfloat16()
    first = None

    def gemm(name, fn, M_, N, K, groups=1):
        t.op(name, fn, 2.0 * (M_ * N + M_ * K + groups * N * K), 2.0 * M_ * N * K)

    for i, kind in ((0, "chunked"), (1, "windowed")):
        mix = model.layers[i].mix
        L, a = mix.layout, mix.spec
        lay = step.chunk_layout(a.size) if a.chunked else step.layout(a.size - 1)
        inp = ops.linear(h, mix.w_in[:, :E])
        tr = mix._transform(cfg.mixes_values(i), cache.rope, first)
        first = inp[:, L.off_v:L.off_v + L.v_width] if first is None else first
        kv = torch.empty(lay.total, L.ld_kv, dtype=torch.bfloat16, device="cuda")
        prep = lambda: G.qkv_prep_(L, inp, tr, step, lay.sidx, cache.data[i, "kv"], kv)  # noqa: E731
        prep()
        if i == 0:
            gemm("qkv projection", lambda: ops.linear(h, mix.w_in[:, :E]), T, L.width_in, E)
        ring = sum(min(n, cache.data[i, "kv"].shape[1]) for n in seqs) * L.ld_kv
        t.op(f"{kind}: qkv_prep", prep, 2.0 * (T * (2 * a.heads * a.dim + 2 * L.ld_kv + (L.v_width if tr.lam is not None else 0)) + ring), 0)
        o = G.stream_attention(L, a, inp, kv, lay, mix.sink)
        pairs = float(sum(m * (m + 1) / 2 + m * f for _, m, _, f in lay.seqs)) if a.chunked else visible_pairs(seqs, a.size)
        t.op(f"{kind}: attention", lambda: G.stream_attention(L, a, inp, kv, lay, mix.sink), 2.0 * T * (a.heads * (a.dim + a.vdim) + L.ld_kv),
             2.0 * pairs * a.heads * (a.dim + a.vdim))
    gemm("output projection", lambda: ops.linear(o, mix.w_o[:, :a.heads * a.vdim]), T, E, a.heads * a.vdim)
    norms = model.layers[1].norms
    out = ops.linear(o, mix.w_o[:, :a.heads * a.vdim])
    t.op("sandwich_norm", lambda: M.sandwich_norm_(x, out, norms["norm1b"].pair, None, norms["norm2"].pair, 1e-6, torch.bfloat16), T * E * 12.0, 0)
    w = model.layers[1].mlp.weights
    s = w.spec
    z = X.router_logits(h, w.router)
    gemm("moe: router product (fp32)", lambda: X.router_logits(h, w.router), T, w.router.shape[0], E)
    rows = X.tile_rows(s, T, torch.bfloat16)
    p = X.plan(w, z, rows)
    n = int((p.idx < s.experts).sum())
    t.op("moe: route + plan", lambda: X.plan(w, z, rows), 4.0 * T * (s.outputs + 4 * s.top), 0)
    xs = X.dispatch(w, h, p)
    t.op("moe: dispatch", lambda: X.dispatch(w, h, p), 2.0 * E * (T + n), 0)
    g = X.grouped_linear(xs, w.up, s.ff, p, s.act)
    gemm(f"moe: up (grouped, {rows}-row tiles)", lambda: X.grouped_linear(xs, w.up, s.ff, p, s.act), n, s.ff, E, s.experts)
    y = X.grouped_linear(g, w.down, E, p)
    gemm("moe: down (grouped)", lambda: X.grouped_linear(g, w.down, E, p), n, E, s.ff, s.experts)
    a_s = ops.linear(h, w.up_s, None, "relu2")
    gemm("shared expert: up", lambda: ops.linear(h, w.up_s, None, "relu2"), T, s.shared, E)
    ys = ops.linear(a_s, w.down_s)
    gemm("shared expert: down", lambda: ops.linear(a_s, w.down_s), T, E, s.shared)
    mixed = M.RowSum(y, p.slot, p.weight, h, ys)
    t.op("moe: combine", lambda: X.combine(mixed), 2.0 * E * (n + 3 * T), 0)
    t.op("moe: whole", lambda: X.mixture(w, h), 4.0 * E * (T + s.experts * s.ff + s.shared), 4.0 * E * (n * s.ff + T * s.shared))
    mlp = model.layers[0].mlp
    ff = mlp.spec.ff
    gemm("gate-up projection + swiglu", lambda: M.glu_linear(h, mlp.w_gu[:, :E], ff, "silu"), T, 2 * ff, E)
    d = M.glu_linear(h, mlp.w_gu[:, :E], ff, "silu")
    gemm("down projection", lambda: ops.linear(d, mlp.w_down[:, :ff]), T, E, ff)
    return t.take()


def routed_ops_decode(model, B: int, context: int, t: Timer) -> list:
    from ..engine.layered import LayeredEngine
    from ..ops import grouped as G
    from ..ops import memory as M
    from ..ops import moe as X

    cfg, E = model.config, model.config.width
    eng = LayeredEngine(model, B, context + 1, use_graphs=False)
    cache = eng.cache
    for d in cache.data.values():
        d.normal_(std=0.1)
    pos = torch.full((B,), context, dtype=torch.int32, device="cuda")
    row = torch.arange(B, dtype=torch.int32, device="cuda")
    x = torch.randn(B, E, device="cuda")
    h = x.bfloat16()

    def skinny(name, xin, w):
        N, K = w.shape
        t.op(name, lambda: eng._dense(xin, w, 1 if N * B <= eng._work[1].numel() else 0), 2.0 * (N * K + B * K + B * N), 2.0 * B * N * K)

    for i, kind in ((0, "chunked"), (1, "windowed")):
        mix = model.layers[i].mix
        L, a = mix.layout, mix.spec
        if i == 0:
            skinny("qkv projection", h, mix.w_in[:, :E])
        inp = torch.randn(B, L.width_in, device="cuda")
        first = torch.randn(B, M.pad8(L.v_width), device="cuda")[:, :L.v_width]
        tr = mix._transform(cfg.mixes_values(i), cache.rope, first)
        o = torch.empty(B, M.pad8(a.heads * a.vdim), dtype=torch.bfloat16, device="cuda")[:, :a.heads * a.vdim]
        splits = eng._splits(mix, B)
        attend, merge = G.ring_attention_pieces(L, a, inp, tr, cache.data[i, "kv"], mix.sink, None, pos, row, splits, o)
        keys = context % a.size + 1 if a.chunked else min(a.size, context + 1)
        t.op(f"{kind}: decode attention ({splits} splits)", attend, 2.0 * B * (keys * L.ld_kv + a.heads * (a.dim + a.vdim)),
             2.0 * B * a.heads * keys * (a.dim + a.vdim))
        if splits > 1:
            t.op(f"{kind}: merge", merge, B * a.heads * a.vdim * (4.0 * splits + 2), 0)
    skinny("output projection", o, mix.w_o[:, :a.heads * a.vdim])
    norms = model.layers[1].norms
    acc = torch.zeros(B, E, device="cuda")
    t.op("sandwich_norm", lambda: M.sandwich_norm_(x, acc, norms["norm1b"].pair, None, norms["norm2"].pair, 1e-6, torch.bfloat16), B * E * 14.0, 0)
    w = model.layers[1].mlp.weights
    s = w.spec
    parts = X.mixture_rows_pieces(w, h)
    for f in parts[:-1]:
        f()
    idx = X.plan(w, X.router_logits(h, w.router), 128).idx
    real = idx[idx < s.experts]
    n, used = real.numel(), real.unique().numel()
    weights = 2.0 * E * (used * s.ff + s.shared)
    R = w.router.shape[0]
    for name, f, b in (("moe: router product", parts[0], 2.0 * E * (R + B)), ("moe: route", parts[1], 4.0 * B * R),
                       (f"moe: up ({used} experts + shared)", parts[2], weights + 2.0 * B * E + 2.0 * (n * s.ff + B * s.shared)),
                       ("moe: down", parts[3], weights + 2.0 * (n * s.ff + B * s.shared) + 4.0 * E * (n + B)),
                       ("sandwich_norm with the sum of the experts",
                        lambda: M.sandwich_norm_(x, parts[4], norms["norm2b"].pair, None, norms["norm1"].pair, 1e-6, torch.bfloat16),
                        E * (4.0 * n + 16.0 * B))):
        t.op(name, f, b, 0)
    mlp = model.layers[0].mlp
    ff = mlp.spec.ff
    skinny("gate-up projection", h, mlp.w_gu[:, :E])
    work = torch.zeros(B, 2 * ff, device="cuda")
    t.op("swiglu", lambda: M.glu(work, ff, "silu", torch.bfloat16), B * ff * 10.0, 0)
    skinny("down projection", torch.randn(B, ff, device="cuda").bfloat16(), mlp.w_down[:, :ff])
    return t.take()


def _moe_ops_prefill(w, h, t: Timer) -> None:
    """Pieces of a mixture without identity and shared experts on the rows h."""
    from ..ops import memory as M
    from ..ops import moe as X

    s, (T, E) = w.spec, h.shape

    def gemm(name, fn, M_, N, K, groups=1):
        t.op(name, fn, 2.0 * (M_ * (N if s.act != "silu" or N == E else N // 2) + M_ * K + groups * N * K), 2.0 * M_ * N * K)

    z = X.router_logits(h, w.router)
    gemm("moe: router product (fp32)", lambda: X.router_logits(h, w.router), T, w.router.shape[0], E)
    rows = X.tile_rows(s, T, torch.bfloat16)
    p = X.plan(w, z, rows)
    n = T * s.top
    t.op("moe: route + plan", lambda: X.plan(w, z, rows), 4.0 * T * (s.outputs + 4 * s.top), 0)
    xs = X.dispatch(w, h, p)
    t.op("moe: dispatch", lambda: X.dispatch(w, h, p), 2.0 * E * (T + n), 0)
    g = X.grouped_linear(xs, w.up, s.ff, p, s.act)
    gemm(f"moe: gate-up (grouped, {rows}-row tiles)", lambda: X.grouped_linear(xs, w.up, s.ff, p, s.act), n, 2 * s.ff, E, s.experts)
    y = X.grouped_linear(g, w.down, E, p)
    gemm("moe: down (grouped)", lambda: X.grouped_linear(g, w.down, E, p), n, E, s.ff, s.experts)
    mixed = M.RowSum(y, p.slot, p.weight, h)
    t.op("moe: combine", lambda: X.combine(mixed), 2.0 * E * (n + T), 0)
    t.op("moe: whole", lambda: X.mixture(w, h), 4.0 * E * T + 6.0 * E * s.experts * s.ff, 6.0 * E * n * s.ff)


def depth_ops_prefill(model, seqs: list, t: Timer) -> list:
    """Kernels of a delta memory, a windowed layer and both kinds of feed-forward of a packed step of fresh prompts ``seqs``."""
    from ..models.layered import PackedStep
    from ..ops import delta as DL
    from ..ops import delta_kernels as DK
    from ..ops import depth as DP
    from ..ops import grouped as G
    from ..ops import latent as ops
    from ..ops import memory as M

    cfg, E, T = model.config, model.config.width, sum(seqs)
    kinds = {layer.type: i for i, layer in reversed(list(enumerate(cfg.layers)))}
    cache = model.new_cache(len(seqs), max(seqs))
    step = PackedStep([(r, 0, [1] * n) for r, n in enumerate(seqs)], "cuda")
    h = torch.randn(T, E, device="cuda").bfloat16()

    def gemm(name, fn, M_, N, K):
        t.op(name, fn, 2.0 * (M_ * N + M_ * K + N * K), 2.0 * M_ * N * K)

    i = kinds["delta"]
    mix = model.layers[i].mix
    L, a, w = mix.layout, mix.spec, mix.weights
    ring, state = cache.data[i, "conv"], cache.data[i, "state"]
    w_ba = mix.w_in[L.off_ba:L.off_ba + 2 * a.heads, :E]
    inp, ba = ops.linear(h, mix.w_in[:L.off_ba, :E]), M.gate_projections(h, w_ba)
    gemm("delta: input projection", lambda: ops.linear(h, mix.w_in[:L.off_ba, :E]), T, L.off_ba, E)
    gemm("delta: step size and decay projection (fp32)", lambda: M.gate_projections(h, w_ba), T, 2 * a.heads, E)
    act = DL.short_conv(L, inp, mix.conv, ring, step)
    t.op("delta: short convolution", lambda: DL.short_conv(L, inp, mix.conv, ring, step), 4.0 * T * L.channels, 0)
    out = torch.empty(T, a.heads * a.vdim, dtype=torch.bfloat16, device="cuda")
    run = DK.delta_prompt(L, w, act, inp, ba, state, step, out)
    nbytes = 2.0 * T * (L.channels + 2 * a.heads * a.vdim) + 8.0 * T * a.heads
    t.op("delta: memory (3 kernels)", run, nbytes, 6.0 * T * a.heads * a.dim * a.vdim)
    for part, name in ((1, "single chunks"), (2, "recurrence"), (4, "read-outs + norm + gate")):
        t.op("  delta: " + name, lambda part=part: run(part), nbytes, 0)
    gemm("delta: output projection", lambda: ops.linear(out, mix.w_o[:, :a.heads * a.vdim]), T, E, a.heads * a.vdim)
    i = kinds["attention"]
    mix = model.layers[i].mix
    L, a = mix.layout, mix.spec
    lay = step.layout(a.size - 1, a.keep)
    gemm("attention: qkv projection + bias", lambda: ops.linear(h, mix.w_in[:, :E], mix.b_in), T, L.width_in, E)
    inp = ops.linear(h, mix.w_in[:, :E], mix.b_in)
    tr = mix._transform(None, cache.rope, None)
    kv = torch.empty(lay.total, L.ld_kv, dtype=torch.bfloat16, device="cuda")
    ring = cache.data[i, "kv"]
    prep = lambda: G.qkv_prep_(L, inp, tr, step, lay.sidx, ring, kv)  # noqa: E731
    prep()
    t.op("attention: qkv_heads", prep, 2.0 * (T * (2 * a.heads * a.dim + 2 * L.ld_kv) + sum(min(n, ring.shape[1]) for n in seqs) * L.ld_kv), 0)
    pairs = visible_pairs(seqs, a.size) + float(sum(min(a.keep, max(0, p - a.size + 1)) for n in seqs for p in range(n)))
    t.op("attention: attention", lambda: G.stream_attention(L, a, inp, kv, lay, None), 2.0 * T * (a.heads * (a.dim + a.vdim) + L.ld_kv),
         2.0 * pairs * a.heads * (a.dim + a.vdim))
    o = G.stream_attention(L, a, inp, kv, lay, None)
    gemm("attention: output projection", lambda: ops.linear(o, mix.w_o[:, :a.heads * a.vdim]), T, E, a.heads * a.vdim)
    sub = ops.linear(o, mix.w_o[:, :a.heads * a.vdim])
    norm, g = model.layers[i].norms["norm1"], cfg.norm_groups
    for past in (0, 1, 8):
        s = DP.DepthStream.begin(torch.randn(past + 1, T, E, device="cuda"))
        weights = torch.full((past + 1,), 0.3, device="cuda") if past else None
        t.op(f"depth_norm (sum over {past})" if past else "depth_norm", lambda s=s, weights=weights: DP.depth_norm_(s, sub, norm, g, 1e-6, torch.bfloat16, weights=weights),
             T * E * (12.0 + (4.0 * past + 4.0 if past else 0)), 0)
        del s
    _moe_ops_prefill(next(layer.mlp for layer in model.layers if layer.mlp is not None and layer.mlp.wide == 0).weights, h, t)
    mlp = model.layers[0].mlp
    ff = mlp.spec.ff
    gemm("gate-up projection + geglu", lambda: M.glu_linear(h, mlp.w_gu[:, :E], ff, "gelu"), T, 2 * ff, E)
    d = M.glu_linear(h, mlp.w_gu[:, :E], ff, "gelu")
    gemm("down projection", lambda: ops.linear(d, mlp.w_down[:, :ff]), T, E, ff)
    return t.take()


def depth_ops_decode(model, B: int, context: int, t: Timer) -> list:
    from ..engine.layered import LayeredEngine
    from ..ops import delta as DL
    from ..ops import depth as DP
    from ..ops import grouped as G
    from ..ops import memory as M
    from ..ops import moe as X

    cfg, E = model.config, model.config.width
    kinds = {layer.type: i for i, layer in reversed(list(enumerate(cfg.layers)))}
    eng = LayeredEngine(model, B, context + 1, use_graphs=False)
    cache = eng.cache
    for d in cache.data.values():
        d.normal_(std=0.1)
    pos = torch.full((B,), context, dtype=torch.int32, device="cuda")
    row = torch.arange(B, dtype=torch.int32, device="cuda")
    h = torch.randn(B, E, device="cuda").bfloat16()

    def skinny(name, xin, w):
        N, K = w.shape
        t.op(name, lambda: eng._dense(xin, w, 1 if N * B <= eng._work[1].numel() else 0), 2.0 * (N * K + B * K + B * N), 2.0 * B * N * K)

    i = kinds["delta"]
    mix = model.layers[i].mix
    L, a = mix.layout, mix.spec
    skinny("delta: input projection", h, mix.w_in[:, :E])
    inp = torch.randn(B, L.width_in, device="cuda")
    ring, state = cache.data[i, "conv"], cache.data[i, "state"]
    t.op("delta: conv, update, norm, gate", lambda: DL.delta_decode(L, mix.weights, inp, ring, state, pos, row, torch.bfloat16),
         8.0 * B * a.heads * a.dim * a.vdim + B * (4.0 * L.width_in + 2.0 * a.conv * L.channels + 2.0 * a.heads * a.vdim), 0)
    skinny("delta: output projection", torch.randn(B, a.heads * a.vdim, device="cuda").bfloat16(), mix.w_o[:, :a.heads * a.vdim])
    i = kinds["attention"]
    mix = model.layers[i].mix
    L, a = mix.layout, mix.spec
    skinny("attention: qkv projection", h, mix.w_in[:, :E])
    inp = torch.randn(B, L.width_in, device="cuda")
    tr = mix._transform(None, cache.rope, None, raw=True)
    o = torch.empty(B, M.pad8(a.heads * a.vdim), dtype=torch.bfloat16, device="cuda")[:, :a.heads * a.vdim]
    splits = eng._splits(mix, B)
    attend, merge = G.ring_attention_pieces(L, a, inp, tr, cache.data[i, "kv"], None, None, pos, row, splits, o)
    keys = min(a.slots, context + 1)
    t.op(f"attention: decode attention ({splits} splits)", attend, 2.0 * B * (keys * L.ld_kv + a.heads * (a.dim + a.vdim)),
         2.0 * B * a.heads * keys * (a.dim + a.vdim))
    if splits > 1:
        t.op("attention: merge", merge, B * a.heads * a.vdim * (4.0 * splits + 2), 0)
    norm, g = model.layers[i].norms["norm1"], cfg.norm_groups
    acc = torch.zeros(B, E, device="cuda")
    for past in (0, 8):
        s = DP.DepthStream.begin(torch.randn(past + 1, B, E, device="cuda"))
        weights = torch.full((past + 1,), 0.3, device="cuda") if past else None
        t.op(f"depth_norm (sum over {past})" if past else "depth_norm", lambda s=s, weights=weights: DP.depth_norm_(s, acc, norm, g, 1e-6, torch.bfloat16, weights=weights),
             B * E * (14.0 + (4.0 * past + 4.0 if past else 0)), 0)
    w = next(layer.mlp for layer in model.layers if layer.mlp is not None and layer.mlp.wide == 0).weights
    s = w.spec
    parts = X.mixture_rows_pieces(w, h)
    for f in parts[:-1]:
        f()
    used = X.plan(w, X.router_logits(h, w.router), 128).idx.unique().numel()
    n, R = B * s.top, w.router.shape[0]
    for name, f, b in (("moe: router product", parts[0], 2.0 * E * (R + B)), ("moe: route", parts[1], 4.0 * B * R),
                       (f"moe: gate-up ({used} experts)", parts[2], 4.0 * E * used * s.ff + 2.0 * B * E + 2.0 * n * s.ff),
                       ("moe: down", parts[3], 2.0 * E * used * s.ff + 2.0 * n * s.ff + 4.0 * E * n)):
        t.op(name, f, b, 0)
    st = DP.DepthStream.begin(torch.randn(9, B, E, device="cuda"))
    weights = torch.full((9,), 0.3, device="cuda")
    t.op("depth_norm with the sum of the experts (sum over 8)", lambda: DP.depth_norm_(st, parts[4], norm, g, 1e-6, torch.bfloat16, weights=weights),
         E * (4.0 * n + 46.0 * B), 0)
    mlp = model.layers[0].mlp
    ff = mlp.spec.ff
    skinny("gate-up projection", h, mlp.w_gu[:, :E])
    work = torch.zeros(B, 2 * ff, device="cuda")
    t.op("geglu", lambda: M.glu(work, ff, "gelu", torch.bfloat16), B * ff * 10.0, 0)
    skinny("down projection", torch.randn(B, ff, device="cuda").bfloat16(), mlp.w_down[:, :ff])
    return t.take()


def closest_ops_prefill(model, B: int, S: int, t: Timer) -> list:
    from ..ops import attention as A
    from ..ops import cuda as K

    c = model.config
    block = model.transformer.core_block[0]
    H, D, E, T = c.n_heads, c.head_dim, c.n_embd, B * S
    x = torch.randn(T, E, device="cuda").bfloat16()
    cos, sin = model._rope(S)

    def gemm(name, fn, M, N, Kd):
        t.op(name, fn, 2.0 * (M * N + M * Kd + N * Kd), 2.0 * M * N * Kd)

    qkv = K.gemm_nt(x, block.attn.Wqkv.weight)
    gemm("qkv projection", lambda: K.gemm_nt(x, block.attn.Wqkv.weight), T, 3 * H * D, E)
    q3 = qkv.view(B, S, -1)
    bias = block.attn.qk_bias
    r = K.rope_fwd(q3, bias, cos, sin, H, H, D)
    t.op("rope", lambda: K.rope_fwd(q3, bias, cos, sin, H, H, D), 2.0 * 2 * T * 3 * H * D, 0)
    t.op("attention", lambda: A.fwd(r, H, H, D, D ** -0.5), 2.0 * T * 4 * H * D, 2.0 * visible_pairs([S] * B, S) * H * 2 * D)
    o = torch.randn(T, H * D, device="cuda").bfloat16()
    gemm("output projection", lambda: K.gemm_nt(o, block.attn.proj.weight), T, E, H * D)
    t.op("add + rmsnorm", lambda: K.add_rmsnorm_fwd(o, x, block.norm_2.weight, 1e-6), 2.0 * 4 * T * E, 0)
    I = block.mlp.proj.weight.shape[1]
    g = torch.randn(T, I, device="cuda").bfloat16()
    gemm("gate-up projection + swiglu", lambda: K.gemm(x, block.mlp.fc.weight, out_mode=K.OUT_SWIGLU), T, 2 * I, E)
    gemm("down projection", lambda: K.gemm_nt(g, block.mlp.proj.weight), T, E, I)
    return t.take()


def closest_ops_decode(model, B: int, context: int, t: Timer) -> list:
    from ..engine import decode as D_
    from ..engine.decode import DecodeEngine
    from ..ops import cuda as K

    c = model.config
    block = model.transformer.core_block[0]
    H, D, E = c.n_heads, c.head_dim, c.n_embd
    eng = DecodeEngine(model, B, context + 1, num_steps=1, use_graphs=False)
    eng.pos.fill_(context)
    eng.lens.fill_(context + 1)
    kc, vc = eng.cache.k[0].normal_(), eng.cache.v[0].normal_()
    x = torch.randn(B, E, device="cuda").bfloat16()
    I = block.mlp.proj.weight.shape[1]

    def skinny(name, xin, w):
        N, Kd = w.shape
        t.op(name, lambda: eng._linear(xin, w, keep_f32=True), 2.0 * (N * Kd + B * Kd + B * N), 2.0 * B * N * Kd)

    skinny("qkv projection", x, block.attn.Wqkv.weight)
    qkv = torch.randn(B, 3 * H * D, device="cuda").bfloat16()
    q = torch.empty(B, H * D, dtype=torch.bfloat16, device="cuda")
    o = torch.empty_like(q)
    t.op("rope_append", lambda: K._check(D_._rope_append(
        qkv.data_ptr(), 0, eng.cos.data_ptr(), eng.sin.data_ptr(), eng.pos.data_ptr(), q.data_ptr(), kc.data_ptr(), vc.data_ptr(), B, H, H, D,
        eng.Lmax, K._stream(), 0), "rope_append"), 2.0 * B * 6 * H * D, 0)
    t.op("decode attention", lambda: K._check(D_._decode_attn(
        q.data_ptr(), kc.data_ptr(), vc.data_ptr(), eng.lens.data_ptr(), o.data_ptr(), eng.part_o.data_ptr(), eng.part_ml.data_ptr(), B, H, H, D,
        eng.Lmax, eng.splits, D ** -0.5, K._stream()), "decode_attention"), 2.0 * B * H * D * (2 * (context + 1) + 2), 4.0 * B * H * D * context)
    skinny("output projection", o, block.attn.proj.weight)
    t.op("add + rmsnorm pair", lambda: eng._pair(o, x, block.norm_2, block.norm_3), 2.0 * 4 * B * E, 0)
    skinny("gate-up projection", x, block.mlp.fc.weight)
    gu = torch.randn(B, 2 * I, device="cuda")
    g = torch.empty(B, I, dtype=torch.bfloat16, device="cuda")
    t.op("swiglu", lambda: K._check(D_._swiglu_acc(gu.data_ptr(), g.data_ptr(), B, I, K._stream()), "swiglu_acc"), B * I * 18.0, 0)
    skinny("down projection", torch.randn(B, I, device="cuda").bfloat16(), block.mlp.proj.weight)
    return t.take()


# ------------------------------------------------------------------------------------------
# whole models
# ------------------------------------------------------------------------------------------
def model_rates(cfg, prompt: int, new: int, batches) -> dict:
    from ..engine.decode import DecodeEngine
    from ..engine.layered import LayeredEngine
    from ..models.layered import LayeredForCausalLM

    out: dict = {"prompt": prompt, "new_tokens": new, "ours": {}, "closest": {}}
    model = LayeredForCausalLM(cfg, torch.bfloat16, "cuda").init_weights()
    out["ours"]["parameters"] = cfg.param_count()
    for B in batches:
        eng = LayeredEngine(model, B, prompt + new + 1, prefill_tokens=65536)
        prompts = torch.randint(0, cfg.vocab, (B, prompt)).tolist()

        def pre():
            rows = [eng.open() for _ in prompts]
            eng.prefill(rows, prompts)
            for r in rows:
                eng.close(r)

        eng.generate(prompts, 4)
        t_pre, t_all = time_calls(pre, 3), time_calls(lambda: eng.generate(prompts, new), 2)
        out["ours"][str(B)] = {"prefill_tok_s": round(B * prompt / t_pre * 1e3), "decode_tok_s": round(B * (new - 1) / (t_all - t_pre) * 1e3, 1),
                               "decode_ms_per_token": round((t_all - t_pre) / (new - 1), 3), "cache_mib": round(eng.cache.get_memory_usage(), 1)}
        del eng
    del model
    torch.cuda.empty_cache()
    model = closest_model(cfg)
    out["closest"]["parameters"] = sum(p.numel() for p in model.parameters())
    for B in batches:
        eng = DecodeEngine(model, B, prompt + new + 1, num_steps=1)
        ids = torch.randint(0, cfg.vocab, (B, prompt), device="cuda")
        if B * prompt > 65536:
            continue                      # its prefill returns the logits of every position
        eng.generate(ids, 4, init_scale=0.0)
        t_pre = time_calls(lambda: eng.prefill(ids, 1, 0.0), 3)
        t_all = time_calls(lambda: eng.generate(ids, new, init_scale=0.0), 2)
        out["closest"][str(B)] = {"prefill_tok_s": round(B * prompt / t_pre * 1e3), "decode_tok_s": round(B * (new - 1) / (t_all - t_pre) * 1e3, 1),
                                  "decode_ms_per_token": round((t_all - t_pre) / (new - 1), 3),
                                  "cache_mib": round(eng.cache.get_memory_usage(), 1)}
        del eng
    return out


SHAPES = ("gasovik-1b", "gasovik-core-5280", "fatudra-1b", "fatudra-core-5280", "dusilorn-2b", "dusilorn-core-5280", "bolovik-3b",
          "bolovik-core-5280")


def run(shapes=SHAPES, batches=(1, 8, 32), prompt: int = 2048, new: int = 128, ops_only: bool = False) -> dict:
    from ..models.layered import LayeredForCausalLM
    from ..models.layered_config import LayeredConfig
    from ..ops import cuda as K

    rec: dict = {}
    for name in shapes:
        cfg = LayeredConfig.from_name(name)
        r: dict = {}
        if not ops_only:
            r["models"] = model_rates(cfg, prompt, new, batches)
            torch.cuda.empty_cache()
        t = Timer()
        ops_prefill, ops_decode = {"post_rms": (layer_ops_prefill, layer_ops_decode), "sandwich": (hybrid_ops_prefill, hybrid_ops_decode),
                                   "sandwich_rms": (routed_ops_prefill, routed_ops_decode), "post_group_rms": (depth_ops_prefill, depth_ops_decode)}[cfg.design.norms]
        kept = 4 if cfg.design.depth_average else 2 if cfg.design.sandwich else 1
        few = replace(cfg, vocab=1024, layers=cfg.layers[:kept], loop=None)
        model = LayeredForCausalLM(few, torch.bfloat16, "cuda").init_weights()
        S = 4096
        r["prefill_ops"] = {"tokens": S, "ours": ops_prefill(model, [S], t)}
        r["decode_ops"] = {f"batch {B}": {"context": S, "ours": ops_decode(model, B, S, t)} for B in (1, 8, 64)}
        del model
        ref = closest_model(replace(cfg, vocab=1024, layers=cfg.layers[:max(3, kept)], loop=None))
        r["prefill_ops"]["closest"] = closest_ops_prefill(ref, 1, S, t)
        for B in (1, 8, 64):
            r["decode_ops"][f"batch {B}"]["closest"] = closest_ops_decode(ref, B, S, t)
            torch.cuda.empty_cache()
        del ref
        rec[name] = r
        torch.cuda.empty_cache()
    rec["device_status"] = K.check_device_status()
    return rec


def main():
    ap = argparse.ArgumentParser(description=__doc__.split("\n\n")[0])
    ap.add_argument("--shapes", default=",".join(SHAPES))
    ap.add_argument("--batches", default="1,8,32")
    ap.add_argument("--prompt", type=int, default=2048)
    ap.add_argument("--new", type=int, default=128)
    ap.add_argument("--ops-only", action="store_true")
    args = ap.parse_args()
    rec = run(args.shapes.split(","), [int(b) for b in args.batches.split(",")], args.prompt, args.new, args.ops_only)
    for name, r in rec.items():
        if not isinstance(r, dict):
            print(name, r)
            continue
        if "models" in r:
            for who in ("ours", "closest"):
                print(name, who, json.dumps(r["models"][who]))
        for title, block in [("prefill", r["prefill_ops"])] + [(f"decode {b}", d) for b, d in r["decode_ops"].items()]:
            for who in ("ours", "closest"):
                for row in block[who]:
                    print(f"{name:18s} {title:16s} {who:8s} {row['op']:42s} {row['us']:9.2f} us  floor {row['roofline_us']:8.2f}  "
                          f"{row['fraction']:.3f} {row['bound']}")


if __name__ == "__main__":
    main()
