"""Layered decoder models with gated delta memories, windows that keep the first tokens, experts chosen within groups and sums over depth
(design ``Bolovik``): every mechanism and the serving path against the plain statements of ``depth_oracle``, on the CPU (fp32) and on the
GPU kernels (fp32, bf16)."""
import io
import json
import math
import os

import pytest
import torch

import depth_oracle as O
from recurrent_pretraining_b200.models import auto, build_model
from recurrent_pretraining_b200.models.layered import LayeredForCausalLM
from recurrent_pretraining_b200.models.layered_config import GroupedMixtureSpec, KeptWindowAttentionSpec, LayeredConfig, RotarySpec, WavelengthScaling
from recurrent_pretraining_b200.models.sublayers import PackedStep, gather_history, rope_tables
from recurrent_pretraining_b200.ops import delta as DL
from recurrent_pretraining_b200.ops import depth as DP
from recurrent_pretraining_b200.ops import grouped as G
from recurrent_pretraining_b200.ops import latent as ops
from recurrent_pretraining_b200.ops import memory as M
from recurrent_pretraining_b200.ops import moe as X

gpu = pytest.mark.gpu
RUNS = [pytest.param(("cpu", torch.float32), id="cpu"), pytest.param(("cuda", torch.float32), marks=gpu, id="gpu-f32"),
        pytest.param(("cuda", torch.bfloat16), marks=gpu, id="gpu-bf16")]
D = torch.float64


@pytest.fixture(params=RUNS)
def run(request):
    return request.param


def load(cfg, w, run):
    model = LayeredForCausalLM(LayeredConfig.from_dict(cfg), run[1], run[0])
    model.load_checkpoint(O.TensorDict(w))
    return model


def make(cfg, run, seed=0, **kw):
    w = O.random_weights(cfg, seed, **kw)
    return load(cfg, w, run), w


def steady(cfg, run):
    """In bf16 all experts are chosen: a router's nearly equal scores may fall either way, and memories carry the difference on.  (The
    choice has its own tests.)"""
    cfg = json.loads(json.dumps(cfg))
    if run[1] == torch.bfloat16:
        for layer in cfg["layers"]:
            if layer["mlp"] is not None and layer["mlp"]["kind"] == "moe":
                r = layer["mlp"]["router"]
                r["top"], r["groups"]["keep"] = r["experts"], r["groups"]["count"]
    return cfg


def engine(model, rows=4, max_len=400, **kw):
    from recurrent_pretraining_b200.engine.layered import LayeredEngine

    return LayeredEngine(model, rows, max_len, **kw)


def tokens(n, vocab=67, seed=0):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(5000 + seed + 7919 * n)).tolist()


def feed(eng, row, seq, cuts):
    """Run ``seq`` in portions of the given sizes (the last one repeats); logits of every position."""
    out, at, k = [], 0, 0
    while at < len(seq):
        n = min(cuts[min(k, len(cuts) - 1)], len(seq) - at)
        out.append(eng.step([(row, seq[at:at + n])], [list(range(n))]).cpu())
        at, k = at + n, k + 1
    return torch.cat(out)


def status_ok(run):
    if run[0] == "cuda":
        from recurrent_pretraining_b200.ops import cuda as K

        assert K.check_device_status() == 0


def agree(got, want, run, what="", bf16=0.1):
    """Logits of every position."""
    d = got.double().cpu() - want
    d = d - d.mean(-1, keepdim=True)
    s = want - want.mean(-1, keepdim=True)
    err = (d.square().mean(-1) / s.square().mean()).sqrt().flatten()
    assert bool(torch.isfinite(err).all()), what
    if run[1] == torch.float32:
        assert float(err.max()) < 4e-5, (what, float(err.max()), int(err.argmax()))
    else:
        assert float(err.max()) < bf16, (what, float(err.max()), int(err.argmax()))


def near(got, want, dtype, f32=2e-5, bf16=8e-3, what=""):
    """rms error over rms."""
    d = got.double().cpu() - want
    err = float(d.square().mean().sqrt() / want.square().mean().sqrt())
    assert bool(torch.isfinite(d).all()) and err < (f32 if dtype == torch.float32 else bf16), (what, err)


def rnd(*shape, seed=0, scale=1.0):
    """Values that bf16 represents exactly."""
    return (torch.randn(*shape, generator=torch.Generator().manual_seed(seed)) * scale).bfloat16()


def pitched(t, dtype, dev, fill=float("nan")):
    """``t`` with a row pitch of a multiple of eight."""
    out = torch.full((t.shape[0], ops.pad8(t.shape[1])), fill, dtype=dtype, device=dev)
    out[:, :t.shape[1]] = t.to(dtype)
    return out[:, :t.shape[1]]


# layers that differ in every size, both kinds first and last, layers without feed-forward, all choices of experts and groups
MIXED = O.config([O.memory(), O.attn(), O.memory(heads=6, kv_heads=1, dim=24, vdim=8, conv=2), O.attn(heads=5, kv_heads=1, dim=8, vdim=72, size=30, keep=0, rot=6, scaling=None),
                  O.attn(heads=3, kv_heads=3, dim=32, vdim=16, size=5, keep=21, rot=32), O.memory(heads=2, kv_heads=2, dim=32, vdim=40, conv=3)],
                 [O.moe(), None, O.mlp(), O.moe(experts=8, top=5, ff=72, count=4, keep=3), O.moe(experts=4, top=4, ff=16, count=1, keep=1)])
# nothing is a multiple of eight
ODD = O.config([O.attn(heads=6, kv_heads=3, dim=11, vdim=13, size=9, keep=5, rot=6), O.memory(heads=6, kv_heads=2, dim=13, vdim=11, conv=5)],
               [O.moe(experts=9, top=2, ff=19, count=3, keep=1), O.mlp(37)], width=45, vocab=61, eps=1e-3, groups=5)
# everything that can be one
ONE = O.config([O.memory(heads=1, kv_heads=1, dim=8, vdim=8, conv=1), O.attn(heads=1, kv_heads=1, dim=8, vdim=8, size=1, keep=1, rot=2, scale=1.0)],
               [O.moe(experts=1, top=1, ff=8, count=1, keep=1), O.moe(experts=2, top=1, ff=1, count=2, keep=1)], width=16, vocab=19, groups=1)
# sizes of the tensor-core kernels
WIDE = O.config([O.attn(heads=20, kv_heads=1, dim=64, vdim=128, size=50, keep=7, rot=32), O.memory(heads=8, kv_heads=2, dim=64, vdim=128),
                 O.memory(heads=2, kv_heads=2, dim=128, vdim=64), O.attn(heads=4, kv_heads=2, dim=128, vdim=64, size=30, keep=33, rot=128, base=1e6)],
                [O.moe(experts=8, top=4, ff=136, count=4, keep=2), O.mlp(520), O.moe(experts=40, top=8, ff=64, count=5, keep=2)], width=520, groups=1)
CONFIGS = {"mixed": MIXED, "odd": ODD, "one": ONE, "wide": WIDE}


# ------------------------------------------------------------------------------------------
# configuration, weights, loading
# ------------------------------------------------------------------------------------------
@pytest.mark.parametrize("name", list(CONFIGS))
def test_config_round_trip_and_dispatch(tmp_path, name):
    d = CONFIGS[name]
    cfg = LayeredConfig.from_dict(d)
    assert json.loads(json.dumps(cfg.to_dict())) == json.loads(json.dumps(d))
    cfg.save(str(tmp_path))
    assert LayeredConfig.from_pretrained(str(tmp_path)).to_dict() == cfg.to_dict()
    model = build_model(cfg, dtype=torch.float32)
    want = O.shapes(d)
    assert {k: tuple(v.shape) for k, v in model.checkpoint_tensors().items()} == want
    assert cfg.param_count() == sum(math.prod(s) for s in want.values())
    idle = sum((m["router"]["experts"] - m["router"]["top"]) * 3 * m["expert"]["ff"] * d["width"]
               for m in (layer["mlp"] for layer in d["layers"]) if m is not None and m["kind"] == "moe")
    assert cfg.param_count() - cfg.active_param_count() == idle


def test_weights_are_loaded_and_saved(tmp_path):
    from recurrent_pretraining_b200.models.weights import save_safetensors

    w = O.random_weights(MIXED, 3)
    with open(tmp_path / "config.json", "w") as f:
        json.dump(MIXED, f)
    save_safetensors(str(tmp_path / "model.safetensors"), w)
    model = auto.load_pretrained(str(tmp_path), torch.float32, torch.device("cpu"))
    assert all(torch.equal(v, w[k].float()) for k, v in model.checkpoint_tensors().items())
    seq = tokens(9)
    agree(model(torch.tensor([seq]))[0], O.forward(MIXED, w, seq), ("cpu", torch.float32))
    again = tmp_path / "again"
    model.save_pretrained(str(again))
    assert torch.equal(auto.load_pretrained(str(again), torch.float32, torch.device("cpu"))(torch.tensor([seq])), model(torch.tensor([seq])))
    for change in (lambda t: t.pop("l0.mlp.e3.up"), lambda t: t.update({"l1.mix.sink": torch.zeros(4)}), lambda t: t.update({"l2.dwa": torch.zeros(3)}),
                   lambda t: t.pop("l0.mix.k.conv"), lambda t: t.update({"l0.mlp.correction": torch.zeros(6)})):
        bad = dict(w)
        change(bad)
        with pytest.raises(ValueError):
            model.load_checkpoint(O.TensorDict(bad))


def _mix(c, i=0):
    return c["layers"][i]["mixer"]


@pytest.mark.parametrize("change", [
    lambda c: c.update(residual_mult=0.5), lambda c: c.update(loop={"start": 0, "stop": 1, "times": 2}), lambda c: c["norm"].update(groups=5), lambda c: c["norm"].update(groups=0),
    lambda c: c["layers"][0].update(type="parallel"), lambda c: c["layers"][0].update(type="attention"), lambda c: _mix(c).update(kv_heads=3),
    lambda c: _mix(c).update(conv=0), lambda c: _mix(c).pop("conv"), lambda c: _mix(c, 1)["mask"].update(size=0), lambda c: _mix(c, 1)["mask"].update(keep_first=-1),
    lambda c: _mix(c, 1).update(softcap=2.0), lambda c: _mix(c, 1).update(v_mix=True), lambda c: _mix(c, 1)["rot"].update(dims=18), lambda c: _mix(c, 1)["rot"].update(dims=7),
    lambda c: _mix(c, 1)["rot"].update(scaling={"factor": 2.0, "original": 64, "fast": 2.0, "slow": 1.0}),
    lambda c: c["layers"][0]["mlp"].update(shared={"ff": 8}), lambda c: c["layers"][0]["mlp"]["router"].update(identity=1),
    lambda c: c["layers"][0]["mlp"]["router"].update(top=5), lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(count=4),
    lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(keep=4), lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(keep=0)])
def test_invalid_configs_are_refused(change):
    cfg = json.loads(json.dumps(MIXED))
    change(cfg)
    with pytest.raises((ValueError, KeyError)):
        LayeredConfig.from_dict(cfg)


def test_registry_shapes_build():
    tiny = build_model(LayeredConfig.from_name("bolovik-tiny"), dtype=torch.float32).init_weights(1)
    out = tiny(torch.tensor([[1, 2, 3], [4, 5, 6]]))
    assert out.shape == (2, 3, 512) and bool(torch.isfinite(out).all())
    for name in ("bolovik-3b", "bolovik-core-5280"):
        c = LayeredConfig.from_name(name)
        assert c.param_count() > 3e9 > c.active_param_count()


# ------------------------------------------------------------------------------------------
# norms and sums over depth
# ------------------------------------------------------------------------------------------
@pytest.mark.parametrize("E,groups", [(45, 5), (45, 1), (48, 2), (264, 3), (2048, 2), (2056, 1), (4096, 16), (9000, 3)])
@pytest.mark.parametrize("past", [0, 1, 6])
def test_group_norms_and_sums_over_depth(run, E, groups, past):
    """Sublayer outputs in operand precision, as accumulators and as sums of experts; results that are kept for later layers or not."""
    dev, dtype = run
    T = 5
    g = torch.Generator().manual_seed(E + past)
    x0, w = torch.randn(T, E, generator=g) * 2, 1 + 0.4 * torch.randn(E, generator=g)
    old, dwa = torch.randn(past, T, E, generator=g), torch.randn(past + 1, generator=g)
    a = rnd(T, E, seed=1, scale=3.0) * torch.linspace(0.1, 3, E).bfloat16()           # groups of different size
    rows, slot = rnd(9, E, seed=2), torch.randint(0, 9, (T, 4), generator=g, dtype=torch.int32)
    weight = torch.rand(T, 5, generator=g)
    mixed = sum(weight[:, k, None].double() * rows[slot[:, k].long()].double() for k in range(4))
    acc = torch.zeros(T, ops.pad8(E), device=dev)[:, :E]
    acc.copy_(a)
    many = M.RowSum(pitched(rows, torch.float32, dev), slot.to(dev), weight.to(dev), pitched(a, dtype, dev))
    for src, value, clear in ((pitched(a, dtype, dev), a.double(), False), (acc, a.double(), dev == "cuda"), (many, mixed, False)):
        for keep in ((True, False) if past else (False,)):
            buf = torch.zeros(past + 1 if keep else max(past, 1), T, E, device=dev)
            buf[:past] = old
            s = DP.DepthStream(buf, x0.to(dev), torch.empty(T, E, device=dev))
            extra = torch.ones(T, 12, device=dev)
            if clear:
                acc.copy_(a)
            h = DP.depth_norm_(s, src, w.to(dev), groups, 1e-4, dtype, clear=clear, zero=extra if dev == "cuda" else None, weights=dwa.to(dev) if past else None)
            own = x0.double() + O.group_norm(value, w.double(), groups, 1e-4)
            want = O.depth_average(list(old.double()) + [own], dwa.double()) if past else own
            near(s.x, want, torch.float32)
            near(h, want, dtype)
            if keep:
                near(buf[past], own, torch.float32)
                assert torch.equal(buf[:past].cpu(), old)
            assert dev == "cpu" or (not extra.any() and (not clear or not acc.any()))
    idx = torch.tensor([3, 1, 3], dtype=torch.int32)
    near(DP.group_norm_rows(x0.to(dev), idx.to(dev), w.to(dev), groups, 1e-5, dtype), O.group_norm(x0.double()[[3, 1, 3]], w.double(), groups, 1e-5), dtype)
    near(DP.group_norm_rows(x0.to(dev), None, w.to(dev), groups, 1e-5, dtype), O.group_norm(x0.double(), w.double(), groups, 1e-5), dtype)


# ------------------------------------------------------------------------------------------
# attention
# ------------------------------------------------------------------------------------------
@pytest.mark.parametrize("scaling", [O.SCALING, {"factor": 8.0, "low": 2.0, "high": 2.0, "original": 100}, {"factor": 5.0, "low": 0.5, "high": 3.0, "original": 1e6}, None], ids=str)
def test_scaled_rotation(scaling):
    rot = {"base": 500.0, "dims": 24, **({"scaling": scaling} if scaling else {})}
    spec = RotarySpec.from_dict(rot, WavelengthScaling)
    want = O.frequencies(rot)
    assert spec.frequencies() == pytest.approx(want, rel=1e-12)
    if scaling == O.SCALING:                                         # all three ranges occur
        ratio = [a / b for a, b in zip(want, O.frequencies({"base": 500.0, "dims": 24}))]
        assert 1.0 in ratio and min(ratio) == pytest.approx(1 / 3.0) and any(1 / 3.0 < r < 1 for r in ratio)
    cos, sin = rope_tables(spec, 300, "cpu")
    x = torch.randn(24, dtype=D)
    for p in (0, 1, 77, 299):
        near(torch.cat([x[:12] * cos[p] - x[12:] * sin[p], x[12:] * cos[p] + x[:12] * sin[p]]), O.rotate_half(x, p, rot), torch.float32)


SIZES = [(4, 2, 16, 24), (6, 2, 64, 64), (3, 1, 128, 128), (10, 2, 96, 96), (20, 1, 64, 128), (3, 3, 12, 13), (3, 3, 11, 5), (2, 1, 200, 128), (2, 2, 256, 256), (1, 1, 8, 8)]
by_name = lambda s: "x".join(map(str, s))  # noqa: E731


def spec_of(size, reach, keep, sharp=1.0, rot=None):
    H, Gk, dim, vdim = size
    return KeptWindowAttentionSpec(H, Gk, dim, vdim, reach, sharp * dim ** -0.5, None, rot=RotarySpec(300.0, rot or max(2, dim // 4 * 2), WavelengthScaling(2.0, 1.0, 4.0, 64.0)), keep=keep)


def transform(a, run, bias=None):
    """The row transform and the same as plain functions of (q, k or v [.., n], position)."""
    tr = G.QkvTransform(None, None, 1e-4, a.rot.dims, rope_tables(a.rot, 700, run[0]), head_norm=True, bias=bias, keep=a.keep)

    def turned(x, heads, pos):
        return O.rms_norm(O.rotate_half(x.double().view(heads, a.dim), pos, a.rot.to_dict()), 1e-4)

    return tr, lambda x, p: turned(x, a.heads, p), lambda x, p: turned(x, a.kv_heads, p), lambda x: O.rms_norm(x.double().view(a.kv_heads, a.vdim), 1e-4)


def attention_want(a, q, k, v, see):
    """q [H, dim] over keys k, v [n, G, .] of which ``see`` are visible -> [H, vdim]."""
    group = a.heads // a.kv_heads
    return torch.stack([O.softmax_weights((k[see, h // group] @ q[h]) * a.scale) @ v[see, h // group] for h in range(a.heads)])


@pytest.mark.parametrize("history,keep", [(10, 4), (10, 0), (1, 30), (0, 5), (200, 200)])
def test_layout_with_kept_positions(history, keep):
    """The stream holds what a portion's tokens can see; a ring that keeps the first positions hands it out."""
    portions = [(0, 0, 50), (3, 13, 1), (1, 16, 40), (2, 399, 3)]
    lay = PackedStep([(r, s, [0] * n) for r, s, n in portions], "cpu").layout(history, keep)
    cap = min(keep + history + 1, 500)
    cache = torch.full((4, cap, 2), -1.0)
    for r, s, _ in portions:
        for p in range(s):
            if p < keep or p >= s - (cap - keep):
                cache[r, G.ring_slots(torch.tensor(p), cap, keep)] = torch.tensor([float(r), float(p)])
    stream = torch.full((lay.total, 2), -2.0)
    gather_history(lay, cache, stream, keep)
    t = 0
    for r, s, n in portions:
        held = sorted({p for p in range(s) if p < keep or p >= s - history})
        at = int(lay.kbase[t])
        assert stream[at:at + len(held)].tolist() == [[r, p] for p in held]
        assert [int(x) for x in lay.sidx[t:t + n]] == list(range(at + len(held), at + len(held) + n))
        t += n


@pytest.mark.parametrize("size", SIZES, ids=by_name)
def test_heads_are_rotated_normed_and_kept(run, size):
    """The projection rows of a packed step: queries in place, keys and values in the stream and in the rings."""
    dev, dtype = run
    H, Gk, dim, vdim = size
    a = spec_of(size, 14, 6)
    L = G.GroupedLayout(H, Gk, dim, vdim)
    step = PackedStep([(2, 0, [0] * 45), (0, 7, [0] * 3), (1, 19, [0] * 1)], dev)
    lay = step.layout(13, 6)
    x = rnd(step.T, L.width_in, seed=4)
    tr, fq, fk, fv = transform(a, run)
    inp = x.to(dtype).to(dev)
    cache, stream = torch.zeros(3, 20, L.ld_kv, dtype=dtype, device=dev), torch.zeros(lay.total, L.ld_kv, dtype=dtype, device=dev)
    G.qkv_prep_(L, inp, tr, step, lay.sidx, cache, stream)
    for t0, n, row, start in step.sequences():
        for i in sorted({0, 1, 5, 6, n // 2, n - 14, n - 1} & set(range(n))):
            t, p = t0 + i, start + i
            near(inp[t, :H * dim], fq(x[t, :H * dim], p).flatten(), dtype)
            kv = stream[int(lay.sidx[t])]
            near(kv[:Gk * dim], fk(x[t, L.off_k:L.off_k + Gk * dim], p).flatten(), dtype)
            near(kv[L.kv_v:L.kv_v + L.v_width], fv(x[t, L.off_v:L.off_v + L.v_width]).flatten(), dtype)
            if p < 6 or i >= n - 14:
                slot = p if p < 20 else 6 + (p - 6) % 14
                for at, m in ((0, Gk * dim), (L.kv_v, L.v_width)):
                    assert torch.equal(cache[row, slot, at:at + m], kv[at:at + m])


@pytest.mark.parametrize("size", SIZES, ids=by_name)
@pytest.mark.parametrize("reach,keep,sharp", [(129, 20, 6.0), (1, 3, 1.0), (300, 1, 3.0), (64, 0, 2.0), (17, 150, 4.0), (100, 128, 30.0), (5, 300, 1.0)])
def test_prompt_attention(run, size, reach, keep, sharp):
    """Queries of several sequences (fresh, continued, one token) over a key stream; some keys stand out, around tile borders and the edges of
    windows and kept positions; scores that are bounded and scores that are not."""
    dev, dtype = run
    if dev == "cpu" and size not in SIZES[:1] + SIZES[5:6]:
        pytest.skip("two sizes on the CPU")
    H, Gk, dim, vdim = size
    a = spec_of(size, reach, keep, sharp)
    L = G.GroupedLayout(H, Gk, dim, vdim)
    portions = [(2, 0, 300), (0, 0, 1), (5, 117, 70), (3, 200, 140), (6, 600, 5)]
    step = PackedStep([(r, s, [0] * n) for r, s, n in portions], dev)
    lay = step.layout(reach - 1, keep)
    inp = rnd(step.T, L.width_in, seed=8)
    qs = O.rms_norm(inp[:, :H * dim].double().view(-1, H, dim), 0.0).bfloat16()
    inp[:, :H * dim] = qs.flatten(1)
    full = {r: rnd(s + n, L.ld_kv, seed=10 + r) for r, s, n in portions}       # keys and values of whole sequences
    for kv in full.values():
        k = O.rms_norm(kv[:, :Gk * dim].double().view(-1, Gk, dim), 0.0)
        needles = [i for i in (0, 1, 2, 3, 19, 20, 63, 64, 127, 128, 149, 150, 199, 255, 256, 299) if i < len(kv)]
        k[needles] = O.rms_norm(k[needles] + 0.7, 0.0)
        kv[:, :Gk * dim] = k.flatten(1).bfloat16()
    inp[:, :H * dim] = O.rms_norm((inp[:, :H * dim].double() + 0.4).view(-1, H, dim), 0.0).flatten(1).bfloat16()   # queries lean towards them
    stream = torch.empty(lay.total, L.ld_kv, dtype=torch.bfloat16)
    at = 0
    for r, s, n in portions:
        held = sorted({p for p in range(s) if p < keep or p >= s - reach + 1})
        stream[at:at + len(held)] = full[r][held]
        stream[at + len(held):at + len(held) + n] = full[r][s:s + n]
        at += len(held) + n
    assert at == lay.total
    got = G.stream_attention(L, a, inp.to(dtype).to(dev), stream.to(dtype).to(dev), lay, None)
    for t0, n, r, s in step.sequences():
        kv = full[r].double()
        k, v = kv[:, :Gk * dim].view(-1, Gk, dim), kv[:, L.kv_v:L.kv_v + Gk * vdim].view(-1, Gk, vdim)
        some = sorted({0, 1, 2, 3, 16, 17, 19, 20, 63, 64, 127, 128, 129, 130, 148, 149, 150, 200, 256, 299, n - 1} & set(range(n)))
        want = torch.stack([attention_want(a, inp[t0 + i, :H * dim].double().view(H, dim), k, v, O.visible_keys(s + i, reach, keep)) for i in some])
        near(got[[t0 + i for i in some]], want.flatten(1), dtype, bf16=2e-2, what=(s, n))
        if dev == "cpu":
            break
    status_ok(run)


@pytest.mark.parametrize("size", SIZES, ids=by_name)
@pytest.mark.parametrize("reach,keep,sharp", [(70, 9, 1.0), (70, 0, 6.0), (1, 3, 1.0), (16, 40, 30.0), (500, 5, 2.0), (20, 400, 1.0)])
@pytest.mark.parametrize("splits", [1, 3, 8])
def test_decode_attention(run, size, reach, keep, sharp, splits):
    """One token per sequence at positions around every border, rings that have gone round several times, key splits that are empty."""
    dev, dtype = run
    if dev == "cpu" and (size not in SIZES[:1] + SIZES[5:6] or splits > 1):
        pytest.skip("two sizes on the CPU")
    if splits == 3 and size in SIZES[2:4]:
        pytest.skip("other sizes")
    H, Gk, dim, vdim = size
    a = spec_of(size, reach, keep, sharp)
    L, max_len = G.GroupedLayout(H, Gk, dim, vdim), 300
    ring = min(reach + keep, max_len)
    pos, row = [0, 1, 2, 3, 15, 16, 69, 70, 78, 79, 80, 199, 256, 299], [4, 0, 11, 2, 3, 8, 6, 7, 9, 1, 12, 13, 14, 15]
    B = len(pos)
    x, bias = rnd(B, L.width_in, seed=6), rnd(L.width_in, seed=7)
    old = rnd(17, max_len, L.ld_kv, seed=5)                                      # what the sequences' earlier positions hold
    cache = rnd(17, ring, L.ld_kv, seed=9)                                       # (and what former owners of the rows left)
    slot = lambda p: p if p < ring else keep + (p - keep) % (ring - keep)  # noqa: E731
    for p_, r in zip(pos, row):
        for p in list(range(min(keep, p_))) + list(range(max(0, p_ - reach + 1), p_)):
            cache[r, slot(p)] = old[r, p]
    ip, ir = (torch.tensor(t, dtype=torch.int32, device=dev) for t in (pos, row))
    tr, fq, fk, fv = transform(a, run, bias.float().to(dev))
    full = x.double() + bias.double()
    for src in ([x.float().to(dev)] if dev == "cuda" and dtype == torch.bfloat16 else []) + [x.to(dtype).to(dev)]:
        c = cache.to(dtype).to(dev)
        got = G.ring_attention(L, a, src, tr, c, None, None, ip, ir, splits, dtype)
        for b, (p, r) in enumerate(zip(pos, row)):
            new = torch.zeros(1, L.ld_kv, dtype=D)
            new[0, :Gk * dim] = fk(full[b, L.off_k:L.off_k + Gk * dim], p).flatten()
            new[0, L.kv_v:L.kv_v + L.v_width] = fv(full[b, L.off_v:L.off_v + L.v_width]).flatten()
            kv = torch.cat([old[r, :p].double(), new.to(dtype).double()])
            k, v = kv[:, :Gk * dim].view(-1, Gk, dim), kv[:, L.kv_v:L.kv_v + Gk * vdim].view(-1, Gk, vdim)
            want = attention_want(a, fq(full[b, :H * dim], p), k, v, O.visible_keys(p, reach, keep))
            near(got[b], want.flatten(), dtype, bf16=2.5e-2 * max(1.0, sharp / 10), what=p)     # rounding of q and k grows with the scores
            for at, m in ((0, Gk * dim), (L.kv_v, L.v_width)):
                near(c[r, slot(p), at:at + m], new[0, at:at + m], dtype)
        idle = [5, 10, 16]
        assert torch.equal(c[idle].float().cpu(), cache[idle].float())           # rows of other sequences
    status_ok(run)


# ------------------------------------------------------------------------------------------
# delta memories
# ------------------------------------------------------------------------------------------
@pytest.mark.parametrize("taps", [1, 2, 3, 4, 7])
@pytest.mark.parametrize("size", [(2, 1, 8, 16), (3, 3, 13, 11), (4, 2, 64, 128)], ids=by_name)
def test_short_convolution(run, taps, size):
    """Fresh and continued portions around the taps' and the kernel's borders; what a later portion or decode step needs is kept."""
    dev, dtype = run
    L = DL.DeltaLayout(*size)
    ch = L.channels
    w = rnd(taps, ch, seed=taps).float()
    lengths = {0: 300, 1: 40, 2: 140, 4: 131}
    full = {r: rnd(n, L.off_ba, seed=r) for r, n in lengths.items()}
    want = {r: O.silu(O.short_conv(x[:, :ch].double(), w.T.double())) for r, x in full.items()}
    ring = rnd(5, taps, ch, seed=50).to(dtype).to(dev)               # left by former owners
    cuts = {0: (129, 1, 2, 168), 1: (1, 1, 3, 35), 2: (2, 127, 1, 10), 4: (128, 1, 1, 1)}
    at = dict.fromkeys(lengths, 0)
    for k in range(4):
        portions = [(r, at[r], cuts[r][k]) for r in lengths]
        step = PackedStep([(r, s, [0] * n) for r, s, n in portions], dev)
        x = torch.cat([full[r][s:s + n] for r, s, n in portions]).to(dtype).to(dev)
        got = DL.short_conv(L, x, w.to(dev), ring, step)
        t = 0
        for r, s, n in portions:
            near(got[t:t + n], want[r][s:s + n], dtype, what=(r, s))
            at[r], t = s + n, t + n


def delta_case(size, T, seed=0, kind="random"):
    """Activated rows, gate rows, step size and decay projections of one sequence and what the recurrence makes of them."""
    H, Gk, dim, vdim = size
    L = DL.DeltaLayout(*size)
    act, z = rnd(T, L.channels, seed=seed), rnd(T, L.off_ba, seed=seed + 1)
    ba = torch.randn(T, 2 * H, generator=torch.Generator().manual_seed(seed + 2)) * 2
    a_log, dt = torch.linspace(-4, 1, H), torch.linspace(-1, 1, H)
    if kind == "same keys":                                          # one direction is written over and over
        act[:, L.off_k:L.off_k + Gk * dim] = act[:1, L.off_k:L.off_k + Gk * dim]
        ba[:, :H] = 6.0
        a_log = torch.full((H,), -9.0)
    elif kind == "two keys":
        act[:, L.off_k:L.off_k + Gk * dim] = act[torch.arange(T) % 2, L.off_k:L.off_k + Gk * dim]
        ba[:, :H] = 4.0
    elif kind == "forgets":
        a_log = torch.full((H,), 3.0)
    elif kind == "keeps":
        a_log, ba[:, :H] = torch.full((H,), -12.0), -1.0
    w = DL.DeltaWeights(torch.zeros(4, L.channels), a_log, dt, 1 + 0.3 * torch.randn(vdim, generator=torch.Generator().manual_seed(9)), 1e-5)
    x = act.double()
    q = O.unit(x[:, L.off_q:L.off_q + Gk * dim].view(T, Gk, dim)) * dim ** -0.5
    k = O.unit(x[:, L.off_k:L.off_k + Gk * dim].view(T, Gk, dim))
    v = x[:, L.off_v:L.off_v + H * vdim].view(T, H, vdim)
    beta, log_g = O.sigmoid(ba[:, :H].double()), O.log_decay(ba[:, H:].double(), a_log.double(), dt.double())
    o = torch.stack([O.delta_scan(q[:, h // (H // Gk)], k[:, h // (H // Gk)], v[:, h], beta[:, h], log_g[:, h]) for h in range(H)], dim=1)
    want = O.head_norm_gate(o, w.norm.double(), z[:, L.off_g:L.off_g + H * vdim].double().view(T, H, vdim), 1e-5).flatten(1)
    return L, w, act, z, ba, want, o


def on(w, dev):
    return DL.DeltaWeights(*(t.to(dev) for t in (w.conv, w.a_log, w.dt_bias, w.norm)), w.eps)


DELTAS = [(2, 1, 64, 64), (4, 2, 128, 128), (3, 3, 32, 96), (2, 1, 40, 24), (6, 2, 13, 11), (1, 1, 200, 40), (2, 2, 96, 256), (1, 1, 8, 8)]


@pytest.mark.parametrize("size", DELTAS, ids=by_name)
@pytest.mark.parametrize("kind", ["random", "same keys", "two keys", "forgets", "keeps"])
def test_delta_rule_over_prompts(run, size, kind):
    """Whole sequences and the same in portions around the chunks' borders; the state is carried on, and a row's former state is not seen."""
    dev, dtype = run
    if dev == "cpu" and size not in DELTAS[3:5]:
        pytest.skip("two sizes on the CPU")
    T = 300 if size[0] > 2 else 400
    L, w, act, z, ba, want, o = delta_case(size, T, seed=3, kind=kind)
    w = on(w, dev)
    state = torch.randn(3, L.heads, L.dim, L.ldv, generator=torch.Generator().manual_seed(0)).to(dev)
    # read-outs of nearly nothing are divided by their own size: rounding shows there, and nowhere else
    tiny = o.square().mean(-1).sqrt() < 0.02 * o.square().mean().sqrt()
    for cuts in ([T], [127, 1, 2, T], [1, 128, 129, T], [2, 2, 64, 70, T]):
        outs, at = [], 0
        for c in cuts:
            n = min(c, T - at)
            if n <= 0:
                break
            e = slice(at, at + n)
            other = 1 + at % 7                                       # another sequence beside it
            step = PackedStep([(2, at, [0] * n), (0, 0, [0] * other)], dev)
            cat = lambda t: torch.cat([t[e], t[:other]])  # noqa: E731
            got = DL.delta_prompt(L, w, cat(act).to(dtype).to(dev), cat(z).to(dtype).to(dev), cat(ba).to(dev), state, step)
            outs.append(got[:n].cpu())
            assert dev == "cpu" or bool(torch.isfinite(got).all())
            near(got[n:], want[:other], dtype, bf16=2e-2)
            at += n
        got = torch.cat(outs).double().view(T, L.heads, L.vdim)
        d = (got - want.view(T, L.heads, L.vdim))[~tiny]
        err = float(d.square().mean().sqrt() / want.square().mean().sqrt())
        # alike keys: what is written cancels in the read-out, the rounding of what is written does not
        assert err < (2e-5 if dtype == torch.float32 else 3e-2 if "keys" in kind else 1.2e-2), (cuts, err)
    status_ok(run)


@pytest.mark.parametrize("size", DELTAS, ids=by_name)
@pytest.mark.parametrize("taps", [1, 4])
def test_delta_rule_decoding(run, size, taps):
    """Projection rows of single tokens: convolution from the ring, unit norms, gates, update, head norm and output gate; after a prompt
    portion and from the first token on, several sequences at different positions."""
    dev, dtype = run
    H, Gk, dim, vdim = size
    L = DL.DeltaLayout(*size)
    T, ch, hv = 24, L.channels, H * vdim
    conv, a_log, dt = rnd(taps, ch, seed=1).float(), torch.linspace(-3, 0, H), torch.linspace(-1, 1, H)
    w = DL.DeltaWeights(conv, a_log, dt, 1 + 0.2 * torch.randn(vdim, generator=torch.Generator().manual_seed(4)), 1e-5)
    lags = {1: 0, 3: 5, 0: 17}                                       # row -> tokens that a prompt portion takes
    full = {r: rnd(T, L.width_in, seed=20 + r) for r in lags}
    want = {}
    for r, x in full.items():
        x = x.double()
        act = O.silu(O.short_conv(x[:, :ch], conv.T.double()))
        q = O.unit(act[:, L.off_q:L.off_q + Gk * dim].view(T, Gk, dim)) * dim ** -0.5
        k = O.unit(act[:, L.off_k:L.off_k + Gk * dim].view(T, Gk, dim))
        v = act[:, L.off_v:L.off_v + hv].view(T, H, vdim)
        beta = O.sigmoid(x[:, L.off_ba:L.off_ba + H])
        log_g = O.log_decay(x[:, L.off_ba + H:L.off_ba + 2 * H], a_log.double(), dt.double())
        o = torch.stack([O.delta_scan(q[:, h // (H // Gk)], k[:, h // (H // Gk)], v[:, h], beta[:, h], log_g[:, h]) for h in range(H)], dim=1)
        want[r] = O.head_norm_gate(o, w.norm.double(), x[:, L.off_g:L.off_g + hv].view(T, H, vdim), 1e-5).flatten(1)
    w = on(w, dev)
    for raw in ([torch.float32] if dev == "cuda" else []) + [dtype]:
        ring = rnd(4, taps, ch, seed=30).to(dtype).to(dev)
        state = torch.randn(4, H, dim, L.ldv, generator=torch.Generator().manual_seed(0)).to(dev)
        for r, n in lags.items():
            if n:
                step = PackedStep([(r, 0, [0] * n)], dev)
                x = full[r][:n].to(dtype).to(dev)
                act = DL.short_conv(L, x, w.conv, ring, step)
                got = DL.delta_prompt(L, w, act, x, x[:, L.off_ba:L.off_ba + 2 * H].float(), state, step)
                near(got, want[r][:n], dtype, bf16=3e-2)
        for k in range(7):
            rows, pos = list(lags), [n + k for n in lags.values()]
            x = torch.stack([full[r][p] for r, p in zip(rows, pos)]).to(raw).to(dev)
            ip, ir = (torch.tensor(t, dtype=torch.int32, device=dev) for t in (pos, rows))
            got = DL.delta_decode(L, w, x, ring, state, ip, ir, dtype)
            near(got, torch.stack([want[r][p] for r, p in zip(rows, pos)]), dtype, bf16=3e-2, what=k)
    status_ok(run)


# ------------------------------------------------------------------------------------------
# mixtures
# ------------------------------------------------------------------------------------------
MOES = [(GroupedMixtureSpec(24, 6, 0, 2, None, 3, 2), 48), (GroupedMixtureSpec(19, 9, 0, 2, None, 3, 1), 45), (GroupedMixtureSpec(8, 1, 0, 1, None, 1, 1), 16),
        (GroupedMixtureSpec(136, 8, 0, 4, None, 4, 2), 264), (GroupedMixtureSpec(64, 40, 0, 8, None, 5, 2), 520), (GroupedMixtureSpec(300, 4, 0, 2, None, 4, 3), 136),
        (GroupedMixtureSpec(33, 72, 0, 30, None, 36, 20), 72), (GroupedMixtureSpec(16, 6, 0, 6, None, 1, 1), 24)]


def moe_weights(s, E, run, seed=0):
    """Weights of a mixture as named tensors and as the product holds them."""
    dev, dtype = run
    cfg = O.config([O.attn()], [O.moe(s.experts, s.top, s.ff, s.group_count, s.group_keep)], width=E, groups=1)
    w = {k[7:]: v for k, v in O.random_weights(cfg, seed).items() if k.startswith("l0.mlp.")}
    p = lambda t: torch.nn.functional.pad(t, (0, ops.pad8(t.shape[1]) - t.shape[1])).to(dtype).to(dev)[:, :t.shape[1]]  # noqa: E731
    up = torch.cat([w[f"e{e}.{part}"] for e in range(s.experts) for part in ("gate", "up")])
    return w, cfg["layers"][0]["mlp"], X.MoeWeights(s, p(w["router"]), None, p(up), p(torch.cat([w[f"e{e}.down"] for e in range(s.experts)])), None, None)


@pytest.mark.parametrize("case", range(len(MOES)))
@pytest.mark.parametrize("T", [1, 2, 7, 16, 33, 64, 300, 1100])
def test_mixture_of_gated_experts(run, case, T):
    """Both forms (any rows, the few rows of a decode step) against the tokens one by one."""
    dev, dtype = run
    s, E = MOES[case]
    if T > 64 and (dev == "cpu" or case == 6):
        pytest.skip("many rows: on a GPU")
    named, m, w = moe_weights(s, E, run, seed=case)
    h = rnd(T, E, seed=T)
    some = sorted({0, T // 3, T - 1} | set(range(0, T, max(1, T // 12))))
    want = O.mixture(h[some].double(), {k: v.double() for k, v in named.items()}, "", m)
    x = torch.nn.functional.pad(h, (0, ops.pad8(E) - E)).to(dtype).to(dev)[:, :E]
    for f in [X.mixture] + ([X.mixture_rows] if T <= 64 else []):
        out = f(w, x)
        out = out.sum() if isinstance(out, M.RowSum) else out
        near(out[some], want, dtype, bf16=1.5e-2)
    status_ok(run)


@pytest.mark.parametrize("experts,top,count,keep", [(6, 2, 3, 1), (10, 3, 2, 1), (12, 4, 4, 2), (40, 8, 5, 2), (64, 6, 64, 6), (72, 9, 36, 5), (128, 8, 8, 4), (5, 5, 1, 1)])
def test_choice_within_the_best_groups(run, experts, top, count, keep):
    """Choices and weights of the router alone; the best expert of all may lie in a group that is not among the best."""
    dev, dtype = run
    s = GroupedMixtureSpec(8, experts, 0, top, None, count, keep)
    z = torch.randn(70, experts, generator=torch.Generator().manual_seed(experts)) * 1.5
    z[0, 0] = 6.0                                                    # alone in its group
    if count > 1 and experts > count:
        z[0, 1:experts // count] = -9.0
    chosen = [O.route(r.double(), top, {"count": count, "keep": keep}) for r in z]
    if dev == "cpu":
        from recurrent_pretraining_b200.ops import reference as ref

        idx, weight = ref.route_grouped(z, top, count, keep)
    else:
        w = X.MoeWeights(s, None, None, None, None, None, None)
        p = X.plan(w, z.to(dev), 128)
        idx, weight = p.idx.cpu(), p.weight[:, :top].cpu()
    for t, (e, v) in enumerate(chosen):
        assert idx[t].tolist() == e
        near(weight[t], v, torch.float32)


# ------------------------------------------------------------------------------------------
# models
# ------------------------------------------------------------------------------------------
@pytest.mark.parametrize("name", list(CONFIGS))
def test_prompt_matches_oracle(run, name):
    cfg = steady(CONFIGS[name], run)
    model, w = make(cfg, run, seed=3 if name == "one" else 1)
    seq = tokens(80 if name != "wide" else 60, cfg["vocab"])
    hidden, got_hidden = [], []
    want = O.forward(cfg, w, seq, hidden)
    got = model.forward_step(PackedStep([(0, 0, seq)], run[0]), None, None, got_hidden)
    assert len(hidden) == len(got_hidden)
    for i, (a, b) in enumerate(zip(got_hidden, hidden)):
        agree(a, b, run, f"layer {i}")
    agree(got, want, run)
    status_ok(run)


@pytest.mark.parametrize("name", list(CONFIGS))
@pytest.mark.parametrize("cuts", [[1], [2], [3, 1, 7], [40, 1], [13, 2, 1, 1, 30], [64, 5]], ids=str)
def test_portions_and_decoding_match_the_whole_prompt(run, name, cuts):
    cfg = steady(CONFIGS[name], run)
    if run[0] == "cpu" and name == "wide" and cuts != [13, 2, 1, 1, 30]:
        pytest.skip("one on the CPU")
    model, w = make(cfg, run, seed=2)
    seq = tokens(75, cfg["vocab"])
    want = O.forward(cfg, w, seq)
    eng = engine(model)
    agree(feed(eng, eng.open(), seq, cuts), want, run)
    status_ok(run)


@pytest.mark.parametrize("size,keep", [(20, 6), (128, 3), (131, 0), (9, 130)])
def test_edges_of_windows_and_kept_positions(run, size, keep):
    """One token's key stands out.  In a window: the last position that sees it and the next one, which does not; among the first: the last
    kept position is seen for good, the one behind it like any other.  In prompts, in portions that end there, and decoded alone."""
    cfg = O.config([O.attn(heads=2, kv_heads=1, dim=16, vdim=16, size=size, keep=keep, rot=2, base=1e9, scaling=None, scale=1.0)], [None], groups=1)
    w = {k: v.float() for k, v in O.random_weights(cfg, 5).items()}
    u = torch.randn(16, generator=torch.Generator().manual_seed(1)).sign()
    u[:2] = 0                                                  # not turned by the rotation
    for part in "qkv":
        w[f"l0.mix.{part}.b"].zero_()
    w["embed"][:, :2] = torch.tensor([2.0, 0.0])
    w["embed"][5, 1] = 9.0
    w["l0.mix.q"] *= 0.1
    w["l0.mix.k"] *= 0.3
    w["l0.mix.q"][:, 0] += 2 * u.repeat(2)                     # every query leans towards the key of token 5
    w["l0.mix.k"][:, 1] += 2 * u
    w = {k: v.bfloat16() for k, v in w.items()}
    model = load(cfg, w, run)
    eng = engine(model, max_len=500)
    n = keep + 2 * size + 40
    plain = [t for t in tokens(3 * n) if t != 5][:n]
    for at in [keep + size + 3, keep] + ([keep - 1] if keep else []):
        seq = plain[:at] + [5] + plain[at + 1:]
        last = at + size - 1
        want, other = O.forward(cfg, w, seq), O.forward(cfg, w, plain)
        gone = (want - other).square().mean(-1).sqrt() / want.square().mean().sqrt()
        assert float(gone[last]) > 0.1 and (float(gone[last + 1]) < 1e-9 if at >= keep else float(gone[-1]) > 0.1), gone[last:last + 2]
        for cuts in ([n], [last, 1], [last + 1, 1], [at, 2, last - at - 1, 1], [size + 1, 1]):
            row = eng.open()
            agree(feed(eng, row, seq, [max(1, c) for c in cuts]), want, run, (at, cuts))
            eng.close(row)
    status_ok(run)


def test_every_part_shows(run):
    """Leaving out or changing any part of the design changes the logits far beyond the tolerance: the agreement of the other tests covers
    them."""
    cfg = O.config([O.memory(), O.attn(size=9), O.memory(heads=2, kv_heads=2)], [O.moe(), O.mlp()])
    cfg = steady(cfg, run)
    model, w = make(cfg, run, seed=3)
    seq = tokens(60)
    want = O.forward(cfg, w, seq)
    agree(model(torch.tensor([seq]))[0], want, run)
    if run[0] != "cpu":
        return
    changes = []
    for part, value in (("q.b", 0.0), ("k.b", 0.0), ("v.b", 0.0), ("A_log", -9.0), ("dt_bias", 2.0), (".mix.norm", 1.0), (".norm1", 1.0), ("dwa", 0.5), (".mix.b", 0.0), (".mix.a", 0.0)):
        changes.append(O.forward(cfg, {k: (torch.full_like(v, value) if k.endswith(part) else v) for k, v in w.items()}, seq))
    front = {k: torch.cat([torch.zeros_like(v[:, :1]), v[:, 1:]], 1) if k.endswith(".conv") else v for k, v in w.items()}
    changes.append(O.forward(cfg, front, seq))
    for change in (lambda c: _mix(c, 1)["mask"].update(keep_first=0), lambda c: _mix(c, 1)["mask"].update(size=8), lambda c: _mix(c, 1).update(scale=0.1),
                   lambda c: _mix(c, 1)["rot"].update(scaling=None), lambda c: c["norm"].update(groups=1), lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(keep=3)):
        c = json.loads(json.dumps(cfg))
        change(c)
        changes.append(O.forward(c, w, seq))
    for i, other in enumerate(changes):
        assert O.rel_error(other, want) > 0.01, i


def test_far_tokens_come_through_memories_and_kept_positions(run):
    """Tokens far beyond the window reach later positions, whatever the cuts."""
    cfg = O.config([O.attn(size=12, keep=4), O.memory()], [O.mlp()])
    w = O.random_weights(cfg, 6)
    w["l1.mix.A_log"] = torch.full((4,), -6.0).bfloat16()            # memories that last
    model = load(cfg, w, run)
    seq = tokens(230)
    want = O.forward(cfg, w, seq)
    assert O.rel_error(O.forward(cfg, w, tokens(20, seed=9) + seq[20:])[150:], want[150:]) > 0.02
    eng = engine(model)
    for cuts in ([230], [200, 1], [7, 2, 128, 1], [2]):
        agree(feed(eng, eng.open(), seq, cuts), want, run, cuts)


def test_long_decoding(run):
    """Rings that go round many times; the cache is full at the end."""
    cfg = O.config([O.attn(size=17, keep=5), O.memory(), O.attn(size=25, keep=0)], [O.moe(), O.mlp()])
    cfg = steady(cfg, run)
    model, w = make(cfg, run, seed=8)
    seq = tokens(260)
    want = O.forward(cfg, w, seq)
    eng = engine(model, 1, 260)
    assert eng.cache.data[0, "kv"].shape[1] == 22 and eng.cache.data[2, "kv"].shape[1] == 25       # a sequence holds a bounded amount
    agree(feed(eng, eng.open(), seq, [4, 1]), want, run)
    with pytest.raises(ValueError):
        eng.step([(0, [1])])


def test_first_tokens(run):
    cfg = steady(MIXED, run)
    model, w = make(cfg, run, seed=9)
    eng = engine(model)
    for t in (0, 66):
        agree(eng.step([(eng.open(), [t])]), O.forward(cfg, w, [t]), run)
    seq = tokens(6)
    want = O.forward(cfg, w, seq)
    for n in range(1, 6):
        row = eng.open()
        got = torch.cat([eng.step([(row, seq[:n])], [list(range(n))]), eng.step([(row, seq[n:])], [list(range(6 - n))])])
        agree(got, want, run)


def test_unequal_batches_match_each_alone(run):
    cfg = steady(MIXED, run)
    model, w = make(cfg, run, seed=10)
    seqs = [tokens(n, seed=n) for n in (1, 33, 130, 5, 64)]
    more = [tokens(7, seed=100 + n) for n in range(5)]
    wants = [O.forward(cfg, w, s + m) for s, m in zip(seqs, more)]
    eng = engine(model, rows=2)                                    # grows on demand
    rows = [eng.open() for _ in seqs]
    got = [[x] for x in eng.step(list(zip(rows, seqs)), [[len(s) - 1] for s in seqs]).split(1)]
    alive = list(range(5))
    for k in range(7):
        if k == 3:                                                 # the batch shrinks while it decodes
            eng.close(rows[1])
            alive.remove(1)
        lg = eng.step([(rows[i], [more[i][k]]) for i in alive])
        for i, x in zip(alive, lg.split(1)):
            got[i].append(x)
    for i, (s, want) in enumerate(zip(seqs, wants)):
        g = torch.cat(got[i])
        agree(g, want[len(s) - 1:len(s) - 1 + len(g)], run, i)
    # mixed steps: portions of different sizes and single tokens in one batch
    eng = engine(model, rows=5)
    rows = [eng.open() for _ in seqs]
    eng.step(list(zip(rows, seqs)), [[] for _ in seqs])
    sizes = (1, 4, 2, 7, 1)
    lg = eng.step([(r, m[:n]) for r, m, n in zip(rows, more, sizes)])
    agree(lg, torch.stack([wants[i][len(seqs[i]) + n - 1] for i, n in enumerate(sizes)]), run)
    status_ok(run)


def test_rows_are_freed_and_used_again(run):
    """A row's keys, convolution inputs and states of its former sequence are not seen by the next one, which may be shorter or a single token."""
    cfg = steady(MIXED, run)
    model, w = make(cfg, run, seed=11)
    eng = engine(model, rows=2)
    for k in range(4):
        a, b = eng.open(), eng.open()
        assert {a, b} == {0, 1} and eng.cache.rows == 2
        for row, n in ((a, 70 - 22 * k), (b, 1 + 20 * k)):
            seq = tokens(n + 4, seed=k)
            agree(feed(eng, row, seq, [n, 1]), O.forward(cfg, w, seq), run)
        eng.close(b)
        eng.close(a)


def test_greedy_generation_through_the_scheduler(run):
    from recurrent_pretraining_b200.engine import server as S

    cfg = O.config([O.memory(), O.attn()], [O.moe(), O.mlp()])
    cfg = steady(cfg, run)
    model, w = make(cfg, run, seed=12)
    prompts = [tokens(n, seed=n) for n in (3, 12, 1, 7)]
    sched = S.BatchScheduler(S.make_backend(model, max_batch=4, max_len=64), window_ms=200.0, stop_ids=())
    try:
        reqs = [sched.submit(p, S.DecodeOptions(max_tokens=10)) for p in prompts]
        for p, r in zip(prompts, reqs):
            assert r.done.wait(120) and r.error is None, r.error
            seq, off = list(p), 0
            for t in r.tokens:                                     # every choice is (nearly) the oracle's best
                lg = O.forward(cfg, w, seq)[-1]
                off += float(lg[t]) < float(lg.max()) - (1e-4 if run[1] == torch.float32 else 0.25 * float(lg.std()))
                seq.append(t)
            assert off <= (0 if run[1] == torch.float32 else 1)
        assert sched.stats["batches"] < 4                          # unequal prompts share a batch
        out = S.handle_completion(sched, {"prompt": prompts[1], "max_tokens": 10, "do_sample": True, "top_k": 1})
        assert out["choices"][0]["token_ids"] == reqs[1].tokens or run[1] == torch.bfloat16
    finally:
        sched.close()


def test_generation_stops_and_prefills_in_portions(run):
    cfg = steady(MIXED, run)
    model, w = make(cfg, run, seed=13)
    eng = engine(model)
    prompts = [tokens(9), tokens(4)]
    plain = eng.generate(prompts, 20)
    stop = plain[0][5]
    cut = eng.generate(prompts, 20, stop_ids=[stop], check_every=2)
    for p, c in zip(plain, cut):
        end = p.index(stop) + 1 if stop in p else len(p)
        assert c == p[:end]
    small = engine(model, prefill_tokens=5)                        # prompts in portions, several sequences per step
    assert small.generate(prompts, 6) == [p[:6] for p in plain] or run[1] == torch.bfloat16
    assert not eng.cache.length                                    # every row went back


@gpu
@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_trace_command(tmp_path, dtype):
    import subprocess

    import numpy as np
    from recurrent_pretraining_b200.models.weights import save_safetensors

    w = O.random_weights(ODD, 21)
    folder, out = tmp_path / "model", tmp_path / "out"
    os.makedirs(folder)
    with open(folder / "config.json", "w") as f:
        json.dump(ODD, f)
    save_safetensors(str(folder / "model.safetensors"), w)
    a, b = tokens(30, 61, seed=3), tokens(12, 61, seed=4)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": a[:29], "want": [0, 28]}, {"id": "y", "tokens": b[:11], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": a[29:], "want": [0]}, {"id": "y", "tokens": b[11:], "want": [0]}], "end": ["x", "y"]}]
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    r = subprocess.run([os.path.join(root, "bin", "trace_run"), "--model", str(folder), "--dtype", dtype, "--out", str(out),
                        "--max-tokens", "64"], input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    wa, wb = O.forward(ODD, w, a), O.forward(ODD, w, b)
    got = torch.cat([torch.from_numpy(np.fromfile(out / f"{n}.f32", dtype="<f4")).view(2, -1) for n in (0, 1)])
    agree(got, torch.stack([wa[0], wa[28], wa[29], wb[11]]), ("cuda", getattr(torch, dtype)))


def test_trace_replay(run, tmp_path):
    import numpy as np
    from recurrent_pretraining_b200.engine.trace import replay

    cfg = steady(MIXED, run)
    model, w = make(cfg, run, seed=14)
    a, b = tokens(20, seed=1), tokens(9, seed=8)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:18], "want": [0, 17]}, {"id": "b", "tokens": b[:8], "want": [7]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[18:19], "want": []}, {"id": "b", "tokens": b[8:], "want": []}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": a[19:], "want": [0]}], "end": ["a"]}]
    answer = io.StringIO()
    eng = engine(model, 1, 64)
    replay(eng, [json.dumps(s) + "\n" for s in steps], str(tmp_path), answer)
    assert answer.getvalue() == "done 0\ndone 1\ndone 2\n" and not eng.cache.length
    wa, wb = O.forward(cfg, w, a), O.forward(cfg, w, b)
    agree(torch.from_numpy(np.fromfile(tmp_path / "0.f32", dtype="<f4")).view(3, -1), torch.stack([wa[0], wa[17], wb[7]]), run)
    agree(torch.from_numpy(np.fromfile(tmp_path / "2.f32", dtype="<f4")).view(1, -1), wa[19:], run)


def test_serve_command_completes_a_prompt(tmp_path, capsys):
    import serve

    cfg = O.config([O.memory(), O.attn()], [O.moe()])
    model, w = make(cfg, ("cpu", torch.float32), seed=22)
    model.save_pretrained(str(tmp_path))
    prompt = tokens(5)
    serve.main(["--model", str(tmp_path), "--cpu", "--prompt-ids", ",".join(map(str, prompt)), "--max-tokens", "6", "--max-len", "64"])
    out = json.loads(capsys.readouterr().out.strip().splitlines()[-1])
    assert out["choices"][0]["token_ids"] == O.greedy(cfg, w, prompt, 6)


@gpu
@pytest.mark.parametrize("graphs", [False, True])
def test_decode_steps_on_a_cache_that_grows(graphs):
    """A graph is not replayed on the storage of a cache that has grown; accumulators are handed back cleared."""
    run = ("cuda", torch.bfloat16)
    cfg = O.config([O.memory(heads=8, kv_heads=4, dim=32, vdim=64), O.attn(heads=8, kv_heads=2, dim=32, vdim=64, size=25, keep=4)],
                   [O.mlp(1024), O.moe(10, 4, 128, 2, 1)], width=656, groups=2)
    cfg = steady(cfg, run)
    model, w = make(cfg, run, seed=15)
    eng = engine(model, rows=1, use_graphs=graphs)
    seq = tokens(60)
    want = O.forward(cfg, w, seq)
    first = eng.open()
    a = feed(eng, first, seq[:30], [3, 1])
    other = eng.open()                                             # the cache is reallocated
    assert eng.cache.rows == 2
    feed(eng, other, tokens(30, seed=5), [5, 1])
    b = feed(eng, first, seq[30:], [1])
    agree(torch.cat([a, b]), want, run)
    torch.cuda.synchronize()
    assert not any(bool(t.any()) for t in eng._work)
    status_ok(run)


@gpu
@pytest.mark.parametrize("name", ["mixed", "wide"])
def test_large_batches_decode_in_groups(name):
    run = ("cuda", torch.bfloat16)
    cfg = steady(CONFIGS[name], run)
    model, w = make(cfg, run, seed=16)
    eng = engine(model, rows=70)
    seqs = [tokens(3 + i % 9, seed=i) for i in range(70)]
    rows = [eng.open() for _ in seqs]
    eng.step([(r, s[:-1]) for r, s in zip(rows, seqs)], [[] for _ in seqs])
    lg = eng.step([(r, s[-1:]) for r, s in zip(rows, seqs)])
    agree(lg[::9], torch.stack([O.forward(cfg, w, seqs[i])[-1] for i in range(0, 70, 9)]), run)


@gpu
def test_many_prompt_tokens_against_fp32(run=("cuda", torch.bfloat16)):
    """A long packed step (whole tiles of the tensor-core kernels, both tile heights of the grouped products) against the same in fp32,
    whose kernels share nothing with it but the layouts."""
    cfg = O.config([O.memory(heads=4, kv_heads=2, dim=64, vdim=64), O.attn(heads=8, kv_heads=2, dim=64, vdim=64, size=333, keep=40, rot=32), O.memory(heads=2, kv_heads=1, dim=128, vdim=128)],
                   [O.moe(6, 3, 96, 2, 1), O.mlp(200)], width=256, groups=2)
    w = O.random_weights(cfg, 18, router=6.0)
    seqs = [tokens(n, seed=n) for n in (1500, 900, 3, 257)]
    cfg, outs = steady(cfg, run), []
    for dtype in (torch.bfloat16, torch.float32):
        eng = engine(load(cfg, w, ("cuda", dtype)), max_len=1600)
        rows = [eng.open() for _ in seqs]
        a = eng.step([(r, s) for r, s in zip(rows, seqs)], [list(range(0, len(s), 7)) for s in seqs])
        b = eng.step([(r, [1, 2, 3, 4]) for r in rows], [[3] for _ in rows])
        outs.append(torch.cat([a, b]).double().cpu())
    agree(outs[0], outs[1], run)
    status_ok(run)
