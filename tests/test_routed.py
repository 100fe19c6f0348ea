"""Layered decoder models with chunked and windowed capped attention and mixtures of experts (design ``Dusilorn``): every mechanism
and the serving path against the plain statements of ``routed_oracle``, on the CPU (fp32) and on the GPU kernels (fp32, bf16)."""
import io
import json
import math
import os

import pytest
import torch

import routed_oracle as O
from recurrent_pretraining_b200.models import auto, build_model
from recurrent_pretraining_b200.models.layered import LayeredForCausalLM
from recurrent_pretraining_b200.models.layered_config import ChunkAttentionSpec, LayeredConfig, MixtureSpec, RotarySpec, WindowAttentionSpec
from recurrent_pretraining_b200.models.sublayers import PackedStep, rope_tables
from recurrent_pretraining_b200.ops import grouped as G
from recurrent_pretraining_b200.ops import latent as ops
from recurrent_pretraining_b200.ops import memory as M
from recurrent_pretraining_b200.ops import moe as X

gpu = pytest.mark.gpu
RUNS = [pytest.param(("cpu", torch.float32), id="cpu"), pytest.param(("cuda", torch.float32), marks=gpu, id="gpu-f32"),
        pytest.param(("cuda", torch.bfloat16), marks=gpu, id="gpu-bf16")]
GPU_RUNS = RUNS[1:]
D = torch.float64


@pytest.fixture(params=RUNS)
def run(request):
    return request.param


def load(cfg, w, run):
    model = LayeredForCausalLM(LayeredConfig.from_dict(cfg), run[1], run[0])
    model.load_checkpoint(O.TensorDict(w))
    return model


def make(cfg, run, seed=0, sharp=1.0):
    w = O.random_weights(cfg, seed, sharp)
    return load(cfg, w, run), w


def engine(model, rows=4, max_len=400, **kw):
    from recurrent_pretraining_b200.engine.layered import LayeredEngine

    return LayeredEngine(model, rows, max_len, **kw)


def tokens(n, vocab=67, seed=0):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(3000 + seed + 7919 * n)).tolist()


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


def agree(got, want, run, what="", bf16=6e-2):
    """Logits of every position.  In bf16 a router's nearly equal scores may fall either way: one position in ten may differ more."""
    d = got.double().cpu() - want
    d = d - d.mean(-1, keepdim=True)
    s = want - want.mean(-1, keepdim=True)
    err = (d.square().mean(-1) / s.square().mean()).sqrt().flatten()
    assert bool(torch.isfinite(err).all()), what
    if run[1] == torch.float32:
        assert float(err.max()) < 4e-5, (what, float(err.max()), int(err.argmax()))
    else:
        bad = int((err > bf16).sum())
        assert bad <= max(1, len(err) // 10), (what, bad, float(err.max()), int(err.argmax()))


def near(got, want, dtype, f32=2e-5, bf16=8e-3):
    """rms error over rms."""
    d = got.double().cpu() - want
    err = float(d.square().mean().sqrt() / want.square().mean().sqrt())
    ok = bool(torch.isfinite(d).all()) and err < (f32 if dtype == torch.float32 else bf16)
    assert ok, err


def rnd(*shape, seed=0, scale=1.0):
    """Values that bf16 represents exactly."""
    return (torch.randn(*shape, generator=torch.Generator().manual_seed(seed)) * scale).bfloat16()


def pitched(t, dtype, dev):
    """``t`` with a row pitch of a multiple of eight, the padding not a number."""
    out = torch.full((t.shape[0], ops.pad8(t.shape[1])), float("nan"), dtype=dtype, device=dev)
    out[:, :t.shape[1]] = t.to(dtype)
    return out[:, :t.shape[1]]


# layers that differ in every size, both kinds first and last, layers without feed-forward or value mixing, all choices of experts
MIXED = O.config([O.windowed(), O.chunked(heads=6, kv_heads=6, dim=24, vdim=8, size=14, softcap=3.0),
                  O.chunked(heads=5, kv_heads=1, dim=8, vdim=72, size=33, v_mix=False), O.windowed(heads=2, kv_heads=1, dim=32, vdim=48, size=27, rot=32, base=1e4)],
                 [O.moe(), O.mlp(), None, O.moe(experts=3, identity=5, top=2, ff=72, shared=None)])
# nothing is a multiple of eight
ODD = O.config([O.chunked(heads=3, kv_heads=3, dim=11, vdim=13, size=9, softcap=5.0), O.windowed(heads=6, kv_heads=3, dim=10, vdim=13, size=7, rot=6)],
               [O.moe(experts=5, identity=1, top=4, ff=19, shared=21), O.mlp(37)], width=45, vocab=61, eps=1e-3, scale=0.7, logit_scale=0.3)
# everything that can be one
ONE = O.config([O.chunked(heads=1, kv_heads=1, dim=8, vdim=8, size=1, scale=1.0, softcap=1.0), O.windowed(heads=1, kv_heads=1, dim=8, vdim=8, size=1, rot=2, v_mix=False)],
               [O.moe(experts=1, identity=0, top=1, ff=8, shared=8), O.moe(experts=1, identity=1, top=1, ff=1, shared=1)], width=16, vocab=19, scale=1.0, logit_scale=1.0)
# sizes of the tensor-core kernels, every expert chosen
WIDE = O.config([O.chunked(heads=20, kv_heads=1, dim=64, vdim=128, size=50, softcap=30.0), O.windowed(heads=4, kv_heads=2, dim=128, vdim=64, size=30, rot=64, softcap=50.0)],
                [O.moe(experts=6, identity=2, top=8, ff=136, shared=520), O.moe(experts=40, identity=0, top=8, ff=64, shared=None)], width=520)
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
    idle = sum((m["router"]["experts"] - min(m["router"]["top"], m["router"]["experts"])) * 2 * m["expert"]["ff"] * d["width"]
               for m in (layer["mlp"] for layer in d["layers"]) if m is not None and m["kind"] == "moe")
    assert cfg.active_param_count() <= cfg.param_count() and cfg.param_count() - cfg.active_param_count() <= idle


def test_weights_are_loaded_and_saved(tmp_path):
    from recurrent_pretraining_b200.models.weights import save_safetensors

    w = O.random_weights(MIXED, 3)
    w["l2.mix.vmix"] = torch.tensor(0.3)                             # a layer that does not mix may have the number all the same
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
    for change in (lambda t: t.pop("l0.mlp.e3.up"), lambda t: t.update({"l0.mix.sink": torch.zeros(4)}), lambda t: t.update({"l1.mix.sink": torch.zeros(5)})):
        bad = dict(w)
        change(bad)
        with pytest.raises(ValueError):
            model.load_checkpoint(O.TensorDict(bad))


def _mix(c, i=0):
    return c["layers"][i]["mixer"]


@pytest.mark.parametrize("change", [
    lambda c: c.update(architecture="Unknown"), lambda c: c.update(residual_mult=0.5), lambda c: c.update(loop=None) or c.update(loop={"start": 0}),
    lambda c: c["layers"][0].update(type="parallel"), lambda c: c["layers"][0].update(type="attention"), lambda c: _mix(c).update(kv_heads=3),
    lambda c: _mix(c).update(window=3), lambda c: _mix(c)["mask"].update(size=0), lambda c: _mix(c).update(softcap=0.0), lambda c: _mix(c).update(dim=-8),
    lambda c: _mix(c)["rot"].update(dims=18), lambda c: _mix(c)["rot"].update(dims=7), lambda c: _mix(c).update(vdim=16),
    lambda c: c["layers"][0]["mlp"].update(kind="sparse"), lambda c: c["layers"][0]["mlp"]["router"].update(top=9),
    lambda c: c["layers"][0]["mlp"]["router"].update(experts=0), lambda c: c["layers"][0]["mlp"]["expert"].update(act="silu"),
    lambda c: c["layers"][0]["mlp"]["shared"].update(ff=0), lambda c: c.pop("logit_scale"), lambda c: c["norm"].update(kind="layer")])
def test_invalid_configs_are_refused(change):
    cfg = json.loads(json.dumps(MIXED))
    change(cfg)
    with pytest.raises((ValueError, KeyError)):
        LayeredConfig.from_dict(cfg)


def test_registry_shapes_build():
    tiny = build_model(LayeredConfig.from_name("dusilorn-tiny"), dtype=torch.float32).init_weights(1)
    assert tiny(torch.tensor([[1, 2, 3], [4, 5, 6]])).shape == (2, 3, 512)
    for name in ("dusilorn-2b", "dusilorn-core-5280"):
        c = LayeredConfig.from_name(name)
        assert c.param_count() > 2e9 > c.active_param_count()


def test_which_layers_mix_values():
    cfg = LayeredConfig.from_dict(MIXED)
    assert [cfg.mixes_values(i) for i in range(4)] == ["first", "mix", None, "mix"]


# ------------------------------------------------------------------------------------------
# mechanisms alone
# ------------------------------------------------------------------------------------------
@pytest.mark.parametrize("E", [45, 48, 2056, 9000])
def test_centred_rms_norms_around_sublayers(run, E):
    dev, dtype = run
    g = torch.Generator().manual_seed(E)
    x, w1, w2 = torch.randn(5, E, generator=g) * 3 + 0.5, torch.randn(E, generator=g) * 0.5, torch.randn(E, generator=g) * 0.5
    a = rnd(5, E, seed=1) + 0.25
    put = lambda t: t.to(dev)  # noqa: E731
    acc = torch.zeros(5, ops.pad8(E), device=dev)[:, :E]
    want = x.double() + O.rms_norm(a.double(), 1e-4, 1 + w1.double())
    for src, clear in ((pitched(a, dtype, dev), False), (acc, dev == "cuda")):
        src.copy_(a)
        y, extra = x.to(dev).clone(), torch.ones(5, 12, device=dev)
        h = M.sandwich_norm_(y, src, (put(w1), None), None, (put(w2), None), 1e-4, dtype, clear=clear, zero=extra if dev == "cuda" else None, out_mult=0.3)
        near(y, want, torch.float32)
        near(h, 0.3 * O.rms_norm(want, 1e-4, 1 + w2.double()), dtype)
        assert dev == "cpu" or (not extra.any() and (not clear or not src.any()))
    y = x.to(dev).clone()
    near(M.sandwich_norm_(y, None, None, None, (put(w2), None), 1e-4, dtype), O.rms_norm(x.double(), 1e-4, 1 + w2.double()), dtype)
    assert torch.equal(y.cpu(), x)
    idx = torch.tensor([3, 1, 3], dtype=torch.int32)
    near(M.norm_rows(x.to(dev), idx.to(dev), put(w2), None, 1e-5, dtype, 2.5), 2.5 * O.rms_norm(x.double()[[3, 1, 3]], 1e-5, 1 + w2.double()), dtype)


@pytest.mark.parametrize("E,top", [(45, 3), (48, 1), (264, 6), (2056, 9)])
def test_norm_of_a_sum_of_experts(run, E, top):
    """The output of a mixture is formed where it is normed: picked rows, the input itself, the gated shared row."""
    dev, dtype = run
    T, n = 7, 11
    g = torch.Generator().manual_seed(top)
    x, w1 = torch.randn(T, E, generator=g), torch.randn(E, generator=g) * 0.3
    rows, h, shared = rnd(n, E, seed=2), rnd(T, E, seed=3), rnd(T, E, seed=4)
    slot = torch.randint(-1, n, (T, top), generator=g, dtype=torch.int32)
    weight = torch.rand(T, top + 1, generator=g)
    for with_shared in (True, False):
        s = torch.zeros(T, E, dtype=D)
        for t in range(T):
            for k in range(top):
                s[t] += weight[t, k].double() * (h[t] if slot[t, k] < 0 else rows[slot[t, k]]).double()
            if with_shared:
                s[t] += weight[t, top].double() * shared[t].double()
        want = x.double() + O.rms_norm(s, 1e-4, 1 + w1.double())
        for kind in {dtype, torch.float32}:
            y = x.to(dev).clone()
            a = M.RowSum(pitched(rows, kind, dev), slot.to(dev), weight.to(dev), pitched(h, dtype, dev), pitched(shared, kind, dev) if with_shared else None)
            if kind == dtype:
                near(X.combine(a), s, dtype)
            if kind != torch.float32:
                continue
            out = M.sandwich_norm_(y, a, (w1.to(dev), None), None, (w1.to(dev), None), 1e-4, dtype)
            near(y, want, torch.float32)
            near(out, O.rms_norm(want, 1e-4, 1 + w1.double()), dtype)


@pytest.mark.parametrize("T,n,Kd", [(1, 40, 48), (7, 37, 45), (300, 264, 100)])
def test_silu_feed_forward(run, T, n, Kd):
    dev, dtype = run
    x, w = rnd(T, Kd, seed=3, scale=2.0), rnd(2 * n, Kd, seed=4, scale=Kd ** -0.5)
    z = x.double() @ w.double().T
    want = O.silu(z[:, :n]) * z[:, n:]
    near(M.glu_linear(pitched(x, dtype, dev), pitched(w, dtype, dev), n, "silu"), want, dtype)
    acc = z.float().to(dev)
    near(M.glu(acc, n, "silu", dtype, dev == "cuda"), want, dtype)
    assert dev == "cpu" or not acc.any()


def spec_of(kind, H, Gk, dim, vdim, size, cap, scale=1.0, rot=None):
    args = (H, Gk, dim, vdim, size, scale * dim ** -0.5, cap)
    return ChunkAttentionSpec(*args) if kind == "chunk" else WindowAttentionSpec(*args, rot=RotarySpec(300.0, rot or dim // 2 * 2))


def transform(a, run, first=None, lam=0.35, seed=0):
    """A row transform with random norms and the same as plain functions of (q or k [.., dim], position)."""
    dev, dtype = run
    g = torch.Generator().manual_seed(seed)
    qn, kn = (1 + 0.4 * torch.randn(n * a.dim, generator=g) if a.qk_norm else None for n in (a.heads, a.kv_heads))
    put = lambda t: None if t is None else t.to(dev)  # noqa: E731
    rope = None if a.rot is None else rope_tables(a.rot, 700, dev)
    tr = G.QkvTransform(put(qn), put(kn), 1e-4, 0 if a.rot is None else a.rot.dims, rope, None if first is None else torch.tensor(lam, device=dev), first)

    def plain(x, heads, norm, pos):
        x = x.double()
        if norm is not None:
            x = O.rms_norm(x, 1e-4, norm.double())
        x = x.view(heads, a.dim)
        return x if a.rot is None else O.rotate_half(x, pos, {"base": a.rot.base, "dims": a.rot.dims})

    return tr, lambda x, pos: plain(x, a.heads, qn, pos), lambda x, pos: plain(x, a.kv_heads, kn, pos)


def attention_want(a, q, k, v, see, sink):
    """q [H, dim] over keys k, v [n, G, .] of which the slice ``see`` is visible -> [H, vdim]."""
    out = []
    for h in range(a.heads):
        g = h // (a.heads // a.kv_heads)
        s = (k[see, g] @ q[h]) * a.scale
        s = s if a.softcap is None else O.cap_score(s, a.softcap)
        out.append(O.softmax_weights(s, None if sink is None else sink[h].double()) @ v[see, g])
    return torch.stack(out)


def visible(a, pos):
    r = O.chunk_keys(pos, a.size) if a.chunked else O.window_keys(pos, a.size)
    return slice(r.start, r.stop)


SIZES = [(4, 2, 16, 24), (6, 2, 64, 64), (3, 1, 128, 128), (10, 2, 96, 96), (20, 1, 64, 128), (3, 3, 12, 13), (3, 3, 11, 5), (2, 1, 200, 128), (2, 2, 256, 256), (1, 1, 8, 8)]


@pytest.mark.parametrize("size", SIZES, ids=lambda s: "x".join(map(str, s)))
@pytest.mark.parametrize("kind,reach", [("chunk", 100), ("window", 130)])
def test_rows_are_normed_rotated_mixed_and_kept(run, size, kind, reach):
    """The projection rows of a packed step: queries in place, keys and mixed values in the stream and in the rings."""
    dev, dtype = run
    H, Gk, dim, vdim = size
    a = spec_of(kind, H, Gk, dim, vdim, 20, 9.0, rot=max(2, dim // 4 * 2))
    L = G.GroupedLayout(H, Gk, dim, vdim)
    step = PackedStep([(2, 0, [0] * 45), (0, 7, [0] * 3), (1, 19, [0] * 1)], dev)
    lay = step.chunk_layout(20) if a.chunked else step.layout(19)
    x, first = rnd(step.T, L.width_in, seed=4), rnd(step.T, L.v_width, seed=5)
    dst = pitched(first, dtype, dev)
    tr, fq, fk = transform(a, run, dst, seed=dim)
    inp = x.to(dtype).to(dev)
    cache, stream = torch.zeros(3, 20, L.ld_kv, dtype=dtype, device=dev), torch.zeros(lay.total, L.ld_kv, dtype=dtype, device=dev)
    G.qkv_prep_(L, inp, tr, step, lay.sidx, cache, stream)
    lam = torch.tensor(0.35).double()
    for t0, n, row, start in step.sequences():
        for i in sorted({0, 1, n // 2, n - 1} & set(range(n))):
            t, p = t0 + i, start + i
            near(inp[t, :H * dim], fq(x[t, :H * dim], p).flatten(), dtype)
            kv = stream[int(lay.sidx[t])]
            near(kv[:Gk * dim], fk(x[t, L.off_k:L.off_k + Gk * dim], p).flatten(), dtype)
            near(kv[L.kv_v:L.kv_v + L.v_width], O.mix_values(x[t, L.off_v:L.off_v + L.v_width].double(), first[t].double(), lam), dtype)
            if i >= n - 20:
                for at, m in ((0, Gk * dim), (L.kv_v, L.v_width)):
                    assert torch.equal(cache[row, p % 20, at:at + m], kv[at:at + m])
    assert torch.equal(inp[:, L.off_v:].cpu().float(), x[:, L.off_v:].float())      # the values of the layer itself stay as they are


@pytest.mark.parametrize("size", SIZES, ids=lambda s: "x".join(map(str, s)))
@pytest.mark.parametrize("kind,reach,cap,sharp", [("chunk", 150, 30.0, 1.0), ("chunk", 64, 2.0, 6.0), ("window", 129, 50.0, 6.0), ("window", 1, 9.0, 1.0),
                                                  ("window", 300, 400.0, 3.0), ("chunk", 1000, None, 1.0)])
def test_prompt_attention(run, size, kind, reach, cap, sharp):
    """Queries of several sequences (fresh, continued, one token) over a key stream; some keys stand out, around tile borders and the
    edges of windows and chunks; scores below, around and far above the cap."""
    dev, dtype = run
    if dev == "cpu" and size not in SIZES[:1] + SIZES[5:6]:
        pytest.skip("two sizes on the CPU")
    H, Gk, dim, vdim = size
    a = spec_of(kind, H, Gk, dim, vdim, reach, cap, sharp)
    L = G.GroupedLayout(H, Gk, dim, vdim)
    portions = [(2, 0, 300), (0, 0, 1), (5, 117, 70), (3, 200, 140)]
    step = PackedStep([(r, s, [0] * n) for r, s, n in portions], dev)
    lay = step.chunk_layout(reach) if a.chunked else step.layout(reach - 1)
    sink = torch.randn(H, generator=torch.Generator().manual_seed(1)) * 2 + 1
    inp = rnd(step.T, L.width_in, seed=8)
    full = {r: rnd(s + n, L.ld_kv, seed=10 + r) for r, s, n in portions}       # keys and values of whole sequences
    for kv in full.values():
        needles = [i for i in (0, 1, 63, 64, 99, 100, 127, 128, 149, 150, 199, 255, 256, 299) if i < len(kv)]
        kv[needles, :Gk * dim] *= 3
    stream = torch.empty(lay.total, L.ld_kv, dtype=torch.bfloat16)
    at = 0
    for r, s, n in portions:                                                    # what the layout says lies in the stream
        front = s % reach if a.chunked else min(s, reach - 1)
        stream[at:at + front + n] = full[r][s - front:]
        at += front + n
    assert at == lay.total
    for use_sink in (True, False):
        out = G.stream_attention(L, a, inp.to(dtype).to(dev), stream.to(dtype).to(dev), lay, sink.to(dev) if use_sink else None)
        for t0, n, row, start in step.sequences():
            k, v = full[row][:, :Gk * dim].double().view(-1, Gk, dim), full[row][:, L.kv_v:L.kv_v + Gk * vdim].double().view(-1, Gk, vdim)
            picks = {0, 1, n // 2, n - 2, n - 1, 63, 64, 127, 128, 129, reach - 1, reach, reach - start % reach, reach - start % reach - 1}
            for i in sorted(picks & set(range(n))):
                p = start + i
                want = attention_want(a, inp[t0 + i, :H * dim].double().view(H, dim), k, v, visible(a, p), sink if use_sink else None)
                near(out[t0 + i], want.flatten(), dtype, bf16=1e-2)
        if dev == "cpu":
            break
    status_ok(run)


@pytest.mark.parametrize("size", SIZES, ids=lambda s: "x".join(map(str, s)))
@pytest.mark.parametrize("kind,reach,cap", [("chunk", 70, 30.0), ("window", 70, 2.0), ("window", 500, 400.0), ("chunk", 16, None)])
@pytest.mark.parametrize("splits", [1, 3, 8])
def test_decode_attention(run, size, kind, reach, cap, splits):
    """One token per sequence at positions around every border, rings that have gone round several times, key splits that are empty."""
    dev, dtype = run
    if dev == "cpu" and (size not in SIZES[:1] + SIZES[5:6] or splits > 1):
        pytest.skip("two sizes on the CPU")
    H, Gk, dim, vdim = size
    a = spec_of(kind, H, Gk, dim, vdim, reach, cap, 3.0, rot=max(2, dim // 4 * 2))
    L, max_len = G.GroupedLayout(H, Gk, dim, vdim), 300
    ring = min(reach, max_len)
    pos, row = [0, 1, 15, 16, 69, 70, 199, 130, 139, 140], [4, 0, 11, 2, 3, 8, 6, 7, 9, 1]
    B = len(pos)
    x, first = rnd(B, L.width_in, seed=6), torch.randn(B, L.v_width, generator=torch.Generator().manual_seed(2))
    old = rnd(12, max_len, L.ld_kv, seed=5)                                      # what the sequences' earlier positions hold
    cache = torch.zeros(12, ring, L.ld_kv, dtype=torch.bfloat16)
    for r in range(12):
        for p in range(max_len):                                                 # rings as a long decoding leaves them ...
            cache[r, p % ring] = old[r, p]
    for p_, r in zip(pos, row):
        for p in range(max(0, p_ - ring), p_):                                   # ... and the rows in use at their own positions
            cache[r, p % ring] = old[r, p]
    sink = torch.randn(H, generator=torch.Generator().manual_seed(3)) + 1
    ip, ir = (torch.tensor(t, dtype=torch.int32, device=dev) for t in (pos, row))
    lam = torch.tensor(0.35).double()
    for src in ([x.float().to(dev)] if dev == "cuda" and dtype == torch.bfloat16 else []) + [x.to(dtype).to(dev)]:
        tr, fq, fk = transform(a, run, first.to(dev), seed=dim)
        c, kept = cache.to(dtype).to(dev), torch.zeros(B, L.v_width, device=dev)
        got = G.ring_attention(L, a, src, tr, c, sink.to(dev), kept, ip, ir, splits, dtype)
        near(kept, x[:, L.off_v:L.off_v + L.v_width].double(), torch.float32)
        for b, (p, r) in enumerate(zip(pos, row)):
            new = torch.zeros(1, L.ld_kv, dtype=D)
            new[0, :Gk * dim] = fk(x[b, L.off_k:L.off_k + Gk * dim], p).flatten()
            new[0, L.kv_v:L.kv_v + L.v_width] = O.mix_values(x[b, L.off_v:L.off_v + L.v_width].double(), first[b].double(), lam)
            kv = torch.cat([old[r, :p].double(), new.to(dtype).double()])
            k, v = kv[:, :Gk * dim].view(-1, Gk, dim), kv[:, L.kv_v:L.kv_v + Gk * vdim].view(-1, Gk, vdim)
            want = attention_want(a, fq(x[b, :H * dim], p), k, v, visible(a, p), sink)
            near(got[b], want.flatten(), dtype, bf16=2e-2)
            for at, m in ((0, Gk * dim), (L.kv_v, L.v_width)):
                near(c[r, p % ring, at:at + m], new[0, at:at + m], dtype)
        idle = [5, 10]
        assert torch.equal(c[idle].float().cpu(), cache[idle].float())           # rows of other sequences
    status_ok(run)


@pytest.mark.parametrize("size", [1, 7, 16, 100])
def test_chunk_layout(size):
    portions = [(0, 0, 50), (3, 13, 1), (1, 16, 40), (2, 99, 3)]
    lay = PackedStep([(r, s, [0] * n) for r, s, n in portions], "cpu").chunk_layout(size)
    at = t = 0
    for r, s, n in portions:
        front = s % size
        assert (not front) or (r, s - front, front, at) in lay.history
        for i in range(n):
            assert int(lay.sidx[t]) == at + front + i
            assert int(lay.sidx[t]) - int(lay.kbase[t]) == (s + i) % size
            t += 1
        at += front + n
    assert lay.total == at and sum(m for _, m, _, _ in lay.seqs) == t and all(f + m <= size for _, m, _, f in lay.seqs)
    assert [x[0] for x in lay.seqs] == sorted(x[0] for x in lay.seqs)


def moe_weights(s, E, run, seed=0, router=3.0):
    """Weights of a mixture as named tensors and as the product holds them."""
    dev, dtype = run
    cfg = O.config([O.chunked()], [{"kind": "moe", "expert": {"ff": s.ff}, "router": {"experts": s.experts, "identity": s.identity, "top": s.top},
                                    **({"shared": {"ff": s.shared}} if s.shared else {})}], width=E)
    w = {k[7:]: v for k, v in O.random_weights(cfg, seed, router=router).items() if k.startswith("l0.mlp.")}
    cat = lambda part: torch.cat([w[f"e{e}.{part}"] for e in range(s.experts)])  # noqa: E731
    rows = torch.cat([w["router"]] + ([w["shared.sg"]] if s.shared else []))
    p = lambda t: torch.nn.functional.pad(t, (0, ops.pad8(t.shape[1]) - t.shape[1])).to(dtype).to(dev)[:, :t.shape[1]]  # noqa: E731
    return w, cfg["layers"][0]["mlp"], X.MoeWeights(s, p(rows), w["correction"].float().to(dev), p(cat("up")), p(cat("down")),
                                                    p(w["shared.up"]) if s.shared else None, p(w["shared.down"]) if s.shared else None)


def as_rows(out):
    return out.sum() if isinstance(out, M.RowSum) else out


MOES = [(MixtureSpec(24, 6, 2, 3, 40), 48), (MixtureSpec(19, 5, 1, 4, 21), 45), (MixtureSpec(8, 1, 0, 1, None), 16), (MixtureSpec(136, 6, 2, 8, 520), 264),
        (MixtureSpec(64, 40, 0, 8, None), 520), (MixtureSpec(300, 3, 6, 2, 8), 136), (MixtureSpec(33, 70, 7, 40, 72), 72)]


@pytest.mark.parametrize("case", range(len(MOES)))
@pytest.mark.parametrize("T", [1, 2, 7, 16, 33, 64, 300, 1100])
def test_mixture_of_experts(run, case, T):
    """Both forms (any rows, the few rows of a decode step) against the tokens one by one; identity experts, the shared expert's gate."""
    dev, dtype = run
    s, E = MOES[case]
    if T > 64 and (dev == "cpu" or case == 6):
        pytest.skip("many rows: on a GPU")
    named, m, w = moe_weights(s, E, run, seed=case)
    h = rnd(T, E, seed=T)
    some = sorted({0, T // 3, T - 1} | set(range(0, T, max(1, T // 12))))
    want = O.mixture(h[some].double(), {k: v.double() for k, v in named.items()}, "", m)
    x = pitched(h, dtype, dev) if dev == "cpu" else torch.nn.functional.pad(h, (0, ops.pad8(E) - E)).to(dtype).to(dev)[:, :E]
    forms = [X.mixture] + ([X.mixture_rows] if T <= 64 else [])
    # nearly equal scores may fall either way in bf16: tokens whose choice is close are left out
    z = h[some].double() @ named["router"].double().T
    c = torch.sort(torch.softmax(z, -1) + named["correction"].double(), -1, descending=True).values
    sure = torch.ones(len(some), dtype=torch.bool) if s.top == s.outputs else (c[:, s.top - 1] - c[:, s.top]) > (1e-6 if dtype == torch.float32 else 1e-4)
    assert int(sure.sum()) >= len(some) // 2
    for f in forms:
        got = as_rows(f(w, x))[some]
        near(got[sure], want[sure], dtype, bf16=1e-2)
    status_ok(run)


def test_choice_and_weights_of_the_router(run):
    """The correction moves the choice but not the weights; equal scores go to the lower index; identity experts carry weight."""
    dev, dtype = run
    s = MixtureSpec(8, 4, 2, 3, 8)
    z = torch.tensor([[1.0, 2.0, 0.0, 0.5, 0.5, 0.5, 0.3], [0.0] * 6 + [-2.0], [-50.0, 60.0, 0.0, 0.0, 0.0, 59.0, 0.0]])
    correction = torch.tensor([0.0, -0.5, 0.0, 0.2, 0.0, 0.0])
    w = X.MoeWeights(s, None, correction.to(dev), None, None, torch.zeros(1, device=dev), None)
    want = [O.route(t[:6].double(), correction.double(), 3) for t in z]
    assert want[0][0].tolist() == [3, 0, 4] and want[1][0].tolist() == [3, 0, 2] and want[2][0].tolist() == [5, 1, 3]
    if dev == "cpu":
        from recurrent_pretraining_b200.ops import reference as ref

        idx, weight = ref.route(z[:, :6], correction, 3)
    else:
        p = X.plan(w, z.to(dev), 64)
        idx, weight = p.idx.cpu(), p.weight[:, :3]
        near(p.weight[:, 3], O.sigmoid(z[:, 6].double()), torch.float32)
        count = torch.bincount(idx[idx < 4], minlength=4)
        assert int(p.n_tiles) == int((count > 0).sum()) and p.offset.cpu().tolist()[3] == 64 * int((count[:3] > 0).sum())
        assert p.tile_expert[:int(p.n_tiles)].cpu().tolist() == [e for e in range(4) if count[e]]
    for t in range(3):
        assert idx[t].tolist() == want[t][0].tolist()
        near(weight[t], want[t][1], torch.float32)


@gpu
@pytest.mark.parametrize("dtype,rows", [(torch.float32, 64), (torch.bfloat16, 128), (torch.bfloat16, 256)])
@pytest.mark.parametrize("N,Kd", [(72, 45), (264, 136), (520, 64)])
def test_grouped_products(dtype, rows, N, Kd):
    """Every slot is multiplied with its own expert's rows; experts without a token and tiles past the last one are left out."""
    s = MixtureSpec(N, 9, 3, 2, None)
    T = 700
    z = torch.randn(T, 12, generator=torch.Generator().manual_seed(1))
    z[:, 4] = -30.0                                                  # an expert that nobody chooses
    z[:400, 7] += 9.0                                                # one that many do
    w = X.MoeWeights(s, None, torch.zeros(12, device="cuda"), None, None, None, None)
    p = X.plan(w, z.cuda(), rows)
    h, wt = rnd(T, Kd, seed=2), rnd(9 * N, Kd, seed=3, scale=Kd ** -0.5)
    pad = lambda t: torch.nn.functional.pad(t, (0, ops.pad8(Kd) - Kd)).to(dtype).cuda()[:, :Kd]  # noqa: E731
    y = X.grouped_linear(X.dispatch(w, pad(h), p), pad(wt), N, p, "relu2")
    idx, slot = p.idx.cpu(), p.slot.cpu()
    assert bool(((slot < 0) == (idx >= 9)).all()) and len(set(slot[slot >= 0].tolist())) == int((idx < 9).sum())
    for t in range(0, T, 37):
        for k in range(2):
            if idx[t, k] < 9:
                e = int(idx[t, k])
                near(y[int(slot[t, k])], O.relu2(wt[e * N:(e + 1) * N].double() @ h[t].double()), dtype)
    status_ok(("cuda", dtype))


# ------------------------------------------------------------------------------------------
# whole models
# ------------------------------------------------------------------------------------------
@pytest.mark.parametrize("name", list(CONFIGS))
def test_prompt_matches_oracle(run, name):
    cfg = CONFIGS[name]
    model, w = make(cfg, run, seed=1)
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
    cfg = CONFIGS[name]
    if run[0] == "cpu" and name == "wide" and cuts != [13, 2, 1, 1, 30]:
        pytest.skip("one on the CPU")
    model, w = make(cfg, run, seed=2, sharp=2.0)
    seq = tokens(75, cfg["vocab"])
    want = O.forward(cfg, w, seq)
    eng = engine(model)
    agree(feed(eng, eng.open(), seq, cuts), want, run)
    status_ok(run)


@pytest.mark.parametrize("kind", ["chunk", "window"])
@pytest.mark.parametrize("size", [20, 128, 131])
def test_edges_of_windows_and_chunks(run, kind, size):
    """One token's key stands out.  The last position that sees it and the next one, which does not, in prompts, in portions that end
    there, and decoded alone; a mask that is one position off would show."""
    layer = O.chunked(heads=2, kv_heads=1, dim=16, vdim=16, size=size, softcap=40.0) if kind == "chunk" else \
        O.windowed(heads=2, kv_heads=1, dim=16, vdim=16, size=size, softcap=40.0, rot=2, base=1e9)
    cfg = O.config([layer], [None])
    w = {k: v.float() for k, v in O.random_weights(cfg, 5).items()}
    u = torch.randn(16, generator=torch.Generator().manual_seed(1)).sign()
    u[:2] = 0                                                  # not turned by the rotation
    w["embed"][:, :2] = torch.tensor([2.0, 0.0])
    w["embed"][5, 1] = 9.0
    w["l0.norm1"].zero_()
    w["l0.mix.q"] *= 0.1
    w["l0.mix.k"] *= 0.1
    w["l0.mix.q"][:, 0] += 2 * u.repeat(2)                     # every query leans towards the key of token 5
    w["l0.mix.k"][:, 1] += 2 * u
    if kind == "chunk":
        w["l0.mix.q.norm"].fill_(3.0)
        w["l0.mix.k.norm"].fill_(1.0)
        w["l0.mix.sink"].zero_()
    w = {k: v.bfloat16() for k, v in w.items()}
    at = size + 3                                              # in the second chunk; the window of its last viewer starts there
    seq = [t for t in tokens(3 * size + 60) if t != 5][:2 * size + 12]
    seq[at] = 5
    last = 2 * size - 1 if kind == "chunk" else at + size - 1
    want, other = O.forward(cfg, w, seq), O.forward(cfg, w, seq[:at] + [6] + seq[at + 1:])
    gone = (want - other).square().mean(-1).sqrt() / want.square().mean().sqrt()
    assert float(gone[last]) > 0.1 and float(gone[last + 1]) < 1e-9
    model = load(cfg, w, run)
    eng = engine(model)
    for cuts in ([len(seq)], [last, 1], [last + 1, 1], [at, 2, last - at - 1, 1], [size + 1, 1]):
        row = eng.open()
        agree(feed(eng, row, seq, cuts), want, run, cuts)
        eng.close(row)
    status_ok(run)


def test_sinks_and_caps_show(run):
    """Leaving out a sink, a cap, the value mixing or the correction changes the logits far beyond the tolerance: the agreement of the
    other tests covers them."""
    cfg = O.config([O.chunked(softcap=2.0), O.windowed(softcap=2.0), O.chunked(size=9, softcap=2.0)], [O.moe()])
    model, w = make(cfg, run, seed=3, sharp=4.0)
    seq = tokens(60)
    want = O.forward(cfg, w, seq)
    agree(model(torch.tensor([seq]))[0], want, run)
    loose = json.loads(json.dumps(cfg))
    for layer in loose["layers"]:
        layer["mixer"]["softcap"] = 1e6
    changes = [O.forward(loose, w, seq)]
    for part, value in (("sink", -40.0), ("vmix", 0.0), ("correction", 0.0), ("k.norm", 1.0), ("norm1b", 0.0)):
        changes.append(O.forward(cfg, {k: (torch.full_like(v, value) if k.endswith(part) else v) for k, v in w.items()}, seq))
    for other in changes:
        assert O.rel_error(other, want) > 0.05
    if run[0] == "cpu":
        for key in ("scale",):
            c = json.loads(json.dumps(cfg))
            c["layers"][1]["mixer"][key] *= 1.3
            assert O.rel_error(O.forward(c, w, seq), want) > 0.01


def test_far_tokens_come_through_the_layers(run):
    """Tokens beyond one window or chunk reach later positions through several layers, whatever the cuts."""
    cfg = O.config([O.windowed(size=40), O.chunked(size=90), O.windowed(size=40)], [O.mlp()])
    model, w = make(cfg, run, seed=6, sharp=3.0)
    seq = tokens(150)
    want = O.forward(cfg, w, seq)
    assert O.rel_error(O.forward(cfg, w, tokens(20, seed=9) + seq[20:])[75:90], want[75:90]) > 0.05
    eng = engine(model)
    for cuts in ([150], [100, 1], [7, 2, 90, 1], [2]):
        agree(feed(eng, eng.open(), seq, cuts), want, run, cuts)


def test_long_decoding(run):
    """Rings that go round many times; the cache is full at the end."""
    cfg = O.config([O.windowed(size=17), O.chunked(size=25)], [O.moe(), O.mlp()])
    model, w = make(cfg, run, seed=8, sharp=2.0)
    seq = tokens(260)
    want = O.forward(cfg, w, seq)
    eng = engine(model, 1, 260)
    assert eng.cache.data[0, "kv"].shape[1] == 17 and eng.cache.data[1, "kv"].shape[1] == 25       # a sequence holds a bounded amount
    agree(feed(eng, eng.open(), seq, [4, 1]), want, run)
    with pytest.raises(ValueError):
        eng.step([(0, [1])])


def test_first_tokens(run):
    model, w = make(MIXED, run, seed=9)
    eng = engine(model)
    for t in (0, 66):
        agree(eng.step([(eng.open(), [t])]), O.forward(MIXED, w, [t]), run)
    seq = tokens(6)
    want = O.forward(MIXED, w, seq)
    for n in range(1, 6):
        row = eng.open()
        got = torch.cat([eng.step([(row, seq[:n])], [list(range(n))]), eng.step([(row, seq[n:])], [list(range(6 - n))])])
        agree(got, want, run)


def test_unequal_batches_match_each_alone(run):
    model, w = make(MIXED, run, seed=10, sharp=2.0)
    seqs = [tokens(n, seed=n) for n in (1, 33, 90, 5, 64)]
    more = [tokens(7, seed=100 + n) for n in range(5)]
    wants = [O.forward(MIXED, w, s + m) for s, m in zip(seqs, more)]
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
    """A row's keys of its former sequence are not seen by the next one, which may be shorter or a single token."""
    model, w = make(MIXED, run, seed=11, sharp=2.0)
    eng = engine(model, rows=2)
    for k in range(4):
        a, b = eng.open(), eng.open()
        assert {a, b} == {0, 1} and eng.cache.rows == 2
        for row, n in ((a, 70 - 22 * k), (b, 1 + 20 * k)):
            seq = tokens(n + 4, seed=k)
            agree(feed(eng, row, seq, [n, 1]), O.forward(MIXED, w, seq), run)
        eng.close(b)
        eng.close(a)
    with pytest.raises(KeyError):
        eng.close(a)


def test_greedy_generation_through_the_scheduler(run):
    from recurrent_pretraining_b200.engine import server as S

    cfg = O.config([O.windowed(), O.chunked()], [O.moe(), O.mlp()])
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
    model, w = make(MIXED, run, seed=13)
    eng = engine(model)
    prompts = [tokens(9), tokens(4)]
    plain = eng.generate(prompts, 20)
    stop = plain[0][5]
    cut = eng.generate(prompts, 20, stop_ids=[stop], check_every=2)
    for p, c in zip(plain, cut):
        end = p.index(stop) + 1 if stop in p else len(p)
        assert c == p[:end]
    assert model.generate(prompts, 5) == [p + o[:5] for p, o in zip(prompts, plain)] or run[1] == torch.bfloat16
    small = engine(model, prefill_tokens=5)                        # prompts in portions, several sequences per step
    assert small.generate(prompts, 6) == [p[:6] for p in plain] or run[1] == torch.bfloat16
    assert not eng.cache.length                                    # every row went back


def test_trace_replay(run, tmp_path):
    import numpy as np
    from recurrent_pretraining_b200.engine.trace import replay

    model, w = make(MIXED, run, seed=14)
    a, b = tokens(20, seed=1), tokens(9, seed=2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:18], "want": [0, 17]}, {"id": "b", "tokens": b[:8], "want": [7]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[18:19], "want": []}, {"id": "b", "tokens": b[8:], "want": []}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": a[19:], "want": [0]}], "end": ["a"]}]
    answer = io.StringIO()
    eng = engine(model, 1, 64)
    replay(eng, [json.dumps(s) + "\n" for s in steps], str(tmp_path), answer)
    assert answer.getvalue() == "done 0\ndone 1\ndone 2\n" and not eng.cache.length
    wa, wb = O.forward(MIXED, w, a), O.forward(MIXED, w, b)
    got = torch.from_numpy(np.fromfile(tmp_path / "0.f32", dtype="<f4")).view(3, -1)
    agree(got, torch.stack([wa[0], wa[17], wb[7]]), run)
    got = torch.from_numpy(np.fromfile(tmp_path / "2.f32", dtype="<f4")).view(1, -1)
    agree(got, wa[19:], run)


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


def test_serve_command_completes_a_prompt(tmp_path, capsys):
    import serve

    cfg = O.config([O.windowed(), O.chunked()], [O.moe()])
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
    cfg = O.config([O.windowed(heads=8, kv_heads=2, dim=32, vdim=64, size=30), O.chunked(heads=8, kv_heads=2, dim=32, vdim=64, size=25)],
                   [O.mlp(1024), O.moe(8, 2, 3, 128, 640)], width=640)
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
    cfg = CONFIGS[name]
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
    cfg = O.config([O.chunked(heads=4, kv_heads=2, dim=64, vdim=64, size=700, softcap=20.0), O.windowed(heads=8, kv_heads=2, dim=64, vdim=64, size=333, rot=32, softcap=30.0)],
                   [O.moe(6, 2, 3, 96, 128)], width=256)
    w = O.random_weights(cfg, 18, router=6.0)
    seqs = [tokens(n, seed=n) for n in (1500, 900, 3, 257)]
    outs = []
    for dtype in (torch.bfloat16, torch.float32):
        eng = engine(load(cfg, w, ("cuda", dtype)), max_len=1600)
        outs.append(eng.step([(eng.open(), s) for s in seqs], [list(range(0, len(s), 7)) for s in seqs]).double().cpu())
    agree(outs[0], outs[1], run)
    status_ok(run)
