"""Layered decoder models that mix distance-biased attention with recurrent memories (design ``Fatudra``): every mechanism and
the serving path against the plain statements of ``hybrid_oracle``, on the CPU (fp32) and on the GPU kernels (fp32 and bf16)."""
import io
import json
import math
import os

import pytest
import torch

import hybrid_oracle as O
from recurrent_pretraining_b200.models import build_model
from recurrent_pretraining_b200.models.layered import LayeredForCausalLM
from recurrent_pretraining_b200.models.layered_config import BiasedAttentionSpec, LayeredConfig, QueryTemperature
from recurrent_pretraining_b200.models.sublayers import PackedStep
from recurrent_pretraining_b200.ops import latent as ops
from recurrent_pretraining_b200.ops import memory as M
from recurrent_pretraining_b200.ops.memory import MemoryLayout, ParallelLayout

gpu = pytest.mark.gpu
RUNS = [pytest.param(("cpu", torch.float32), id="cpu"), pytest.param(("cuda", torch.float32), marks=gpu, id="gpu-f32"),
        pytest.param(("cuda", torch.bfloat16), marks=gpu, id="gpu-bf16")]
TOL = {torch.float32: 3e-5, torch.bfloat16: 8e-2}     # rms of the logit error over the rms of the logits


@pytest.fixture(params=RUNS)
def run(request):
    return request.param


def make(cfg, run, seed=0, sharp=1.0):
    dev, dtype = run
    w = O.random_weights(cfg, seed, sharp)
    model = LayeredForCausalLM(LayeredConfig.from_dict(cfg), dtype, dev)
    model.load_checkpoint(O.TensorDict(w))
    return model, w


def engine(model, rows=4, max_len=400, **kw):
    from recurrent_pretraining_b200.engine.layered import LayeredEngine

    return LayeredEngine(model, rows, max_len, **kw)


def tokens(n, vocab=67, seed=0):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(2000 + seed + 7919 * n)).tolist()


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


def close(got, want, dtype, scale=1.0):
    err = float((got.double().cpu() - want).abs().max())
    assert err <= (5e-6 if dtype == torch.float32 else 1.2e-2) * scale * (1 + float(want.abs().max())), err


def near(got, want, dtype, f32=2e-5, bf16=8e-3):
    """rms error over rms."""
    d = got.double().cpu() - want
    err = float(d.square().mean().sqrt() / want.square().mean().sqrt())
    ok = bool(torch.isfinite(d).all()) and err < (f32 if dtype == torch.float32 else bf16)
    assert ok, err


def rnd(*shape, seed=0, scale=1.0):
    """Values that bf16 represents exactly."""
    return (torch.randn(*shape, generator=torch.Generator().manual_seed(seed)) * scale).bfloat16()


# layers that differ in every size, a loop over a layer of each kind, a layer without feed-forward
MIXED = O.config([O.par(), O.mem(), O.par(heads=6, kv_heads=6, dim=24, vdim=8, rows=7, bias_max=31.5, q_temp=None, r_heads=1, r_dim=24, r_vdim=40),
                  O.mem(heads=3, dim=40, vdim=8, gate_cap=4.0), O.par(heads=5, kv_heads=1, dim=8, vdim=72, rows=2, bias_max=9, q_temp=(1.0, 1), r_heads=2)],
                 ff=(40, None, 88), loop=(1, 3, 3))
# nothing is a multiple of eight
ODD = O.config([O.par(heads=3, kv_heads=3, dim=11, vdim=13, rows=5, bias_max=20, r_heads=3, r_dim=7, r_vdim=5), O.mem(heads=3, dim=9, vdim=21),
                O.par(heads=6, kv_heads=2, dim=5, vdim=3, rows=9, r_heads=1, r_dim=13, r_vdim=11)], ff=(37,), width=45, vocab=61, eps=1e-3, loop=(0, 3, 2))
ONE = O.config([O.par(heads=1, kv_heads=1, dim=8, vdim=8, rows=1, r_heads=1, r_dim=8, r_vdim=8, left_scale=1.0, right_scale=1.0, decay=[1.0]),
                O.mem(heads=1, dim=8, vdim=8)], ff=(8,), width=16, vocab=19, scale=1.0, loop=(1, 2, 1))
WIDE = O.config([O.par(heads=20, kv_heads=1, dim=64, vdim=128, rows=12, r_heads=9, r_dim=64, r_vdim=72), O.mem(heads=5, dim=128, vdim=96)],
                ff=(600,), width=520)
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
    assert [(r.layer, r.loop_pass) for r in cfg.runs()] == O.layer_runs(d)


def test_table_height_comes_from_the_tensors(tmp_path):
    """A stored configuration does not name the rows of the distance-bias tables; layers may differ in them."""
    from recurrent_pretraining_b200.models import auto
    from recurrent_pretraining_b200.models.weights import save_safetensors

    w = O.random_weights(MIXED, 3)
    with open(tmp_path / "config.json", "w") as f:
        json.dump(O.stored(MIXED), f)
    save_safetensors(str(tmp_path / "model.safetensors"), w)
    model = auto.load_pretrained(str(tmp_path), torch.float32, torch.device("cpu"))
    assert [layer.mix.spec.left.bias_rows for layer in model.layers[::2]] == [10, 7, 2]
    assert all(torch.equal(v, w[k].float()) for k, v in model.checkpoint_tensors().items())
    seq = tokens(9)
    assert O.rel_error(model(torch.tensor([seq]))[0], O.forward(MIXED, w, seq)) < TOL[torch.float32]
    with pytest.raises(ValueError):
        build_model(LayeredConfig.from_dict(O.stored(MIXED)))
    again = tmp_path / "again"
    model.save_pretrained(str(again))
    assert torch.equal(auto.load_pretrained(str(again), torch.float32, torch.device("cpu"))(torch.tensor([seq])), model(torch.tensor([seq])))


def _left(c):
    return c["layers"][0]["mixer"]["left"]


@pytest.mark.parametrize("change", [
    lambda c: c.update(architecture="Unknown"), lambda c: c.update(residual_mult=0.5), lambda c: c["layers"][0].update(type="latent_attention"),
    lambda c: c["layers"][0].update(type="other"), lambda c: _left(c).update(window=3), lambda c: _left(c).update(kv_heads=3),
    lambda c: _left(c).update(bias_max=5), lambda c: _left(c)["q_temp"].update(every=0), lambda c: c["layers"][0]["mixer"]["right"]["decay"].append(0.5),
    lambda c: c["layers"][0]["mixer"]["right"]["decay"].__setitem__(0, 1.5), lambda c: c["layers"][1]["mixer"].update(gate_cap=0.0),
    lambda c: c["layers"][1]["mixer"].update(dim=0), lambda c: c["loop"].update(stop=9), lambda c: c["loop"].update(times=0),
    lambda c: c["loop"].update(start=3), lambda c: c["layers"][0]["mlp"].update(kind="gated"), lambda c: c["norm"].update(kind="rms"),
    lambda c: c["embedding"].update(tied=True)])
def test_invalid_configs_are_refused(change):
    cfg = json.loads(json.dumps(MIXED))
    change(cfg)
    with pytest.raises((ValueError, KeyError)):
        LayeredConfig.from_dict(cfg)


def test_registry_shapes_build():
    tiny = build_model(LayeredConfig.from_name("fatudra-tiny"), dtype=torch.float32).init_weights(1)
    assert tiny(torch.tensor([[1, 2, 3], [4, 5, 6]])).shape == (2, 3, 512) and len(tiny.runs) == 6
    for name in ("fatudra-1b", "fatudra-core-5280"):
        assert LayeredConfig.from_name(name).param_count() > 1e9


# ------------------------------------------------------------------------------------------
# mechanisms alone
# ------------------------------------------------------------------------------------------
@pytest.mark.parametrize("rows,reach", [(1, 5), (2, 2), (2, 50), (3, 40), (7, 31.5), (10, 6), (16, 250), (32, 128), (32, 1000), (64, 33)])
def test_distance_buckets(rows, reach):
    spec = BiasedAttentionSpec(1, 1, 8, 8, 1.0, reach).with_rows(rows)
    ids = spec.buckets()
    far = len(ids) - 1
    for n in range(3 * int(reach) + 10):
        assert ids[min(n, far)] == O.bucket(n, rows, reach)
    assert ids[-1] == rows - 1 and sorted(ids) == ids
    rel = torch.randn(rows, 3)
    assert torch.equal(M.BiasTable.build(rel, ids).values, rel[ids].T)


def test_query_temperature():
    spec = QueryTemperature(0.3, 7)
    for p in (0, 5, 6, 7, 12, 13, 14, 699, 700):
        assert spec.at(p) == pytest.approx(O.query_temperature(p, {"coef": 0.3, "every": 7}))
    assert spec.at(5) == 1.0 and spec.at(6) == pytest.approx(1 + 0.3 * math.log(2))


@pytest.mark.parametrize("E", [45, 48, 2056, 9000])
def test_layer_norms_around_sublayers(run, E):
    dev, dtype = run
    g = torch.Generator().manual_seed(E)
    x, bias, step = torch.randn(5, E, generator=g) * 3 + 1.5, torch.randn(E, generator=g), torch.randn(E, generator=g)
    a, w1, b1, w2, b2 = rnd(5, E, seed=1) + 0.7, *(torch.randn(E, generator=g) for _ in range(4))
    a = a.bfloat16()
    put = lambda t: t.to(dev)  # noqa: E731
    post, pre = (put(w1), put(b1)), (put(w2), put(b2))
    acc = torch.zeros(5, ops.pad8(E), device=dev)[:, :E]             # the fp32 accumulator of a weight-streaming product
    for src, clear in ((a.to(dev).to(dtype), False), (acc, dev == "cuda")):
        for use_bias, use_step, use_pre in ((True, True, True), (False, False, True), (True, False, False)):
            src.copy_(a)
            y = x.to(dev).clone()
            extra = torch.ones(5, 12, device=dev)
            s = a.double() + (0.6 * bias.double() if use_bias else 0)
            want = x.double() + O.layer_norm(s, 1e-4, w1.double(), b1.double()) + (step.double() if use_step else 0)
            h = M.sandwich_norm_(y, src, post, put(step) if use_step else None, pre if use_pre else None, 1e-4, dtype, put(bias) if use_bias else None,
                                 0.6, clear, extra if dev == "cuda" else None)
            close(y, want, torch.float32)
            if use_pre:
                close(h, O.layer_norm(want, 1e-4, w2.double(), b2.double()), dtype)
            else:
                assert h is None
            assert dev == "cpu" or (not extra.any() and (not clear or not src.any()))
    y = x.to(dev).clone()
    h = M.sandwich_norm_(y, None, None, put(step), pre, 1e-4, dtype)
    close(h, O.layer_norm(x.double() + step.double(), 1e-4, w2.double(), b2.double()), dtype)
    close(y, x.double() + step.double(), torch.float32)
    idx = torch.tensor([3, 1, 3], dtype=torch.int32)
    close(M.norm_rows(x.to(dev), idx.to(dev), *pre, 1e-5, dtype), O.layer_norm(x.double()[[3, 1, 3]], 1e-5, w2.double(), b2.double()), dtype)


@pytest.mark.parametrize("T,n,Kd", [(1, 40, 48), (7, 37, 45), (130, 264, 100), (300, 600, 520), (513, 250, 72)])
def test_gated_feed_forward(run, T, n, Kd):
    dev, dtype = run
    x, w = rnd(T, Kd, seed=3, scale=2.0), rnd(2 * n, Kd, seed=4, scale=Kd ** -0.5)
    pitch = lambda t: torch.nn.functional.pad(t, (0, ops.pad8(Kd) - Kd)).to(dtype).to(dev)[:, :Kd]  # noqa: E731
    z = x.double() @ w.double().T
    want = O.gelu_tanh(z[:, :n]) * z[:, n:]
    close(M.glu_linear(pitch(x), pitch(w), n, "gelu"), want, dtype)
    acc = z.float().to(dev)
    close(M.glu(acc, n, "gelu", dtype, dev == "cuda"), want, dtype)
    assert dev == "cpu" or not acc.any()
    # the projection of a parallel layer: a bias on all columns, silu on some
    y = ops.linear(pitch(x), pitch(w), torch.arange(2 * n, device=dev, dtype=torch.float32) / n, "silu", act_cols=(8, ops.pad8(n)))
    h = z + torch.arange(2 * n, dtype=torch.float64) / n
    h[:, 8:ops.pad8(n)] = O.silu(h[:, 8:ops.pad8(n)])
    close(y, h, dtype)
    # silu gates are not disturbed by the option
    if dtype == torch.bfloat16:
        from recurrent_pretraining_b200.ops import cuda as K

        close(K.gemm(pitch(x), pitch(w), out=torch.empty(T, ops.pad8(n), dtype=dtype, device=dev)[:, :n], out_mode=K.OUT_SWIGLU),
              O.silu(z[:, :n]) * z[:, n:], dtype)


def test_gate_projections(run):
    dev, dtype = run
    for T, n, Kd in ((5, 6, 40), (300, 10, 520), (700, 64, 1024), (300, 70, 512)):
        h, w = rnd(T, Kd, seed=1).to(dtype).to(dev), rnd(n, Kd, seed=2, scale=Kd ** -0.5).to(dtype).to(dev)
        got = M.gate_projections(h, w)
        assert got.dtype == torch.float32
        near(got, h.double().cpu() @ w.double().cpu().T, torch.float32)


def attention_case(size, rows, reach, temp, seed):
    H, G, dim, vdim = size
    spec = BiasedAttentionSpec(H, G, dim, vdim, 1.1 * dim ** -0.5, reach, QueryTemperature(*temp) if temp else None).with_rows(rows)
    L = ParallelLayout(H, G, dim, vdim, 2, 8, 16)
    return spec, L, torch.randn(rows, H, generator=torch.Generator().manual_seed(seed)) * 2


def attention_want(spec, rel, q, k, v, pos):
    """q [H, dim] at ``pos`` over keys [pos + 1, G, .] -> [H, vdim]."""
    t = O.query_temperature(pos, None if spec.q_temp is None else {"coef": spec.q_temp.coef, "every": spec.q_temp.every})
    bias = rel.double()[[O.bucket(pos - j, len(rel), spec.bias_max) for j in range(pos + 1)]]
    out = []
    for h in range(spec.heads):
        g = h // (spec.heads // spec.kv_heads)
        s = (k[:, g] @ (q[h] * t)) * spec.scale + bias[:, h]
        e = torch.exp(s - s.max())
        out.append((e / e.sum()) @ v[:, g])
    return torch.stack(out)


ATT = [(4, 2, 16, 24), (6, 2, 64, 64), (3, 1, 128, 128), (10, 2, 96, 96), (20, 1, 64, 128), (3, 3, 11, 13), (2, 1, 200, 128), (2, 2, 256, 256), (1, 1, 8, 8)]


@pytest.mark.parametrize("size", ATT, ids=lambda s: "x".join(map(str, s)))
@pytest.mark.parametrize("rows,reach,temp", [(16, 60, (0.5, 40)), (7, 300.0, None), (1, 9, (0.2, 1))])
def test_prompt_attention(run, size, rows, reach, temp):
    """Queries of several sequences (fresh, continued, one token) over the cached keys; a few keys stand out, some far away and
    some around tile borders and bucket edges."""
    dev, dtype = run
    if dev == "cpu" and size not in ATT[:1] + ATT[5:6]:
        pytest.skip("two sizes on the CPU")
    spec, L, rel = attention_case(size, rows, reach, temp, seed=size[2] + rows)
    H, G, dim, vdim = size
    portions = [(2, 0, [0] * 300), (0, 0, [0]), (5, 117, [0] * 70), (3, 200, [0] * 129)]
    step = PackedStep(portions, dev)
    cap = 350
    cache = rnd(6, cap, L.ld_kv, seed=7)
    needles = [0, 1, 63, 64, 127, 128, 129, 255, 256, 299]
    keys = cache[:, :, :G * dim].view(6, cap, G, dim)
    keys[:, needles] = keys[:, needles] * 3
    inp = rnd(step.T, L.width_in, seed=8)
    cache_dev, table = cache.to(dtype).to(dev), M.BiasTable.build(rel.to(dev), spec.buckets())
    x = inp.to(dtype).to(dev)
    M.kv_append(L, x, None, cache_dev, step.pos, step.row)
    for t0, n, row, start in step.sequences():
        cache[row, start:start + n] = inp[t0:t0 + n, L.off_k:L.off_k + L.ld_kv]
    assert torch.equal(cache_dev.float().cpu(), cache.float())
    out = torch.full((step.T, L.width_o), 7.0, dtype=dtype, device=dev)
    out = torch.nn.functional.pad(out, (0, ops.pad8(L.width_o) - L.width_o))[:, :L.width_o]
    M.prompt_attention(L, spec, x, cache_dev, table, step, 0.7, out)
    for t0, n, row, start in step.sequences():
        for i in sorted({0, 1, n // 2, n - 2, n - 1, 127, 128, 129} & set(range(n))):
            p = start + i
            k = cache[row, :p + 1, :G * dim].double().view(p + 1, G, dim)
            v = cache[row, :p + 1, L.kv_v:L.kv_v + G * vdim].double().view(p + 1, G, vdim)
            want = attention_want(spec, rel, inp[t0 + i, :H * dim].double().view(H, dim), k, v, p)
            want = want * O.sigmoid(inp[t0 + i, L.off_lg:L.off_lg + H].double())[:, None] * 0.7
            near(out[t0 + i, :H * vdim], want.flatten(), dtype)
    assert bool((out[:, L.off_r:] == 7).all())
    status_ok(run)


@pytest.mark.parametrize("size", ATT, ids=lambda s: "x".join(map(str, s)))
@pytest.mark.parametrize("splits", [1, 3, 8])
def test_parallel_decode(run, size, splits):
    """One token per sequence at different positions: both halves, their gates and the merge of key splits."""
    dev, dtype = run
    if dev == "cpu" and (size not in ATT[:1] + ATT[5:6] or splits > 1):
        pytest.skip("two sizes on the CPU")
    from recurrent_pretraining_b200.models.layered_config import DecayMemorySpec, ParallelSpec

    H, G, dim, vdim = size
    spec, L, rel = attention_case(size, 9, 70, (0.4, 30), seed=3)
    decay = (0.0, 0.97)
    both = ParallelSpec(spec, DecayMemorySpec(2, 8, 16, decay), 0.7, 1.2)
    pos, row = [0, 1, 15, 16, 69, 70, 199, 130], [4, 0, 11, 2, 3, 8, 6, 7]
    B, cap = len(pos), 200
    cache, state = rnd(12, cap, L.ld_kv, seed=5), torch.randn(12, 2, 8, 16, generator=torch.Generator().manual_seed(1))
    inp, bias = rnd(B, L.width_in, seed=6), torch.randn(L.width_in, generator=torch.Generator().manual_seed(2)) * 0.3
    bias[L.off_lg:] = 0                                            # only q, k and v have biases
    norm_w = torch.rand(32) + 0.5
    x = inp.double() + bias.double()
    want = []
    for b, (p, r) in enumerate(zip(pos, row)):
        rounded = x[b, L.off_k:L.off_k + L.ld_kv].to(dtype).double()
        kv = torch.cat([cache[r, :p].double(), rounded[None]])
        k, v = kv[:, :G * dim].view(p + 1, G, dim), kv[:, L.kv_v:L.kv_v + G * vdim].view(p + 1, G, vdim)
        o = attention_want(spec, rel, x[b, :H * dim].view(H, dim), k, v, p) * O.sigmoid(x[b, L.off_lg:L.off_lg + H])[:, None] * 0.7
        m = []
        for h in range(2):
            q, kk = (O.silu(x[b, o_ + 8 * h:o_ + 8 * h + 8]) for o_ in (L.off_rq, L.off_rk))
            S = (0 if p == 0 else decay[h]) * state[r, h].double() + torch.outer(kk, O.silu(x[b, L.off_rv + 16 * h:L.off_rv + 16 * h + 16]))
            m.append(S.T @ q)
        m = O.rms_norm(torch.cat(m), 1e-4, norm_w.double()) * O.sigmoid(x[b, L.off_rg:L.off_rg + 32]) * 1.2
        want.append((o.flatten(), m))
    put = lambda t: t.to(dev)  # noqa: E731
    table = M.BiasTable.build(put(rel), spec.buckets())
    ip, ir = (torch.tensor(t, dtype=torch.int32, device=dev) for t in (pos, row))
    for src in ([put(inp).float()] if dev == "cuda" and dtype == torch.bfloat16 else []) + [put(inp).to(dtype)]:
        c, s = put(cache).to(dtype), put(state).clone()
        got = M.parallel_decode(L, both, src, put(bias), c, s, table, torch.tensor(decay, device=dev), put(norm_w), 1e-4, ip, ir, splits, dtype)
        for b, (o, m) in enumerate(want):
            near(got[b, :H * vdim], o, dtype, bf16=1.2e-2)
            near(got[b, L.off_r:], m, dtype, bf16=1.2e-2)
        near(c[ir.long(), ip.long()], x[:, L.off_k:L.off_k + L.ld_kv], dtype)
        assert torch.equal(s[[1, 5, 9, 10]].cpu(), state[[1, 5, 9, 10]])          # rows of other sequences
    status_ok(run)


MEM = [(2, 16, 24), (2, 64, 64), (3, 128, 128), (2, 96, 192), (2, 24, 40), (2, 7, 9), (1, 200, 72), (1, 8, 8)]
PORTIONS = [(3, 0, 300), (1, 5, 1), (0, 0, 2), (4, 77, 129), (2, 128, 128)]


def memory_inputs(size, seed):
    H, dim, vdim = size
    L = MemoryLayout(H, dim, vdim)
    step_rows = 5
    T = sum(n for _, _, n in PORTIONS)
    inp = rnd(T, L.width_in, seed=seed)
    g = torch.Generator().manual_seed(seed)
    state, stab = torch.randn(step_rows, H, dim, L.ldv, generator=g) * 0.5, torch.rand(step_rows, H, dim + 1, generator=g)
    state[..., vdim:] = 0
    x = inp.double()
    q, k, v = (x[:, o:o + H * n].reshape(T, H, n) for o, n in ((L.off_q, dim), (L.off_k, dim), (L.off_v, vdim)))
    return L, inp, q, k, v, state, stab


@pytest.mark.parametrize("size", MEM, ids=lambda s: "x".join(map(str, s)))
def test_decaying_memory_of_a_prompt(run, size):
    dev, dtype = run
    if dev == "cpu" and size not in MEM[:1] + MEM[5:6]:
        pytest.skip("two sizes on the CPU")
    H, dim, vdim = size
    base, inp, q, k, v, state, _ = memory_inputs(size, seed=4)
    L = ParallelLayout(1, 1, 8, 8, H, dim, vdim)
    x = torch.zeros(inp.shape[0], L.width_in, dtype=torch.bfloat16)
    for at, o, n in ((L.off_rq, base.off_q, dim), (L.off_rk, base.off_k, dim), (L.off_rv, base.off_v, vdim)):
        x[:, at:at + H * n] = inp[:, o:o + H * n]
    decay = torch.tensor([1.0, 0.6, 0.999][:H])
    step = PackedStep([(r, s, [0] * n) for r, s, n in PORTIONS], dev)
    s = state.clone().to(dev)
    logs = torch.log2(decay).to(dev)
    got = M.decay_memory_prompt(L, x.to(dtype).to(dev), decay.to(dev), logs, s, step)
    after = state.double()
    for t0, n, row, start in step.sequences():
        S0 = state[row, :, :, :vdim].double() if start else torch.zeros(H, dim, vdim, dtype=torch.float64)
        o = O.decayed_memory(q[t0:t0 + n], k[t0:t0 + n], v[t0:t0 + n], decay.double())
        for h in range(H):                                         # what the state in front still contributes
            for t in range(n):
                o[t, h] += decay[h].double() ** (t + 1) * (S0[h].T @ q[t0 + t, h])
        near(got[t0:t0 + n], o.flatten(1), dtype)
        w = decay.double()[None] ** torch.arange(n - 1, -1, -1)[:, None]
        after[row, :, :, :vdim] = decay.double()[:, None, None] ** n * S0 + torch.einsum("th,thd,the->hde", w, k[t0:t0 + n], v[t0:t0 + n])
    near(s, after, torch.float32)
    status_ok(run)


def gated_want(L, size, inp, q, k, v, li, lf, state, stab, norm_w, t0, n, row, start):
    H, dim, vdim = size
    out = []
    S, N, m = state[row, :, :, :vdim], stab[row, :, :dim], stab[row, :, dim]
    if start == 0:
        S.zero_(), N.zero_(), m.zero_()
    for t in range(t0, t0 + n):
        o = []
        for h in range(H):
            mn = max(float(lf[t, h] + m[h]), float(li[t, h]))
            a, b = math.exp(float(lf[t, h] + m[h]) - mn), math.exp(float(li[t, h]) - mn)
            S[h] = a * S[h] + b * torch.outer(k[t, h], v[t, h])
            N[h], m[h] = a * N[h] + b * k[t, h], mn
            qq = q[t, h] * dim ** -0.5
            o.append(O.rms_norm(S[h].T @ qq / (max(abs(float(N[h] @ qq)), math.exp(-mn)) + 1e-6), 1e-4))
        out.append(torch.cat(o) * norm_w.double() * O.sigmoid(inp[t, L.off_g:L.off_g + H * vdim].double()))
    return torch.stack(out)


@pytest.mark.parametrize("size", MEM, ids=lambda s: "x".join(map(str, s)))
def test_gated_memory(run, size):
    """A packed step with fresh and continued sequences, then one token per row; outputs, states, normalisers, maxima."""
    dev, dtype = run
    if dev == "cpu" and size not in MEM[:1] + MEM[5:6]:
        pytest.skip("two sizes on the CPU")
    H, dim, vdim = size
    L, inp, q, k, v, state, stab = memory_inputs(size, seed=5)
    g = torch.Generator().manual_seed(9)
    T, E = inp.shape[0], 40
    h, w = rnd(T, E, seed=1), rnd(2 * H, E, seed=2, scale=2 * E ** -0.5)
    gb = torch.randn(2 * H, generator=g)
    gb[H:] += 3
    norm_w = torch.rand(H * vdim, generator=g) + 0.5
    z = h.double() @ w.double().T
    z = 5.0 * torch.tanh((z + gb.double()) / 5.0)
    li, lf = z[:, :H], -torch.log1p(torch.exp(-z[:, H:]))
    put = lambda t: t.to(dev)  # noqa: E731
    step = PackedStep([(r, s, [0] * n) for r, s, n in PORTIONS], dev)
    s, e = put(state).clone(), put(stab).clone()
    gates = M.gate_projections(put(h).to(dtype), put(w).to(dtype))
    got = M.gated_memory(L, put(inp).to(dtype), gates, put(gb), 5.0, s, e, put(norm_w), 1e-4, dtype, step=step)
    st, sb = state.double(), stab.double()
    for t0, n, row, start in step.sequences():
        near(got[t0:t0 + n], gated_want(L, size, inp, q, k, v, li, lf, st, sb, norm_w, t0, n, row, start), dtype, f32=1e-4, bf16=1.2e-2)
    near(s, st, torch.float32, f32=1e-4)
    near(e, sb, torch.float32, f32=1e-4)
    pos, row = [9, 0, 300], [2, 0, 4]
    ip, ir = (torch.tensor(t, dtype=torch.int32, device=dev) for t in (pos, row))
    s, e = put(st.float()), put(sb.float())
    for src in ([put(inp[:3]).float()] if dev == "cuda" and dtype == torch.bfloat16 else []) + [put(inp[:3]).to(dtype)]:
        s1, e1, st1, sb1 = s.clone(), e.clone(), st.clone(), sb.clone()
        got = M.gated_memory(L, src, None, put(gb), 5.0, s1, e1, put(norm_w), 1e-4, dtype, rows=(ip, ir), h=put(h[:3]).to(dtype), w_gate=put(w).to(dtype))
        for b in range(3):
            near(got[b:b + 1], gated_want(L, size, inp, q, k, v, li, lf, st1, sb1, norm_w, b, 1, row[b], pos[b]), dtype, f32=1e-4, bf16=1.2e-2)
        near(s1, st1, torch.float32, f32=1e-4)
        near(e1, sb1, torch.float32, f32=1e-4)
    status_ok(run)


@pytest.mark.parametrize("i_shift,f_shift", [(8.0, -6.0), (-8.0, 9.0), (0.0, 12.0)])
def test_gated_memory_with_extreme_gates(run, i_shift, f_shift):
    """Memories that forget at once, hardly write, or never forget: the running maximum and the normaliser's floor decide."""
    dev, dtype = run
    size = (2, 16, 24)
    L, inp, q, k, v, state, stab = memory_inputs(size, seed=6)
    T = inp.shape[0]
    z = rnd(T, 4, seed=3).double() + torch.tensor([i_shift] * 2 + [f_shift] * 2)
    gates, gb = z.float().to(dev), torch.zeros(4, device=dev)
    z = 12.0 * torch.tanh(z / 12.0)
    norm_w = torch.ones(48)
    step = PackedStep([(r, s, [0] * n) for r, s, n in PORTIONS], dev)
    s, e = state.clone().to(dev), stab.clone().to(dev)
    st, sb = state.double(), stab.double()
    got = M.gated_memory(L, inp.to(dtype).to(dev), gates, gb, 12.0, s, e, norm_w.to(dev), 1e-4, dtype, step=step)
    for t0, n, row, start in step.sequences():
        want = gated_want(L, size, inp, q, k, v, z[:, :2], -torch.log1p(torch.exp(-z[:, 2:])), st, sb, norm_w, t0, n, row, start)
        near(got[t0:t0 + n], want, dtype, f32=1e-4, bf16=2e-2)
    near(e, sb, torch.float32, f32=1e-4)


# ------------------------------------------------------------------------------------------
# whole models
# ------------------------------------------------------------------------------------------
@pytest.mark.parametrize("name", list(CONFIGS))
def test_prompt_matches_oracle(run, name):
    cfg = CONFIGS[name]
    model, w = make(cfg, run, seed=1)
    seq = tokens(61 if name != "wide" else 40, cfg["vocab"])
    hidden, got_hidden = [], []
    want = O.forward(cfg, w, seq, hidden)
    got = model.forward_step(PackedStep([(0, 0, seq)], run[0]), None, None, got_hidden)
    tol = TOL[run[1]]
    assert len(hidden) == len(got_hidden)
    for i, (a, b) in enumerate(zip(got_hidden, hidden)):
        assert float((a.double().cpu() - b).square().mean().sqrt() / b.square().mean().sqrt()) < tol, f"execution {i}"
    assert O.rel_error(got, want) < tol
    status_ok(run)


@pytest.mark.parametrize("name", ["mixed", "odd", "one"])
@pytest.mark.parametrize("cuts", [[1], [2], [3, 1, 7], [40, 1], [13, 2, 1, 1, 30], [64, 5]], ids=str)
def test_portions_and_decoding_match_the_whole_prompt(run, name, cuts):
    cfg = CONFIGS[name]
    model, w = make(cfg, run, seed=2, sharp=2.0)
    seq = tokens(75, cfg["vocab"])
    want = O.forward(cfg, w, seq)
    eng = engine(model)
    assert O.rel_error(feed(eng, eng.open(), seq, cuts), want) < TOL[run[1]] * 1.5
    status_ok(run)


def test_chunk_and_tile_borders(run):
    """Portions that end just before, on and just behind the chunks of the memories and the tiles of the attention."""
    cfg = O.config([O.par(heads=2, kv_heads=1, dim=16, vdim=16, rows=12, bias_max=200, q_temp=(0.3, 128), r_heads=1), O.mem(heads=1)], ff=(None,))
    model, w = make(cfg, run, seed=4, sharp=3.0)
    seq = tokens(300)
    want = O.forward(cfg, w, seq)
    eng = engine(model)
    for cuts in ([300], [250, 1], [126, 2, 3, 129, 1], [127, 1, 128, 44], [129, 127, 2, 42], [1, 255, 40]):
        row = eng.open()
        assert O.rel_error(feed(eng, row, seq, cuts), want) < TOL[run[1]] * 1.5, cuts
        eng.close(row)
    status_ok(run)


def test_far_keys_are_found(run):
    """A first token whose key stands out for every later query: its value has to come through over hundreds of positions and over
    every cut, whatever bucket its distance falls into."""
    cfg = O.config([O.par(heads=2, kv_heads=2, dim=16, vdim=16, rows=8, bias_max=40, r_heads=1)], ff=(None,))
    model, w = make(cfg, run, seed=5)
    w = dict(w)
    w["embed"] = w["embed"].clone()
    w["embed"][5] *= 0.2
    w["embed"][5, :4] = 12.0
    w["l0.mix.left.q.b"] = torch.full_like(w["l0.mix.left.q.b"], 1.5)
    w["l0.mix.left.k"] = w["l0.mix.left.k"].clone()
    w["l0.mix.left.k"][:, :4] += 0.8
    model.load_checkpoint(O.TensorDict(w))
    seq = [5] + [t for t in tokens(420) if t != 5][:330]
    want = O.forward(cfg, w, seq)
    other = O.forward(cfg, w, [6] + seq[1:])
    assert O.rel_error(other[100:], want[100:]) > 0.3              # the token matters
    eng = engine(model)
    for cuts in ([331], [200, 1], [7, 2, 150, 1]):
        assert O.rel_error(feed(eng, eng.open(), seq, cuts), want) < TOL[run[1]] * 1.5, cuts


def test_memories_reach_back(run):
    """With attention scaled away, what is left of early tokens comes through the recurrent state alone."""
    cfg = O.config([O.par(left_scale=1e-6, decay=[1.0, 0.999, 0.99]), O.mem()], ff=(None,), loop=(0, 2, 2))
    model, w = make(cfg, run, seed=6)
    w = {k: (v + 4 if k.endswith("mix.f.b") else v) for k, v in w.items()}
    model.load_checkpoint(O.TensorDict(w))
    seq = tokens(150)
    want = O.forward(cfg, w, seq)
    assert O.rel_error(O.forward(cfg, w, tokens(20, seed=9) + seq[20:])[100:], want[100:]) > 0.1
    eng = engine(model)
    for cuts in ([150], [20, 1], [70, 2, 1, 40]):
        assert O.rel_error(feed(eng, eng.open(), seq, cuts), want) < TOL[run[1]] * 1.5, cuts


def test_passes_of_a_loop_keep_their_own_state(run):
    """A model that runs a layer three times differs from one that has the layer three times only in the vectors added in front of
    the passes; decoded token by token the two agree when those vectors are zero."""
    loop = O.config([O.par(), O.mem()], ff=(40,), loop=(0, 2, 3))
    flat = O.config([O.par(), O.mem()] * 3, ff=(40,))
    model, w = make(loop, run, seed=7)
    w = dict(w, **{"loop.step": torch.zeros_like(w["loop.step"])})
    model.load_checkpoint(O.TensorDict(w))
    wf = {}
    for k, v in w.items():
        if k[0] == "l" and k[1].isdigit():
            wf.update({f"l{int(k[1]) + 2 * t}{k[2:]}": v for t in range(3)})
        elif k != "loop.step":
            wf[k] = v
    other = LayeredForCausalLM(LayeredConfig.from_dict(flat), run[1], run[0])
    other.load_checkpoint(O.TensorDict(wf))
    seq = tokens(40)
    a, b = (feed(e, e.open(), seq, [17, 1]) for e in (engine(model), engine(other)))
    assert float((a - b).abs().max()) <= 1e-5 * float(a.abs().max()) or run[1] == torch.bfloat16
    assert O.rel_error(a, O.forward(loop, w, seq)) < TOL[run[1]] * 1.5


def test_long_decoding(run):
    cfg = O.config([O.par(rows=10, bias_max=90, q_temp=(0.3, 50)), O.mem()], ff=(40,))
    model, w = make(cfg, run, seed=8, sharp=2.0)
    seq = tokens(330)
    want = O.forward(cfg, w, seq)
    eng = engine(model, 1, 330)
    assert O.rel_error(feed(eng, eng.open(), seq, [4, 1]), want) < TOL[run[1]] * 1.5
    with pytest.raises(ValueError):
        eng.step([(0, [1])])


def test_first_tokens(run):
    model, w = make(MIXED, run, seed=9)
    eng = engine(model)
    for t in (0, 66):
        assert O.rel_error(eng.step([(eng.open(), [t])]), O.forward(MIXED, w, [t])) < TOL[run[1]]
    seq = tokens(6)
    want = O.forward(MIXED, w, seq)
    for n in range(1, 6):
        row = eng.open()
        got = torch.cat([eng.step([(row, seq[:n])], [list(range(n))]), eng.step([(row, seq[n:])], [list(range(6 - n))])])
        assert O.rel_error(got, want) < TOL[run[1]] * 1.5


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
        assert O.rel_error(g, want[len(s) - 1:len(s) - 1 + len(g)]) < TOL[run[1]] * 1.5, i
    # mixed steps: portions of different sizes and single tokens in one batch
    eng = engine(model, rows=5)
    rows = [eng.open() for _ in seqs]
    eng.step(list(zip(rows, seqs)), [[] for _ in seqs])
    lg = eng.step([(r, m[:n]) for r, m, n in zip(rows, more, (1, 4, 2, 7, 1))])
    for i, n in enumerate((1, 4, 2, 7, 1)):
        assert O.rel_error(lg[i:i + 1], wants[i][len(seqs[i]) + n - 1:len(seqs[i]) + n]) < TOL[run[1]] * 1.5
    status_ok(run)


def test_rows_are_freed_and_used_again(run):
    """A row's keys and states of its former sequence are not seen by the next one, which may be shorter or a single token."""
    model, w = make(MIXED, run, seed=11, sharp=2.0)
    eng = engine(model, rows=2)
    for k in range(4):
        a, b = eng.open(), eng.open()
        assert {a, b} == {0, 1} and eng.cache.rows == 2
        for row, n in ((a, 70 - 22 * k), (b, 1 + 20 * k)):
            seq = tokens(n + 4, seed=k)
            assert O.rel_error(feed(eng, row, seq, [n, 1]), O.forward(MIXED, w, seq)) < TOL[run[1]] * 1.5
        eng.close(b)
        eng.close(a)
    with pytest.raises(KeyError):
        eng.close(a)


def test_greedy_generation_through_the_scheduler(run):
    from recurrent_pretraining_b200.engine import server as S

    cfg = O.config([O.par(), O.mem()], ff=(40,), loop=(0, 2, 2))
    model, w = make(cfg, run, seed=12)
    prompts = [tokens(n, seed=n) for n in (3, 12, 1, 7)]
    sched = S.BatchScheduler(S.make_backend(model, max_batch=4, max_len=64), window_ms=200.0, stop_ids=())
    try:
        reqs = [sched.submit(p, S.DecodeOptions(max_tokens=10)) for p in prompts]
        for p, r in zip(prompts, reqs):
            assert r.done.wait(120) and r.error is None, r.error
            seq = list(p)
            for t in r.tokens:                                     # every choice is (nearly) the oracle's best
                lg = O.forward(cfg, w, seq)[-1]
                slack = 1e-4 if run[1] == torch.float32 else 0.2 * float(lg.std())
                assert float(lg[t]) >= float(lg.max()) - slack
                seq.append(t)
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
    assert model.generate(prompts, 5) == [p + o[:5] for p, o in zip(prompts, plain)]
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
    assert O.rel_error(got, torch.stack([wa[0], wa[17], wb[7]])) < TOL[run[1]]
    got = torch.from_numpy(np.fromfile(tmp_path / "2.f32", dtype="<f4")).view(1, -1)
    assert O.rel_error(got, wa[19:]) < TOL[run[1]]


@gpu
@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_trace_command(tmp_path, dtype):
    """bin/trace_run on a model folder whose configuration leaves the table heights to the tensors."""
    import subprocess

    import numpy as np
    from recurrent_pretraining_b200.models.weights import save_safetensors

    w = O.random_weights(ODD, 21)
    folder, out = tmp_path / "model", tmp_path / "out"
    os.makedirs(folder)
    with open(folder / "config.json", "w") as f:
        json.dump(O.stored(ODD), f)
    save_safetensors(str(folder / "model.safetensors"), w)
    a, b = tokens(30, 61, seed=3), tokens(12, 61, seed=4)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": a[:29], "want": [0, 28]}, {"id": "y", "tokens": b[:11], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": a[29:], "want": [0]}, {"id": "y", "tokens": b[11:], "want": [0]}], "end": ["x", "y"]}]
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    r = subprocess.run([os.path.join(root, "bin", "trace_run"), "--model", str(folder), "--dtype", dtype, "--out", str(out),
                        "--max-tokens", "64"], input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    wa, wb = O.forward(ODD, w, a), O.forward(ODD, w, b)
    tol = TOL[getattr(torch, dtype)]
    got = [torch.from_numpy(np.fromfile(out / f"{n}.f32", dtype="<f4")).view(2, -1) for n in (0, 1)]
    assert O.rel_error(got[0], wa[[0, 28]]) < tol and O.rel_error(got[1], torch.stack([wa[29], wb[11]])) < tol


def test_serve_command_completes_a_prompt(tmp_path, capsys):
    import serve

    cfg = O.config([O.par(), O.mem()], ff=(40,), loop=(0, 1, 2))
    model, w = make(cfg, ("cpu", torch.float32), seed=22)
    model.save_pretrained(str(tmp_path))
    prompt = tokens(5)
    serve.main(["--model", str(tmp_path), "--cpu", "--prompt-ids", ",".join(map(str, prompt)), "--max-tokens", "6", "--max-len", "64"])
    out = json.loads(capsys.readouterr().out.strip().splitlines()[-1])
    assert out["choices"][0]["token_ids"] == O.greedy(cfg, w, prompt, 6)


@gpu
@pytest.mark.parametrize("graphs", [False, True])
def test_every_decode_step_takes_effect_once(graphs):
    """Recording a graph must not advance the recurrent state; a graph is not replayed on the storage of a cache that has grown;
    accumulators are handed back cleared."""
    run = ("cuda", torch.bfloat16)
    cfg = O.config([O.par(heads=8, kv_heads=2, dim=32, vdim=64, r_heads=3, r_dim=32, r_vdim=64), O.mem(heads=5, dim=40, vdim=64)], ff=(1024,), width=640)
    model, w = make(cfg, run, seed=15)
    eng = engine(model, rows=1, use_graphs=graphs)
    seq = tokens(40)
    want = O.forward(cfg, w, seq)
    first = eng.open()
    a = feed(eng, first, seq[:20], [3, 1])
    other = eng.open()                                             # the cache is reallocated
    assert eng.cache.rows == 2
    feed(eng, other, tokens(30, seed=5), [5, 1])
    b = feed(eng, first, seq[20:], [1])
    assert O.rel_error(torch.cat([a, b]), want) < 1.5 * TOL[torch.bfloat16]
    torch.cuda.synchronize()
    assert not any(bool(t.any()) for t in eng._work)
    status_ok(run)


@gpu
def test_large_batches_decode_in_groups():
    run = ("cuda", torch.bfloat16)
    model, w = make(MIXED, run, seed=16)
    eng = engine(model, rows=70)
    seqs = [tokens(3 + i % 9, seed=i) for i in range(70)]
    rows = [eng.open() for _ in seqs]
    eng.step([(r, s[:-1]) for r, s in zip(rows, seqs)], [[] for _ in seqs])
    lg = eng.step([(r, s[-1:]) for r, s in zip(rows, seqs)])
    for i in range(0, 70, 9):
        assert O.rel_error(lg[i:i + 1], O.forward(MIXED, w, seqs[i])[-1:]) < 1.5 * TOL[torch.bfloat16]
