"""Layered decoder models (latent attention, sliding window): every mechanism and the serving path against the plain
statements of ``layered_oracle``, on the CPU (fp32) and on the GPU kernels (fp32 and bf16)."""
import io
import json
import math
import os

import pytest
import torch

import layered_oracle as O
from recurrent_pretraining_b200.models import build_model
from recurrent_pretraining_b200.models.layered import LayeredForCausalLM, PackedStep
from recurrent_pretraining_b200.models.layered_config import LayeredConfig, RotarySpec
from recurrent_pretraining_b200.ops import latent as ops
from recurrent_pretraining_b200.ops.latent import LatentLayout

gpu = pytest.mark.gpu
RUNS = [pytest.param(("cpu", torch.float32), id="cpu"), pytest.param(("cuda", torch.float32), marks=gpu, id="gpu-f32"),
        pytest.param(("cuda", torch.bfloat16), marks=gpu, id="gpu-bf16")]
GPU_RUNS = RUNS[1:]
TOL = {torch.float32: 2e-5, torch.bfloat16: 6e-2}     # rms of the logit error over the rms of the logits


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
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(1000 + seed + 7919 * n)).tolist()


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


# layers that differ in every size, share latents under narrower and wider windows, and leave the feed-forward out
MIXED = O.config([O.mixer(), O.mixer(heads=3, dim=24, rot_dim=8, vdim=16, kv_rank=32, window=5, kv_from=0),
                  O.mixer(heads=1, dim=8, rot_dim=16, vdim=40, kv_rank=56, window=19, scaling=None),
                  O.mixer(heads=5, dim=16, rot_dim=8, vdim=8, kv_rank=32, window=29, kv_from=0),
                  O.mixer(heads=2, dim=40, rot_dim=16, vdim=72, kv_rank=56, window=8, scaling=None, kv_from=2)], ff=(40, None, 88))
# nothing is a multiple of eight
ODD = O.config([O.mixer(heads=3, dim=11, rot_dim=6, vdim=13, kv_rank=27, window=9, base=90.0),
                O.mixer(heads=2, dim=5, rot_dim=6, vdim=21, kv_rank=27, window=14, base=90.0, kv_from=0)],
               ff=(37,), width=45, vocab=61, mult=1.0, eps=1e-3)
ONE = O.config([O.mixer(heads=1, dim=8, rot_dim=8, vdim=8, kv_rank=8, window=1)], ff=(8,), width=16, vocab=19)
WIDE = O.config([O.mixer(heads=20, dim=64, rot_dim=32, vdim=128, kv_rank=136, window=150),
                 O.mixer(heads=20, dim=72, rot_dim=32, vdim=64, kv_rank=136, window=70, kv_from=0)], ff=(600,), width=520)
CONFIGS = {"mixed": MIXED, "odd": ODD, "one": ONE, "wide": WIDE}


# ------------------------------------------------------------------------------------------
# configuration, weights, loading
# ------------------------------------------------------------------------------------------
def test_config_round_trip_and_dispatch(tmp_path):
    cfg = LayeredConfig.from_dict(MIXED)
    assert cfg.to_dict() == MIXED
    cfg.save(str(tmp_path))
    assert LayeredConfig.from_pretrained(str(tmp_path)).to_dict() == MIXED
    model = build_model(cfg, dtype=torch.float32)
    assert isinstance(model, LayeredForCausalLM)
    want = O.shapes(MIXED)
    assert {k: tuple(v.shape) for k, v in model.checkpoint_tensors().items()} == want
    assert cfg.param_count() == sum(math.prod(s) for s in want.values())
    assert cfg.latent_windows() == {0: 29, 2: 19} and [cfg.kv_source(i) for i in range(5)] == [0, 0, 2, 0, 2]


@pytest.mark.parametrize("change", [
    lambda c: c.update(architecture="Unknown"), lambda c: c.update(extra=1), lambda c: c["layers"][0].update(type="other"),
    lambda c: c["layers"][0]["mixer"].update(sinks=2), lambda c: c["layers"][0]["mixer"].update(kv_from=3),
    lambda c: c["layers"][1]["mixer"].update(kv_from=1), lambda c: c["layers"][1]["mixer"].update(kv_rank=24),
    lambda c: c["layers"][3]["mixer"].update(kv_from=1), lambda c: c["layers"][0]["mixer"]["rot"].update(dims=4),
    lambda c: c["layers"][0]["mlp"].update(kind="gated"), lambda c: c["layers"][0]["mixer"]["mask"].update(size=0)])
def test_invalid_configs_are_refused(change):
    cfg = json.loads(json.dumps(MIXED))
    change(cfg)
    with pytest.raises((ValueError, KeyError)):
        LayeredConfig.from_dict(cfg)


@pytest.mark.parametrize("scaling", [None, {"factor": 4.0, "original": 64, "fast": 32.0, "slow": 1.0},
                                     {"factor": 2.0, "original": 4, "fast": 2.0, "slow": 1.0},          # lo clamps at 0
                                     {"factor": 8.0, "original": 10 ** 9, "fast": 4.0, "slow": 1e-9},   # hi clamps at dims - 1
                                     {"factor": 1.0, "original": 4096, "fast": 32.0, "slow": 1.0},
                                     {"factor": 3.0, "original": 628, "fast": 5.0, "slow": 5.0}])
@pytest.mark.parametrize("dims,base", [(2, 10.0), (8, 500.0), (64, 10000.0)])
def test_rotation_frequencies(scaling, dims, base):
    rot = {"base": base, "dims": dims}
    if scaling:
        rot["scaling"] = scaling
    want, mag = O.yarn_frequencies(rot)
    spec = RotarySpec.from_dict(rot)
    assert spec.frequencies() == pytest.approx(want, rel=1e-12) and spec.magnitude == pytest.approx(mag, rel=1e-12)


def test_checkpoint_files_and_loader_choice(tmp_path):
    from recurrent_pretraining_b200.models import auto
    from recurrent_pretraining_b200.models.weights import SafetensorsFile, save_safetensors

    w = O.random_weights(MIXED, 3)
    LayeredConfig.from_dict(MIXED).save(str(tmp_path))
    path = os.path.join(str(tmp_path), "model.safetensors")
    save_safetensors(path, w)
    f = SafetensorsFile(path)
    assert all(torch.equal(f.tensor(k), v) for k, v in w.items()) and set(f.keys()) == set(w)
    model = auto.load_pretrained(str(tmp_path), torch.float32, torch.device("cpu"))
    assert isinstance(model, LayeredForCausalLM)
    assert all(torch.equal(v, w[k].float()) for k, v in model.checkpoint_tensors().items())
    again = tmp_path / "again"
    model.save_pretrained(str(again))
    assert all(torch.equal(SafetensorsFile(str(again / "model.safetensors")).tensor(k), v) for k, v in w.items())
    for bad in ({**w, "l9.norm1": w["l0.norm1"]}, {k: v for k, v in w.items() if k != "l2.mix.dkv"},
                {**w, "l1.mix.uk": w["l1.mix.uk"][:-1]}):
        with pytest.raises(ValueError):
            model.load_checkpoint(O.TensorDict(bad))
    with open(path, "r+b") as fh:
        fh.truncate(os.path.getsize(path) - 2)
    with pytest.raises(ValueError):
        SafetensorsFile(path)


def test_registry_shapes_build():
    from recurrent_pretraining_b200 import registry

    for name in registry.layered_configs:
        cfg = LayeredConfig.from_name(name)
        assert cfg.name == name and cfg.param_count() > 0
    tiny = build_model(LayeredConfig.from_name("gasovik-tiny"), dtype=torch.float32).init_weights(1)
    assert tiny(torch.tensor([[1, 2, 3], [4, 5, 6]])).shape == (2, 3, 512)


# ------------------------------------------------------------------------------------------
# mechanisms alone
# ------------------------------------------------------------------------------------------
def close(got, want, dtype, scale=1.0):
    err = float((got.double().cpu() - want).abs().max())
    assert err <= (3e-6 if dtype == torch.float32 else 1.2e-2) * scale * (1 + float(want.abs().max())), err


def rnd(*shape, seed=0, scale=1.0):
    """Values that bf16 represents exactly."""
    return (torch.randn(*shape, generator=torch.Generator().manual_seed(seed)) * scale).bfloat16()


@pytest.mark.parametrize("E", [45, 48, 2056, 9000])
def test_embedding_and_residual_norm(run, E):
    dev, dtype = run
    table, ids = rnd(23, E, seed=1), torch.tensor([5, 0, 22, 5])
    t = torch.zeros(23, ops.pad8(E), dtype=dtype, device=dev)
    t[:, :E] = table
    x, xb = ops.embed(ids.to(dev), t[:, :E])
    assert x.dtype == torch.float32 and torch.equal(x.cpu(), table[ids].float()) and torch.equal(xb.float().cpu(), x.cpu())
    a, bias, w = rnd(4, E, seed=2), torch.randn(E), torch.rand(E) + 0.5
    want = x.cpu().double() + 0.7 * O.rms_norm(a.double() + bias.double(), 1e-4, w.double())
    acc = torch.zeros(4, ops.pad8(E), device=dev)[:, :E]            # the fp32 accumulator of a weight-streaming product
    for src, clear in ((a.to(dev).to(dtype), False), (acc, True)):
        src.copy_(a)
        y = x.clone()
        extra = torch.ones(4, 12, device=dev)
        yb = ops.rms_residual_(y, src, bias.to(dev), w.to(dev), 1e-4, 0.7, dtype, clear and dev == "cuda",
                               extra if dev == "cuda" else None)
        close(y, want, torch.float32)
        close(yb, want, dtype)
        if dev == "cuda":
            assert not extra.any() and (not clear or not src.any())
    idx = torch.tensor([3, 1, 3], dtype=torch.int32)
    close(ops.rmsnorm_rows(x, idx.to(dev), w.to(dev), 1e-5, dtype), O.rms_norm(x.cpu().double()[[3, 1, 3]], 1e-5, w.double()), dtype)


@pytest.mark.parametrize("M,N,Kd", [(1, 40, 48), (7, 37, 45), (130, 264, 100), (300, 600, 520), (513, 250, 72)])
def test_products_with_bias_and_activation(run, M, N, Kd):
    dev, dtype = run
    x, w, bias = rnd(M, Kd, seed=3), rnd(N, Kd, seed=4, scale=Kd ** -0.5), torch.randn(N)
    pitch = lambda t: torch.nn.functional.pad(t, (0, ops.pad8(Kd) - Kd)).to(dtype).to(dev)[:, :Kd]  # noqa: E731
    z = x.double() @ w.double().T
    xs, ws = pitch(x), pitch(w)
    close(ops.linear(xs, ws), z, dtype)
    f = ops.linear(xs, ws, out_f32=True)
    assert f.dtype == torch.float32
    close(f, z, torch.float32, 3.0)
    h = z + bias.double()
    close(ops.linear(xs, ws, bias.to(dev)), h, dtype)
    h = torch.where(h > 0, h * h, torch.zeros_like(h))
    close(ops.linear(xs, ws, bias.to(dev), "relu2"), h, dtype)
    close(ops.bias_act(f, bias.to(dev), "relu2", dtype), h, dtype)


class _Step:
    def __init__(self, pos, row, end, dev):
        self.pos, self.row, self.end = (torch.tensor(t, dtype=torch.int32, device=dev) for t in (pos, row, end))


@pytest.mark.parametrize("size", [(2, 16, 8, 24, 32), (3, 11, 6, 13, 27), (5, 64, 32, 8, 200)])
def test_latent_rows_and_rotation(run, size):
    dev, dtype = run
    H, dim, rot_dim, vdim, rank = size
    L = LatentLayout(H, dim, rot_dim, vdim, rank, True)
    rot = O.mixer(rot_dim=rot_dim)["rot"]
    pos, row, end = [130, 131, 0, 257, 258], [2, 2, 0, 1, 1], [132, 132, 1, 387, 387]
    inp = rnd(5, L.width_in, seed=5)
    w = torch.rand(rank) + 0.5
    from recurrent_pretraining_b200.models.layered import rope_tables

    tables = rope_tables(RotarySpec.from_dict(rot), 400, dev)
    cache = torch.full((3, 128, L.ld_lat), 7.0, dtype=dtype, device=dev)
    stream = torch.full((9, L.ld_lat), 7.0, dtype=dtype, device=dev)
    sidx = [3, 4, 0, 7, 8]
    got = inp.to(dtype).to(dev)
    ops.latent_prep_(L, got, w.to(dev), 1e-4, tables, _Step(pos, row, end, dev), torch.tensor(sidx, dtype=torch.int32, device=dev), cache, stream)
    hd = dim + rot_dim
    for t, p in enumerate(pos):
        q = inp[t, :H * hd].double().view(H, hd)
        want = torch.cat([q[:, :dim], O.rotate(q[:, dim:], p, rot)], 1)
        close(got[t, :H * hd], want.flatten(), dtype)
        d = inp[t, L.off_d:].double()
        lat = torch.zeros(L.ld_lat, dtype=torch.float64)
        lat[:rank] = O.rms_norm(d[:rank], 1e-4, w.double())
        lat[L.rank_pad:L.rank_pad + rot_dim] = O.rotate(d[rank:rank + rot_dim], p, rot)
        close(stream[sidx[t]], lat, dtype)
        if p >= end[t] - 128:                       # only the newest slots' worth of a portion reaches the ring
            close(cache[row[t], p % 128], lat, dtype)
    assert torch.equal(got[:, H * hd:].float().cpu(), inp[:, H * hd:].float())          # gate and latent columns untouched
    assert bool((stream[[1, 2, 5, 6]] == 7).all()) and bool((cache[1, 257 % 128] == 7).all()) and bool((cache[0, 1:] == 7).all())


def _attention_case(L, T, window, portions, needles, seed):
    """Random projection rows, keys and values of a packed stream, with needle keys that every query that sees them rests on."""
    K = max(k0 + h + n for _, n, k0, h in portions)
    inp, kv, stream = rnd(T, L.width_in, seed=seed), rnd(K, L.width_kv, seed=seed + 1), rnd(K, L.ld_lat, seed=seed + 2)
    hd = L.dim + L.rot
    u = torch.ones(L.heads, L.dim)
    inp[:, :L.heads * hd].view(T, L.heads, hd)[..., :L.dim] = (0.1 * torch.randn(T, L.heads, L.dim) + u).bfloat16()
    k = kv[:, :L.heads * L.dim].view(K, L.heads, L.dim)
    v = kv[:, L.off_v:L.off_v + L.heads * L.vdim].view(K, L.heads, L.vdim)
    for j in needles:
        k[j] = 2.5
        v[j] = 40.0 + j % 7
    return inp, kv, stream


def _attention_want(L, inp, kv, stream, seqs, window, scale, hd):
    T = inp.shape[0]
    q = inp[:, :L.heads * hd].double().view(T, L.heads, hd)
    k = kv[:, :L.heads * L.dim].double().view(-1, L.heads, L.dim)
    v = kv[:, L.off_v:L.off_v + L.heads * L.vdim].double().view(-1, L.heads, L.vdim)
    kr = stream[:, L.rank_pad:L.rank_pad + L.rot].double()
    out = torch.zeros(T, L.heads, L.vdim, dtype=torch.float64)
    for t0, n, k0, h in seqs:
        for i in range(n):
            at = h + i
            keys = [k0 + j for j in O.visible_keys(at, window)]
            for g in range(L.heads):
                s = (k[keys, g] @ q[t0 + i, g, :L.dim] + kr[keys] @ q[t0 + i, g, L.dim:]) * scale
                out[t0 + i, g] = O.attend(s, v[keys, g])
    g = inp[:, L.off_g:L.off_g + L.heads * L.vdim].double()
    return out.flatten(1) / (1 + torch.exp(-g))


ATT_SIZES = [(2, 16, 8, 24, 16), (1, 128, 64, 128, 64), (2, 96, 32, 96, 40), (1, 64, 64, 64, 32), (2, 72, 16, 160, 24),
             (1, 192, 64, 128, 16), (3, 11, 6, 13, 27), (1, 8, 8, 256, 16), (1, 200, 64, 200, 16)]


@pytest.mark.parametrize("size", ATT_SIZES, ids=lambda s: "x".join(map(str, s)))
@pytest.mark.parametrize("window", [1, 40, 128, 193, 5000])
def test_stream_attention(run, size, window):
    """Queries of several sequences (fresh, with history, one token) over one key stream; needles lie just inside and just
    outside the windows of queries at tile borders."""
    dev, dtype = run
    if dev == "cpu" and (size not in ATT_SIZES[:1] or window not in (40, 193)):
        pytest.skip("one size on the CPU")
    H, dim, rot, vdim, rank = size
    L = LatentLayout(H, dim, rot, vdim, rank, True)
    seqs, t0, k0 = [], 0, 0
    for n, h in ((300, 0), (1, 0), (70, min(window - 1, 90)), (129, min(window - 1, 500))):
        seqs.append((t0, n, k0, h))
        t0, k0 = t0 + n, k0 + h + n
    needles = {0, 63, 64, 127, 128, 255, 256, max(0, 255 - window), max(0, 256 - window), max(0, 257 - window)}
    needles = sorted(j for j in needles if j < 300) + [seqs[2][2], seqs[3][2] + seqs[3][3]]
    inp, kv, stream = _attention_case(L, t0, window, seqs, needles, seed=size[1] + window)
    scale = 1.0 / dim
    want = _attention_want(L, inp, kv, stream, seqs, window, scale, dim + rot)

    class Layout:
        pass

    lay = Layout()
    lay.seqs = seqs
    put = lambda t: t.to(dtype).to(dev)  # noqa: E731
    lay.sidx = torch.tensor([k + h + i for _, n, k, h in seqs for i in range(n)], dtype=torch.int32, device=dev)
    lay.kbase = torch.tensor([k for _, n, k, h in seqs for _ in range(n)], dtype=torch.int32, device=dev)
    got = ops.stream_attention(L, put(inp), put(kv), put(stream), lay, window, scale)
    assert torch.isfinite(got).all()
    d = got.double().cpu() - want
    assert float(d.abs().max()) < (2e-4 if dtype == torch.float32 else 0.35), float(d.abs().max())     # values reach 46
    assert float(d.square().mean().sqrt()) < (2e-5 if dtype == torch.float32 else 0.06)
    status_ok(run)


DEC_SIZES = [(2, 16, 8, 24, 32), (16, 128, 64, 128, 512), (55, 24, 32, 16, 136), (20, 40, 16, 72, 200), (3, 11, 6, 13, 27),
             (70, 16, 8, 8, 64), (33, 8, 16, 8, 900)]


@pytest.mark.parametrize("size", DEC_SIZES, ids=lambda s: "x".join(map(str, s)))
@pytest.mark.parametrize("window,cap,splits", [(1, 128, 1), (40, 128, 1), (128, 128, 2), (130, 256, 3), (300, 384, 2), (384, 384, 5)])
def test_ring_attention(run, size, window, cap, splits):
    """One token per sequence against ring caches at different fill levels and wrap positions; a needle sits on the oldest
    visible key of every sequence and a larger one on the key just outside."""
    dev, dtype = run
    if dev == "cpu" and (size not in DEC_SIZES[:1] or splits > 3):
        pytest.skip("one size on the CPU")
    H, dim, rot_dim, vdim, rank = size
    L = LatentLayout(H, dim, rot_dim, vdim, rank, True)
    rot = O.mixer(rot_dim=rot_dim)["rot"]
    from recurrent_pretraining_b200.models.layered import rope_tables

    tables = rope_tables(RotarySpec.from_dict(rot), 2000, dev)
    pos = [0, 5, window - 1, window, 127, 128, cap - 1, cap, cap + 130, 3 * cap + 77]
    row = [4, 0, 11, 2, 3, 8, 6, 7, 1, 9]
    B = len(pos)
    inp = rnd(B, L.width_in, seed=9)
    inp[:, L.off_d:] = 0.3 * inp[:, L.off_d:]
    w_kv = torch.zeros(L.width_kv, ops.pad8(rank), dtype=torch.bfloat16)
    w_kv[:H * dim, :rank] = rnd(H * dim, rank, seed=10, scale=rank ** -0.5)
    w_kv[L.off_v:L.off_v + H * vdim, :rank] = rnd(H * vdim, rank, seed=11, scale=rank ** -0.5)
    nw = torch.ones(rank)
    cache = rnd(12, cap, L.ld_lat, seed=12)
    cache[..., rank:L.rank_pad] = 0
    cache[..., L.rank_pad + rot_dim:] = 0
    hd, scale = dim + rot_dim, dim ** -0.5
    q = inp[:, :H * hd].double().view(B, H, hd)
    for b, (p, r) in enumerate(zip(pos, row)):      # the oldest visible key and the one before it stand out for head 0
        need = (w_kv[:dim, :rank].double().T @ q[b, 0, :dim]).float()
        need = need / need.norm() * rank ** 0.5
        if window > 1 and p >= window - 1:
            cache[r, (p - window + 1) % cap, :rank] = (2 * need).bfloat16()
        if p >= window and cap > window:
            cache[r, (p - window) % cap, :rank] = (4 * need).bfloat16()
    want = torch.zeros(B, H, vdim, dtype=torch.float64)
    for b, (p, r) in enumerate(zip(pos, row)):
        d = inp[b, L.off_d:].double()
        own = torch.zeros(L.ld_lat, dtype=torch.float64)
        own[:rank] = O.rms_norm(d[:rank], 1e-4)
        own[L.rank_pad:L.rank_pad + rot_dim] = O.rotate(d[rank:rank + rot_dim], p, rot)
        keys = torch.stack([own if j == p else cache[r, j % cap].double() for j in O.visible_keys(p, window)])
        c, kr = keys[:, :rank], keys[:, L.rank_pad:L.rank_pad + rot_dim]
        for g in range(H):
            k = c @ w_kv[g * dim:(g + 1) * dim, :rank].double().T
            s = (k @ q[b, g, :dim] + kr @ O.rotate(q[b, g, dim:], p, rot)) * scale
            want[b, g] = O.attend(s, c @ w_kv[L.off_v + g * vdim:L.off_v + (g + 1) * vdim, :rank].double().T)
    want = want.flatten(1) / (1 + torch.exp(-inp[:, L.off_g:L.off_g + H * vdim].double()))
    put = lambda t: t.to(dtype).to(dev)  # noqa: E731
    ip, ir = (torch.tensor(t, dtype=torch.int32, device=dev) for t in (pos, row))
    for src in ([inp.to(dev).float()] if dev == "cuda" and dtype == torch.bfloat16 else []) + [put(inp)]:
        got = ops.ring_attention(L, src, put(w_kv), nw.to(dev), 1e-4, tables, ip, ir, put(cache), window, scale, splits, dtype)
        d = got.double().cpu() - want
        err, rms = float(d.abs().max()), float(want.square().mean().sqrt())
        assert torch.isfinite(got).all() and err < (1e-4 if dtype == torch.float32 else 0.08) * (1 + rms), (err, rms)
    status_ok(run)


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
    for i, (a, b) in enumerate(zip(got_hidden, hidden)):
        assert float((a.double().cpu() - b).square().mean().sqrt() / b.square().mean().sqrt()) < tol, f"layer {i}"
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


@pytest.mark.parametrize("window", [127, 128, 129])
def test_windows_at_ring_borders(run, window):
    """Ring capacity, window edge and tile edge fall together; prompts, portions and decoding cross the border."""
    cfg = O.config([O.mixer(window=window, heads=2), O.mixer(window=window - 90, kv_from=0)], ff=(None,))
    model, w = make(cfg, run, seed=4, sharp=3.0)
    seq = tokens(300)
    want = O.forward(cfg, w, seq)
    eng = engine(model)
    tol = TOL[run[1]] * 1.5
    for cuts in ([300], [250, 1], [126, 2, 3, 129, 1], [1, 255, 40]):
        row = eng.open()
        assert O.rel_error(feed(eng, row, seq, cuts), want) < tol, cuts
        eng.close(row)
    status_ok(run)


def test_long_decoding_wraps_the_ring(run):
    cfg = O.config([O.mixer(window=100), O.mixer(window=60, kv_from=0)], ff=(40,))
    model, w = make(cfg, run, seed=5, sharp=2.0)
    seq = tokens(330)
    want = O.forward(cfg, w, seq)
    eng = engine(model, 1, 330)
    assert eng.cache.caps == {0: 128}
    assert O.rel_error(feed(eng, eng.open(), seq, [4, 1]), want) < TOL[run[1]] * 1.5


def test_reader_with_the_wider_window(run):
    """The cache of a layer keeps what the widest window among its readers still needs."""
    cfg = O.config([O.mixer(window=3), O.mixer(window=140, kv_from=0)], ff=(None,))
    model, w = make(cfg, run, seed=6, sharp=2.5)
    seq = tokens(200)
    want = O.forward(cfg, w, seq)
    eng = engine(model)
    for cuts in ([200], [150, 1], [60, 2, 90, 1]):
        assert O.rel_error(feed(eng, eng.open(), seq, cuts), want) < TOL[run[1]] * 1.5, cuts


def test_first_tokens(run):
    """One-token prompts, and the first positions of a prompt, against the oracle."""
    model, w = make(MIXED, run, seed=7)
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
    model, w = make(MIXED, run, seed=8, sharp=2.0)
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
    model, w = make(MIXED, run, seed=9, sharp=2.0)
    eng = engine(model, rows=2)
    for k in range(4):
        a, b = eng.open(), eng.open()
        assert {a, b} == {0, 1} and eng.cache.rows == 2
        for row, n in ((a, 70 - 9 * k), (b, 3 + 20 * k)):
            seq = tokens(n + 4, seed=k)
            assert O.rel_error(feed(eng, row, seq, [n, 1]), O.forward(MIXED, w, seq)) < TOL[run[1]] * 1.5
        eng.close(b)
        eng.close(a)
    with pytest.raises(KeyError):
        eng.close(a)
    row = eng.open()
    with pytest.raises(ValueError):
        eng.step([(row, tokens(401))])
    with pytest.raises(ValueError):
        eng.step([(row, [67])])


def test_greedy_generation_through_the_scheduler(run):
    from recurrent_pretraining_b200.engine import server as S

    cfg = O.config([O.mixer(window=6), O.mixer(window=9, kv_from=0)], ff=(40,))
    model, w = make(cfg, run, seed=10)
    prompts = [tokens(n, seed=n) for n in (3, 12, 1, 7)]
    sched = S.BatchScheduler(S.make_backend(model, max_batch=4, max_len=64), window_ms=200.0, stop_ids=())
    try:
        reqs = [sched.submit(p, S.DecodeOptions(max_tokens=10)) for p in prompts]
        for p, r in zip(prompts, reqs):
            assert r.done.wait(120) and r.error is None, r.error
            seq = list(p)
            for t in r.tokens:                                     # every choice is (nearly) the oracle's best
                lg = O.forward(cfg, w, seq)[-1]
                slack = 0 if run[1] == torch.float32 else 0.15 * float(lg.std())
                assert float(lg[t]) >= float(lg.max()) - slack
                seq.append(t)
            if run[1] == torch.float32:
                assert r.tokens == O.greedy(cfg, w, p, 10)
        assert sched.stats["batches"] < 4                          # unequal prompts share a batch
        out = S.handle_completion(sched, {"prompt": prompts[1], "max_tokens": 10, "do_sample": True, "top_k": 1})
        assert out["choices"][0]["token_ids"] == reqs[1].tokens     # sampling from the single best token
        with pytest.raises(RuntimeError):
            S.handle_completion(sched, {"prompt": prompts[1], "num_steps": 4})
    finally:
        sched.close()


def test_generation_stops_and_sampling_options(run):
    model, w = make(MIXED, run, seed=11)
    eng = engine(model)
    prompts = [tokens(9), tokens(4)]
    plain = eng.generate(prompts, 20)
    stop = plain[0][5]
    cut = eng.generate(prompts, 20, stop_ids=[stop], check_every=2)
    for p, c in zip(plain, cut):
        end = p.index(stop) + 1 if stop in p else len(p)
        assert c == p[:end]
    assert model.generate(torch.tensor([prompts[0]], device=run[0]), 5)[0].tolist() == prompts[0] + plain[0][:5]
    assert model.generate(prompts, 5) == [p + o[:5] for p, o in zip(prompts, plain)]
    small = engine(model, prefill_tokens=5)                        # prompts in portions, several sequences per step
    assert small.generate(prompts, 6) == [p[:6] for p in plain] or run[1] == torch.bfloat16
    torch.manual_seed(0)
    sampled = eng.generate(prompts, 20, do_sample=True, temperature=1.5, top_p=0.9)
    assert sampled != plain and all(0 <= t < 67 for s in sampled for t in s)
    rep = eng.generate(prompts, 20, repetition_penalty=1e9)
    assert all(len(set(p + r)) == len(p + r) - (len(p) - len(set(p))) for p, r in zip(prompts, rep))
    assert not eng.cache.length                                    # every row went back


def test_trace_replay(run, tmp_path):
    from recurrent_pretraining_b200.engine.trace import replay

    import numpy as np

    model, w = make(MIXED, run, seed=12)
    a, b = tokens(20, seed=1), tokens(9, seed=2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:18], "want": [0, 17]}, {"id": "b", "tokens": b[:8], "want": [7]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[18:19], "want": []}, {"id": "b", "tokens": b[8:], "want": []}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": a[19:], "want": [0]}], "end": ["a"]}]
    answer = io.StringIO()
    eng = engine(model, 1, 64)
    replay(eng, [json.dumps(s) + "\n" for s in steps] + ["\n"], str(tmp_path), answer)
    assert answer.getvalue() == "done 0\ndone 1\ndone 2\n" and not eng.cache.length
    assert sorted(os.listdir(tmp_path)) == ["0.f32", "2.f32"]
    wa, wb = O.forward(MIXED, w, a), O.forward(MIXED, w, b)
    got = torch.from_numpy(np.fromfile(tmp_path / "0.f32", dtype="<f4")).view(3, -1)
    assert O.rel_error(got, torch.stack([wa[0], wa[17], wb[7]])) < TOL[run[1]]
    got = torch.from_numpy(np.fromfile(tmp_path / "2.f32", dtype="<f4")).view(1, -1)
    assert O.rel_error(got, wa[19:]) < TOL[run[1]]


@gpu
@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_trace_command(tmp_path, dtype):
    """bin/trace_run on a model folder: steps in, one answer per step, logits in the output folder."""
    import subprocess

    import numpy as np
    from recurrent_pretraining_b200.models.weights import save_safetensors

    w = O.random_weights(ODD, 21)
    folder, out = tmp_path / "model", tmp_path / "out"
    LayeredConfig.from_dict(ODD).save(str(folder))
    save_safetensors(str(folder / "model.safetensors"), w)
    a, b = tokens(30, 61, seed=3), tokens(12, 61, seed=4)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": a[:29], "want": [0, 28]}, {"id": "y", "tokens": b[:11], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": a[29:], "want": [0]}, {"id": "y", "tokens": b[11:], "want": [0]}], "end": ["x", "y"]}]
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    r = subprocess.run([os.path.join(root, "bin", "trace_run"), "--model", str(folder), "--dtype", dtype, "--out", str(out),
                        "--max-tokens", "64"], input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [x for x in r.stdout.splitlines() if x.startswith("done")] == ["done 0", "done 1"]
    wa, wb = O.forward(ODD, w, a), O.forward(ODD, w, b)
    tol = TOL[getattr(torch, dtype)]
    got = [torch.from_numpy(np.fromfile(out / f"{n}.f32", dtype="<f4")).view(2, -1) for n in (0, 1)]
    assert O.rel_error(got[0], wa[[0, 28]]) < tol and O.rel_error(got[1], torch.stack([wa[29], wb[11]])) < tol


def test_serve_command_completes_a_prompt(tmp_path, capsys):
    import serve

    cfg = O.config([O.mixer(window=6)], ff=(40,))
    model, w = make(cfg, ("cpu", torch.float32), seed=22)
    model.save_pretrained(str(tmp_path))
    prompt = tokens(5)
    serve.main(["--model", str(tmp_path), "--cpu", "--prompt-ids", ",".join(map(str, prompt)), "--max-tokens", "6", "--max-len", "64"])
    out = json.loads(capsys.readouterr().out.strip().splitlines()[-1])
    assert out["choices"][0]["token_ids"] == O.greedy(cfg, w, prompt, 6)


@gpu
def test_graphs_follow_a_cache_that_moves():
    """A captured decode step is not replayed on the storage of a cache that has grown."""
    run = ("cuda", torch.bfloat16)
    model, w = make(MIXED, run, seed=13)
    eng = engine(model, rows=1)
    seq = tokens(40)
    want = O.forward(MIXED, w, seq)
    first = eng.open()
    feed(eng, first, seq[:20], [10, 1])
    other = eng.open()                                             # the cache is reallocated
    assert eng.cache.rows == 2
    feed(eng, other, tokens(30, seed=5), [5, 1])
    assert O.rel_error(feed(eng, first, seq[20:], [1]), want[20:]) < 2 * TOL[torch.bfloat16]
    status_ok(run)


@gpu
def test_large_batches_decode_in_groups():
    run = ("cuda", torch.bfloat16)
    model, w = make(MIXED, run, seed=14)
    eng = engine(model, rows=70)
    seqs = [tokens(3 + i % 9, seed=i) for i in range(70)]
    rows = [eng.open() for _ in seqs]
    eng.step([(r, s[:-1]) for r, s in zip(rows, seqs)], [[] for _ in seqs])
    lg = eng.step([(r, s[-1:]) for r, s in zip(rows, seqs)])
    for i in range(0, 70, 9):
        assert O.rel_error(lg[i:i + 1], O.forward(MIXED, w, seqs[i])[-1:]) < 1.5 * TOL[torch.bfloat16]


@gpu
def test_accumulators_are_handed_back_cleared():
    run = ("cuda", torch.bfloat16)
    cfg = O.config([O.mixer(heads=8, dim=32, rot_dim=16, vdim=64, kv_rank=64)], ff=(1024,), width=640)
    model, w = make(cfg, run, seed=15)
    for graphs in (False, True):
        eng = engine(model, use_graphs=graphs)
        seq = tokens(24)
        assert O.rel_error(feed(eng, eng.open(), seq, [3, 1]), O.forward(cfg, w, seq)) < 1.5 * TOL[torch.bfloat16]
        torch.cuda.synchronize()
        assert not any(bool(t.any()) for t in eng._work)
