"""Plain, slow statements of the layered decoder's mechanisms in double precision, one function each, and small random
models to compare the framework with.  Nothing here comes from the package: a model is a configuration dict and a dict of
named tensors."""
import math

import torch

D = torch.float64


def rms_norm(x, eps, w=None):
    y = x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)
    return y if w is None else y * w


def yarn_frequencies(rot):
    """Per pair (2 i, 2 i + 1): radians per position, and the factor on cos and sin."""
    n, base, sc = rot["dims"], rot["base"], rot.get("scaling")
    freqs = []
    for i in range(n // 2):
        f = base ** (-2.0 * i / n)
        if sc is not None:
            edge = [n * math.log(sc["original"] / (2 * math.pi * t)) / (2 * math.log(base)) for t in (sc["fast"], sc["slow"])]
            lo, hi = max(math.floor(edge[0]), 0), min(math.ceil(edge[1]), n - 1)
            ramp = (i - lo) / max(hi - lo, 0.001)
            ramp = 0.0 if ramp < 0 else 1.0 if ramp > 1 else ramp
            f = f / sc["factor"] * ramp + f * (1 - ramp)
        freqs.append(f)
    return freqs, 1.0 if sc is None else 0.1 * math.log(sc["factor"]) + 1.0


def rotate(vec, position, rot):
    """One vector (or a stack of vectors of one position): interleaved pairs turned by position * frequency."""
    freqs, mag = yarn_frequencies(rot)
    out = vec.clone()
    for i, f in enumerate(freqs):
        c, s = math.cos(position * f) * mag, math.sin(position * f) * mag
        out[..., 2 * i] = vec[..., 2 * i] * c - vec[..., 2 * i + 1] * s
        out[..., 2 * i + 1] = vec[..., 2 * i + 1] * c + vec[..., 2 * i] * s
    return out


def latents(h, w, name, a, eps):
    """Normed latent c [T, rank] and rotated shared key part [T, rot_dim] of a layer."""
    d = h @ w[name + "dkv"].T
    c = rms_norm(d[:, :a["kv_rank"]], eps, w[name + "dkv.norm"])
    kr = torch.stack([rotate(d[t, a["kv_rank"]:], t, a["rot"]) for t in range(len(d))])
    return c, kr


def visible_keys(i, window):
    return range(max(0, i - window + 1), i + 1)


def attend(scores, values):
    """softmax(scores) . values for one query of one head."""
    e = torch.exp(scores - scores.max())
    return (e / e.sum()) @ values


def latent_attention(h, c, kr, w, name, a):
    """Concatenated heads [T, heads * vdim] before the gate."""
    T, H = len(h), a["heads"]
    q = (h @ w[name + "q"].T).view(T, H, a["dim"] + a["rot_dim"])
    k = (c @ w[name + "uk"].T).view(T, H, a["dim"])
    v = (c @ w[name + "uv"].T).view(T, H, a["vdim"])
    out = torch.zeros(T, H, a["vdim"], dtype=D)
    for i in range(T):
        keys = list(visible_keys(i, a["mask"]["size"]))
        qr = rotate(q[i, :, a["dim"]:], i, a["rot"])
        for g in range(H):
            s = (k[keys, g] @ q[i, g, :a["dim"]] + kr[keys] @ qr[g]) * a["scale"]
            out[i, g] = attend(s, v[keys, g])
    return out.flatten(1)


def gate(o, h, w_g):
    return o / (1 + torch.exp(-(h @ w_g.T)))


def feed_forward(h, w, name):
    z = h @ w[name + "up"].T + w[name + "up.b"]
    return torch.where(z > 0, z * z, torch.zeros_like(z)) @ w[name + "down"].T + w[name + "down.b"]


def forward(cfg, w, tokens, hidden=None):
    """Logits [T, vocab] of one whole sequence."""
    w = {k: v.to(D) for k, v in w.items()}
    eps, m, kept = cfg["norm"]["eps"], cfg["residual_mult"], {}
    x = w["embed"][torch.tensor(tokens)]
    for i, layer in enumerate(cfg["layers"]):
        a, name = layer["mixer"], f"l{i}."
        if a.get("kv_from") is None:
            kept[i] = latents(x, w, name + "mix.", a, eps)
        c, kr = kept[i if a.get("kv_from") is None else a["kv_from"]]
        o = gate(latent_attention(x, c, kr, w, name + "mix.", a), x, w[name + "mix.g"]) @ w[name + "mix.o"].T
        x = x + m * rms_norm(o, eps, w[name + "norm1"])
        if layer["mlp"] is not None:
            x = x + m * rms_norm(feed_forward(x, w, name + "mlp."), eps, w[name + "norm2"])
        if hidden is not None:
            hidden.append(x)
    return rms_norm(x, eps, w["final.norm"]) @ w["head"].T


def greedy(cfg, w, prompt, new):
    seq = list(prompt)
    for _ in range(new):
        seq.append(int(forward(cfg, w, seq)[-1].argmax()))
    return seq[len(prompt):]


# ------------------------------------------------------------------------------------------
# small models
# ------------------------------------------------------------------------------------------
def mixer(heads=2, dim=16, rot_dim=8, vdim=24, kv_rank=32, window=11, base=500.0, scaling="default", kv_from=None, scale=None):
    rot = {"base": base, "dims": rot_dim}
    if scaling == "default":
        scaling = {"factor": 2.5, "original": 48, "fast": 6.0, "slow": 1.0}
    if scaling is not None:
        rot["scaling"] = scaling
    out = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "mask": {"size": window},
           "scale": (dim + rot_dim) ** -0.5 * 1.3 if scale is None else scale, "rot": rot}
    if kv_from is not None:
        out["kv_from"] = kv_from
    return out


def config(mixers, ff=(40,), vocab=67, width=48, eps=1e-5, mult=0.4):
    """One layer per mixer; ``ff`` is cycled (None: a layer without feed-forward)."""
    return {"architecture": "Gasovik", "vocab": vocab, "width": width, "norm": {"eps": eps}, "residual_mult": mult,
            "layers": [{"type": "latent_attention", "mixer": a,
                        "mlp": None if ff[i % len(ff)] is None else {"kind": "dense", "ff": ff[i % len(ff)]}}
                       for i, a in enumerate(mixers)]}


def shapes(cfg):
    E, V = cfg["width"], cfg["vocab"]
    out = {"embed": (V, E), "final.norm": (E,), "head": (V, E)}
    for i, layer in enumerate(cfg["layers"]):
        a, n = layer["mixer"], f"l{i}."
        out.update({n + "norm1": (E,), n + "mix.q": (a["heads"] * (a["dim"] + a["rot_dim"]), E),
                    n + "mix.uk": (a["heads"] * a["dim"], a["kv_rank"]), n + "mix.uv": (a["heads"] * a["vdim"], a["kv_rank"]),
                    n + "mix.g": (a["heads"] * a["vdim"], E), n + "mix.o": (E, a["heads"] * a["vdim"])})
        if a.get("kv_from") is None:
            out.update({n + "mix.dkv": (a["kv_rank"] + a["rot_dim"], E), n + "mix.dkv.norm": (a["kv_rank"],)})
        if layer["mlp"] is not None:
            f = layer["mlp"]["ff"]
            out.update({n + "norm2": (E,), n + "mlp.up": (f, E), n + "mlp.up.b": (f,), n + "mlp.down": (E, f), n + "mlp.down.b": (E,)})
    return out


def random_weights(cfg, seed=0, sharp=1.0):
    """bf16-representable weights.  ``sharp`` scales the queries: large values make attention rest on few keys."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in shapes(cfg).items():
        if len(shape) == 1:
            t = torch.randn(shape, generator=g) * 0.3 + (0.0 if name.endswith(".b") else 1.0)
        else:
            t = torch.randn(shape, generator=g) * (1.0 if name == "embed" else shape[1] ** -0.5)
        if name.endswith("mix.q"):
            t = t * sharp
        out[name] = t.bfloat16()
    return out


class TensorDict:
    """The interface of a weight file over a dict of tensors."""

    def __init__(self, tensors):
        self.t = tensors

    def keys(self):
        return self.t.keys()

    def shape(self, name):
        return tuple(self.t[name].shape)

    def tensor(self, name):
        return self.t[name]


def rel_error(got, want):
    """rms of the difference (mean over the vocabulary taken off) over the rms of the expected logits, worst row."""
    d = got.double().cpu() - want
    d = d - d.mean(-1, keepdim=True)
    s = want - want.mean(-1, keepdim=True)
    return float((d.square().mean(-1).sqrt() / s.square().mean().sqrt()).max())
