"""Plain, slow statements of the mechanisms of the design ``Bolovik`` in double precision, one function each, and small random models
to compare the framework with.  Nothing here comes from the package: a model is a configuration dict and a dict of named
tensors."""
import math

import torch

from layered_oracle import TensorDict, rel_error, rms_norm  # noqa: F401

D = torch.float64


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


# ------------------------------------------------------------------------------------------
# norms and the sums over depth
# ------------------------------------------------------------------------------------------
def group_norm(x, w, groups, eps):
    """Every one of ``groups`` equal parts of a vector is divided by its own root mean square."""
    parts = x.unflatten(-1, (groups, x.shape[-1] // groups))
    return rms_norm(parts, eps).flatten(-2) * w


def depth_average(past, weights):
    """``past``: embedding output and layer results so far."""
    assert len(past) == len(weights)
    return sum(w * x for w, x in zip(weights, past))


# ------------------------------------------------------------------------------------------
# gated delta rule
# ------------------------------------------------------------------------------------------
def short_conv(x, taps):
    """x [T, channels], taps [channels, n]: the last column meets the current token."""
    n = taps.shape[1]
    out = torch.zeros_like(x)
    for t in range(len(x)):
        for j in range(n):
            if t - j >= 0:
                out[t] += taps[:, n - 1 - j] * x[t - j]
    return out


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def log_decay(z, a_log, dt_bias):
    return -torch.exp(a_log) * softplus(z + dt_bias)


def delta_scan(q, k, v, beta, log_g):
    """q, k [T, d], v [T, e], beta and log_g [T] of one head -> read-outs [T, e]."""
    S = torch.zeros(q.shape[1], v.shape[1], dtype=D)
    out = []
    for t in range(len(q)):
        S = torch.exp(log_g[t]) * S
        u = beta[t] * (v[t] - S.T @ k[t])
        S = S + torch.outer(k[t], u)
        out.append(S.T @ q[t])
    return torch.stack(out)


def head_norm_gate(o, w, z, eps):
    """o, z [T, H, e]."""
    return rms_norm(o, eps) * w * silu(z)


def delta(h, w, name, a, eps):
    T, H, G = len(h), a["heads"], a["kv_heads"]
    q, k, v = (silu(short_conv(h @ w[name + s].T, w[name + s + ".conv"])) for s in "qkv")
    q, k, v = unit(q.view(T, G, -1)) * a["dim"] ** -0.5, unit(k.view(T, G, -1)), v.view(T, H, -1)
    beta = sigmoid(h @ w[name + "b"].T)
    log_g = log_decay(h @ w[name + "a"].T, w[name + "A_log"], w[name + "dt_bias"])
    o = torch.stack([delta_scan(q[:, i // (H // G)], k[:, i // (H // G)], v[:, i], beta[:, i], log_g[:, i]) for i in range(H)], dim=1)
    o = head_norm_gate(o, w[name + "norm"], (h @ w[name + "g"].T).view(T, H, -1), eps)
    return o.flatten(1) @ w[name + "o"].T


# ------------------------------------------------------------------------------------------
# attention
# ------------------------------------------------------------------------------------------
def frequencies(rot):
    """Radians per position of every pair; long wavelengths are stretched, those between the two bounds in part."""
    out, sc = [], rot.get("scaling")
    for i in range(rot["dims"] // 2):
        f = rot["base"] ** (-2.0 * i / rot["dims"])
        if sc is not None:
            length = 2 * math.pi / f
            if length > sc["original"] / sc["low"]:
                f = f / sc["factor"]
            elif length >= sc["original"] / sc["high"]:
                s = (sc["original"] / length - sc["low"]) / (sc["high"] - sc["low"])
                f = (1 - s) * f / sc["factor"] + s * f
        out.append(f)
    return out


def rotate_half(vec, position, rot):
    """One vector (or a stack of one position): entry i of the first half of the leading entries turns with entry i of the
    second half."""
    n = rot["dims"]
    out = vec.clone()
    for i, f in enumerate(frequencies(rot)):
        c, s = math.cos(position * f), math.sin(position * f)
        out[..., i] = vec[..., i] * c - vec[..., i + n // 2] * s
        out[..., i + n // 2] = vec[..., i + n // 2] * c + vec[..., i] * s
    return out


def visible_keys(i, size, keep):
    """Positions that position ``i`` sees: the last ``size`` and the first ``keep``."""
    return [j for j in range(i + 1) if i - j < size or j < keep]


def softmax_weights(s):
    e = torch.exp(s - s.max())
    return e / e.sum()


def attend(q, k, v, a):
    """q [T, H, d], k, v [T, G, .] of one sequence -> [T, H, vdim]."""
    T, H = q.shape[:2]
    m = a["mask"]
    out = torch.zeros(T, H, v.shape[2], dtype=D)
    for i in range(T):
        see = visible_keys(i, m["size"], m["keep_first"])
        for h in range(H):
            g = h // (H // k.shape[1])
            out[i, h] = softmax_weights((k[see, g] @ q[i, h]) * a["scale"]) @ v[see, g]
    return out


def attention(h, w, name, a, eps):
    T, H, G = len(h), a["heads"], a["kv_heads"]
    q, k, v = (h @ w[name + s].T + w[name + s + ".b"] for s in "qkv")
    q, k, v = q.view(T, H, -1), k.view(T, G, -1), v.view(T, G, -1)
    q = rms_norm(torch.stack([rotate_half(q[t], t, a["rot"]) for t in range(T)]), eps)
    k = rms_norm(torch.stack([rotate_half(k[t], t, a["rot"]) for t in range(T)]), eps)
    return attend(q, k, rms_norm(v, eps), a).flatten(1) @ w[name + "o"].T


# ------------------------------------------------------------------------------------------
# feed-forward
# ------------------------------------------------------------------------------------------
def gated(h, w, name, act):
    return (act(h @ w[name + "gate"].T) * (h @ w[name + "up"].T)) @ w[name + "down"].T


def route(z, top, groups):
    """Router logits of one token -> chosen experts and their weights."""
    s = sigmoid(z)
    n = len(s) // groups["count"]
    strength = [sum(sorted(s[g * n:(g + 1) * n].tolist(), reverse=True)[:2]) for g in range(groups["count"])]
    best = sorted(range(groups["count"]), key=lambda g: -strength[g])[:groups["keep"]]
    allowed = [e for e in range(len(s)) if e // n in best]
    chosen = sorted(allowed, key=lambda e: -float(s[e]))[:top]
    return chosen, s[chosen]


def mixture(h, w, name, m):
    r = m["router"]
    out = torch.zeros_like(h)
    for t in range(len(h)):
        for c, p in zip(*route(w[name + "router"] @ h[t], r["top"], r["groups"])):
            out[t] += p * gated(h[t], w, f"{name}e{c}.", silu)
    return out


def feed_forward(h, w, name, m):
    return gated(h, w, name, gelu_tanh) if m["kind"] == "dense" else mixture(h, w, name, m)


# ------------------------------------------------------------------------------------------
# the model
# ------------------------------------------------------------------------------------------
def forward(cfg, w, tokens, hidden=None):
    """Logits [T, vocab] of one whole sequence."""
    w = {k: v.to(D) for k, v in w.items()}
    eps, groups = cfg["norm"]["eps"], cfg["norm"]["groups"]
    x = w["embed"][torch.tensor(tokens)]
    past = [x]
    for i, layer in enumerate(cfg["layers"]):
        n = f"l{i}."
        mixer = {"delta": delta, "attention": attention}[layer["type"]]
        x = x + group_norm(mixer(x, w, n + "mix.", layer["mixer"], eps), w[n + "norm1"], groups, eps)
        if layer["mlp"] is not None:
            x = x + group_norm(feed_forward(x, w, n + "mlp.", layer["mlp"]), w[n + "norm2"], groups, eps)
        past.append(x)
        x = depth_average(past, w[n + "dwa"])
        if hidden is not None:
            hidden.append(x)
    return group_norm(x, w["final.norm"], groups, eps) @ w["head"].T


def greedy(cfg, w, prompt, new):
    seq = list(prompt)
    for _ in range(new):
        seq.append(int(forward(cfg, w, seq)[-1].argmax()))
    return seq[len(prompt):]


# ------------------------------------------------------------------------------------------
# small models
# ------------------------------------------------------------------------------------------
SCALING = {"factor": 3.0, "low": 1.0, "high": 5.0, "original": 60}


def attn(heads=4, kv_heads=2, dim=16, vdim=24, size=11, keep=3, scale=None, rot=8, base=500.0, scaling=SCALING):
    rot = {"base": base, "dims": rot}
    if scaling is not None:
        rot["scaling"] = dict(scaling)
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": size, "keep_first": keep},
                                           "scale": 1.3 * dim ** -0.5 if scale is None else scale, "rot": rot}}


def memory(heads=4, kv_heads=2, dim=16, vdim=24, conv=4):
    return {"type": "delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}}


def moe(experts=6, top=2, ff=24, count=3, keep=2):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "groups": {"count": count, "keep": keep}, "top": top}}


def mlp(ff=40):
    return {"kind": "dense", "ff": ff}


def config(mixers, mlps, vocab=67, width=48, eps=1e-5, groups=3):
    """One layer per mixer; ``mlps`` is cycled (None: a layer without feed-forward)."""
    return {"architecture": "Bolovik", "vocab": vocab, "width": width, "norm": {"eps": eps, "groups": groups},
            "layers": [{**m, "mlp": mlps[i % len(mlps)]} for i, m in enumerate(mixers)]}


def shapes(cfg):
    E, V = cfg["width"], cfg["vocab"]
    out = {"embed": (V, E), "final.norm": (E,), "head": (V, E)}
    for i, layer in enumerate(cfg["layers"]):
        a, m, n = layer["mixer"], layer["mlp"], f"l{i}."
        for s in ("norm1",) + (() if m is None else ("norm2",)):
            out[n + s] = (E,)
        out[n + "dwa"] = (i + 2,)
        x, H, G = n + "mix.", a["heads"], a["kv_heads"]
        out[x + "o"] = (E, H * a["vdim"])
        if layer["type"] == "attention":
            for s, r in (("q", H * a["dim"]), ("k", G * a["dim"]), ("v", G * a["vdim"])):
                out.update({x + s: (r, E), x + s + ".b": (r,)})
        else:
            for s, r in (("q", G * a["dim"]), ("k", G * a["dim"]), ("v", H * a["vdim"])):
                out.update({x + s: (r, E), x + s + ".conv": (r, a["conv"])})
            out.update({x + "g": (H * a["vdim"], E), x + "b": (H, E), x + "a": (H, E), x + "A_log": (H,), x + "dt_bias": (H,), x + "norm": (a["vdim"],)})
        f = n + "mlp."
        if m is not None:
            parts = [("", m["ff"])] if m["kind"] == "dense" else [(f"e{e}.", m["expert"]["ff"]) for e in range(m["router"]["experts"])]
            if m["kind"] == "moe":
                out[f + "router"] = (m["router"]["experts"], E)
            for p, ff in parts:
                out.update({f + p + "gate": (ff, E), f + p + "up": (ff, E), f + p + "down": (E, ff)})
    return out


def random_weights(cfg, seed=0, sharp=1.0, router=3.0):
    """bf16-representable weights.  ``sharp`` scales step sizes and decays, ``router`` the router, so that choices are seldom close.  Memories
    reach from a few tokens to hundreds.  Sublayers add a part of the stream's size: rounding is not blown up from layer to layer."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in shapes(cfg).items():
        t = torch.randn(shape, generator=g)
        if name.endswith(".A_log"):
            t = t * 0.7 - 2.0
        elif name.endswith(".dt_bias"):
            t = t * 0.5 - 1.5
        elif name.endswith(".dwa"):
            t = 0.15 * t
            t[-1] = 0.9
        elif name.endswith(".conv"):
            t = t * shape[1] ** -0.5
        elif name.endswith((".q.b", ".k.b", ".v.b")):
            t = t * 0.5
        elif name.endswith((".norm1", ".norm2")):
            t = 0.35 + 0.1 * t
        elif len(shape) == 1:
            t = 1 + 0.3 * t
        elif name != "embed":
            t = t * shape[1] ** -0.5
        if name.endswith(".router"):
            t = t * router
        if name.endswith((".mix.b", ".mix.a")):
            t = t * sharp
        out[name] = t.bfloat16()
    return out
