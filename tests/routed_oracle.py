"""Plain, slow statements of the routed decoder's mechanisms (design ``Dusilorn``) in double precision, one function each, and
small random models to compare the framework with.  Nothing here comes from the package: a model is a configuration dict
and a dict of named tensors."""
import math

import torch

from layered_oracle import TensorDict, rel_error, rms_norm  # noqa: F401

D = torch.float64


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def relu2(z):
    return torch.clamp(z, min=0) ** 2


# ------------------------------------------------------------------------------------------
# attention
# ------------------------------------------------------------------------------------------
def rotate_half(vec, position, rot):
    """One vector (or a stack of one position): entry i of the first half of the leading ``dims`` entries turns with entry i of
    the second half."""
    n = rot["dims"]
    out = vec.clone()
    for i in range(n // 2):
        a = position * rot["base"] ** (-2.0 * i / n)
        c, s = math.cos(a), math.sin(a)
        out[..., i] = vec[..., i] * c - vec[..., i + n // 2] * s
        out[..., i + n // 2] = vec[..., i + n // 2] * c + vec[..., i] * s
    return out


def cap_score(s, cap):
    return cap * torch.tanh(s / cap)


def chunk_keys(i, size):
    """Positions that position ``i`` sees: those of its own chunk up to itself."""
    return range(i // size * size, i + 1)


def window_keys(i, size):
    """The last ``size`` positions, itself included."""
    return range(max(0, i - size + 1), i + 1)


def softmax_weights(s, sink=None):
    """Softmax of one query's scores; ``sink`` adds one term to the denominator."""
    m = s.max() if sink is None else torch.maximum(s.max(), sink)
    e = torch.exp(s - m)
    return e / (e.sum() + (0 if sink is None else torch.exp(sink - m)))


def mix_values(v, first, lam):
    return (1 - lam) * v + lam * first


def attend(q, k, v, kind, a, sink=None):
    """q [T, H, d], k, v [T, G, .] of one sequence -> [T, H, vdim]."""
    T, H = q.shape[:2]
    keys = {"attention": chunk_keys, "attention_2": window_keys}[kind]
    out = torch.zeros(T, H, v.shape[2], dtype=D)
    for i in range(T):
        see = keys(i, a["mask"]["size"])
        see = slice(see.start, see.stop)
        for h in range(H):
            g = h // (H // k.shape[1])
            s = cap_score((k[see, g] @ q[i, h]) * a["scale"], a["softcap"])
            out[i, h] = softmax_weights(s, None if sink is None else sink[h]) @ v[see, g]
    return out


def attention(h, w, name, kind, a, eps, first):
    """Sublayer output [T, width] and the values that later layers mix in."""
    T, H, G = len(h), a["heads"], a["kv_heads"]
    q, k, v = (h @ w[name + s].T for s in "qkv")
    if kind == "attention":
        q, k = rms_norm(q, eps, w[name + "q.norm"]), rms_norm(k, eps, w[name + "k.norm"])
    q, k = q.view(T, H, a["dim"]), k.view(T, G, a["dim"])
    if kind == "attention_2":
        q = torch.stack([rotate_half(q[t], t, a["rot"]) for t in range(T)])
        k = torch.stack([rotate_half(k[t], t, a["rot"]) for t in range(T)])
    if a.get("v_mix"):
        if first is None:
            first = v
        else:
            v = mix_values(v, first, w[name + "vmix"])
    o = attend(q, k, v.view(T, G, a["vdim"]), kind, a, w[name + "sink"] if kind == "attention" else None)
    return o.flatten(1) @ w[name + "o"].T, first


# ------------------------------------------------------------------------------------------
# feed-forward
# ------------------------------------------------------------------------------------------
def dense(h, w, name):
    return (silu(h @ w[name + "gate"].T) * (h @ w[name + "up"].T)) @ w[name + "down"].T


def expert(h, w, name):
    return relu2(h @ w[name + "up"].T) @ w[name + "down"].T


def route(z, correction, top):
    """Router logits of one token -> chosen outputs (best first) and their weights."""
    s = torch.exp(z - z.max())
    s = s / s.sum()
    chosen = torch.argsort(s + correction, descending=True, stable=True)[:top]
    return chosen, s[chosen] / (s[chosen].sum() + 1e-20)


def mixture(h, w, name, m):
    r = m["router"]
    out = torch.zeros_like(h)
    for t in range(len(h)):
        chosen, weights = route(w[name + "router"] @ h[t], w[name + "correction"], r["top"])
        for c, p in zip(chosen.tolist(), weights):
            out[t] += p * (h[t] if c >= r["experts"] else expert(h[t], w, f"{name}e{c}."))
    if m.get("shared") is not None:
        out = out + sigmoid(h @ w[name + "shared.sg"].T) * expert(h, w, name + "shared.")
    return out


def feed_forward(h, w, name, m):
    return dense(h, w, name) if m["kind"] == "dense" else mixture(h, w, name, m)


# ------------------------------------------------------------------------------------------
# the model
# ------------------------------------------------------------------------------------------
def forward(cfg, w, tokens, hidden=None):
    """Logits [T, vocab] of one whole sequence."""
    w = {k: v.to(D) for k, v in w.items()}
    eps = cfg["norm"]["eps"]

    def norm(x, name):
        return rms_norm(x, eps, 1 + w[name])

    x = w["embed"][torch.tensor(tokens)] * cfg["embedding"]["scale"]
    first = None
    for i, layer in enumerate(cfg["layers"]):
        n = f"l{i}."
        o, first = attention(norm(x, n + "norm1"), w, n + "mix.", layer["type"], layer["mixer"], eps, first)
        x = x + norm(o, n + "norm1b")
        if layer["mlp"] is not None:
            x = x + norm(feed_forward(norm(x, n + "norm2"), w, n + "mlp.", layer["mlp"]), n + "norm2b")
        if hidden is not None:
            hidden.append(x)
    return norm(x, "final.norm") @ w["head"].T * cfg["logit_scale"]


def greedy(cfg, w, prompt, new):
    seq = list(prompt)
    for _ in range(new):
        seq.append(int(forward(cfg, w, seq)[-1].argmax()))
    return seq[len(prompt):]


# ------------------------------------------------------------------------------------------
# small models
# ------------------------------------------------------------------------------------------
def chunked(heads=4, kv_heads=2, dim=16, vdim=24, size=20, scale=None, softcap=12.0, v_mix=True):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": size},
                                           "scale": 1.3 * dim ** -0.5 if scale is None else scale, "softcap": softcap, "v_mix": v_mix}}


def windowed(heads=4, kv_heads=2, dim=16, vdim=24, size=11, scale=None, softcap=9.0, v_mix=True, rot=8, base=500.0):
    layer = chunked(heads, kv_heads, dim, vdim, size, scale, softcap, v_mix)
    layer["mixer"]["rot"] = {"base": base, "dims": rot}
    return dict(layer, type="attention_2")


def moe(experts=6, identity=2, top=3, ff=24, shared=40):
    out = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "identity": identity, "top": top}}
    if shared is not None:
        out["shared"] = {"ff": shared}
    return out


def mlp(ff=40):
    return {"kind": "dense", "ff": ff}


def config(mixers, mlps, vocab=67, width=48, eps=1e-5, scale=2.5, logit_scale=1.7):
    """One layer per mixer; ``mlps`` is cycled (None: a layer without feed-forward)."""
    return {"architecture": "Dusilorn", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale},
            "logit_scale": logit_scale, "layers": [{**m, "mlp": mlps[i % len(mlps)]} for i, m in enumerate(mixers)]}


def shapes(cfg):
    E, V = cfg["width"], cfg["vocab"]
    out = {"embed": (V, E), "final.norm": (E,), "head": (V, E)}
    for i, layer in enumerate(cfg["layers"]):
        a, m, n = layer["mixer"], layer["mlp"], f"l{i}."
        for s in ("norm1", "norm1b") + (() if m is None else ("norm2", "norm2b")):
            out[n + s] = (E,)
        x, H, G = n + "mix.", a["heads"], a["kv_heads"]
        out.update({x + "q": (H * a["dim"], E), x + "k": (G * a["dim"], E), x + "v": (G * a["vdim"], E), x + "o": (E, H * a["vdim"])})
        if layer["type"] == "attention":
            out.update({x + "q.norm": (H * a["dim"],), x + "k.norm": (G * a["dim"],), x + "sink": (H,)})
        if a.get("v_mix"):
            out[x + "vmix"] = ()
        f = n + "mlp."
        if m is not None and m["kind"] == "dense":
            out.update({f + "gate": (m["ff"], E), f + "up": (m["ff"], E), f + "down": (E, m["ff"])})
        elif m is not None:
            parts = [(f"e{e}.", m["expert"]["ff"]) for e in range(m["router"]["experts"])]
            total = m["router"]["experts"] + m["router"]["identity"]
            out.update({f + "router": (total, E), f + "correction": (total,)})
            if m.get("shared") is not None:
                parts.append(("shared.", m["shared"]["ff"]))
                out[f + "shared.sg"] = (1, E)
            for p, ff in parts:
                out.update({f + p + "up": (ff, E), f + p + "down": (E, ff)})
    return out


def random_weights(cfg, seed=0, sharp=1.0, router=4.0):
    """bf16-representable weights.  ``sharp`` scales the attention scores (through the queries or their norm): large values make
    attention rest on few keys; ``router`` scales the router, so that choices are seldom close."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in shapes(cfg).items():
        t = torch.randn(shape, generator=g)
        if name.endswith(".vmix"):
            t = 0.4 + 0.2 * torch.tanh(t)
        elif name.endswith(".correction"):
            t = t * 0.1
        elif name.endswith((".q.norm", ".k.norm")):
            t = 1 + 0.3 * t
        elif len(shape) == 1 and not name.endswith(".sink"):
            t = t * 0.3
        elif len(shape) == 2 and name != "embed":
            t = t * shape[1] ** -0.5
        if name.endswith(("mix.q", "q.norm")):
            t = t * sharp
        if name.endswith(".router"):
            t = t * router
        out[name] = t.bfloat16()
    return out
