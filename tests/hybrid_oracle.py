"""Plain, slow statements of the hybrid decoder's mechanisms (design ``Fatudra``) in double precision, one function each, and
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


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def layer_norm(x, eps, w, b):
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w + b


# ------------------------------------------------------------------------------------------
# softmax attention with a distance bias
# ------------------------------------------------------------------------------------------
def bucket(n, rows, reach):
    """Row of the bias table for distance ``n``: exact up to half the rows, then logarithmic up to ``reach``."""
    half = rows // 2
    if n < half or rows == 1:
        return min(n, rows - 1)
    return min(rows - 1, half + math.floor(math.log(n / half) / math.log(reach / half) * (rows - half)))


def query_temperature(p, spec):
    return 1.0 if spec is None else 1 + spec["coef"] * math.log((p + 1) // spec["every"] + 1)


def biased_attention(h, w, name, a):
    """Heads [T, H, vdim] before the output gate."""
    T, H, G = len(h), a["heads"], a["kv_heads"]
    q = (h @ w[name + "q"].T + w[name + "q.b"]).view(T, H, a["dim"])
    k = (h @ w[name + "k"].T + w[name + "k.b"]).view(T, G, a["dim"])
    v = (h @ w[name + "v"].T + w[name + "v.b"]).view(T, G, a["vdim"])
    rel = w[name + "rel"]
    rows = torch.tensor([bucket(n, len(rel), a["bias_max"]) for n in range(T)])
    out = torch.zeros(T, H, a["vdim"], dtype=D)
    for i in range(T):
        t = query_temperature(i, a.get("q_temp"))
        bias = rel[rows[torch.arange(i, -1, -1)]]             # [i + 1, H]
        for g in range(H):
            kv = g // (H // G)
            s = (k[:i + 1, kv] @ (q[i, g] * t)) * a["scale"] + bias[:, g]
            e = torch.exp(s - s.max())
            out[i, g] = (e / e.sum()) @ v[:i + 1, kv]
    return out


def gated_attention(h, w, name, a):
    o = biased_attention(h, w, name, a) * sigmoid(h @ w[name + "g"].T)[:, :, None]
    return o.flatten(1) @ w[name + "o"].T + w[name + "o.b"]


# ------------------------------------------------------------------------------------------
# recurrences
# ------------------------------------------------------------------------------------------
def decayed_memory(q, k, v, decay):
    """q, k [T, H, d], v [T, H, e], decay [H] -> [T, H, e]."""
    T, H, _ = q.shape
    out = torch.zeros(T, H, v.shape[2], dtype=D)
    for g in range(H):
        S = torch.zeros(q.shape[2], v.shape[2], dtype=D)
        for t in range(T):
            S = decay[g] * S + torch.outer(k[t, g], v[t, g])
            out[t, g] = S.T @ q[t, g]
    return out


def lightning(h, w, name, a, eps):
    T, H = len(h), a["heads"]
    q = silu(h @ w[name + "q"].T).view(T, H, a["dim"])
    k = silu(h @ w[name + "k"].T).view(T, H, a["dim"])
    v = silu(h @ w[name + "v"].T).view(T, H, a["vdim"])
    o = decayed_memory(q, k, v, a["decay"]).flatten(1)
    return (rms_norm(o, eps, w[name + "norm"]) * sigmoid(h @ w[name + "g"].T)) @ w[name + "o"].T


def matrix_memory(q, k, v, i, f):
    """Gated matrix memory with a normaliser and a running maximum; q already scaled; i, f [T, H] log gates."""
    T, H, _ = q.shape
    out = torch.zeros(T, H, v.shape[2], dtype=D)
    for g in range(H):
        S = torch.zeros(q.shape[2], v.shape[2], dtype=D)
        n = torch.zeros(q.shape[2], dtype=D)
        m = 0.0
        for t in range(T):
            m_new = max(float(f[t, g]) + m, float(i[t, g]))
            a, b = math.exp(float(f[t, g]) + m - m_new), math.exp(float(i[t, g]) - m_new)
            S, n, m = a * S + b * torch.outer(k[t, g], v[t, g]), a * n + b * k[t, g], m_new
            out[t, g] = (S.T @ q[t, g]) / (max(abs(float(n @ q[t, g])), math.exp(-m)) + 1e-6)
    return out


def memory_gates(h, w, name, cap):
    """Log input gate and log forget gate [T, H]."""
    i = cap * torch.tanh((h @ w[name + "i"].T + w[name + "i.b"]) / cap)
    z = cap * torch.tanh((h @ w[name + "f"].T + w[name + "f.b"]) / cap)
    return i, -torch.log1p(torch.exp(-z))


def mlstm(h, w, name, a, eps):
    T, H = len(h), a["heads"]
    q = (h @ w[name + "q"].T).view(T, H, a["dim"]) * a["dim"] ** -0.5
    k = (h @ w[name + "k"].T).view(T, H, a["dim"])
    v = (h @ w[name + "v"].T).view(T, H, a["vdim"])
    o = matrix_memory(q, k, v, *memory_gates(h, w, name, a["gate_cap"]))
    o = rms_norm(o, eps).flatten(1) * w[name + "norm"] * sigmoid(h @ w[name + "g"].T)
    return o @ w[name + "o"].T


def parallel(h, w, name, a, eps):
    return a["left_scale"] * gated_attention(h, w, name + "left.", a["left"]) + \
        a["right_scale"] * lightning(h, w, name + "right.", a["right"], eps)


MIX = {"parallel": parallel, "mlstm": mlstm}


def feed_forward(h, w, name):
    return (gelu_tanh(h @ w[name + "gate"].T) * (h @ w[name + "up"].T)) @ w[name + "down"].T


# ------------------------------------------------------------------------------------------
# the model
# ------------------------------------------------------------------------------------------
def layer_runs(cfg):
    """(layer, pass or None) in the order of execution; the pass number stands at the first layer of a pass."""
    n, lp = len(cfg["layers"]), cfg.get("loop")
    if lp is None:
        return [(i, None) for i in range(n)]
    body = [(i, t if i == lp["start"] else None) for t in range(lp["times"]) for i in range(lp["start"], lp["stop"])]
    return [(i, None) for i in range(lp["start"])] + body + [(i, None) for i in range(lp["stop"], n)]


def forward(cfg, w, tokens, hidden=None):
    """Logits [T, vocab] of one whole sequence."""
    w = {k: v.to(D) for k, v in w.items()}
    eps = cfg["norm"]["eps"]

    def norm(x, name):
        return layer_norm(x, eps, w[name], w[name + ".b"])

    x = w["embed"][torch.tensor(tokens)] * cfg["embedding"]["scale"]
    for i, t in layer_runs(cfg):
        layer, n = cfg["layers"][i], f"l{i}."
        if t is not None:
            x = x + w["loop.step"][t]
        x = x + norm(MIX[layer["type"]](norm(x, n + "norm1"), w, n + "mix.", layer["mixer"], eps), n + "norm1b")
        if layer["mlp"] is not None:
            x = x + norm(feed_forward(norm(x, n + "norm2"), w, n + "mlp."), n + "norm2b")
        if hidden is not None:
            hidden.append(x)
    return norm(x, "final.norm") @ w["head"].T


def greedy(cfg, w, prompt, new):
    seq = list(prompt)
    for _ in range(new):
        seq.append(int(forward(cfg, w, seq)[-1].argmax()))
    return seq[len(prompt):]


# ------------------------------------------------------------------------------------------
# small models
# ------------------------------------------------------------------------------------------
def par(heads=4, kv_heads=2, dim=16, vdim=24, bias_max=50, q_temp=(0.4, 7), scale=None, rows=10, r_heads=3, r_dim=8, r_vdim=16,
        decay=None, left_scale=0.7, right_scale=1.1):
    """A ``parallel`` layer; ``rows`` is the height of its bias table (a tensor's size, not part of a stored configuration)."""
    left = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "bias_max": bias_max,
            "scale": 1.2 * dim ** -0.5 if scale is None else scale, "bias_rows": rows}
    if q_temp is not None:
        left["q_temp"] = {"coef": q_temp[0], "every": q_temp[1]}
    decay = [1 - 0.4 / 4 ** k for k in range(r_heads)] if decay is None else decay
    return {"type": "parallel", "mixer": {"left": left, "right": {"heads": r_heads, "dim": r_dim, "vdim": r_vdim, "decay": decay},
                                          "left_scale": left_scale, "right_scale": right_scale}}


def mem(heads=2, dim=16, vdim=24, gate_cap=9.0):
    return {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": gate_cap}}


def config(mixers, ff=(40,), vocab=67, width=48, eps=1e-5, scale=3.0, loop=None):
    """One layer per mixer; ``ff`` is cycled (None: a layer without feed-forward); ``loop``: (start, stop, times)."""
    out = {"architecture": "Fatudra", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale},
           "layers": [{**m, "mlp": None if ff[i % len(ff)] is None else {"kind": "dense", "ff": ff[i % len(ff)]}}
                      for i, m in enumerate(mixers)]}
    if loop is not None:
        out["loop"] = dict(zip(("start", "stop", "times"), loop))
    return out


def stored(cfg):
    """The configuration as a model folder holds it: without the sizes that only the tensors give."""
    layers = []
    for layer in cfg["layers"]:
        layer = dict(layer, mixer=dict(layer["mixer"]))
        if layer["type"] == "parallel":
            layer["mixer"]["left"] = {k: v for k, v in layer["mixer"]["left"].items() if k != "bias_rows"}
        layers.append(layer)
    return dict(cfg, layers=layers)


def shapes(cfg):
    E, V = cfg["width"], cfg["vocab"]
    out = {"embed": (V, E), "final.norm": (E,), "final.norm.b": (E,), "head": (V, E)}
    if cfg.get("loop"):
        out["loop.step"] = (cfg["loop"]["times"], E)
    for i, layer in enumerate(cfg["layers"]):
        a, n = layer["mixer"], f"l{i}."
        for s in ("norm1", "norm1b") + (() if layer["mlp"] is None else ("norm2", "norm2b")):
            out[n + s] = out[n + s + ".b"] = (E,)
        if layer["type"] == "parallel":
            b, c, l, r = a["left"], a["right"], n + "mix.left.", n + "mix.right."
            for s, m in (("q", b["heads"] * b["dim"]), ("k", b["kv_heads"] * b["dim"]), ("v", b["kv_heads"] * b["vdim"])):
                out[l + s], out[l + s + ".b"] = (m, E), (m,)
            out.update({l + "rel": (b["bias_rows"], b["heads"]), l + "g": (b["heads"], E), l + "o": (E, b["heads"] * b["vdim"]), l + "o.b": (E,)})
            hd, hv = c["heads"] * c["dim"], c["heads"] * c["vdim"]
            out.update({r + "q": (hd, E), r + "k": (hd, E), r + "v": (hv, E), r + "g": (hv, E), r + "o": (E, hv), r + "norm": (hv,)})
        else:
            m, hd, hv = n + "mix.", a["heads"] * a["dim"], a["heads"] * a["vdim"]
            out.update({m + "q": (hd, E), m + "k": (hd, E), m + "v": (hv, E), m + "g": (hv, E), m + "o": (E, hv), m + "norm": (hv,)})
            for s in ("i", "f"):
                out[m + s], out[m + s + ".b"] = (a["heads"], E), (a["heads"],)
        if layer["mlp"] is not None:
            f = layer["mlp"]["ff"]
            out.update({n + "mlp.gate": (f, E), n + "mlp.up": (f, E), n + "mlp.down": (E, f)})
    return out


def random_weights(cfg, seed=0, sharp=1.0):
    """bf16-representable weights.  ``sharp`` scales the attention queries: large values make attention rest on few keys."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in shapes(cfg).items():
        t = torch.randn(shape, generator=g)
        if name.endswith("mix.f.b"):
            t = t + 2.5                                     # forget gates near one: memories reach far back
        elif len(shape) == 1:
            t = t * 0.3 + (0.0 if name.endswith(".b") else 1.0)
        elif not name.endswith((".rel", "loop.step", "embed")):
            t = t * shape[1] ** -0.5
        if name.endswith("mix.left.q"):
            t = t * sharp
        out[name] = t.bfloat16()
    return out
