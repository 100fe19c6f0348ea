"""Configuration of decoder-only models that are described layer by layer.

``config.json`` of such a model names its ``architecture`` and lists its layers; every entry carries the layer's mixer
``type``, the mixer's own sizes and constants and its feed-forward (or null).  The classes here validate that
description and derive shapes; ``models/layered.py`` builds the modules from it.

Architectures:

* ``Gasovik``: latent attention under a sliding window (optionally on the latents of an earlier layer), gated heads,
  biased squared-ReLU feed-forward, norms on the sublayer outputs only.
* ``Fatudra``: layers that run grouped-query attention with a learned distance bias beside a memory with fixed decay, or a
  gated matrix memory; tanh-GELU gated feed-forward; layer norms before and after every sublayer; a range of layers may run
  several times in a row with the same weights.
* ``Dusilorn``: grouped-query attention, either inside chunks (normed queries and keys, no rotation, an attention sink) or under
  a sliding window (rotated), scores capped, values mixed with those of the first such layer; a gated feed-forward or a mixture
  of experts with identity experts and a gated shared expert; RMS norms before and after every sublayer.
* ``Bolovik``: gated delta-rule memories behind short convolutions, or grouped-query attention under a sliding window that keeps the
  first tokens (biased, rotated, then normed per head); a gated feed-forward or a mixture of gated experts chosen within the best groups;
  RMS norms over groups of columns on the sublayer outputs only; a weighted sum of all earlier results after every layer.
"""
from __future__ import annotations

import json
import math
import os
from dataclasses import asdict, dataclass, field, fields, replace
from typing import ClassVar, Optional


def _take(d: dict, known: tuple, where: str) -> None:
    unknown = set(d) - set(known)
    if unknown:
        raise ValueError(f"{where}: unknown keys {sorted(unknown)}")


@dataclass(frozen=True)
class YarnScaling:
    """Frequency interpolation of a rotary embedding (YaRN, Peng et al.)."""

    factor: float
    original: float
    fast: float
    slow: float

    def ramp(self, dims: int, base: float) -> list:
        """Per pair: 0 keeps the frequency, 1 divides it by ``factor``."""
        def turns(t):
            return dims * math.log(self.original / (2 * math.pi * t)) / (2 * math.log(base))

        lo, hi = max(math.floor(turns(self.fast)), 0), min(math.ceil(turns(self.slow)), dims - 1)
        return [min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0) for i in range(dims // 2)]

    @property
    def magnitude(self) -> float:
        """Factor on both cos and sin."""
        return 0.1 * math.log(self.factor) + 1.0

    def stretched(self, f: list, dims: int, base: float) -> list:
        return [v / self.factor * r + v * (1 - r) for v, r in zip(f, self.ramp(dims, base))]


@dataclass(frozen=True)
class WavelengthScaling:
    """Frequency scaling by wavelength: those of at most ``original / high`` positions stay, those beyond ``original / low`` are
    divided by ``factor``, the ones between are interpolated."""

    factor: float
    low: float
    high: float
    original: float
    magnitude = 1.0

    def stretched(self, f: list, dims: int, base: float) -> list:
        out = []
        for v in f:
            length = 2 * math.pi / v
            if length < self.original / self.high:
                out.append(v)
            elif length > self.original / self.low:
                out.append(v / self.factor)
            else:
                s = (self.original / length - self.low) / (self.high - self.low) if self.high != self.low else 1.0
                out.append((1 - s) * v / self.factor + s * v)
        return out


@dataclass(frozen=True)
class RotarySpec:
    base: float
    dims: int
    scaling: Optional[object] = None         # YarnScaling or WavelengthScaling

    def frequencies(self) -> list:
        """Radians per position of every pair."""
        f = [self.base ** (-2 * i / self.dims) for i in range(self.dims // 2)]
        if self.scaling is None:
            return f
        return self.scaling.stretched(f, self.dims, self.base)

    @property
    def magnitude(self) -> float:
        return 1.0 if self.scaling is None else self.scaling.magnitude

    @classmethod
    def from_dict(cls, d: dict, scaling=YarnScaling) -> "RotarySpec":
        """``scaling``: the kind of scaling that the mixer may have."""
        _take(d, ("base", "dims", "scaling"), "rot")
        sc = d.get("scaling")
        if sc is not None:
            names = [f.name for f in fields(scaling)]
            _take(sc, tuple(names), "rot.scaling")
            sc = scaling(**{k: float(sc[k]) for k in names})
        if d["dims"] <= 0 or d["dims"] % 2:
            raise ValueError(f"rot.dims must be a positive even number, not {d['dims']}")
        return cls(float(d["base"]), int(d["dims"]), sc)

    def to_dict(self) -> dict:
        out = {"base": self.base, "dims": self.dims}
        if self.scaling is not None:
            out["scaling"] = asdict(self.scaling)
        return out


@dataclass(frozen=True)
class LatentAttentionSpec:
    """``heads`` heads of ``dim`` unrotated + ``rot_dim`` rotated query / key dimensions and ``vdim`` value dimensions over
    a latent of ``kv_rank`` numbers per token; ``window`` keys are visible (the query's own position included).
    ``kv_from`` names the layer whose latents are used instead of an own down-projection."""

    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    window: int
    scale: float
    rot: RotarySpec
    kv_from: Optional[int] = None

    @classmethod
    def from_dict(cls, d: dict) -> "LatentAttentionSpec":
        _take(d, ("heads", "dim", "rot_dim", "vdim", "kv_rank", "mask", "scale", "rot", "kv_from"), "mixer")
        _take(d["mask"], ("size",), "mixer.mask")
        spec = cls(int(d["heads"]), int(d["dim"]), int(d["rot_dim"]), int(d["vdim"]), int(d["kv_rank"]),
                   int(d["mask"]["size"]), float(d["scale"]), RotarySpec.from_dict(d["rot"]),
                   None if d.get("kv_from") is None else int(d["kv_from"]))
        if min(spec.heads, spec.dim, spec.rot_dim, spec.vdim, spec.kv_rank, spec.window) <= 0:
            raise ValueError(f"latent attention sizes must be positive: {d}")
        if spec.rot.dims != spec.rot_dim:
            raise ValueError(f"rot.dims {spec.rot.dims} differs from rot_dim {spec.rot_dim}")
        return spec

    def to_dict(self) -> dict:
        out = {"heads": self.heads, "dim": self.dim, "rot_dim": self.rot_dim, "vdim": self.vdim, "kv_rank": self.kv_rank,
               "mask": {"size": self.window}, "scale": self.scale, "rot": self.rot.to_dict()}
        if self.kv_from is not None:
            out["kv_from"] = self.kv_from
        return out


@dataclass(frozen=True)
class QueryTemperature:
    """Queries at position p are multiplied by ``1 + coef * ln(floor((p + 1) / every) + 1)``."""

    coef: float
    every: int

    def at(self, p: int) -> float:
        return 1.0 + self.coef * math.log((p + 1) // self.every + 1)


@dataclass(frozen=True)
class BiasedAttentionSpec:
    """Causal grouped-query attention without rotation: ``heads`` query heads over ``kv_heads`` key / value heads, a learned
    bias per head and distance bucket, one output gate per head.  ``bias_rows`` (buckets of the table) is a tensor's size:
    None until a checkpoint or a registry shape gives it."""

    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    bias_max: float
    q_temp: Optional[QueryTemperature] = None
    bias_rows: Optional[int] = None

    def bucket(self, n: int) -> int:
        """Table row of distance ``n``: one per distance up to half the rows, then logarithmic up to ``bias_max``."""
        half = self.bias_rows // 2
        if n < half or self.bias_rows == 1:
            return min(n, self.bias_rows - 1)
        return min(self.bias_rows - 1,
                   half + math.floor(math.log(n / half) / math.log(self.bias_max / half) * (self.bias_rows - half)))

    def buckets(self) -> list:
        """Buckets of the distances 0, 1, .. up to the first one of the last row (every farther distance shares it)."""
        out = [0]
        while out[-1] != self.bias_rows - 1:
            out.append(self.bucket(len(out)))
        return out

    @classmethod
    def from_dict(cls, d: dict) -> "BiasedAttentionSpec":
        _take(d, ("heads", "kv_heads", "dim", "vdim", "scale", "bias_max", "q_temp", "bias_rows"), "mixer.left")
        t = d.get("q_temp")
        if t is not None:
            _take(t, ("coef", "every"), "mixer.left.q_temp")
            t = QueryTemperature(float(t["coef"]), int(t["every"]))
            if t.every <= 0:
                raise ValueError("q_temp.every must be positive")
        spec = cls(int(d["heads"]), int(d["kv_heads"]), int(d["dim"]), int(d["vdim"]), float(d["scale"]), d["bias_max"], t,
                   None if d.get("bias_rows") is None else int(d["bias_rows"]))
        if min(spec.heads, spec.kv_heads, spec.dim, spec.vdim) <= 0 or spec.heads % spec.kv_heads:
            raise ValueError(f"attention sizes must be positive, kv_heads a divisor of heads: {d}")
        return spec if spec.bias_rows is None else spec.with_rows(spec.bias_rows)

    def with_rows(self, rows: int) -> "BiasedAttentionSpec":
        if rows < 1 or (rows > 1 and self.bias_max <= rows // 2):
            raise ValueError(f"a distance bias of {rows} rows needs a reach above {rows // 2}, not {self.bias_max}")
        return replace(self, bias_rows=int(rows))

    def to_dict(self) -> dict:
        out = {k: getattr(self, k) for k in ("heads", "kv_heads", "dim", "vdim", "scale", "bias_max")}
        if self.q_temp is not None:
            out["q_temp"] = {"coef": self.q_temp.coef, "every": self.q_temp.every}
        if self.bias_rows is not None:
            out["bias_rows"] = self.bias_rows
        return out

    def param_count(self, E: int) -> int:
        qkv = self.heads * self.dim + self.kv_heads * (self.dim + self.vdim)
        return qkv * (E + 1) + self.heads * (self.bias_rows or 0) + self.heads * E + E * self.heads * self.vdim + E


@dataclass(frozen=True)
class GroupedAttentionSpec:
    """Grouped-query attention with capped scores: ``softcap * tanh(q . k * scale / softcap)`` (None: not capped); ``size`` tokens of a window or a
    chunk are visible, under a window the first ``keep`` of the sequence as well.  Subclasses fix the kind of mask, how q, k and v are formed and
    whether a learned sink takes part in the softmax.  ``v_mix``: values are mixed with those of the first layer that mixes."""

    chunked = False                  # visible: the own chunk (counted from position 0); else the last ``size`` positions
    keeps = False                    # the first tokens may be kept visible
    capped = True                    # scores may be capped, values mixed
    biased = False                   # q, k and v have biases
    qk_norm = False                  # RMS norms with weights over all of q and of k
    head_norm = False                # RMS norms without weights over every head of q and k (after their rotation) and of v
    sink = False
    rotated = False
    scaling: ClassVar = None         # kind of frequency scaling that the rotation may have

    heads: int
    kv_heads: int
    dim: int
    vdim: int
    size: int
    scale: float
    softcap: Optional[float]
    v_mix: bool = False
    rot: Optional[RotarySpec] = None
    keep: int = 0

    @classmethod
    def from_dict(cls, d: dict) -> "GroupedAttentionSpec":
        _take(d, ("heads", "kv_heads", "dim", "vdim", "mask", "scale") + (("softcap", "v_mix") if cls.capped else ()) + (("rot",) if cls.rotated else ()), "mixer")
        _take(d["mask"], ("size",) + (("keep_first",) if cls.keeps else ()), "mixer.mask")
        rot = None
        if cls.rotated:
            if cls.scaling is None and d["rot"].get("scaling") is not None:
                raise ValueError(f"rot must not be scaled: {d['rot']}")
            rot = RotarySpec.from_dict(d["rot"], cls.scaling or YarnScaling)
        spec = cls(int(d["heads"]), int(d["kv_heads"]), int(d["dim"]), int(d["vdim"]), int(d["mask"]["size"]), float(d["scale"]),
                   None if d.get("softcap") is None else float(d["softcap"]), bool(d.get("v_mix", False)), rot, int(d["mask"].get("keep_first", 0)))
        if min(spec.heads, spec.kv_heads, spec.dim, spec.vdim, spec.size) <= 0 or spec.heads % spec.kv_heads:
            raise ValueError(f"attention sizes must be positive, kv_heads a divisor of heads: {d}")
        if spec.softcap is not None and not spec.softcap > 0:
            raise ValueError(f"softcap must be positive: {d}")
        if spec.rot is not None and spec.rot.dims > spec.dim:
            raise ValueError(f"rot must turn at most {spec.dim} dimensions: {d['rot']}")
        if spec.keep < 0:
            raise ValueError(f"mask.keep_first must not be negative: {d}")
        return spec

    def to_dict(self) -> dict:
        out = {k: getattr(self, k) for k in ("heads", "kv_heads", "dim", "vdim", "scale") + (("v_mix",) if self.capped else ())}
        if self.softcap is not None:
            out["softcap"] = self.softcap
        out["mask"] = {"size": self.size, **({"keep_first": self.keep} if self.keeps else {})}
        if self.rot is not None:
            out["rot"] = self.rot.to_dict()
        return out

    @property
    def v_width(self) -> int:
        return self.kv_heads * self.vdim

    @property
    def slots(self) -> int:
        """Positions that a sequence holds: the kept ones and a window or chunk."""
        return self.keep + self.size

    @property
    def score_bound(self) -> Optional[float]:
        """Largest magnitude of a score, where the design bounds it."""
        if self.softcap is not None:
            return self.softcap
        return abs(self.scale) * self.dim if self.head_norm else None

    def param_count(self, E: int) -> int:
        n = self.heads * (self.dim + self.vdim) * E + self.kv_heads * (self.dim + self.vdim) * E + int(self.v_mix)
        n += ((self.heads + self.kv_heads) * self.dim + self.v_width) * self.biased
        return n + (self.heads + self.kv_heads) * self.dim * self.qk_norm + self.heads * self.sink


class ChunkAttentionSpec(GroupedAttentionSpec):
    chunked = qk_norm = sink = True


class WindowAttentionSpec(GroupedAttentionSpec):
    rotated = True


class KeptWindowAttentionSpec(GroupedAttentionSpec):
    keeps = biased = head_norm = rotated = True
    capped = False
    scaling = WavelengthScaling


@dataclass(frozen=True)
class DeltaMemorySpec:
    """Matrix memory with the gated delta rule (Gated DeltaNet, Yang et al.): ``heads`` memories of ``dim`` keys and ``vdim`` values, whose
    queries and keys come from ``kv_heads`` heads; q, k and v pass a causal convolution over ``conv`` tokens."""

    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int

    @classmethod
    def from_dict(cls, d: dict) -> "DeltaMemorySpec":
        names = ("heads", "kv_heads", "dim", "vdim", "conv")
        _take(d, names, "mixer")
        spec = cls(*(int(d[k]) for k in names))
        if min(spec.heads, spec.kv_heads, spec.dim, spec.vdim, spec.conv) <= 0 or spec.heads % spec.kv_heads:
            raise ValueError(f"memory sizes must be positive, kv_heads a divisor of heads: {d}")
        return spec

    def to_dict(self) -> dict:
        return asdict(self)

    def param_count(self, E: int) -> int:
        qk, v = 2 * self.kv_heads * self.dim, self.heads * self.vdim
        return (qk + v) * (E + self.conv) + (2 * v + 2 * self.heads) * E + 2 * self.heads + self.vdim


@dataclass(frozen=True)
class DecayMemorySpec:
    """Linear attention with one fixed decay per head."""

    heads: int
    dim: int
    vdim: int
    decay: tuple

    @classmethod
    def from_dict(cls, d: dict) -> "DecayMemorySpec":
        _take(d, ("heads", "dim", "vdim", "decay"), "mixer.right")
        spec = cls(int(d["heads"]), int(d["dim"]), int(d["vdim"]), tuple(float(x) for x in d["decay"]))
        if min(spec.heads, spec.dim, spec.vdim) <= 0 or len(spec.decay) != spec.heads or not all(0 <= x <= 1 for x in spec.decay):
            raise ValueError(f"a decaying memory needs positive sizes and one decay in [0, 1] per head: {d}")
        return spec

    def to_dict(self) -> dict:
        return {"heads": self.heads, "dim": self.dim, "vdim": self.vdim, "decay": list(self.decay)}

    def param_count(self, E: int) -> int:
        return self.heads * (2 * self.dim + 3 * self.vdim) * E + self.heads * self.vdim


@dataclass(frozen=True)
class ParallelSpec:
    """Attention (left) and a decaying memory (right) on the same input, their outputs added with fixed weights."""

    left: BiasedAttentionSpec
    right: DecayMemorySpec
    left_scale: float
    right_scale: float

    @classmethod
    def from_dict(cls, d: dict) -> "ParallelSpec":
        _take(d, ("left", "right", "left_scale", "right_scale"), "mixer")
        return cls(BiasedAttentionSpec.from_dict(d["left"]), DecayMemorySpec.from_dict(d["right"]), float(d["left_scale"]),
                   float(d["right_scale"]))

    def to_dict(self) -> dict:
        return {"left": self.left.to_dict(), "right": self.right.to_dict(), "left_scale": self.left_scale,
                "right_scale": self.right_scale}

    def param_count(self, E: int) -> int:
        return self.left.param_count(E) + self.right.param_count(E)


@dataclass(frozen=True)
class GatedMemorySpec:
    """Matrix memory with exponential input gate, sigmoid forget gate, normaliser and running maximum (mLSTM of xLSTM, Beck et
    al.); ``gate_cap`` bounds the gates' logarithms."""

    heads: int
    dim: int
    vdim: int
    gate_cap: float

    @classmethod
    def from_dict(cls, d: dict) -> "GatedMemorySpec":
        _take(d, ("heads", "dim", "vdim", "gate_cap"), "mixer")
        spec = cls(int(d["heads"]), int(d["dim"]), int(d["vdim"]), float(d["gate_cap"]))
        if min(spec.heads, spec.dim, spec.vdim) <= 0 or spec.gate_cap <= 0:
            raise ValueError(f"a gated memory needs positive sizes: {d}")
        return spec

    def to_dict(self) -> dict:
        return {"heads": self.heads, "dim": self.dim, "vdim": self.vdim, "gate_cap": self.gate_cap}

    def param_count(self, E: int) -> int:
        return self.heads * (2 * self.dim + 3 * self.vdim + 2) * E + self.heads * (self.vdim + 2)


@dataclass(frozen=True)
class LoopSpec:
    """Layers ``start`` .. ``stop - 1`` run ``times`` times in a row, each pass with a cache of its own; a learned vector per
    pass is added to the residual stream in front of it."""

    start: int
    stop: int
    times: int

    @classmethod
    def from_dict(cls, d: dict) -> "LoopSpec":
        _take(d, ("start", "stop", "times"), "loop")
        return cls(int(d["start"]), int(d["stop"]), int(d["times"]))

    def to_dict(self) -> dict:
        return {"start": self.start, "stop": self.stop, "times": self.times}


@dataclass(frozen=True)
class DenseMLPSpec:
    ff: int

    @classmethod
    def from_dict(cls, d: dict) -> "DenseMLPSpec":
        _take(d, ("kind", "ff"), "mlp")
        if d["ff"] <= 0:
            raise ValueError(f"mlp.ff must be positive: {d}")
        return cls(int(d["ff"]))

    def to_dict(self) -> dict:
        return {"kind": "dense", "ff": self.ff}

    def param_count(self, E: int) -> int:
        """Matrices of the gated form."""
        return 3 * self.ff * E


@dataclass(frozen=True)
class MixtureSpec:
    """``experts`` feed-forwards of ``ff`` hidden units and ``identity`` experts that return their input, of which each token uses
    ``top``; ``shared``: hidden units of an expert that runs for every token behind a gate (None: there is none).  With ``group_count`` the
    experts form groups of neighbours, and only those of the ``group_keep`` groups whose two best scores add up to most can be chosen.
    Subclasses fix the experts' form and how scores become weights."""

    act: ClassVar = "relu2"          # "relu2": two matrices; "silu": gated, three
    scores: ClassVar = "softmax"     # of the router's outputs, or "sigmoid"
    corrected: ClassVar = True       # a correction is added to the scores for the choice
    normalized: ClassVar = True      # the chosen scores are divided by their sum
    grouped: ClassVar = False

    ff: int
    experts: int
    identity: int
    top: int
    shared: Optional[int] = None
    group_count: int = 1
    group_keep: int = 1

    @property
    def outputs(self) -> int:
        """Router outputs."""
        return self.experts + self.identity

    @property
    def gated(self) -> bool:
        return self.act == "silu"

    @classmethod
    def from_dict(cls, d: dict) -> "MixtureSpec":
        _take(d, ("kind", "expert", "router") + (() if cls.grouped else ("shared",)), "mlp")
        _take(d["expert"], ("ff",), "mlp.expert")
        r = d["router"]
        _take(r, ("experts", "top") + (("groups",) if cls.grouped else ("identity",)), "mlp.router")
        shared, groups = d.get("shared"), r.get("groups") or {"count": 1, "keep": 1}
        _take(groups, ("count", "keep"), "mlp.router.groups")
        if shared is not None:
            _take(shared, ("ff",), "mlp.shared")
        spec = cls(int(d["expert"]["ff"]), int(r["experts"]), int(r.get("identity", 0)), int(r["top"]), None if shared is None else int(shared["ff"]),
                   int(groups["count"]), int(groups["keep"]))
        if min(spec.ff, spec.experts, spec.top, 1 if spec.shared is None else spec.shared) <= 0 or spec.identity < 0 or spec.top > spec.outputs:
            raise ValueError(f"a mixture needs positive sizes and at most as many chosen experts as there are: {d}")
        n, k = spec.group_count, spec.group_keep
        if n < 1 or spec.outputs % n or not 1 <= k <= n or spec.top > spec.outputs // n * k:
            raise ValueError(f"groups must be equal and hold the chosen experts: {d}")
        return spec

    def to_dict(self) -> dict:
        r = {"experts": self.experts, "top": self.top}
        r.update({"groups": {"count": self.group_count, "keep": self.group_keep}} if self.grouped else {"identity": self.identity})
        out = {"kind": "moe", "expert": {"ff": self.ff}, "router": r}
        if self.shared is not None:
            out["shared"] = {"ff": self.shared}
        return out

    def _count(self, E: int, experts: int) -> int:
        return (3 if self.gated else 2) * experts * self.ff * E + self.outputs * (E + self.corrected) + \
            (0 if self.shared is None else (2 * self.shared + 1) * E)

    def param_count(self, E: int) -> int:
        return self._count(E, self.experts)

    def active_params(self, E: int) -> int:
        """Parameters that a token meets when all its experts have tensors."""
        return self._count(E, self.top)


class GroupedMixtureSpec(MixtureSpec):
    act = "silu"
    scores = "sigmoid"
    corrected = normalized = False
    grouped = True


@dataclass(frozen=True)
class Design:
    """What an architecture fixes beside its configuration."""

    mixers: dict                     # mixer types a layer may have -> their specs
    norms: str                       # "post_rms": x += mult * rms(f(x)); "sandwich": x += ln(f(ln(x))); "sandwich_rms": the
                                     # same with RMS norms whose weights are stored around zero; "post_group_rms": x += rms(f(x)) with
                                     # norms over groups of columns, then a weighted sum of all earlier results
    mlps: dict                       # feed-forward kinds a layer may have -> (form, spec); forms: "relu2": biased, two matrices; "geglu" /
                                     # "swiglu": gated by tanh-GELU / silu, no biases; "moe": mixture of experts
    keys: tuple                      # keys of config.json beside the common ones

    @property
    def sandwich(self) -> bool:
        return self.norms.startswith("sandwich")

    @property
    def latent(self) -> bool:
        """Whether layers share rings of latents."""
        return LatentAttentionSpec in self.mixers.values()

    @property
    def depth_average(self) -> bool:
        return self.norms == "post_group_rms"


DESIGNS = {
    "Gasovik": Design({"latent_attention": LatentAttentionSpec}, "post_rms", {"dense": ("relu2", DenseMLPSpec)}, ("residual_mult",)),
    "Fatudra": Design({"parallel": ParallelSpec, "mlstm": GatedMemorySpec}, "sandwich", {"dense": ("geglu", DenseMLPSpec)}, ("embedding", "loop")),
    "Dusilorn": Design({"attention": ChunkAttentionSpec, "attention_2": WindowAttentionSpec}, "sandwich_rms",
                       {"dense": ("swiglu", DenseMLPSpec), "moe": ("moe", MixtureSpec)}, ("embedding", "logit_scale")),
    "Bolovik": Design({"delta": DeltaMemorySpec, "attention": KeptWindowAttentionSpec}, "post_group_rms",
                      {"dense": ("geglu", DenseMLPSpec), "moe": ("moe", GroupedMixtureSpec)}, ()),
}
ARCHITECTURES = tuple(DESIGNS)


def is_layered(config: dict) -> bool:
    """Whether a parsed ``config.json`` describes a model of this family."""
    return config.get("architecture") in ARCHITECTURES


@dataclass(frozen=True)
class LayerSpec:
    type: str
    mixer: object                    # one of the specs of the design's ``mixers``
    mlp: Optional[object] = None     # one of the specs of its ``mlps``

    @classmethod
    def from_dict(cls, d: dict, design: Design) -> "LayerSpec":
        _take(d, ("type", "mixer", "mlp"), "layer")
        if d["type"] not in design.mixers:
            raise ValueError(f"unknown mixer type {d['type']!r}")
        mlp = d.get("mlp")
        if mlp is not None and mlp.get("kind") not in design.mlps:
            raise ValueError(f"unknown feed-forward kind {mlp.get('kind')!r}")
        return cls(d["type"], design.mixers[d["type"]].from_dict(d["mixer"]), None if mlp is None else design.mlps[mlp["kind"]][1].from_dict(mlp))

    @property
    def mlp_kind(self) -> str:
        return "moe" if isinstance(self.mlp, MixtureSpec) else "dense"

    def to_dict(self) -> dict:
        return {"type": self.type, "mixer": self.mixer.to_dict(), "mlp": None if self.mlp is None else self.mlp.to_dict()}


@dataclass(frozen=True)
class LayerRun:
    """One execution of a layer: ``index`` counts executions (caches belong to them), ``loop_pass`` is set on the first layer
    of a pass of the loop."""

    index: int
    layer: int
    loop_pass: Optional[int] = None


@dataclass
class LayeredConfig:
    architecture: str
    vocab: int
    width: int
    norm_eps: float
    residual_mult: float = 1.0
    layers: list = field(default_factory=list)
    name: str = ""
    embed_scale: float = 1.0
    loop: Optional[LoopSpec] = None
    logit_scale: float = 1.0
    norm_groups: int = 1

    def __post_init__(self):
        if self.architecture not in ARCHITECTURES:
            raise ValueError(f"Invalid architecture {self.architecture} provided.")
        if not self.layers:
            raise ValueError("a model needs at least one layer")
        for i, layer in enumerate(self.layers):
            if not isinstance(layer.mixer, self.design.mixers.get(layer.type, ())):
                raise ValueError(f"layer {i}: {self.architecture} has no mixer {layer.type!r}")
            if layer.mlp is not None and layer.mlp_kind not in self.design.mlps:
                raise ValueError(f"layer {i}: {self.architecture} has no feed-forward {layer.mlp_kind!r}")
            j = getattr(layer.mixer, "kv_from", None)
            if j is None:
                continue
            if not 0 <= j < i or self.layers[j].mixer.kv_from is not None:
                raise ValueError(f"layer {i}: kv_from {j} must name an earlier layer with latents of its own")
            a, b = layer.mixer, self.layers[j].mixer
            if (a.kv_rank, a.rot_dim, a.rot) != (b.kv_rank, b.rot_dim, b.rot):
                raise ValueError(f"layer {i}: latent size and rotation must equal those of layer {j}")
        if len({layer.mixer.v_width for layer in self.layers if getattr(layer.mixer, "v_mix", False)}) > 1:
            raise ValueError("layers that mix their values need equally many value rows")
        if self.norm_groups < 1 or self.width % self.norm_groups:
            raise ValueError(f"norm.groups must divide the width, {self.norm_groups} does not divide {self.width}")
        lp = self.loop
        if lp is not None and not (0 <= lp.start < lp.stop <= len(self.layers) and lp.times >= 1):
            raise ValueError(f"loop {lp} does not lie inside {len(self.layers)} layers")

    @property
    def architecture_class_name(self) -> str:
        return self.architecture

    @property
    def design(self) -> Design:
        return DESIGNS[self.architecture]

    @property
    def latent(self) -> bool:
        return self.design.latent

    def runs(self) -> list:
        """The executions of layers, in order."""
        lp, order = self.loop, []
        for i in range(len(self.layers)):
            if lp is not None and lp.start <= i < lp.stop:
                if i == lp.start:
                    order += [(k, t if k == lp.start else None) for t in range(lp.times) for k in range(lp.start, lp.stop)]
            else:
                order.append((i, None))
        return [LayerRun(n, i, t) for n, (i, t) in enumerate(order)]

    def mixes_values(self, i: int) -> Optional[str]:
        """"first": layer ``i`` provides the values that later layers mix in, "mix": it mixes them into its own, None: neither."""
        mixing = [k for k, layer in enumerate(self.layers) if getattr(layer.mixer, "v_mix", False)]
        return None if i not in mixing else "first" if i == mixing[0] else "mix"

    def kv_source(self, i: int) -> int:
        """The layer whose latents layer ``i`` attends to."""
        j = self.layers[i].mixer.kv_from
        return i if j is None else j

    def latent_windows(self) -> dict:
        """Source layer -> widest window among the layers that read its latents."""
        out: dict = {}
        for i, layer in enumerate(self.layers):
            s = self.kv_source(i)
            out[s] = max(out.get(s, 0), layer.mixer.window)
        return out

    def with_tensor_shapes(self, shape) -> "LayeredConfig":
        """Fill in the sizes that only the tensors give; ``shape(name)`` returns a checkpoint tensor's shape."""
        layers = []
        for i, layer in enumerate(self.layers):
            a = layer.mixer
            if isinstance(a, ParallelSpec) and a.left.bias_rows is None:
                a = replace(a, left=a.left.with_rows(shape(f"l{i}.mix.left.rel")[0]))
            layers.append(replace(layer, mixer=a))
        return replace(self, layers=layers)

    # -- construction ------------------------------------------------------------------------------------------------
    @classmethod
    def from_dict(cls, d: dict) -> "LayeredConfig":
        if not is_layered(d):
            raise ValueError(f"Invalid architecture {d.get('architecture')} provided.")
        design = DESIGNS[d["architecture"]]
        keys, groups = design.keys, 1
        _take(d, ("architecture", "vocab", "width", "norm", "layers", "name") + keys, "config")
        _take(d["norm"], ("eps",) + (("groups",) if design.depth_average else ()), "norm")
        if design.depth_average:
            groups = int(d["norm"].get("groups", 1))
        scale, loop = 1.0, None
        if "embedding" in keys:
            _take(d["embedding"], ("scale",), "embedding")
            scale = float(d["embedding"]["scale"])
        if d.get("loop") is not None:
            loop = LoopSpec.from_dict(d["loop"])
        mult = float(d["residual_mult"]) if "residual_mult" in keys else 1.0
        logit = float(d["logit_scale"]) if "logit_scale" in keys else 1.0
        return cls(d["architecture"], int(d["vocab"]), int(d["width"]), float(d["norm"]["eps"]), mult,
                   [LayerSpec.from_dict(x, design) for x in d["layers"]], d.get("name", ""), scale, loop, logit, groups)

    def to_dict(self) -> dict:
        out = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps}}
        keys = self.design.keys
        if self.design.depth_average:
            out["norm"]["groups"] = self.norm_groups
        if "residual_mult" in keys:
            out["residual_mult"] = self.residual_mult
        if "embedding" in keys:
            out["embedding"] = {"scale": self.embed_scale}
        if "logit_scale" in keys:
            out["logit_scale"] = self.logit_scale
        if self.loop is not None:
            out["loop"] = self.loop.to_dict()
        out["layers"] = [x.to_dict() for x in self.layers]
        if self.name:
            out["name"] = self.name
        return out

    @classmethod
    def from_name(cls, name: str) -> "LayeredConfig":
        from .. import registry

        return cls.from_dict(registry.lookup(name))

    @classmethod
    def from_pretrained(cls, path: str) -> "LayeredConfig":
        with open(os.path.join(path, "config.json"), encoding="utf-8") as f:
            return cls.from_dict(json.load(f))

    def save(self, path: str) -> None:
        os.makedirs(path, exist_ok=True)
        with open(os.path.join(path, "config.json"), "w", encoding="utf-8") as f:
            json.dump(self.to_dict(), f, indent=1)

    def construct_model(self, **kwargs):
        from . import build_model

        return build_model(self, **kwargs)

    # -- counts ------------------------------------------------------------------------------------------------------
    def active_param_count(self) -> int:
        """Parameters that a token meets: of a mixture of experts only those it can choose."""
        idle = (layer.mlp for layer in self.layers if isinstance(layer.mlp, MixtureSpec))
        return self.param_count() - sum(m.param_count(self.width) - m.active_params(self.width) for m in idle)

    def param_count(self) -> int:
        E = self.width
        if self.design.sandwich:
            norm = 2 * E if self.design.norms == "sandwich" else E
            n = 2 * self.vocab * E + norm + (0 if self.loop is None else self.loop.times * E)
            for layer in self.layers:
                n += layer.mixer.param_count(E) + 2 * norm + (0 if layer.mlp is None else layer.mlp.param_count(E) + 2 * norm)
            return n
        n = 2 * self.vocab * E + E
        if self.design.depth_average:
            for i, layer in enumerate(self.layers):
                n += layer.mixer.param_count(E) + E + i + 2 + (0 if layer.mlp is None else layer.mlp.param_count(E) + E)
            return n
        for i, layer in enumerate(self.layers):
            a = layer.mixer
            n += a.heads * ((a.dim + a.rot_dim) * E + 2 * a.vdim * E + (a.dim + a.vdim) * a.kv_rank) + E
            if a.kv_from is None:
                n += (a.kv_rank + a.rot_dim) * E + a.kv_rank
            if layer.mlp is not None:
                n += 2 * layer.mlp.ff * E + layer.mlp.ff + E + E
        return n
