"""Configuration of decoder-only models that are described layer by layer.

``config.json`` of such a model names its ``architecture`` and lists its layers; every entry carries the layer's mixer
``type``, the mixer's own sizes and constants and its feed-forward (or null).  The classes here validate that
description and derive shapes; ``models/layered.py`` builds the modules from it.

Architectures:

* ``Gasovik``: latent attention under a sliding window (optionally on the latents of an earlier layer), gated heads,
  biased squared-ReLU feed-forward, norms on the sublayer outputs only.
"""
from __future__ import annotations

import json
import math
import os
from dataclasses import dataclass, field
from typing import Optional

ARCHITECTURES = ("Gasovik",)


def is_layered(config: dict) -> bool:
    """Whether a parsed ``config.json`` describes a model of this family."""
    return config.get("architecture") in ARCHITECTURES


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


@dataclass(frozen=True)
class RotarySpec:
    base: float
    dims: int
    scaling: Optional[YarnScaling] = None

    def frequencies(self) -> list:
        """Radians per position of every interleaved pair."""
        f = [self.base ** (-2 * i / self.dims) for i in range(self.dims // 2)]
        if self.scaling is None:
            return f
        return [v / self.scaling.factor * r + v * (1 - r) for v, r in zip(f, self.scaling.ramp(self.dims, self.base))]

    @property
    def magnitude(self) -> float:
        return 1.0 if self.scaling is None else self.scaling.magnitude

    @classmethod
    def from_dict(cls, d: dict) -> "RotarySpec":
        _take(d, ("base", "dims", "scaling"), "rot")
        sc = d.get("scaling")
        if sc is not None:
            _take(sc, ("factor", "original", "fast", "slow"), "rot.scaling")
            sc = YarnScaling(float(sc["factor"]), float(sc["original"]), float(sc["fast"]), float(sc["slow"]))
        if d["dims"] <= 0 or d["dims"] % 2:
            raise ValueError(f"rot.dims must be a positive even number, not {d['dims']}")
        return cls(float(d["base"]), int(d["dims"]), sc)

    def to_dict(self) -> dict:
        out = {"base": self.base, "dims": self.dims}
        if self.scaling is not None:
            s = self.scaling
            out["scaling"] = {"factor": s.factor, "original": s.original, "fast": s.fast, "slow": s.slow}
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
class DenseMLPSpec:
    ff: int

    @classmethod
    def from_dict(cls, d: dict) -> "DenseMLPSpec":
        _take(d, ("kind", "ff"), "mlp")
        if d.get("kind") != "dense":
            raise ValueError(f"unknown feed-forward kind {d.get('kind')!r}")
        return cls(int(d["ff"]))

    def to_dict(self) -> dict:
        return {"kind": "dense", "ff": self.ff}


MIXERS = {"latent_attention": LatentAttentionSpec}


@dataclass(frozen=True)
class LayerSpec:
    type: str
    mixer: LatentAttentionSpec
    mlp: Optional[DenseMLPSpec] = None

    @classmethod
    def from_dict(cls, d: dict) -> "LayerSpec":
        _take(d, ("type", "mixer", "mlp"), "layer")
        if d["type"] not in MIXERS:
            raise ValueError(f"unknown mixer type {d['type']!r}")
        mlp = d.get("mlp")
        return cls(d["type"], MIXERS[d["type"]].from_dict(d["mixer"]), None if mlp is None else DenseMLPSpec.from_dict(mlp))

    def to_dict(self) -> dict:
        return {"type": self.type, "mixer": self.mixer.to_dict(), "mlp": None if self.mlp is None else self.mlp.to_dict()}


@dataclass
class LayeredConfig:
    architecture: str
    vocab: int
    width: int
    norm_eps: float
    residual_mult: float
    layers: list = field(default_factory=list)
    name: str = ""

    def __post_init__(self):
        if self.architecture not in ARCHITECTURES:
            raise ValueError(f"Invalid architecture {self.architecture} provided.")
        if not self.layers:
            raise ValueError("a model needs at least one layer")
        for i, layer in enumerate(self.layers):
            j = layer.mixer.kv_from
            if j is None:
                continue
            if not 0 <= j < i or self.layers[j].mixer.kv_from is not None:
                raise ValueError(f"layer {i}: kv_from {j} must name an earlier layer with latents of its own")
            a, b = layer.mixer, self.layers[j].mixer
            if (a.kv_rank, a.rot_dim, a.rot) != (b.kv_rank, b.rot_dim, b.rot):
                raise ValueError(f"layer {i}: latent size and rotation must equal those of layer {j}")

    @property
    def architecture_class_name(self) -> str:
        return self.architecture

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

    # -- construction ------------------------------------------------------------------------------------------------
    @classmethod
    def from_dict(cls, d: dict) -> "LayeredConfig":
        _take(d, ("architecture", "vocab", "width", "norm", "residual_mult", "layers", "name"), "config")
        _take(d["norm"], ("eps",), "norm")
        return cls(d["architecture"], int(d["vocab"]), int(d["width"]), float(d["norm"]["eps"]), float(d["residual_mult"]),
                   [LayerSpec.from_dict(x) for x in d["layers"]], d.get("name", ""))

    def to_dict(self) -> dict:
        out = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
               "residual_mult": self.residual_mult, "layers": [x.to_dict() for x in self.layers]}
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
    def param_count(self) -> int:
        n = 2 * self.vocab * self.width + self.width
        for i, layer in enumerate(self.layers):
            a, E = layer.mixer, self.width
            n += a.heads * ((a.dim + a.rot_dim) * E + 2 * a.vdim * E + (a.dim + a.vdim) * a.kv_rank) + E
            if a.kv_from is None:
                n += (a.kv_rank + a.rot_dim) * E + a.kv_rank
            if layer.mlp is not None:
                n += 2 * layer.mlp.ff * E + layer.mlp.ff + E + E
        return n
