"""Decoder-only models described layer by layer (``models/layered_config.py``).

A layer is a mixer and an optional feed-forward (``models/sublayers.py``).  How they read and add to the fp32 residual stream
is the design's norm style:

* "post_rms": a sublayer reads the stream itself; ``x += mult * rmsnorm(sublayer(x))``;
* "sandwich": ``x += layernorm(sublayer(layernorm(x)))``; one kernel adds a sublayer's output and norms the next one's input;
* "sandwich_rms": the same with RMS norms whose weights are stored around zero;
* "post_group_rms": as "post_rms", with norms over groups of columns, and at the end of a layer the stream is replaced by a weighted
  sum of the embedding output and all layer results so far.

The residual stream, norms, rotations, scores, softmax, gates of recurrences and recurrent state are fp32; matrix operands are
bf16 (serving) or fp32.  A range of layers may be executed several times (``LayeredConfig.runs``); every execution has its own
cache.

Execution forms, both over sequence rows of a ``RowCache``:

* ``forward_step``: packed prompt portions of any lengths;
* ``decode_step``: one token per row.
"""
from __future__ import annotations

import math
import os
from typing import Optional

import torch
import torch.nn as nn

from ..ops import depth as depth_ops
from ..ops import latent as ops
from ..ops import memory as mem_ops
from .kv_cache import HybridCache, LatentRingCache, RowCache
from .layered_config import LayeredConfig
from .sublayers import MIXERS, MLPS, DecodeContext, PackedStep, StepContext, rope_tables, vector, weight
from .weights import SafetensorsFile, save_safetensors


class LayerNorm(nn.Module):
    def __init__(self, width: int, device):
        super().__init__()
        self.w, self.b = vector(width, device), vector(width, device)

    @property
    def pair(self) -> tuple:
        return self.w, self.b

    def checkpoint_tensors(self, name: str) -> dict:
        return {name: self.w, name + ".b": self.b}


class CentredRMSNorm(nn.Module):
    """RMS norm times 1 + w."""

    def __init__(self, width: int, device):
        super().__init__()
        self.w = vector(width, device)

    @property
    def pair(self) -> tuple:
        return self.w, None

    def checkpoint_tensors(self, name: str) -> dict:
        return {name: self.w}


NORMS = {"sandwich": LayerNorm, "sandwich_rms": CentredRMSNorm}


class Layer(nn.Module):
    def __init__(self, cfg: LayeredConfig, i: int, dtype, device):
        super().__init__()
        spec = cfg.layers[i]
        self.mix = MIXERS[type(spec.mixer)](spec.mixer, cfg.width, cfg.norm_eps, dtype, device)
        self.mlp = None if spec.mlp is None else MLPS[cfg.design.mlps[spec.mlp_kind][0]](spec.mlp, cfg.width, dtype, device)
        names = ("norm1",) if self.mlp is None else ("norm1", "norm2")
        if cfg.design.sandwich:
            norm = NORMS[cfg.design.norms]
            self.norms = nn.ModuleDict({n + side: norm(cfg.width, device) for n in names for side in ("", "b")})   # before and after
        else:
            self.norms = nn.ParameterDict({n: vector(cfg.width, device) for n in names})
        self.dwa = vector(i + 2, device) if cfg.design.depth_average else None

    def checkpoint_tensors(self) -> dict:
        out: dict = {}
        for name, n in self.norms.items():
            out.update(n.checkpoint_tensors(name) if isinstance(n, nn.Module) else {name: n})
        if self.dwa is not None:
            out["dwa"] = self.dwa
        out.update({f"mix.{k}": v for k, v in self.mix.checkpoint_tensors().items()})
        if self.mlp is not None:
            out.update({f"mlp.{k}": v for k, v in self.mlp.checkpoint_tensors().items()})
        return out


# ------------------------------------------------------------------------------------------
# the model
# ------------------------------------------------------------------------------------------
class LayeredForCausalLM(nn.Module):
    def __init__(self, config: LayeredConfig, dtype: torch.dtype = torch.bfloat16, device="cpu"):
        super().__init__()
        assert dtype in (torch.bfloat16, torch.float32), dtype
        self.config, self.dtype = config, dtype
        self.embed = weight(config.vocab, config.width, dtype, device)
        self.layers = nn.ModuleList(Layer(config, i, dtype, device) for i in range(len(config.layers)))
        self.sandwich, self.depth_average = config.design.sandwich, config.design.depth_average
        self.final_norm = NORMS[config.design.norms](config.width, device) if self.sandwich else vector(config.width, device)
        self.head = weight(config.vocab, config.width, dtype, device)
        self.loop_step = None if config.loop is None else nn.Parameter(
            torch.zeros(config.loop.times, config.width, dtype=torch.float32, device=device), requires_grad=False)
        self.runs = config.runs()

    @property
    def device(self) -> torch.device:
        return self.embed.device

    # -- weights -----------------------------------------------------------------------------------------------------
    def checkpoint_tensors(self) -> dict:
        """Checkpoint name -> the view of this model's storage that holds it."""
        E = self.config.width
        out = {"embed": self.embed[:, :E], "head": self.head[:, :E]}
        out.update(self.final_norm.checkpoint_tensors("final.norm") if self.sandwich else {"final.norm": self.final_norm})
        if self.loop_step is not None:
            out["loop.step"] = self.loop_step
        for i, layer in enumerate(self.layers):
            out.update({f"l{i}.{k}": v for k, v in layer.checkpoint_tensors().items()})
        return out

    @torch.no_grad()
    def load_checkpoint(self, source) -> None:
        """``source``: a ``SafetensorsFile`` (or anything with ``keys``, ``shape`` and ``tensor``)."""
        want = self.checkpoint_tensors()
        unused = {f"l{i}.mix.{k}" for i, layer in enumerate(self.layers) for k in getattr(layer.mix, "unused_tensors", ())}
        missing, extra = sorted(set(want) - set(source.keys())), sorted(set(source.keys()) - set(want) - unused)
        if missing or extra:
            raise ValueError(f"checkpoint does not fit the configuration: missing {missing[:8]}, unexpected {extra[:8]}")
        for name, dst in want.items():
            if tuple(source.shape(name)) != tuple(dst.shape):
                raise ValueError(f"{name}: shape {tuple(source.shape(name))} in the checkpoint, {tuple(dst.shape)} in the configuration")
            dst.copy_(source.tensor(name))
        self.weights_changed()

    def weights_changed(self) -> None:
        """To be called after the stored tensors were written: what is derived from them follows."""
        for layer in self.layers:
            if hasattr(layer.mix, "weights_changed"):
                layer.mix.weights_changed()

    @classmethod
    def from_pretrained(cls, path: str, torch_dtype: torch.dtype = torch.bfloat16, device="cpu") -> "LayeredForCausalLM":
        source = SafetensorsFile(os.path.join(path, "model.safetensors"))
        model = cls(LayeredConfig.from_pretrained(path).with_tensor_shapes(source.shape), torch_dtype, device)
        model.load_checkpoint(source)
        return model

    def save_pretrained(self, path: str) -> None:
        """``config.json`` and ``model.safetensors`` with bf16 tensors."""
        self.config.save(path)
        save_safetensors(os.path.join(path, "model.safetensors"),
                         {k: v.to(torch.bfloat16) for k, v in self.checkpoint_tensors().items()})

    @torch.no_grad()
    def init_weights(self, seed: int = 0) -> "LayeredForCausalLM":
        """Random weights: matrices normal with deviation 1 / sqrt(fan in), norm factors one, biases zero (forget gates: spread
        over 3 .. 6, decays of delta memories: 1/16 .. 1 at a step of softplus(-2), so that memories of different length exist), mixed values half and
        half, sums over depth mostly the layer's own result."""
        g = torch.Generator(device=self.device).manual_seed(seed)
        zero = (".b", ".sink", ".correction") + ((".norm1", ".norm2", "b", "final.norm") if self.config.design.norms == "sandwich_rms" else ())
        for name, t in self.checkpoint_tensors().items():
            if name.endswith(".mix.f.b"):
                t.copy_(torch.linspace(3.0, 6.0, t.numel(), device=t.device))
            elif name.endswith(".mix.A_log"):
                t.copy_(torch.linspace(math.log(1 / 16), 0.0, t.numel(), device=t.device))
            elif name.endswith(".mix.dt_bias"):
                t.fill_(-2.0)
            elif name.endswith(".dwa"):
                t.fill_(0.5 / max(1, t.numel() - 1))
                t[-1] = 0.5
            elif t.dim() == 0:
                t.fill_(0.5)
            elif t.dim() == 1:
                t.fill_(0.0 if name.endswith(zero) else 1.0)
            else:
                std = 1.0 if name == "embed" else t.shape[1] ** -0.5
                t.copy_(torch.randn(t.shape, generator=g, device=self.device, dtype=torch.float32) * std)
        self.weights_changed()
        return self

    # -- plumbing ----------------------------------------------------------------------------------------------------
    def new_cache(self, max_rows: int, max_len: int) -> RowCache:
        if not self.config.latent:
            shapes = {(run.index, name): shape for run in self.runs
                      for name, shape in self.layers[run.layer].mix.cache_shapes(max_len).items()}
            cache = HybridCache(shapes, max_rows, max_len, self.device)
            cache.rope = self._rope(max_len)
            return cache
        windows = self.config.latent_windows()
        cache = LatentRingCache({i: self.layers[i].mix.layout for i in windows}, windows, max_rows, max_len, self.dtype, self.device)
        # kept with the cache: captured graphs hold the addresses of both
        cache.rope = self._rope(max_len)
        return cache

    def _rope(self, length: int) -> dict:
        specs = {rot: None for rot in (getattr(layer.mix.spec, "rot", None) for layer in self.layers) if rot is not None}
        return {rot: rope_tables(rot, length, self.device) for rot in specs}

    # -- execution ---------------------------------------------------------------------------------------------------
    def _step_vector(self, n: int):
        """What is added to the stream in front of execution ``n``."""
        t = self.runs[n].loop_pass if n < len(self.runs) else None
        return None if t is None else self.loop_step[t]

    def _start(self, tok):
        """Residual stream and the first sublayer's input."""
        c = self.config
        if self.depth_average:
            past = torch.empty(len(self.layers), tok.numel(), c.width, dtype=torch.float32, device=tok.device)
            _, h = ops.embed(tok, self.embed[:, :c.width], out=past[0])
            return depth_ops.DepthStream.begin(past), h
        if not self.sandwich:
            return ops.embed(tok, self.embed[:, :c.width])
        x, _ = ops.embed(tok, self.embed[:, :c.width], c.embed_scale, copy=False)
        first = self.layers[self.runs[0].layer].norms["norm1"].pair
        return x, mem_ops.sandwich_norm_(x, None, None, self._step_vector(0), first, c.norm_eps, self.dtype)

    def _add(self, x, n: int, name: str, out, part, clear=False, zero=None, final=False):
        """Add the output of sublayer ``name`` ("norm1": mixer, "norm2": feed-forward) of execution ``n`` to the stream; returns
        the next sublayer's input (after the last one: the normed input of the head with ``final``)."""
        c, layer = self.config, self.layers[self.runs[n].layer]
        if self.depth_average:
            end = name == ("norm1" if layer.mlp is None else "norm2")
            return depth_ops.depth_norm_(x, out, layer.norms[name], c.norm_groups, c.norm_eps, self.dtype, part.out_bias, clear, zero,
                                         layer.dwa if end else None)
        if not self.sandwich:
            return ops.rms_residual_(x, out, part.out_bias, layer.norms[name], c.norm_eps, c.residual_mult, self.dtype, clear, zero)
        step, pre = None, None
        if name == "norm1" and layer.mlp is not None:
            pre = layer.norms["norm2"].pair
        elif n + 1 < len(self.runs):
            step, pre = self._step_vector(n + 1), self.layers[self.runs[n + 1].layer].norms["norm1"].pair
        elif final:
            pre = self.final_norm.pair
        last = name == ("norm1" if layer.mlp is None else "norm2") and n + 1 == len(self.runs)
        return mem_ops.sandwich_norm_(x, out, layer.norms[name + "b"].pair, step, pre, c.norm_eps, self.dtype, part.out_bias,
                                      part.out_bias_mult, clear, zero, c.logit_scale if last else 1.0)

    def _logits(self, x, idx, h=None):
        """``h``: the final norm of all rows, where it is formed already.  The logits' factor is part of that norm."""
        c = self.config
        if self.depth_average:
            h = depth_ops.group_norm_rows(x.x, idx, self.final_norm, c.norm_groups, c.norm_eps, self.dtype)
        elif h is None:
            h = mem_ops.norm_rows(x, idx, *self.final_norm.pair, c.norm_eps, self.dtype, c.logit_scale) if self.sandwich else \
                ops.rmsnorm_rows(x, idx, self.final_norm, c.norm_eps, self.dtype)
        return ops.linear(h, self.head[:, :c.width], out_f32=True)

    @torch.no_grad()
    def forward_step(self, step: PackedStep, cache: Optional[RowCache], want: Optional[list] = None,
                     hidden: Optional[list] = None) -> Optional[torch.Tensor]:
        """Run the portions of ``step``; fp32 logits [len(want), vocab] of the packed token indices ``want`` (None: all tokens;
        empty: nothing is computed past the last layer).  ``hidden`` collects the residual stream after every execution of a
        layer.  Without a cache the portions are whole sequences and nothing is kept."""
        ctx = StepContext(self.config, step, cache)
        if not self.config.latent and cache is None:
            ctx.cache = self.new_cache(1 + max(r for r, _, _ in step.portions), max(n for _, _, n in step.portions))
        elif self.config.latent:
            ctx.windows = self.config.latent_windows()
        ctx.rope = ctx.cache.rope if ctx.cache is not None else self._rope(max(s + n for _, s, n in step.portions))
        x, h = self._start(step.tok)
        for n, run in enumerate(self.runs):
            layer = self.layers[run.layer]
            before = None if hidden is None else self._step_vector(n + 1)
            h = self._add(x, n, "norm1", layer.mix.stream(h, run, ctx), layer.mix)
            if layer.mlp is not None:
                h = self._add(x, n, "norm2", layer.mlp(h), layer.mlp)
            if hidden is not None:
                stream = x.x if self.depth_average else x
                hidden.append(stream.clone() if before is None else stream - before)     # the stream already holds the next pass's vector
        if want is not None and not len(want):
            return None
        idx = None if want is None else torch.tensor(want, dtype=torch.int32).to(self.device)
        return self._logits(x, idx)

    @torch.no_grad()
    def decode_step(self, tok, pos, row, cache: RowCache, dense, splits) -> torch.Tensor:
        """One token per row: ids [B] at positions [B] of cache rows [B] -> fp32 logits [B, vocab]."""
        ctx = DecodeContext(self.config, pos, row, cache, dense, splits)
        x, h = self._start(tok)
        for n, run in enumerate(self.runs):
            layer = self.layers[run.layer]
            out, clear, acc = layer.mix.decode(h, run, ctx)
            h = self._add(x, n, "norm1", out, layer.mix, clear, acc, final=True)
            if layer.mlp is not None:
                out, clear = layer.mlp.decode(h, dense)
                h = self._add(x, n, "norm2", out, layer.mlp, clear, final=True)
        return self._logits(x, None, h if self.sandwich else None)

    @torch.no_grad()
    def forward(self, input_ids: torch.Tensor) -> torch.Tensor:
        """fp32 logits [B, S, vocab] of whole sequences, without a cache."""
        B, S = input_ids.shape
        step = PackedStep([(b, 0, input_ids[b].tolist()) for b in range(B)], self.device)
        return self.forward_step(step, None).view(B, S, -1)

    @torch.no_grad()
    def generate(self, input_ids, max_new_tokens: int = 20, stop_ids=(), **sampling):
        """Continuations through the serving engine.  ``input_ids``: [B, S] tensor (result: [B, S + new], every row of the same
        length) or a list of token lists of any lengths (result: list of token lists)."""
        from ..engine.layered import LayeredEngine

        ragged = not torch.is_tensor(input_ids)
        prompts = [list(p) for p in input_ids] if ragged else input_ids.tolist()
        engine = LayeredEngine(self, max_batch=len(prompts), max_len=max(len(p) for p in prompts) + max_new_tokens)
        outs = engine.generate(prompts, max_new_tokens, stop_ids=stop_ids if ragged else (), **sampling)
        if ragged:
            return [p + o for p, o in zip(prompts, outs)]
        return torch.cat([input_ids, torch.tensor(outs, dtype=input_ids.dtype, device=input_ids.device)], dim=1)
