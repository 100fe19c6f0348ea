"""Decoder-only models described layer by layer (``models/layered_config.py``).

A layer is a mixer and an optional feed-forward, each reading the residual stream itself; a sublayer's output is normed,
scaled by ``residual_mult`` and added: ``x += mult * norm(sublayer(x))``.  The residual stream, norms, rotations, scores
and softmax are fp32; matrix operands are bf16 (serving) or fp32.

Execution forms, both over sequence rows of a ``LatentRingCache``:

* ``forward_step``: packed prompt portions of any lengths.  Keys and values are up-projected from the step's latent
  stream (the portion's own latents behind the cached ones its windows reach back to).
* ``decode_step``: one token per row.  Scores are taken against the cached latents themselves (q is carried through the key
  up-projection, the weighted latents through the value up-projection), so a step reads one latent row per key for all
  heads.

Weights are stored as they are executed: the projections that read the same input are one matrix ([q | gate | latent],
[key | value] up-projection), with row pitches padded to eight elements.  ``checkpoint_tensors`` names the views that
make up a checkpoint.
"""
from __future__ import annotations

import os
from dataclasses import dataclass
from typing import Optional

import torch
import torch.nn as nn

from ..ops import latent as ops
from ..ops.latent import LatentLayout, pad8
from .kv_cache import LatentRingCache
from .layered_config import DenseMLPSpec, LatentAttentionSpec, LayeredConfig, RotarySpec
from .weights import SafetensorsFile, save_safetensors


def _weight(rows: int, cols: int, dtype, device) -> nn.Parameter:
    """[rows, cols] matrix with a zero-filled row pitch that is a multiple of eight."""
    return nn.Parameter(torch.zeros(rows, pad8(cols), dtype=dtype, device=device), requires_grad=False)


def _vector(n: int, device) -> nn.Parameter:
    return nn.Parameter(torch.zeros(n, dtype=torch.float32, device=device), requires_grad=False)


def rope_tables(rot: RotarySpec, length: int, device) -> tuple:
    """cos / sin [length, dims / 2] of the spec's (interpolated) frequencies, times its magnitude.  The angles are formed in
    double precision and stored as fp32."""
    ang = torch.outer(torch.arange(length, dtype=torch.float64), torch.tensor(rot.frequencies(), dtype=torch.float64))
    return tuple((f(ang) * rot.magnitude).float().contiguous().to(device) for f in (torch.cos, torch.sin))


# ------------------------------------------------------------------------------------------
# one packed step
# ------------------------------------------------------------------------------------------
@dataclass
class StreamLayout:
    """Where the keys of a packed step lie for a given history length: per sequence first the cached positions its portion can
    still see, then the portion itself."""

    sidx: torch.Tensor        # [T] stream index of every token
    kbase: torch.Tensor       # [T] stream index of the first key of its sequence
    seqs: list                # (first token, tokens, first key, history) per sequence
    total: int
    history: list             # (row, first position, count, first key) of the sequences with history


class PackedStep:
    """Token ids and positions of a batch of prompt portions; ``portions`` are (row, first position, token ids)."""

    def __init__(self, portions: list, device):
        self.device, self.portions = torch.device(device), [(r, s, len(t)) for r, s, t in portions]
        tok, pos, row, end = [], [], [], []
        for r, s, t in portions:
            n = len(t)
            tok.extend(t)
            pos.extend(range(s, s + n))
            row.extend([r] * n)
            end.extend([s + n] * n)
        self.tok = torch.tensor(tok, dtype=torch.int64).to(self.device)
        meta = torch.tensor([pos, row, end], dtype=torch.int32).to(self.device)
        self.pos, self.row, self.end = meta[0], meta[1], meta[2]
        self.T = len(tok)
        self._layouts: dict = {}

    def layout(self, history: int) -> StreamLayout:
        """Layout with up to ``history`` cached positions in front of every portion."""
        if all(s == 0 for _, s, _ in self.portions):
            history = 0
        if history not in self._layouts:
            seqs, sidx, kbase, hist = [], [], [], []
            t0 = k0 = 0
            for r, s, n in self.portions:
                h = min(s, history)
                seqs.append((t0, n, k0, h))
                sidx.extend(range(k0 + h, k0 + h + n))
                kbase.extend([k0] * n)
                if h:
                    hist.append((r, s - h, h, k0))
                t0, k0 = t0 + n, k0 + h + n
            idx = torch.tensor([sidx, kbase], dtype=torch.int32).to(self.device)
            self._layouts[history] = StreamLayout(idx[0], idx[1], seqs, k0, hist)
        return self._layouts[history]


def gather_history(layout: StreamLayout, cache: torch.Tensor, stream: torch.Tensor) -> None:
    """Copy the cached latents in front of every portion from the ring ``cache`` [rows, cap, ld] into the stream."""
    if not layout.history:
        return
    cap = cache.shape[1]
    src, dst = [], []
    for row, p0, n, k0 in layout.history:
        src.extend(row * cap + (p % cap) for p in range(p0, p0 + n))
        dst.extend(range(k0, k0 + n))
    idx = torch.tensor([src, dst], dtype=torch.int32).to(cache.device)
    ops.gather_rows(cache.view(-1, cache.shape[2]), idx[0], stream, idx[1])


# ------------------------------------------------------------------------------------------
# sublayers
# ------------------------------------------------------------------------------------------
class LatentAttention(nn.Module):
    """Windowed attention over per-token latents with gated heads; see ``LatentAttentionSpec``."""

    def __init__(self, spec: LatentAttentionSpec, width: int, eps: float, dtype, device):
        super().__init__()
        a = spec
        self.spec, self.width, self.eps, self.dtype = spec, width, eps, dtype
        L = self.layout = LatentLayout(a.heads, a.dim, a.rot_dim, a.vdim, a.kv_rank, a.kv_from is None)
        self.w_in = _weight(L.width_in, width, dtype, device)
        self.w_kv = _weight(L.width_kv, a.kv_rank, dtype, device)
        self.w_o = _weight(width, a.heads * a.vdim, dtype, device)
        self.latent_norm = _vector(a.kv_rank, device) if L.own else None

    def checkpoint_tensors(self) -> dict:
        a, L, E = self.spec, self.layout, self.width
        out = {"q": self.w_in[:a.heads * (a.dim + a.rot_dim), :E], "g": self.w_in[L.off_g:L.off_g + a.heads * a.vdim, :E],
               "uk": self.w_kv[:a.heads * a.dim, :a.kv_rank], "uv": self.w_kv[L.off_v:L.off_v + a.heads * a.vdim, :a.kv_rank],
               "o": self.w_o[:, :a.heads * a.vdim]}
        if L.own:
            out["dkv"] = self.w_in[L.off_d:L.off_d + a.kv_rank + a.rot_dim, :E]
            out["dkv.norm"] = self.latent_norm
        return out

    def project_stream(self, xb, step: PackedStep, cache, stream, lay: StreamLayout, rope):
        """The portion's projection rows (q rotated); appends the latents of an own layer to ``stream`` and the ring."""
        inp = ops.linear(xb, self.w_in[:, :self.width])
        if self.layout.own and cache is not None:
            gather_history(lay, cache, stream)     # before the ring slots of the oldest positions are written again
        ops.latent_prep_(self.layout, inp, self.latent_norm, self.eps, rope, step, lay.sidx, cache if self.layout.own else None,
                         stream)
        return inp

    def stream(self, xb, step: PackedStep, cache, stream, lay: StreamLayout, rope):
        a = self.spec
        inp = self.project_stream(xb, step, cache, stream, lay, rope)
        kv = ops.linear(stream[:, :a.kv_rank], self.w_kv[:, :a.kv_rank])
        o = ops.stream_attention(self.layout, inp, kv, stream, lay, a.window, a.scale)
        return ops.linear(o, self.w_o[:, :a.heads * a.vdim])

    def decode(self, xb, pos, row, cache, rope, dense, splits: int):
        """One token per row; ``dense(x, w, which)`` is the engine's narrow-batch product.  Returns the sublayer
        output, whether it is an accumulator that the next kernel clears, and the projection's accumulator or None."""
        a = self.spec
        inp, acc = dense(xb, self.w_in[:, :self.width], 0)
        o = ops.ring_attention(self.layout, inp, self.w_kv, self.latent_norm, self.eps, rope, pos, row, cache,
                               min(a.window, cache.shape[1]), a.scale, splits, self.dtype)
        out, clear = dense(o, self.w_o[:, :a.heads * a.vdim], 1)
        return out, clear, inp if acc else None


class DenseMLP(nn.Module):
    """down(relu(up x)^2) with biases; the bias of the down projection is added by the norm that follows."""

    act = "relu2"

    def __init__(self, spec: DenseMLPSpec, width: int, dtype, device):
        super().__init__()
        self.spec, self.width, self.dtype = spec, width, dtype
        self.w_up, self.b_up = _weight(spec.ff, width, dtype, device), _vector(spec.ff, device)
        self.w_down, self.b_down = _weight(width, spec.ff, dtype, device), _vector(width, device)

    def checkpoint_tensors(self) -> dict:
        return {"up": self.w_up[:, :self.width], "up.b": self.b_up, "down": self.w_down[:, :self.spec.ff], "down.b": self.b_down}

    def forward(self, xb):
        return ops.linear(ops.linear(xb, self.w_up[:, :self.width], self.b_up, self.act), self.w_down[:, :self.spec.ff])

    def decode(self, xb, dense):
        h, clear = dense(xb, self.w_up[:, :self.width], 1)
        h = ops.bias_act(h, self.b_up, self.act, self.dtype, clear)
        return dense(h, self.w_down[:, :self.spec.ff], 1)


class Layer(nn.Module):
    def __init__(self, cfg: LayeredConfig, i: int, dtype, device):
        super().__init__()
        spec = cfg.layers[i]
        self.mix = LatentAttention(spec.mixer, cfg.width, cfg.norm_eps, dtype, device)
        self.norm1 = _vector(cfg.width, device)
        self.mlp = None if spec.mlp is None else DenseMLP(spec.mlp, cfg.width, dtype, device)
        self.norm2 = None if spec.mlp is None else _vector(cfg.width, device)

    def checkpoint_tensors(self) -> dict:
        out = {"norm1": self.norm1}
        out.update({f"mix.{k}": v for k, v in self.mix.checkpoint_tensors().items()})
        if self.mlp is not None:
            out["norm2"] = self.norm2
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
        self.embed = _weight(config.vocab, config.width, dtype, device)
        self.layers = nn.ModuleList(Layer(config, i, dtype, device) for i in range(len(config.layers)))
        self.final_norm = _vector(config.width, device)
        self.head = _weight(config.vocab, config.width, dtype, device)

    @property
    def device(self) -> torch.device:
        return self.embed.device

    # -- weights -----------------------------------------------------------------------------------------------------
    def checkpoint_tensors(self) -> dict:
        """Checkpoint name -> the view of this model's storage that holds it."""
        E = self.config.width
        out = {"embed": self.embed[:, :E], "final.norm": self.final_norm, "head": self.head[:, :E]}
        for i, layer in enumerate(self.layers):
            out.update({f"l{i}.{k}": v for k, v in layer.checkpoint_tensors().items()})
        return out

    @torch.no_grad()
    def load_checkpoint(self, source) -> None:
        """``source``: a ``SafetensorsFile`` (or anything with ``keys``, ``shape`` and ``tensor``)."""
        want = self.checkpoint_tensors()
        missing, extra = sorted(set(want) - set(source.keys())), sorted(set(source.keys()) - set(want))
        if missing or extra:
            raise ValueError(f"checkpoint does not fit the configuration: missing {missing[:8]}, unexpected {extra[:8]}")
        for name, dst in want.items():
            if tuple(source.shape(name)) != tuple(dst.shape):
                raise ValueError(f"{name}: shape {tuple(source.shape(name))} in the checkpoint, {tuple(dst.shape)} in the configuration")
            dst.copy_(source.tensor(name))

    @classmethod
    def from_pretrained(cls, path: str, torch_dtype: torch.dtype = torch.bfloat16, device="cpu") -> "LayeredForCausalLM":
        model = cls(LayeredConfig.from_pretrained(path), torch_dtype, device)
        model.load_checkpoint(SafetensorsFile(os.path.join(path, "model.safetensors")))
        return model

    def save_pretrained(self, path: str) -> None:
        """``config.json`` and ``model.safetensors`` with bf16 tensors."""
        self.config.save(path)
        save_safetensors(os.path.join(path, "model.safetensors"),
                         {k: v.to(torch.bfloat16) for k, v in self.checkpoint_tensors().items()})

    @torch.no_grad()
    def init_weights(self, seed: int = 0) -> "LayeredForCausalLM":
        """Random weights: matrices normal with deviation 1 / sqrt(fan in), norm weights one, biases zero."""
        g = torch.Generator(device=self.device).manual_seed(seed)
        for name, t in self.checkpoint_tensors().items():
            if t.dim() == 1:
                t.fill_(0.0 if name.endswith(".b") else 1.0)
            else:
                std = 1.0 if name == "embed" else t.shape[1] ** -0.5
                t.copy_(torch.randn(t.shape, generator=g, device=self.device, dtype=torch.float32) * std)
        return self

    # -- plumbing ----------------------------------------------------------------------------------------------------
    def new_cache(self, max_rows: int, max_len: int) -> LatentRingCache:
        windows = self.config.latent_windows()
        cache = LatentRingCache({i: self.layers[i].mix.layout for i in windows}, windows, max_rows, max_len, self.dtype, self.device)
        # kept with the cache: captured graphs hold the addresses of both
        cache.rope = {layer.mix.spec.rot: None for layer in self.layers}
        for rot in cache.rope:
            cache.rope[rot] = rope_tables(rot, max_len, self.device)
        return cache

    # -- execution ---------------------------------------------------------------------------------------------------
    def _residual(self, layer_norm, x, out, bias, clear=False, zero=None):
        c = self.config
        return ops.rms_residual_(x, out, bias, layer_norm, c.norm_eps, c.residual_mult, self.dtype, clear, zero)

    def _logits(self, x, idx):
        h = ops.rmsnorm_rows(x, idx, self.final_norm, self.config.norm_eps, self.dtype)
        return ops.linear(h, self.head[:, :self.config.width], out_f32=True)

    @torch.no_grad()
    def forward_step(self, step: PackedStep, cache: Optional[LatentRingCache], want: Optional[list] = None,
                     hidden: Optional[list] = None) -> Optional[torch.Tensor]:
        """Run the portions of ``step``; fp32 logits [len(want), vocab] of the packed token indices ``want`` (None: all tokens;
        empty: nothing is computed past the last layer).  ``hidden`` collects the residual stream after every layer."""
        c = self.config
        last = max(s + n for _, s, n in step.portions)
        windows, streams = c.latent_windows(), {}
        tables = cache.rope if cache is not None else \
            {rot: rope_tables(rot, last, self.device) for rot in {layer.mix.spec.rot for layer in self.layers}}
        x, xb = ops.embed(step.tok, self.embed[:, :c.width])
        for i, layer in enumerate(self.layers):
            src = c.kv_source(i)
            lay = step.layout(windows[src] - 1)
            if src == i:
                streams[i] = torch.empty(lay.total, layer.mix.layout.ld_lat, dtype=self.dtype, device=self.device)
            out = layer.mix.stream(xb, step, cache.data[src] if cache is not None else None, streams[src], lay,
                                   tables[layer.mix.spec.rot])
            xb = self._residual(layer.norm1, x, out, None)
            if layer.mlp is not None:
                xb = self._residual(layer.norm2, x, layer.mlp(xb), layer.mlp.b_down)
            if hidden is not None:
                hidden.append(x.clone())
        if want is not None and not len(want):
            return None
        idx = None if want is None else torch.tensor(want, dtype=torch.int32).to(self.device)
        return self._logits(x, idx)

    @torch.no_grad()
    def decode_step(self, tok, pos, row, cache: LatentRingCache, dense, splits) -> torch.Tensor:
        """One token per row: ids [B] at positions [B] of cache rows [B] -> fp32 logits [B, vocab]."""
        c = self.config
        x, xb = ops.embed(tok, self.embed[:, :c.width])
        for i, layer in enumerate(self.layers):
            src = c.kv_source(i)
            out, clear, acc = layer.mix.decode(xb, pos, row, cache.data[src], cache.rope[layer.mix.spec.rot], dense,
                                               splits(layer.mix, tok.numel()))
            xb = self._residual(layer.norm1, x, out, None, clear, acc)
            if layer.mlp is not None:
                out, clear = layer.mlp.decode(xb, dense)
                xb = self._residual(layer.norm2, x, out, layer.mlp.b_down, clear)
        return self._logits(x, None)

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
