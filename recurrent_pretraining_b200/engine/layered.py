"""Serving engine of the layered decoder models: sequence rows, packed prompt steps, graph-replayed decode steps, sampling.

A batch may mix sequences of any lengths.  ``step`` takes each sequence's next tokens -- a prompt, a portion of one, or
a single token -- and returns the logits that were asked for; ``generate`` is a loop over the same steps.

* Prompt portions are packed without padding (``forward_step``).
* One token per sequence is a decode step: weight-streaming GEMMs with fp32 accumulators that fused consumers read and
  clear, attention over the cache and updates of recurrent state, everything captured as one CUDA graph per batch size.
"""
from __future__ import annotations

from typing import Optional

import torch

from ..models.layered import LayeredForCausalLM, PackedStep
from ..models.sampling import SamplingOptions, apply_repetition_penalty, sample_next_token
from .base import SKINNY_ROWS, GraphRunner, skinny_linear


class LayeredEngine(GraphRunner):
    def __init__(self, model: LayeredForCausalLM, max_batch: int = 8, max_len: int = 4096, use_graphs: bool = True,
                 prefill_tokens: int = 16384):
        self.model, self.cfg = model, model.config
        self.dev = model.device
        self.max_len, self.prefill_tokens = max_len, prefill_tokens
        self.cache = model.new_cache(max_batch, max_len)
        self.on_gpu = self.dev.type == "cuda"
        self.use_graphs = use_graphs and self.on_gpu
        self._graphs: dict = {}
        self._generation = self.cache.generation
        n = SKINNY_ROWS
        self._tok = torch.zeros(n, dtype=torch.int64, device=self.dev)
        self._meta = torch.zeros(2, n, dtype=torch.int32, device=self.dev)      # positions, cache rows
        # accumulators of the stream-K GEMMs, zero between uses: 0 = the mixer's input projection (read until the end of the
        # attention), 1 = every other product (cleared by its one consumer)
        self._work = [None, None]
        if self.on_gpu and model.dtype == torch.bfloat16:
            widths = [max(m.mix.layout.width_in for m in model.layers),
                      max([self.cfg.width] + [m.mlp.spec.ff * m.mlp.wide for m in model.layers if m.mlp is not None])]
            self._work = [torch.zeros(n * w, dtype=torch.float32, device=self.dev) for w in widths]

    # -- sequences ---------------------------------------------------------------------------------------------------
    def open(self) -> int:
        """A cache row for a new sequence."""
        return self.cache.alloc()

    def close(self, row: int) -> None:
        self.cache.free(row)

    # -- steps -------------------------------------------------------------------------------------------------------
    def step(self, entries: list, want: Optional[list] = None) -> Optional[torch.Tensor]:
        """Run each entry's next tokens: ``entries`` are (row, token ids), ``want`` the places among an entry's tokens whose
        logits are returned, in order, as fp32 [n, vocab] (default: the last place of every entry)."""
        if want is None:
            want = [[len(t) - 1] for _, t in entries]
        for (row, toks), places in zip(entries, want):
            if not toks or min(toks) < 0 or max(toks) >= self.cfg.vocab:
                raise ValueError("an entry needs at least one token, all inside the vocabulary")
            if any(not 0 <= w < len(toks) for w in places):
                raise ValueError("a wanted place lies outside the entry's tokens")
        if len({row for row, _ in entries}) != len(entries):
            raise ValueError("a sequence appears twice in one step")
        portions = [(row, self.cache.advance(row, len(t)), t) for row, t in entries]
        if all(len(t) == 1 for _, _, t in portions):
            logits = [self._decode(portions[i:i + SKINNY_ROWS]) for i in range(0, len(portions), SKINNY_ROWS)]
            picks = [i for i, w in enumerate(want) for _ in w]
            if not picks:
                return None
            logits = logits[0] if len(logits) == 1 else torch.cat(logits)
            return logits[torch.tensor(picks, device=self.dev)] if picks != list(range(len(portions))) else logits
        flat, t0 = [], 0
        for (_, _, t), w in zip(portions, want):
            flat.extend(t0 + k for k in w)
            t0 += len(t)
        return self.model.forward_step(PackedStep(portions, self.dev), self.cache, flat)

    def _decode(self, portions: list) -> torch.Tensor:
        B = len(portions)
        host = torch.tensor([[t[0] for _, _, t in portions], [s for _, s, _ in portions], [r for r, _, _ in portions]])
        self._tok[:B].copy_(host[0])
        self._meta[:, :B].copy_(host[1:])
        out = self._decode_graph(B)
        return out.clone() if self.use_graphs else out      # the graph's output buffer is written again by its next replay

    def _decode_graph(self, B: int) -> torch.Tensor:
        if self._generation != self.cache.generation:       # the cache has moved
            self._graphs.clear()
            self._generation = self.cache.generation
        tok, pos, row = self._tok[:B], self._meta[0, :B], self._meta[1, :B]
        return self._run(("decode", B), lambda: self.model.decode_step(tok, pos, row, self.cache, self._dense, self._splits),
                         once=True)

    def _dense(self, x, w, which: int):
        """Narrow-batch product -> (result, whether it is a persistent accumulator that its consumer has to clear)."""
        if not self.on_gpu or x.dtype != torch.bfloat16:
            from ..ops import latent as ops

            return ops.linear(x, w), False
        y = skinny_linear(x, w, self._work[which], keep_f32=True, ld_out=(w.shape[0] + 7) // 8 * 8)
        return y, y.dtype == torch.float32

    def _splits(self, mix, B: int) -> int:
        """Key splits of the decode attention."""
        return mix.decode_splits(B, self.max_len, self.on_gpu and self.model.dtype == torch.bfloat16)

    # -- generation --------------------------------------------------------------------------------------------------
    def prefill(self, rows: list, prompts: list) -> torch.Tensor:
        """Process the prompts (in portions of at most ``prefill_tokens`` packed tokens); logits of their last tokens."""
        last = [None] * len(rows)
        done = [0] * len(rows)
        while any(d < len(p) for d, p in zip(done, prompts)):
            entries, who, room = [], [], self.prefill_tokens
            for i, p in enumerate(prompts):
                n = min(len(p) - done[i], room)
                if n > 0:
                    entries.append((rows[i], p[done[i]:done[i] + n]))
                    who.append(i)
                    done[i] += n
                    room -= n
            ends = [i for i in who if done[i] == len(prompts[i])]
            want = [[len(t) - 1] if done[i] == len(prompts[i]) else [] for i, (_, t) in zip(who, entries)]
            logits = self.step(entries, want)
            for k, i in enumerate(ends):
                last[i] = logits[k]
        return torch.stack(last)

    @torch.no_grad()
    def generate(self, prompts: list, max_new_tokens: int, stop_ids=(), check_every: int = 8, generator=None, **sampling) -> list:
        """Continuations (lists of new token ids) of prompts of any lengths.  A sequence ends after ``max_new_tokens`` or with
        its first stop id (which is returned).  Greedy unless ``do_sample`` / ``repetition_penalty`` say otherwise."""
        opt = SamplingOptions(**sampling)
        prompts = [list(p) for p in prompts]
        if any(not p or len(p) + max_new_tokens > self.max_len for p in prompts):
            raise ValueError(f"prompts must hold 1 .. {self.max_len - max_new_tokens} tokens")
        if max_new_tokens <= 0:
            return [[] for _ in prompts]
        outs: list = []
        for i in range(0, len(prompts), SKINNY_ROWS):
            outs += self._generate(prompts[i:i + SKINNY_ROWS], max_new_tokens, set(stop_ids), check_every, opt)
        return outs

    def _generate(self, prompts, new, stops, check_every, opt) -> list:
        rows = [self.open() for _ in prompts]
        try:
            logits = self.prefill(rows, prompts)
            B = len(prompts)
            tokens: list = []                 # [B] tensors, one per generated position
            seqs = [list(p) for p in prompts]
            live = set(range(B))
            nxt = self._pick(logits, seqs, opt)
            tokens.append(nxt)
            self._meta[:, :B].copy_(torch.tensor([[len(p) for p in prompts], rows], dtype=torch.int32))
            for t in range(1, new):
                if not opt.greedy:            # the penalties read the sequences on the host
                    for s, k in zip(seqs, nxt.tolist()):
                        s.append(k)
                if stops and t % check_every == 0:
                    recent = torch.stack(tokens[-check_every:], dim=1).tolist()
                    live -= {i for i, r in enumerate(recent) if stops.intersection(r)}
                    if not live:
                        break
                for r in rows:
                    self.cache.advance(r, 1)
                self._tok[:B].copy_(nxt)
                logits = self._decode_graph(B)
                self._meta[0, :B].add_(1)
                nxt = self._pick(logits, seqs, opt)
                tokens.append(nxt)
            out = torch.stack(tokens, dim=1).tolist()
        finally:
            for r in rows:
                self.close(r)
        cut = []
        for r in out:
            end = next((k + 1 for k, t in enumerate(r) if t in stops), len(r))
            cut.append(r[:end])
        return cut

    @staticmethod
    def _pick(logits, seqs, opt) -> torch.Tensor:
        if opt.greedy:
            return logits.argmax(-1)
        if opt.repetition_penalty not in (None, 1.0):
            logits = torch.cat([apply_repetition_penalty(logits[i:i + 1], torch.tensor([s], device=logits.device), opt)
                                for i, s in enumerate(seqs)])
            opt = SamplingOptions(opt.do_sample, opt.temperature, opt.top_k, opt.top_p, opt.min_p)
        return sample_next_token(logits, None, opt)[:, 0]
