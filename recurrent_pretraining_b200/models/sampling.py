"""Next-token sampling shared by the models' generation paths.

Order: repetition / DRY penalty -> temperature -> softmax -> top-k -> top-p -> min-p -> renormalise -> multinomial;
greedy argmax when ``do_sample`` is false."""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

import torch
import torch.nn.functional as F


@dataclass
class SamplingOptions:
    do_sample: bool = False
    temperature: Optional[float] = None
    top_k: Optional[int] = None
    top_p: Optional[float] = None
    min_p: Optional[float] = None
    repetition_penalty: Optional[float] = None

    @property
    def greedy(self) -> bool:
        return not self.do_sample and self.repetition_penalty in (None, 1.0)


def sample_next_token(logits, input_ids, gc):
    if gc.repetition_penalty is not None and gc.repetition_penalty != 1.0:
        logits = apply_repetition_penalty(logits, input_ids, gc)
    if not gc.do_sample:
        return torch.argmax(logits, dim=-1, keepdim=True)
    logits = logits.to(copy=True, dtype=torch.float32)
    if gc.temperature:
        logits = logits / gc.temperature
    probs = F.softmax(logits, dim=-1)
    if gc.top_k:
        kth = torch.topk(probs, gc.top_k, dim=-1)[0][:, -1:]
        probs = torch.where(probs < kth, torch.zeros_like(probs), probs)
    if gc.top_p:
        sp, si = torch.sort(probs, descending=True, dim=-1)
        remove = torch.cumsum(sp, dim=-1) > gc.top_p
        remove[:, 0] = False
        mask = torch.zeros_like(probs, dtype=torch.bool).scatter(1, si, remove)
        probs = torch.where(mask, torch.zeros_like(probs), probs)
    if gc.min_p:
        probs = torch.where(probs < gc.min_p * probs.max(dim=-1, keepdim=True)[0], torch.zeros_like(probs), probs)
    probs = probs / probs.sum(dim=-1, keepdim=True).clamp(min=1e-10)
    return torch.multinomial(probs, num_samples=1)


def apply_repetition_penalty(original_logits, input_ids, gc, use_candidates: bool = False):
    """Classic repetition penalty on every token already in the sequence, or the DRY penalty (exponential in the
    length of the repeated n-gram a token would extend) when ``dry_multiplier`` > 0."""
    two_d = original_logits.dim() == 2
    if two_d:
        logits = (original_logits.unsqueeze(1) if original_logits.shape[0] == input_ids.shape[0]
                  else original_logits.unsqueeze(0)).to(copy=True, dtype=torch.float32)
    else:
        logits = original_logits.clone()
    B, T, V = logits.shape
    dry = getattr(gc, "dry_multiplier", 0) or 0
    for b in range(B):
        seq = input_ids[b]
        if use_candidates:
            seq = torch.cat([seq, logits[b].argmax(dim=-1)])
        if dry > 0:
            base, allowed = getattr(gc, "dry_base", 1.75), getattr(gc, "dry_allowed_length", 2)
            ctx = seq.tolist()
            n = len(ctx)
            best: dict = {}
            for start in range(max(0, n - 128), n - 1):
                m = 0
                while start + m < n and m < 32 and ctx[start + m] == ctx[n - m - 1]:
                    m += 1
                if m > 0 and start + m < n:
                    tok = ctx[start + m]
                    best[tok] = max(best.get(tok, 0), m + 1)
            for tok, match in best.items():
                if match >= allowed:
                    logits[b, :, tok] -= dry * base ** (match - allowed)
        else:
            uniq = torch.unique(seq)
            sel = logits[b][:, uniq]
            logits[b][:, uniq] = torch.where(sel < 0, sel * gc.repetition_penalty, sel / gc.repetition_penalty)
    if two_d:
        return logits.squeeze(1) if original_logits.shape[0] == input_ids.shape[0] else logits.squeeze(0)
    return logits
