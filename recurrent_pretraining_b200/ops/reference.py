"""Plain PyTorch statements of every op the framework uses.

These are the numerical oracles for the CUDA kernels (tests compare a kernel against the
function of the same name evaluated in fp32) and the execution path on CPU.  Each function
names the reference behaviour it restates.
"""
from __future__ import annotations

import math

import torch
import torch.nn.functional as F


def rmsnorm(x: torch.Tensor, weight: torch.Tensor | None, eps: float) -> torch.Tensor:
    """y = cast_x(x32 * rsqrt(mean(x32^2) + eps)) * w   (recpre/norms.py:63-68).  The output keeps the
    dtype of ``x`` (the framework carries a bf16 residual stream on GPU)."""
    x32 = x.float()
    y = x32 * torch.rsqrt(x32.pow(2).mean(-1, keepdim=True) + eps)
    if weight is not None:
        y = y.to(x.dtype).float() * weight.float()
    return y.to(x.dtype)


def add_rmsnorm(a: torch.Tensor, x: torch.Tensor, weight: torch.Tensor | None, eps: float) -> torch.Tensor:
    """Sandwich post-norm: norm(a + x) where the sum is rounded to the stream dtype first
    (recpre/model_dynamic.py:279-282)."""
    return rmsnorm((a.float() + x.float()).to(x.dtype), weight, eps)


def rope_tables(head_dim: int, length: int, base: float = 50000.0, condense: int = 1) -> tuple[torch.Tensor, torch.Tensor]:
    """cos/sin tables [length, head_dim/2] in fp32 (recpre/model_dynamic.py:1438-1443)."""
    inv = 1.0 / (base ** (torch.arange(0, head_dim, 2, dtype=torch.float32) / head_dim))
    t = torch.arange(length, dtype=torch.float32) / condense
    ang = torch.outer(t, inv).float()
    return torch.cos(ang), torch.sin(ang)


def freqs_cis_buffer(cos: torch.Tensor, sin: torch.Tensor) -> torch.Tensor:
    """The state-dict form ``[1, S, 1, hd/2, 2]`` of the tables."""
    return torch.stack([cos[None, :, None, :], sin[None, :, None, :]], dim=4)


def rope_interleaved(x: torch.Tensor, cos: torch.Tensor, sin: torch.Tensor) -> torch.Tensor:
    """Rotate interleaved pairs (2i, 2i+1) of the last dim of ``x`` [B,S,H,hd]; cos/sin are [S, hd/2] (or
    broadcastable [B,S,1,hd/2]); math in fp32, result in x.dtype (recpre/model_dynamic.py:1450-1462)."""
    if cos.ndim == 2:
        cos, sin = cos[None, :, None, :], sin[None, :, None, :]
    xr = x.float().unflatten(-1, (-1, 2))
    a, b = xr[..., 0], xr[..., 1]
    out = torch.stack([a * cos - b * sin, b * cos + a * sin], dim=-1).flatten(-2)
    return out.to(x.dtype)


def qk_bias_rope(qkv: torch.Tensor, qk_bias: torch.Tensor | None, cos: torch.Tensor, sin: torch.Tensor,
                 n_head: int, n_kv: int, head_dim: int):
    """Split fused qkv [B,S,(H+2Hkv)*hd] into q,k,v [B,S,H,hd], add the q/k bias, rotate q and k
    (recpre/model_dynamic.py:349-370)."""
    B, S, _ = qkv.shape
    q, k, v = qkv.split([n_head * head_dim, n_kv * head_dim, n_kv * head_dim], dim=-1)
    q = q.reshape(B, S, n_head, head_dim)
    k = k.reshape(B, S, n_kv, head_dim)
    v = v.reshape(B, S, n_kv, head_dim)
    if qk_bias is not None:
        q = (q.float() + qk_bias[0].float()).to(qkv.dtype)
        k = (k.float() + qk_bias[1].float()).to(qkv.dtype)
    return rope_interleaved(q, cos, sin), rope_interleaved(k, cos, sin), v.contiguous()


def causal_attention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float | None = None,
                     q_offset: int = 0) -> torch.Tensor:
    """softmax(q k^T * scale + causal) v with q,k,v as [B,S,H,hd]; returns [B,Sq,H,hd].  ``q_offset`` is the
    absolute position of the first query row (for cached decode, keys start at position 0)."""
    B, Sq, H, D = q.shape
    Sk, Hk = k.shape[1], k.shape[2]
    scale = 1.0 / math.sqrt(D) if scale is None else scale
    qf, kf, vf = (t.float().transpose(1, 2) for t in (q, k, v))
    if Hk != H:
        kf = kf.repeat_interleave(H // Hk, dim=1)
        vf = vf.repeat_interleave(H // Hk, dim=1)
    s = torch.matmul(qf, kf.transpose(-1, -2)) * scale
    qi = torch.arange(Sq, device=q.device)[:, None] + q_offset
    ki = torch.arange(Sk, device=q.device)[None, :]
    s = s.masked_fill(ki > qi, float("-inf"))
    p = torch.softmax(s, dim=-1)
    return torch.matmul(p, vf).transpose(1, 2).to(q.dtype).contiguous()


def masked_attention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, mask: torch.Tensor,
                     scale: float | None = None) -> torch.Tensor:
    """softmax(q k^T * scale, restricted to ``mask``) v with q,k,v as [B,S,H,hd] and a boolean ``mask`` [B,1,Sq,Sk]
    (True = may attend).  A query row that may attend to nothing (a padding position) returns zeros."""
    B, Sq, H, D = q.shape
    Hk = k.shape[2]
    scale = 1.0 / math.sqrt(D) if scale is None else scale
    qf, kf, vf = (t.float().transpose(1, 2) for t in (q, k, v))
    if Hk != H:
        kf = kf.repeat_interleave(H // Hk, dim=1)
        vf = vf.repeat_interleave(H // Hk, dim=1)
    s = torch.matmul(qf, kf.transpose(-1, -2)) * scale
    s = s.masked_fill(~mask, float("-inf"))
    p = torch.softmax(s, dim=-1)
    p = torch.nan_to_num(p, nan=0.0)
    return torch.matmul(p, vf).transpose(1, 2).to(q.dtype).contiguous()


def swiglu(h: torch.Tensor) -> torch.Tensor:
    """silu(gate) * up with ``h = [gate | up]`` along the last dim (recpre/model_dynamic.py:776-780)."""
    a, b = h.float().chunk(2, dim=-1)
    return (F.silu(a) * b).to(h.dtype)


def linear(x: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    return F.linear(x, w.to(x.dtype))


def adapter(x: torch.Tensor, e: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """Linear(2E -> E) on cat[state, embedding] (recpre/model_dynamic.py:1210)."""
    return F.linear(torch.cat([x, e.to(x.dtype)], dim=-1), w.to(x.dtype))


def embedding(ids: torch.Tensor, w: torch.Tensor, scale: float) -> torch.Tensor:
    return F.embedding(ids, w) * scale


def linear_cross_entropy(x: torch.Tensor, w: torch.Tensor, labels: torch.Tensor, logit_scale: float = 1.0,
                         ignore_index: int = -100, z_reg: float = 0.0) -> torch.Tensor:
    """mean over valid rows of CE(float(x w^T) * logit_scale, label) (+ z_reg * lse^2), the quantities of
    recpre/ops.py:12-20 and recpre/model_dynamic.py:1133-1134."""
    logits = F.linear(x, w.to(x.dtype)).float() * logit_scale
    flat = logits.view(-1, logits.shape[-1])
    lab = labels.reshape(-1)
    loss = F.cross_entropy(flat, lab, ignore_index=ignore_index)
    if z_reg:
        valid = lab != ignore_index
        lse = torch.logsumexp(flat, dim=-1)
        loss = loss + z_reg * (lse.pow(2) * valid).sum() / valid.sum().clamp(min=1)
    return loss


def trunc_normal_state(shape, std: float, generator: torch.Generator | None = None, device="cpu",
                       dtype=torch.float32) -> torch.Tensor:
    """State init: normal(0, std) truncated at +-3 std (recpre/model_dynamic.py:1360-1365)."""
    x = torch.empty(shape, dtype=torch.float32, device=device)
    torch.nn.init.trunc_normal_(x, mean=0.0, std=std, a=-3 * std, b=3 * std, generator=generator)
    return x.to(dtype)


def adamw_step(p, g, m, v, lr, beta1, beta2, eps, wd, step, grad_scale=1.0):
    """Decoupled-weight-decay Adam on fp32 tensors, in place (torch.optim.AdamW semantics)."""
    g = g * grad_scale
    p.mul_(1 - lr * wd)
    m.lerp_(g, 1 - beta1)
    v.mul_(beta2).addcmul_(g, g, value=1 - beta2)
    bc1, bc2 = 1 - beta1 ** step, 1 - beta2 ** step
    denom = (v.sqrt() / math.sqrt(bc2)).add_(eps)
    p.addcdiv_(m, denom, value=-lr / bc1)


# ------------------------------------------------------------------------------------------
# layered decoder models: latent attention, sliding window, fp32 residual stream
# ------------------------------------------------------------------------------------------
def relu2(x: torch.Tensor) -> torch.Tensor:
    return F.relu(x).square()


def linear_act(x: torch.Tensor, w: torch.Tensor, bias: torch.Tensor | None = None, act: str | None = None,
               act_cols: tuple = (0, 0)) -> torch.Tensor:
    """act(x w^T + bias) with an fp32 bias; result in x.dtype.  "silu" applies to the columns ``act_cols``."""
    y = F.linear(x, w).float()
    if bias is not None:
        y = y + bias
    if act == "relu2":
        y = relu2(y)
    elif act == "silu":
        y[:, act_cols[0]:act_cols[1]] = F.silu(y[:, act_cols[0]:act_cols[1]])
    elif act is not None:
        raise ValueError(f"unknown activation {act!r}")
    return y.to(x.dtype)


def rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    x = x.float()
    return x / torch.sqrt(x.square().mean(-1, keepdim=True) + eps)


def rms_residual(x: torch.Tensor, a: torch.Tensor, bias: torch.Tensor | None, w: torch.Tensor, eps: float,
                 mult: float) -> torch.Tensor:
    """x + mult * rmsnorm(a + bias) * w on an fp32 residual stream."""
    s = a.float() if bias is None else a.float() + bias
    return x + mult * rms(s, eps) * w


def rotate_pairs(x: torch.Tensor, cos: torch.Tensor, sin: torch.Tensor) -> torch.Tensor:
    """Rotation of the interleaved pairs of the last dim; cos / sin broadcast against the pairs; fp32 result."""
    u, v = x.float()[..., 0::2], x.float()[..., 1::2]
    return torch.stack([u * cos - v * sin, v * cos + u * sin], dim=-1).flatten(-2)


def window_attention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, visible: torch.Tensor, scale: float) -> torch.Tensor:
    """q [T, H, D]; k, v [K, H, .] shared by all queries or [T, K, H, .] per query; visible [T, K] boolean.  fp32."""
    q, k, v = q.float(), k.float(), v.float()
    per_query = k.dim() == 4
    s = torch.einsum("thd,tkhd->thk" if per_query else "thd,khd->thk", q, k) * scale
    p = torch.softmax(s.masked_fill(~visible[:, None], float("-inf")), dim=-1)
    return torch.einsum("thk,tkhd->thd" if per_query else "thk,khd->thd", p, v)


# ------------------------------------------------------------------------------------------
# layered decoder models: layer norms around sublayers, distance-biased attention, matrix memories
# ------------------------------------------------------------------------------------------
def layer_norm(x: torch.Tensor, w: torch.Tensor, b: torch.Tensor, eps: float) -> torch.Tensor:
    x = x.float()
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt(d.square().mean(-1, keepdim=True) + eps) * w + b


def biased_attention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, bias: torch.Tensor, pos: torch.Tensor, scale: torch.Tensor) -> torch.Tensor:
    """Causal grouped-query attention of one sequence: q [T, H, D] at positions ``pos`` [T], k, v [N, G, .] of the positions
    0 .. N - 1, ``bias`` [H, distances] (its last entry holds for every farther distance), ``scale`` [T] on the products."""
    H, G = q.shape[1], k.shape[1]
    k, v = (t.float().repeat_interleave(H // G, dim=1) for t in (k, v))
    dist = pos[:, None] - torch.arange(k.shape[0])[None]
    s = torch.einsum("thd,khd->thk", q.float(), k) * scale[:, None, None]
    s = s + bias[:, dist.clamp(0, bias.shape[1] - 1)].transpose(0, 1)
    p = torch.softmax(s.masked_fill((dist < 0)[:, None], float("-inf")), dim=-1)
    return torch.einsum("thk,khd->thd", p, v)


def memory_scan(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, state: torch.Tensor, decay: torch.Tensor) -> torch.Tensor:
    """S = decay S + k v^T, o = S^T q per token and head; q, k [T, H, D], v [T, H, E], ``state`` [H, D, E] is updated."""
    out = []
    for t in range(q.shape[0]):
        state.copy_(decay[:, None, None] * state + k[t, :, :, None] * v[t, :, None, :])
        out.append(torch.einsum("hde,hd->he", state, q[t]))
    return torch.stack(out)


def gated_memory_scan(q, k, v, log_i, log_f, state, norm, peak) -> torch.Tensor:
    """Matrix memory with normaliser ``norm`` [H, D] and running maximum ``peak`` [H] of the log gates [T, H]."""
    out = []
    for t in range(q.shape[0]):
        m = torch.maximum(log_f[t] + peak, log_i[t])
        a, b = torch.exp(log_f[t] + peak - m), torch.exp(log_i[t] - m)
        state.copy_(a[:, None, None] * state + b[:, None, None] * k[t, :, :, None] * v[t, :, None, :])
        norm.copy_(a[:, None] * norm + b[:, None] * k[t])
        peak.copy_(m)
        den = torch.maximum((norm * q[t]).sum(-1).abs(), torch.exp(-m)) + 1e-6
        out.append(torch.einsum("hde,hd->he", state, q[t]) / den[:, None])
    return torch.stack(out)


def log_gates(raw: torch.Tensor, bias: torch.Tensor, cap: float):
    """Log input gate and log forget gate [T, H] of raw projections [T, 2H]."""
    i, f = (cap * torch.tanh((raw.float() + bias) / cap)).chunk(2, dim=-1)
    return i, F.logsigmoid(f)


# ------------------------------------------------------------------------------------------
# layered decoder models: capped attention with a sink, mixture of experts
# ------------------------------------------------------------------------------------------
def rotate_halves(x: torch.Tensor, cos: torch.Tensor, sin: torch.Tensor) -> torch.Tensor:
    """Rotation of entry i of the first half of the last dim with entry i of the second; fp32 result."""
    u, v = x.float().chunk(2, dim=-1)
    return torch.cat([u * cos - v * sin, v * cos + u * sin], dim=-1)


def capped_attention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, visible: torch.Tensor, scale: float, softcap: float | None,
                     sink: torch.Tensor | None) -> torch.Tensor:
    """Grouped-query attention: q [T, H, D]; k, v [K, G, .] shared by all queries or [T, K, G, .] per query; visible [T, K]; ``sink``
    [H]: one more term of the softmax's denominator.  fp32."""
    T, H, G = q.shape[0], q.shape[1], k.shape[-2]
    q = q.float().unflatten(1, (G, H // G))
    per_query = k.dim() == 4
    s = torch.einsum("tgrd,tkgd->tgrk" if per_query else "tgrd,kgd->tgrk", q, k.float()).flatten(1, 2) * scale
    if softcap:
        s = softcap * torch.tanh(s / softcap)
    s = s.masked_fill(~visible[:, None], float("-inf"))
    if sink is not None:
        s = torch.cat([s, sink[None, :, None].expand(T, -1, 1)], dim=-1)
    p = torch.softmax(s, dim=-1)
    if sink is not None:
        p = p[..., :-1]
    v = v.float().masked_fill(~visible[:, :, None, None], 0.0) if per_query else v.float()      # slots that were never written
    return torch.einsum("tgrk,tkge->tgre" if per_query else "tgrk,kge->tgre", p.unflatten(1, (G, H // G)), v).flatten(1, 2)


def route(z: torch.Tensor, correction: torch.Tensor, top: int):
    """Router logits [T, outputs] -> chosen outputs [T, top], best first, and their normalised scores."""
    s = torch.softmax(z.float(), dim=-1)
    idx = torch.sort(s + correction, dim=-1, descending=True, stable=True).indices[:, :top]
    w = s.gather(1, idx)
    return idx, w / (w.sum(-1, keepdim=True) + 1e-20)


# ------------------------------------------------------------------------------------------
# layered decoder models: norms over groups of columns, gated delta rule, choice of experts within groups
# ------------------------------------------------------------------------------------------
def group_rms(x: torch.Tensor, groups: int, eps: float) -> torch.Tensor:
    return rms(x.unflatten(-1, (groups, -1)), eps).flatten(-2)


def unit(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt(x.square().sum(-1, keepdim=True) + eps)


def delta_scan(q, k, v, beta, log_g, state) -> torch.Tensor:
    """S = g S, u = beta (v - S^T k), S = S + k u^T, o = S^T q per token and head; q, k [T, H, D], v [T, H, E], beta, log_g [T, H],
    ``state`` [H, D, E] is updated."""
    out = []
    for t in range(q.shape[0]):
        s = torch.exp(log_g[t])[:, None, None] * state
        u = beta[t][:, None] * (v[t] - torch.einsum("hde,hd->he", s, k[t]))
        state.copy_(s + k[t, :, :, None] * u[:, None, :])
        out.append(torch.einsum("hde,hd->he", state, q[t]))
    return torch.stack(out)


def route_grouped(z: torch.Tensor, top: int, groups: int, keep: int):
    """Router logits [T, outputs] -> chosen outputs [T, top] of the best groups, best first, and their sigmoid scores."""
    s = torch.sigmoid(z.float())
    g = s.unflatten(1, (groups, -1))
    strength = g.topk(min(2, g.shape[2]), dim=-1).values.sum(-1)
    best = torch.sort(strength, dim=-1, descending=True, stable=True).indices[:, :keep]
    allowed = torch.zeros_like(strength, dtype=torch.bool).scatter_(1, best, True)[:, :, None].expand_as(g).flatten(1)
    idx = torch.sort(s.masked_fill(~allowed, float("-inf")), dim=-1, descending=True, stable=True).indices[:, :top]
    return idx, s.gather(1, idx)
