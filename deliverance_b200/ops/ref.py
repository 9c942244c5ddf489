"""Plain PyTorch statement of every op in the kernel set.

This is the slow, always-available oracle: the CUDA kernels in ``csrc/`` are tested against these functions evaluated
in fp32, and the CPU execution path of the framework (tests, the fp32 llama oracle) runs on them directly. Math follows
the reference: RMSNorm ``(offset + w) * x * rsqrt(mean(x^2) + eps)`` (core/.../generator/RmsNorm.java:107-121), HF
half-rotation RoPE with pairs ``(i, i + d/2)`` (CausalSelfAttention.java:340-372,429-446), scores
``softmax(softcap(scale * q.k))`` with causal visibility ``j <= pos`` (VectorTensorMathUtils.java:34-78), activations
(math/.../ActivationFunction.java:8-33).
"""
from __future__ import annotations

import math
from typing import Optional

import torch
import torch.nn.functional as F

from ..ckpt.jq4 import q4_dequantize


def act_fn(name: str):
    name = (name or "silu").lower()
    if name in ("silu", "swish"):
        return F.silu
    if name in ("gelu_pytorch_tanh", "gelu_new", "gelu_tanh", "gelu_fast"):
        return lambda x: F.gelu(x, approximate="tanh")
    if name == "gelu":
        return F.gelu
    if name == "relu":
        return F.relu
    if name == "relu2":
        return lambda x: F.relu(x).square()
    if name == "tanh":
        return torch.tanh
    raise ValueError(f"unknown activation '{name}'")


def rmsnorm(x: torch.Tensor, w: torch.Tensor, eps: float, offset: float = 0.0) -> torch.Tensor:
    xf = x.float()
    var = xf.double().pow(2).mean(dim=-1, keepdim=True).float() if x.device.type == "cpu" else xf.pow(2).mean(dim=-1, keepdim=True)
    y = xf * torch.rsqrt(var + eps) * (w.float() + offset)
    return y.to(x.dtype)


def add_rmsnorm(x: torch.Tensor, residual: torch.Tensor, w: torch.Tensor, eps: float, offset: float = 0.0,
                res_mult: float = 1.0) -> torch.Tensor:
    """``residual += x * res_mult`` (in place) and return ``rmsnorm(residual)``."""
    residual.copy_((residual.float() + x.float() * res_mult).to(residual.dtype))
    return rmsnorm(residual, w, eps, offset)


def layernorm(x: torch.Tensor, w: torch.Tensor, b: Optional[torch.Tensor], eps: float) -> torch.Tensor:
    return F.layer_norm(x.float(), (x.shape[-1],), w.float(), None if b is None else b.float(), eps).to(x.dtype)


def linear_dense(x: torch.Tensor, w: torch.Tensor, bias: Optional[torch.Tensor] = None) -> torch.Tensor:
    y = x.float() @ w.float().t()
    if bias is not None:
        y = y + bias.float()
    return y.to(x.dtype)


def linear_q4(x: torch.Tensor, packed: torch.Tensor, scales: torch.Tensor, bias: Optional[torch.Tensor] = None) -> torch.Tensor:
    return linear_dense(x, q4_dequantize(packed, scales, torch.float32), bias)


def rope_tables(head_dim: int, max_pos: int, theta: float, factor: float = 1.0, rot_dim: Optional[int] = None):
    """cos/sin tables ``[max_pos, rot/2]`` fp32: angle = pos * theta^(-2i/rot) / factor (math/.../VectorMathUtils.java:20-41)."""
    rot = rot_dim or head_dim
    i = torch.arange(0, rot // 2, dtype=torch.float64)
    inv = 1.0 / (theta ** (2.0 * i / rot)) / factor
    ang = torch.arange(max_pos, dtype=torch.float64).unsqueeze(1) * inv.unsqueeze(0)
    return torch.cos(ang).float(), torch.sin(ang).float()


def yarn_rope_tables(dims: int, max_pos: int, base: float, scaling: Optional[dict] = None):
    """cos/sin tables ``[max_pos, dims/2]`` fp32 with YaRN frequency interpolation. ``scaling``: ``factor``, ``original`` (context
    length the base frequencies were made for), ``fast`` / ``slow`` (full turns over that context at which a pair is kept as it is /
    fully slowed down by ``factor``; a linear ramp over the pair index lies between). Both tables carry ``0.1 ln(factor) + 1``."""
    if not scaling:
        return rope_tables(dims, max_pos, base, 1.0)
    i = torch.arange(0, dims // 2, dtype=torch.float64)
    f = base ** (-2.0 * i / dims)
    pair_of = lambda turns: dims * math.log(float(scaling["original"]) / (2.0 * math.pi * float(turns))) / (2.0 * math.log(base))  # noqa: E731
    lo = max(math.floor(pair_of(scaling["fast"])), 0)
    hi = min(math.ceil(pair_of(scaling["slow"])), dims - 1)
    ramp = ((i - lo) / max(hi - lo, 0.001)).clamp(0.0, 1.0)
    factor = float(scaling["factor"])
    inv = f / factor * ramp + f * (1.0 - ramp)
    ang = torch.arange(max_pos, dtype=torch.float64).unsqueeze(1) * inv.unsqueeze(0)
    mult = 0.1 * math.log(factor) + 1.0
    return (torch.cos(ang) * mult).float(), (torch.sin(ang) * mult).float()


def banded_rope_tables(dims: int, max_pos: int, base: float, scaling: Optional[dict] = None):
    """cos/sin tables ``[max_pos, dims/2]`` fp32 with Llama-3.1 frequency scaling. ``scaling``: pairs that turn more than ``high`` times
    over ``original`` tokens keep their frequency, those that turn less than ``low`` times are slowed down by ``factor``, the turns in
    between blend the two linearly."""
    i = torch.arange(0, dims // 2, dtype=torch.float64)
    f = float(base) ** (-2.0 * i / dims)
    if scaling:
        factor, low, high = (float(scaling[k]) for k in ("factor", "low", "high"))
        turns = float(scaling["original"]) * f / (2.0 * math.pi)
        keep = ((turns - low) / (high - low)).clamp(0.0, 1.0) if high != low else (turns > low).double()
        f = f / factor * (1.0 - keep) + f * keep
    ang = torch.arange(max_pos, dtype=torch.float64).unsqueeze(1) * f.unsqueeze(0)
    return torch.cos(ang).float(), torch.sin(ang).float()


def apply_rope_pairs(x: torch.Tensor, pos: torch.Tensor, cos: torch.Tensor, sin: torch.Tensor) -> torch.Tensor:
    """x ``[T, heads, d]``; rotates the first ``2 * cos.shape[1]`` dims with neighbouring pairs (2 i, 2 i + 1)."""
    n = 2 * cos.shape[1]
    c, s = cos[pos].unsqueeze(1), sin[pos].unsqueeze(1)
    xf = x.float()
    a, b = xf[..., 0:n:2], xf[..., 1:n:2]
    out = torch.cat([torch.stack([a * c - b * s, b * c + a * s], dim=-1).flatten(-2), xf[..., n:]], dim=-1)
    return out.to(x.dtype)


def apply_rope(x: torch.Tensor, pos: torch.Tensor, cos: torch.Tensor, sin: torch.Tensor) -> torch.Tensor:
    """x ``[T, heads, d]``; rotates the first ``2 * cos.shape[1]`` dims with pairs (i, i + half)."""
    half = cos.shape[1]
    c = cos[pos].unsqueeze(1).float()
    s = sin[pos].unsqueeze(1).float()
    xf = x.float()
    a, b, rest = xf[..., :half], xf[..., half : 2 * half], xf[..., 2 * half :]
    out = torch.cat([a * c - b * s, b * c + a * s, rest], dim=-1)
    return out.to(x.dtype)


def qk_prepare_and_cache(qkv, positions, slots, n_heads, n_kv, head_dim, q_norm_w, k_norm_w, eps, norm_offset,
                         cos, sin, k_cache, v_cache):
    """Split fused qkv ``[T, (H + 2 KV) * D]``, apply optional per-head RMSNorm to q and k, RoPE to q and k, and
    scatter k, v into the paged cache rows ``slots`` (flat row = block * block_size + offset).

    ``k_cache`` / ``v_cache``: ``[num_blocks, KV, block_size, D]``. Returns q ``[T, H, D]``.
    """
    T = qkv.shape[0]
    q, k, v = qkv.split([n_heads * head_dim, n_kv * head_dim, n_kv * head_dim], dim=-1)
    q = q.reshape(T, n_heads, head_dim)
    k = k.reshape(T, n_kv, head_dim)
    v = v.reshape(T, n_kv, head_dim)
    if q_norm_w is not None:
        q = rmsnorm(q, q_norm_w, eps, norm_offset)
        k = rmsnorm(k, k_norm_w, eps, norm_offset)
    if cos is not None:
        q = apply_rope(q, positions, cos, sin)
        k = apply_rope(k, positions, cos, sin)
    nb, kvh, bs, d = k_cache.shape
    blk = torch.div(slots, bs, rounding_mode="floor")
    off = slots % bs
    k_cache[blk, :, off, :] = k.to(k_cache.dtype)
    v_cache[blk, :, off, :] = v.to(v_cache.dtype)
    return q.contiguous()


def paged_attention(q, k_cache, v_cache, block_tables, q_start, q_len, ctx_len, scale, softcap=0.0, window=0,
                    causal=True, keep_first=0, sink=None, mix=None):
    """Attention of ragged query rows against paged K/V.

    q ``[T, H, D]``; sequence ``i`` owns query rows ``[q_start[i], q_start[i] + q_len[i])`` which are the *last*
    ``q_len[i]`` positions of a context of ``ctx_len[i]`` cached tokens. Row at position ``p`` sees keys ``j <= p``
    (and ``j > p - window`` or ``j < keep_first`` when ``window > 0``). Score = ``softmax(softcap * tanh(scale * q.k / softcap))``;
    ``sink`` ``[H]``: a further score per head without a value takes part in the softmax (neither scaled nor capped). ``mix`` ``[H, H]`` (to, from):
    the heads' scores are mixed in front of the softmax. Values may be wider or narrower than keys.
    """
    T, H, D = q.shape
    nb, KV, bs, _ = k_cache.shape
    DV = v_cache.shape[-1]
    group = H // KV
    out = q.new_zeros(T, H, DV)
    for i in range(len(q_len)):
        ql, cl, qs = int(q_len[i]), int(ctx_len[i]), int(q_start[i])
        if ql == 0:
            continue
        nblk = (cl + bs - 1) // bs
        blocks = block_tables[i, :nblk].long()
        k = k_cache[blocks].permute(1, 0, 2, 3).reshape(KV, nblk * bs, D)[:, :cl].float()
        v = v_cache[blocks].permute(1, 0, 2, 3).reshape(KV, nblk * bs, DV)[:, :cl].float()
        qi = q[qs : qs + ql].float().permute(1, 0, 2)  # H, ql, D
        k = k.repeat_interleave(group, dim=0)
        v = v.repeat_interleave(group, dim=0)
        s = torch.matmul(qi, k.transpose(1, 2)) * scale
        if mix is not None:
            s = torch.einsum("hg,gtj->htj", mix.float(), s)
        if softcap and softcap > 0:
            s = torch.tanh(s / softcap) * softcap
        pos = torch.arange(cl - ql, cl, device=q.device).unsqueeze(1)
        j = torch.arange(cl, device=q.device).unsqueeze(0)
        mask = torch.ones(ql, cl, dtype=torch.bool, device=q.device)
        if causal:
            mask &= j <= pos
        if window and window > 0:
            mask &= (j > pos - window) | (j < keep_first)
        s = s.masked_fill(~mask.unsqueeze(0), float("-inf"))
        if sink is not None:
            p = torch.softmax(torch.cat([s, sink.float().view(H, 1, 1).expand(H, ql, 1)], dim=-1), dim=-1)[..., :-1]
        else:
            p = torch.softmax(s, dim=-1)
        out[qs : qs + ql] = torch.matmul(p, v).permute(1, 0, 2).to(q.dtype)
    return out


def act_mul(gate_up: torch.Tensor, act: str) -> torch.Tensor:
    """``act(x[:, :I]) * x[:, I:]`` on a concatenated gate|up projection."""
    I = gate_up.shape[-1] // 2
    g, u = gate_up[..., :I].float(), gate_up[..., I:].float()
    return (act_fn(act)(g) * u).to(gate_up.dtype)


def embedding(table: torch.Tensor, ids: torch.Tensor, scale: float = 1.0, dtype: Optional[torch.dtype] = None) -> torch.Tensor:
    out = table[ids.long()].float() * scale
    return out.to(dtype or table.dtype)


def bigram_embedding(table, bigram, ids, prev, mul_prev: int, mul_cur: int, scale: float) -> torch.Tensor:
    out = table[ids.long()].float() * scale
    if bigram is not None:
        buckets = bigram.shape[0] - 1
        row = torch.remainder(prev.long() * mul_prev + ids.long() * mul_cur, buckets)
        out = out + bigram[torch.where(prev < 0, torch.full_like(row, buckets), row)].float()
    return out


def add_layernorm(residual, delta, norm1, norm2, eps, pitch, dtype):
    if delta is not None:
        residual.add_(delta.float())
    mean = residual.mean(dim=-1, keepdim=True)
    d = residual - mean
    n = d * torch.rsqrt(d.pow(2).mean(dim=-1, keepdim=True) + eps)
    pad = pitch - residual.shape[-1]
    return tuple(None if nb is None else F.pad(n * nb[0] + nb[1], (0, pad)).to(dtype) for nb in (norm1, norm2))


def sandwich_norm(residual, sub, w_sub, mult, w_next, eps, rms=False):
    """fp32 ``residual += mult * norm(sub; w_sub)`` in place, then ``norm(residual; w_next)`` (the plain residual without it); ``rms``: RMS norms
    instead of LayerNorms."""
    def norm(v, w):
        d = v if rms else v - v.mean(dim=-1, keepdim=True)
        return d * torch.rsqrt(d.pow(2).mean(dim=-1, keepdim=True) + eps) * w

    if sub is not None:
        residual.add_(norm(sub.float(), w_sub), alpha=mult)
    return residual if w_next is None else norm(residual, w_next)


def softcap_(logits: torch.Tensor, cap: float) -> torch.Tensor:
    return torch.tanh(logits / cap) * cap if cap and cap > 0 else logits


# ---- MoE -------------------------------------------------------------------------------------------------------------
def moe_route(router_logits: torch.Tensor, k: int, mode: str, renorm: bool, correction=None, groups: int = 1, keep: int = 1, scale: float = 1.0):
    """Return (weights ``[T, k]`` fp32, expert ids ``[T, k]``).

    ``softmax_topk``: softmax over all experts, take top-k, optionally renormalise (Mixtral always renormalises,
    MixtureOfExpertsBlock.java:100-112; Qwen3-MoE by ``norm_topk_prob``, Qwen3MoeFeedForward.java:276-301).
    ``topk_softmax``: take the top-k logits, softmax over those k (GraniteMoeHybridMoeFeedForward.java:112-141).
    ``sigmoid_topk``: scores ``s = sigmoid(z)``; the largest ``s + correction`` among the experts of the ``keep`` best of ``groups`` equal groups
    of neighbours (a group counts the sum of its two largest choice scores); weights ``scale * s / (sum + 1e-20)``.
    """
    lf = router_logits.float()
    if mode == "softmax_topk":
        p = torch.softmax(lf, dim=-1)
        w, idx = torch.topk(p, k, dim=-1)
        if renorm:
            w = w / w.sum(dim=-1, keepdim=True)
    elif mode == "topk_softmax":
        top, idx = torch.topk(lf, k, dim=-1)
        w = torch.softmax(top, dim=-1)
    elif mode == "sigmoid_topk":
        s = torch.sigmoid(lf)
        choice = s if correction is None else s + correction.float()
        if groups > 1 and keep < groups:
            by_group = choice.view(choice.shape[0], groups, -1)
            best = by_group.topk(min(2, by_group.shape[-1]), dim=-1).values.sum(dim=-1)
            kept = torch.zeros_like(best, dtype=torch.bool).scatter_(1, best.topk(keep, dim=-1).indices, True)
            choice = by_group.masked_fill(~kept.unsqueeze(-1), float("-inf")).flatten(1)
        idx = choice.topk(k, dim=-1).indices
        w = s.gather(1, idx)
        w = w / (w.sum(dim=-1, keepdim=True) + 1e-20) * scale
    else:
        raise ValueError(mode)
    return w, idx


def moe_experts(x, weights, idx, gate_up_fn, down_fn, num_experts, act, gated_fn=None):
    """Group tokens by expert, run gate|up -> act*mul -> down per expert, scatter-add with the route weight. ``gated_fn(e, rows)``
    replaces gate|up + act*mul when the expert weights are stored in the interleaved layout of the fused epilogue."""
    T, Hd = x.shape
    out = torch.zeros(T, Hd, dtype=torch.float32, device=x.device)
    for e in range(num_experts):
        tok, slot = torch.nonzero(idx == e, as_tuple=True)
        if tok.numel() == 0:
            continue
        h = gated_fn(e, x[tok]) if gated_fn is not None else act_mul(gate_up_fn(e, x[tok]), act)
        y = down_fn(e, h).float()
        out.index_add_(0, tok, y * weights[tok, slot].unsqueeze(1))
    return out.to(x.dtype)


# ---- Mamba2 ----------------------------------------------------------------------------------------------------------
def short_conv(x, weight, bias, ring, start: int):
    """Causal convolution per channel over the rows ``x [n, C]`` of ONE sequence, whose first row is position ``start``, then silu; fp32 result.
    ``weight [C, taps]`` (last column: the current token's). ``ring [taps, C]`` keeps the inputs of the last positions, position ``p`` at row ``p
    mod taps``, and is advanced."""
    n, taps = x.shape[0], weight.shape[1]
    rows = [ring[p % taps].clone() if p >= 0 else torch.zeros_like(ring[0]) for p in range(start - taps + 1, start)]
    x = x.float()
    seen = torch.cat([torch.stack(rows), x]) if rows else x
    acc = sum(seen[j : j + n] * weight[:, j].float() for j in range(taps))
    if bias is not None:
        acc = acc + bias.float()
    for i in range(max(0, n - taps), n):
        ring[(start + i) % taps] = x[i]
    return F.silu(acc)


def ssd_sequential(x, B, C, dt, neg_a, D, state):
    """Token-by-token state-space recurrence of ONE sequence, fp32: ``S <- exp(neg_a dt) S + dt B x^T``, ``y = S^T C + D x``. x ``[T, H, dv]``, B and C
    ``[T, G, N]`` (head h uses group h // (H / G)), dt ``[T, H]`` positive, neg_a and D ``[H]``; ``state [H, N, dv]`` is updated in place."""
    x, group = x.float(), x.shape[1] // B.shape[1]
    B, C = B.float().repeat_interleave(group, dim=1), C.float().repeat_interleave(group, dim=1)
    y = torch.empty(x.shape, dtype=torch.float32, device=x.device)
    decay = torch.exp(neg_a * dt)
    for t in range(x.shape[0]):
        state.mul_(decay[t].view(-1, 1, 1)).addcmul_((dt[t].unsqueeze(-1) * B[t]).unsqueeze(-1), x[t].unsqueeze(-2))
        y[t] = (state * C[t].unsqueeze(-1)).sum(dim=-2) + D.view(-1, 1) * x[t]
    return y


# ---- gated delta rule --------------------------------------------------------------------------------------------------
def delta_sequential(q, k, v, log_a, beta, state):
    """Token-by-token gated delta rule of ONE sequence, fp32: ``S <- diag(exp(log_a)) S``, ``u = beta (v - S^T k)``, ``S <- S + k u^T``, ``o = S^T q``.
    q, k, log_a ``[T, H, dk]``, v ``[T, H, dv]``, beta ``[T, H]``; ``state [H, dk, dv]`` is updated in place. Returns ``[T, H, dv]``."""
    out = torch.empty(v.shape, dtype=torch.float32, device=v.device)
    a = torch.exp(log_a)
    for t in range(v.shape[0]):
        state.mul_(a[t].unsqueeze(-1))
        u = beta[t].unsqueeze(-1) * (v[t] - (state * k[t].unsqueeze(-1)).sum(dim=-2))
        state.addcmul_(k[t].unsqueeze(-1), u.unsqueeze(-2))
        out[t] = (state * q[t].unsqueeze(-1)).sum(dim=-2)
    return out


# ---- gated linear attention ------------------------------------------------------------------------------------------
def gla_sequential(q, k, v, z, q_scale: float, tau: float, state):
    """Token-by-token gated linear attention of ONE sequence, fp32: ``S <- diag(sigmoid(z)^(1/tau)) S + k v^T``, ``o = S^T (q * q_scale)``.
    q, k, z ``[T, H, dk]``, v ``[T, H, dv]``; ``state [H, dk, dv]`` is updated in place. Returns ``[T, H, dv]``."""
    q, k, v = q.float() * q_scale, k.float(), v.float()
    alpha = torch.exp(F.logsigmoid(z.float()) / tau)
    out = torch.empty(v.shape, dtype=torch.float32, device=v.device)
    for t in range(v.shape[0]):
        state.mul_(alpha[t].unsqueeze(-1)).addcmul_(k[t].unsqueeze(-1), v[t].unsqueeze(-2))
        out[t] = (state * q[t].unsqueeze(-1)).sum(dim=-2)
    return out


def gla_norm_gate(o, g, w, eps: float):
    """``o [T, H, dv]`` RMS-normed over dv with the shared weight ``w [dv]``, times ``silu(g)``."""
    o = o.float()
    return o * torch.rsqrt(o.pow(2).mean(dim=-1, keepdim=True) + eps) * w * F.silu(g.float())


# ---- lightning attention ---------------------------------------------------------------------------------------------
def lightning_sequential(q, k, v, decay, state):
    """Token-by-token linear attention of ONE sequence with a constant decay per head, fp32: ``S <- decay S + k v^T``, ``o = S^T q``.
    q, k ``[T, H, dk]``, v ``[T, H, dv]`` (activated), ``decay [H]``; ``state [H, dk, dv]`` is updated in place. Returns ``[T, H, dv]``."""
    q, k, v = q.float(), k.float(), v.float()
    out = torch.empty(v.shape, dtype=torch.float32, device=v.device)
    d = decay.view(-1, 1, 1)
    for t in range(v.shape[0]):
        state.copy_(state.double() * d + k[t].unsqueeze(-1) * v[t].unsqueeze(-2))
        out[t] = (state * q[t].unsqueeze(-1)).sum(dim=-2)
    return out


# ---- residual streams --------------------------------------------------------------------------------------------------
def layernorm_rows(v, w, eps):
    d = v - v.mean(dim=-1, keepdim=True)
    return d * torch.rsqrt(d.pow(2).mean(dim=-1, keepdim=True) + eps) * w


def stream_write(streams, y, mix, write):
    """In place over ``[T, S, W]``: ``x_t = sum_s mix[s, t] x_s + write[t] y``."""
    streams.copy_(torch.einsum("nsw,st->ntw", streams, mix) + write.view(1, -1, 1) * y.float().unsqueeze(1))


def stream_read(streams, read):
    return streams.sum(dim=1) if read is None else torch.einsum("nsw,s->nw", streams, read)


# ---- sampling helpers --------------------------------------------------------------------------------------------------
def log_softmax_at(logits: torch.Tensor, idx: torch.Tensor) -> torch.Tensor:
    lf = logits.float()
    return lf.gather(-1, idx) - torch.logsumexp(lf, dim=-1, keepdim=True)
