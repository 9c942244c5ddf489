"""Grouped-query softmax attention with per-layer sizes: unequal query / key and value widths, partial rotation of neighbouring pairs or of
the two halves of the rotated columns, per-head query / key norms, values that are the projected keys or a blend with another layer's,
sliding window with kept first tokens, score soft-cap, a sink per head in the denominator (a score that has no value), an output gate per
column or per head, scores of the heads mixed by a matrix in front of the softmax.

One projection row is ``[q (H * dk) | k (G * dk) | v (G * dv) | g]`` with head widths rounded up to multiples of 8 (16-byte rows everywhere);
the columns behind the real ones carry zero weights, so scores, cache rows and outputs are exact whatever the sizes. Tied values have no
columns of their own; ``g`` is there for gated heads. CUDA forms:

* prompts: the tcgen05 / TMA kernel (``attention_tc.cu``) over the paged cache, heads up to 256 wide;
* decode: the split-KV tensor-core kernel (``attention.cu``), heads up to 256 wide;
* fp32 and wider heads: one CTA per (row, head) on CUDA cores.

Mixed scores (``mixed``): a cache row holds all KV heads of a token, ``k [pages, 1, page, G * dk]`` and ``v [pages, 1, page, G * dv]``. Prompts move the mixing to the
query side: head h's mixed score against a key is the product of the whole cache row with ``[sum_(g in group 0) mix[h, g] q_g | sum_(g in group 1) .. | ..]``, so
the prompt kernel runs with queries of ``G * dk`` columns against one wide key (gathered rows). Decode steps take all heads of a row in one CTA and mix the fp32 scores.
"""
from __future__ import annotations

from dataclasses import dataclass

import torch

from .. import ops
from . import ref


def up8(n: int) -> int:
    return (n + 7) // 8 * 8


@dataclass(frozen=True)
class GroupedShape:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    tied: bool = False  # the values are the projected keys
    gate: str = ""  # output gate: "" | "columns" | "heads"
    mixed: bool = False  # the heads' scores are mixed in front of the softmax

    def __post_init__(self):
        if self.heads % self.kv_heads:
            raise ValueError(f"{self.heads} query heads do not divide into {self.kv_heads} groups")
        if self.tied and self.dim != self.vdim:
            raise ValueError(f"keys of {self.dim} columns cannot be values of {self.vdim}")
        if self.gate not in ("", "columns", "heads"):
            raise ValueError(f"unknown output gate '{self.gate}'")
        if self.mixed and self.tied:
            raise ValueError("mixed scores with tied values are not supported")

    @property
    def dk(self) -> int:
        return up8(self.dim)

    @property
    def dv(self) -> int:
        return up8(self.vdim)

    @property
    def q_width(self) -> int:
        return self.heads * self.dk

    @property
    def k_width(self) -> int:
        return self.kv_heads * self.dk

    @property
    def v_at(self) -> int:
        """First value column (tied values: the first key column)."""
        return self.q_width if self.tied else self.q_width + self.k_width

    @property
    def v_width(self) -> int:
        return self.kv_heads * self.dv

    @property
    def gate_at(self) -> int:
        return self.q_width + self.k_width + (0 if self.tied else self.v_width)

    @property
    def gate_logits(self) -> int:
        return {"": 0, "columns": self.out_width, "heads": self.heads}[self.gate]

    @property
    def width(self) -> int:
        return self.gate_at + up8(self.gate_logits)

    @property
    def out_width(self) -> int:
        return self.heads * self.dv

    @property
    def tensor_core(self) -> bool:
        """Widths the tensor-core kernels take (fp32 and wider heads use the CUDA-core rows form)."""
        return max(self.dk, self.dv) <= 256



def pad_head_rows(w: torch.Tensor, heads: int, dim: int, padded: int) -> torch.Tensor:
    """``[heads * dim, K]`` -> ``[heads * padded, K]`` with zero rows behind every head."""
    if dim == padded:
        return w
    return torch.nn.functional.pad(w.reshape(heads, dim, -1), (0, 0, 0, padded - dim)).reshape(heads * padded, -1)


def pad_head_columns(w: torch.Tensor, heads: int, dim: int, padded: int) -> torch.Tensor:
    """``[N, heads * dim]`` -> ``[N, heads * padded]`` with zero columns behind every head."""
    if dim == padded:
        return w
    return torch.nn.functional.pad(w.reshape(w.shape[0], heads, dim), (0, padded - dim)).reshape(w.shape[0], heads * padded)


def rope_pairs_kv(s: GroupedShape, qkv, positions, slots, cos, sin, k_cache, v_cache) -> None:
    """Rotate the queries in place, write the rotated keys and the values into their cache rows."""
    if ops._cuda(qkv):
        ops._count()
        ops.require_ext().rope_pairs_kv(qkv, positions, slots, cos, sin, k_cache, v_cache, s.heads, s.kv_heads, s.dk, s.dv)
        return
    T, p = qkv.shape[0], positions.long()
    q, k, v = qkv.split([s.q_width, s.k_width, s.kv_heads * s.dv], dim=-1)
    q.copy_(ref.apply_rope_pairs(q.reshape(T, s.heads, s.dk), p, cos, sin).reshape(T, -1))
    page = k_cache.shape[2]
    blk, off = torch.div(slots, page, rounding_mode="floor"), slots % page
    k_cache[blk, :, off, :] = ref.apply_rope_pairs(k.reshape(T, s.kv_heads, s.dk), p, cos, sin).to(k_cache.dtype)
    v_cache[blk, :, off, :] = v.reshape(T, s.kv_heads, s.dv).to(v_cache.dtype)


def rope_heads_kv(s: GroupedShape, p, positions, slots, cos, sin, k_cache, v_cache, q_norm=None, k_norm=None, eps: float = 0.0, v_first=None,
                  lam: float = 0.0) -> None:
    """Optional per-head RMS norm of queries and keys (fp32 weights ``[dk]``, mean over the real columns), rotation of the pairs (i, i + half);
    queries in place, keys into their cache rows. The values go to the cache as projected (tied: the keys as projected) or, with ``v_first
    [T, G * dv]``, as ``(1 - lam) v + lam v_first``."""
    if ops._cuda(p):
        ops._count()
        ops.require_ext().rope_heads_kv(p, s.q_width, s.v_at, positions, slots, cos, sin, k_cache, v_cache, s.heads, s.kv_heads, s.dk, s.dv, s.dim, q_norm, k_norm,
                                        eps, v_first, lam)
        return
    T, pos = p.shape[0], positions.long()
    q = p[:, : s.q_width].reshape(T, s.heads, s.dk)
    k = p[:, s.q_width : s.q_width + s.k_width].reshape(T, s.kv_heads, s.dk)
    v = p[:, s.v_at : s.v_at + s.v_width].reshape(T, s.kv_heads, s.dv)
    if v_first is not None:
        v = (1.0 - lam) * v.float() + lam * v_first.float().reshape(T, s.kv_heads, s.dv)
    page = k_cache.shape[2]
    blk, off = torch.div(slots, page, rounding_mode="floor"), slots % page
    cached = lambda c, x: x.reshape(T, c.shape[1], -1).to(c.dtype)  # noqa: E731  (mixed scores: one wide head)
    v_cache[blk, :, off, :] = cached(v_cache, v)

    def normed(x, w):
        if w is None:
            return x
        x = x.float()
        return x * torch.rsqrt(x.pow(2).sum(dim=-1, keepdim=True) / s.dim + eps) * w

    k_cache[blk, :, off, :] = cached(k_cache, ref.apply_rope(normed(k, k_norm), pos, cos, sin))
    p[:, : s.q_width] = ref.apply_rope(normed(q, q_norm), pos, cos, sin).reshape(T, -1).to(p.dtype)


def attention(s: GroupedShape, qkv, batch, k_cache, v_cache, scale: float, softcap: float, window: int, keep_first: int, sink, splits: int, mult: float = 1.0,
              out=None, mix=None):
    """Heads of every row of the batch, ``[T, H * dv]`` (``out``: a column range of wider rows to write to); the batch's keys and values are
    in the cache already. ``sink``: fp32 ``[H]`` or None. Gated shapes multiply with the sigmoid of their logits in ``qkv``, all with ``mult``.
    ``mix``: fp32 ``[H, H]`` of shapes with mixed scores."""
    q = qkv[:, : s.q_width]
    gate = qkv[:, s.gate_at : s.gate_at + s.gate_logits] if s.gate else None
    if not ops._cuda(qkv):
        split = lambda c: c.reshape(c.shape[0], c.shape[2], s.kv_heads, -1).transpose(1, 2) if s.mixed else c  # noqa: E731
        o = ref.paged_attention(q.reshape(-1, s.heads, s.dk), split(k_cache), split(v_cache), batch.block_tables, batch.q_start.tolist(), batch.q_len.tolist(),
                                batch.ctx_len.tolist(), scale, softcap, window, True, keep_first, sink, mix)
        if gate is not None:
            o = o.float() * torch.sigmoid(gate.float()).reshape(o.shape[0], s.heads, -1)
        o = (o * mult).to(qkv.dtype).reshape(-1, s.out_width)
        return o if out is None else out.copy_(o)
    e = ops.require_ext()
    mask = (float(scale), float(softcap), int(window))
    extra = {"keep_first": int(keep_first), "sink": sink, "gate": gate, "out_mult": float(mult), "out": out}
    if s.mixed:
        return _mixed_attention(s, qkv, q, mix, batch, k_cache, v_cache, mask, splits, extra)
    if qkv.dtype == torch.float32 or not s.tensor_core:
        ops._count()
        return e.attention_rows(q, k_cache, v_cache, batch.block_tables, None if batch.is_decode else row_sequence(batch), batch.positions, s.heads, *mask, **extra)
    if batch.is_decode:
        ops._count(1 if splits <= 1 else 2)
        return e.decode_attention(q, k_cache, v_cache, batch.block_tables, batch.ctx_len, s.heads, *mask, splits, 0, **extra)
    ts, t0 = batch.tiles(e.prefill_tc_tile_rows(max(s.dk, s.dv)))
    ops._count()
    return e.prefill_attention_tc(q, k_cache, v_cache, batch.block_tables, batch.q_start, batch.q_len, batch.ctx_len, ts, t0, s.heads, *mask, True, **extra)


def _mixed_attention(s: GroupedShape, qkv, q, mix, batch, k_cache, v_cache, mask: tuple, splits: int, extra: dict):
    e = ops.require_ext()
    if batch.is_decode and qkv.dtype == torch.bfloat16 and e.mixed_decode_ok(s.heads, s.kv_heads, s.dk, s.dv):
        ops._count(1 if splits <= 1 else 2)
        return e.mixed_decode(q, mix, k_cache, v_cache, batch.block_tables, batch.ctx_len, s.heads, s.kv_heads, mask[0], mask[2], splits, gate=extra["gate"],
                              out_mult=extra["out_mult"], out=extra["out"])
    rows = 0 if batch.is_decode or qkv.dtype == torch.float32 else e.prefill_wide_tile_rows(s.k_width, s.dv)
    if not rows:
        ops._count(2)
        return e.attention_rows(e.fold_heads(q, mix, s.heads, s.kv_heads, s.k_width), k_cache, v_cache, batch.block_tables,
                                None if batch.is_decode else row_sequence(batch), batch.positions, s.heads, *mask, kv_heads=s.kv_heads, **extra)
    ops._count(3)
    pitch = (s.k_width + 63) // 64 * 64
    plan = wide_plan(batch, mask[2])
    keys, values = e.latent_gather(k_cache, v_cache, batch.block_tables, plan["seq"], plan["key0"], plan["n_keys"], plan["row0"], plan["max_rows"], plan["total"], pitch,
                                   s.v_width)
    ts, t0 = batch.tiles(rows)
    return e.prefill_wide(e.fold_heads(q, mix, s.heads, s.kv_heads, pitch), keys, values, batch.q_start, batch.q_len, plan["n_keys"], plan["row0"], ts, t0, s.heads,
                          s.kv_heads, mask[0], mask[2], gate=extra["gate"], out_mult=extra["out_mult"], out=extra["out"])


def wide_plan(batch, window: int) -> dict:
    """Visible key range of every sequence of a batch and its place in the gathered rows (built once per batch and window)."""
    key = ("wide", window)
    if key not in batch.plans:
        dev = batch.q_len.device
        n, ctx = torch.tensor(batch.q_len_host), torch.tensor(batch.ctx_len_host)
        first = (ctx - n - window + 1).clamp(min=0) if window > 0 else torch.zeros_like(ctx)
        keys = torch.where(n > 0, ctx - first, torch.zeros_like(ctx))
        row0 = torch.cumsum(keys, 0) - keys
        put = lambda t: t.to(torch.int32).to(dev, non_blocking=True)  # noqa: E731
        batch.plans[key] = {"seq": put(torch.arange(len(n))), "key0": put(first), "n_keys": put(keys), "row0": put(row0), "max_rows": int(keys.max()),
                            "total": int(keys.sum())}
    return batch.plans[key]


def mixed_splits(s: GroupedShape, num_seqs: int, span: int, sms: int = 148) -> int:
    """Split-KV factor of the decode kernel of mixed scores: one CTA per (sequence, split), as many as run at once, at least two 32-key tiles per split."""
    e = ops.ext()
    ctas = e.mixed_decode_ctas(s.heads, s.kv_heads, s.dk, s.dv) if e is not None else 1
    tiles = max(1, (span + 31) // 32)
    return int(max(1, min(sms * max(1, ctas) // max(1, num_seqs), tiles // 2, 64)))


def row_sequence(batch) -> torch.Tensor:
    """Sequence of every row of a batch (int32, built once per batch)."""
    if "row_seq" not in batch.plans and batch.is_decode:
        batch.plans["row_seq"] = torch.arange(batch.num_seqs, dtype=torch.int32, device=batch.q_len.device)
    if "row_seq" not in batch.plans:
        n = torch.tensor(batch.q_len_host)
        batch.plans["row_seq"] = torch.repeat_interleave(torch.arange(len(n)), n).to(torch.int32).to(batch.q_len.device, non_blocking=True)
    return batch.plans["row_seq"]
