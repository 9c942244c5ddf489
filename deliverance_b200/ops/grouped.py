"""Grouped-query softmax attention with per-layer sizes: unequal query / key and value widths, partial rotation of neighbouring pairs,
sliding window with kept first tokens, score soft-cap and a sink in the denominator (a score of 0 that has no value).

One projection row is ``[q (H * dk) | k (G * dk) | v (G * dv)]`` with head widths rounded up to multiples of 8 (16-byte rows everywhere);
the columns behind the real ones carry zero weights, so scores, cache rows and outputs are exact whatever the sizes. CUDA forms:

* prompts: the tcgen05 / TMA kernel (``attention_tc.cu``) over the paged cache, heads up to 256 wide;
* decode: the split-KV tensor-core kernel (``attention.cu``), heads up to 256 wide;
* fp32 and wider heads: one CTA per (row, head) on CUDA cores.
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

    def __post_init__(self):
        if self.heads % self.kv_heads:
            raise ValueError(f"{self.heads} query heads do not divide into {self.kv_heads} groups")

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
    def width(self) -> int:
        return self.q_width + self.k_width + self.kv_heads * self.dv

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


def attention(s: GroupedShape, qkv, batch, k_cache, v_cache, scale: float, softcap: float, window: int, keep_first: int, sink: bool, splits: int):
    """Heads of every row of the batch, ``[T, H * dv]``; the batch's keys and values are in the cache already."""
    q = qkv[:, : s.q_width]
    mask = (float(scale), float(softcap), int(window), int(keep_first), bool(sink))
    if not ops._cuda(qkv):
        o = ref.paged_attention(q.reshape(-1, s.heads, s.dk), k_cache, v_cache, batch.block_tables, batch.q_start.tolist(), batch.q_len.tolist(),
                                batch.ctx_len.tolist(), scale, softcap, window, True, keep_first, sink)
        return o.reshape(-1, s.out_width)
    e = ops.require_ext()
    if qkv.dtype == torch.float32 or not s.tensor_core:
        ops._count()
        return e.attention_rows(q, k_cache, v_cache, batch.block_tables, None if batch.is_decode else row_sequence(batch), batch.positions, s.heads, *mask)
    if batch.is_decode:
        ops._count(1 if splits <= 1 else 2)
        return e.decode_attention(q, k_cache, v_cache, batch.block_tables, batch.ctx_len, s.heads, mask[0], mask[1], mask[2], splits, 0, mask[3], mask[4])
    ts, t0 = batch.tiles(e.prefill_tc_tile_rows(max(s.dk, s.dv)))
    ops._count()
    return e.prefill_attention_tc(q, k_cache, v_cache, batch.block_tables, batch.q_start, batch.q_len, batch.ctx_len, ts, t0, s.heads, mask[0], mask[1],
                                  mask[2], True, mask[3], mask[4])


def row_sequence(batch) -> torch.Tensor:
    """Sequence of every row of a batch (int32, built once per batch)."""
    if "row_seq" not in batch.plans:
        n = torch.tensor(batch.q_len_host)
        batch.plans["row_seq"] = torch.repeat_interleave(torch.arange(len(n)), n).to(torch.int32).to(batch.q_len.device, non_blocking=True)
    return batch.plans["row_seq"]
