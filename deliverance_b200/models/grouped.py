"""Grouped-query attention mixer with per-layer sizes (``ops/grouped.py``): any decoder can use it. Score scale, soft-cap, window, kept
first tokens, sink and rotation tables are parameters; it reads its input rows, keeps its cache in the pair ``kv.layer(i)`` and returns
the output projection."""
from __future__ import annotations

import torch

from .. import ops
from ..ops import LinearWeight, grouped as gop
from ..ops.grouped import GroupedShape, pad_head_columns, pad_head_rows
from .batch import ForwardBatch


class GroupedAttention:
    kind = "sliding"

    def __init__(self, shape: GroupedShape, scale: float, softcap: float, window: int, keep_first: int, sink: bool, cos, sin, device, dtype):
        self.shape, self.scale, self.softcap = shape, float(scale), float(softcap)
        self.window, self.keep_first, self.sink = int(window), int(keep_first), bool(sink)
        self.cos, self.sin = cos, sin
        self.device, self.dtype = device, dtype
        if cos.shape[1] * 2 > shape.dim:
            raise ValueError(f"rotation covers {cos.shape[1] * 2} of {shape.dim} query / key columns")

    def load(self, q, k, v, o, k_pad: int) -> "GroupedAttention":
        """Weights as stored (``[out, in]``); ``k_pad``: padded input width of the rows :meth:`forward` gets."""
        s = self.shape
        for n, t, rows in (("q", q, s.heads * s.dim), ("k", k, s.kv_heads * s.dim), ("v", v, s.kv_heads * s.vdim)):
            if t.shape[0] != rows:
                raise ValueError(f"grouped attention: '{n}' has {t.shape[0]} rows, the configured sizes need {rows}")
        if o.shape[1] != s.heads * s.vdim:
            raise ValueError(f"grouped attention: 'o' has {o.shape[1]} columns, the configured sizes need {s.heads * s.vdim}")
        w = torch.cat([pad_head_rows(q, s.heads, s.dim, s.dk), pad_head_rows(k, s.kv_heads, s.dim, s.dk), pad_head_rows(v, s.kv_heads, s.vdim, s.dv)])
        w = torch.nn.functional.pad(w, (0, k_pad - w.shape[1]))
        put = lambda t: LinearWeight(t.to(device=self.device, dtype=self.dtype).contiguous())  # noqa: E731
        self.w_in, self.w_out = put(w), put(pad_head_columns(o, s.heads, s.vdim, s.dv))
        return self

    def nbytes(self) -> int:
        return self.w_in.nbytes() + self.w_out.nbytes()

    def forward(self, x, batch: ForwardBatch, kv, run: int, stage) -> torch.Tensor:
        s = self.shape
        k_cache, v_cache = kv.layer(run)
        with stage("groupedattention.qkv_projection"):
            qkv = ops.linear(x, self.w_in)
        with stage("groupedattention.rope"):
            gop.rope_pairs_kv(s, qkv, batch.positions, batch.slots, self.cos, self.sin, k_cache, v_cache)
        with stage("groupedattention.score_value"):
            a = gop.attention(s, qkv, batch, k_cache, v_cache, self.scale, self.softcap, self.window, self.keep_first, self.sink, self._splits(batch))
        with stage("groupedattention.output_projection"):
            return ops.linear(a, self.w_out)

    def _splits(self, batch: ForwardBatch) -> int:
        """Split-KV factor of a decode step: a captured step knows the window but not the contexts it will see."""
        if not batch.is_decode:
            return 1
        span = max(batch.ctx_len_host) if batch.ctx_len_host else self.cos.shape[0]
        if self.window > 0:
            span = min(span, self.window + self.keep_first)
        return ops.decode_splits(batch.num_seqs, self.shape.kv_heads * ((self.shape.heads // self.shape.kv_heads + 15) // 16), span)

    def cache_layout(self) -> dict:
        return {"heads": self.shape.kv_heads, "k": self.shape.dk, "v": self.shape.dv, "state": None}
