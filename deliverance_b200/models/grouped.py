"""Grouped-query attention mixer with per-layer sizes (``ops/grouped.py``): any decoder can use it. Score scale, soft-cap, window, kept
first tokens, sink, rotation tables and layout, head norms, mixed scores, value mixing and output gate are parameters; it reads its input rows, keeps its
cache in the pair ``kv.layer(i)`` and returns the output projection (:meth:`forward`), or works between projections that it shares with
another mixer (:meth:`pack`, :meth:`heads`)."""
from __future__ import annotations

from typing import Optional

import torch

from .. import ops
from ..ops import LinearWeight, grouped as gop
from ..ops.grouped import GroupedShape, pad_head_columns, pad_head_rows
from .batch import ForwardBatch


class GroupedAttention:
    def __init__(self, shape: GroupedShape, scale: float, softcap: float, window: int, keep_first: int, sink: bool, cos, sin, device, dtype,
                 rotate: str = "pairs", eps: float = 0.0, mult: float = 1.0, v_mix: bool = False):
        """``sink``: the softmax has a sink, of score 0 unless :meth:`pack` gets learned ones. ``rotate``: ``pairs`` (2 i, 2 i + 1) or ``halves``
        (i, i + half) of the rotated columns. ``mult``: constant factor of the heads. ``v_mix``: the values are blended with those of the
        first such layer of the forward pass."""
        self.shape, self.scale, self.softcap = shape, float(scale), float(softcap)
        self.window, self.keep_first = int(window), int(keep_first)
        self.kind = "sliding" if self.window > 0 else "attention"
        self.sink = torch.zeros(shape.heads, dtype=torch.float32, device=device) if sink else None
        self.cos, self.sin, self.rotate = cos, sin, rotate
        self.eps, self.mult, self.v_mix = float(eps), float(mult), bool(v_mix)
        self.lam = 0.0
        self.q_norm = self.k_norm = self.mix = None
        self.device, self.dtype = device, dtype
        if cos.shape[1] * 2 > shape.dim:
            raise ValueError(f"rotation covers {cos.shape[1] * 2} of {shape.dim} query / key columns")
        if rotate not in ("pairs", "halves") or (rotate == "pairs" and (shape.tied or v_mix or shape.mixed)):
            raise ValueError("tied values, mixed values and mixed scores need the 'halves' rotation")
        if shape.mixed and (softcap or keep_first or sink):
            raise ValueError("mixed scores go without soft-cap, kept tokens and sink")

    def pack(self, q, k, v, o, g=None, sink=None, q_norm=None, k_norm=None, vmix: Optional[float] = None, mix=None) -> tuple:
        """Weights as stored (``[out, in]``) -> (rows of the input projection, columns of the output projection) in the padded layout. ``mix [H, H]`` (to,
        from): head h's score becomes ``sum_g mix[h, g] score_g`` in front of the softmax."""
        s = self.shape
        want = [("q", q, s.heads * s.dim), ("k", k, s.kv_heads * s.dim)]
        if not s.tied:
            want.append(("v", v, s.kv_heads * s.vdim))
        if s.gate:
            want.append(("g", g, s.heads * (s.vdim if s.gate == "columns" else 1)))
        for n, t, rows in want:
            if t.shape[0] != rows:
                raise ValueError(f"grouped attention: '{n}' has {t.shape[0]} rows, the configured sizes need {rows}")
        if o.shape[1] != s.heads * s.vdim:
            raise ValueError(f"grouped attention: 'o' has {o.shape[1]} columns, the configured sizes need {s.heads * s.vdim}")
        rows = [pad_head_rows(q, s.heads, s.dim, s.dk), pad_head_rows(k, s.kv_heads, s.dim, s.dk)]
        if not s.tied:
            rows.append(pad_head_rows(v, s.kv_heads, s.vdim, s.dv))
        if s.gate:
            rows.append(pad_head_rows(g, s.heads, s.vdim, s.dv) if s.gate == "columns" else g)
        w = torch.cat(rows)
        w = torch.nn.functional.pad(w, (0, 0, 0, s.width - w.shape[0]))
        if sink is not None:
            if sink.numel() != s.heads:
                raise ValueError(f"grouped attention: {sink.numel()} sinks for {s.heads} heads")
            self.sink = sink.reshape(-1).to(device=self.device, dtype=torch.float32).contiguous()
        if q_norm is not None:
            if q_norm.numel() != s.dim or k_norm.numel() != s.dim:
                raise ValueError(f"grouped attention: head norms need {s.dim} weights")
            norm = lambda t: torch.nn.functional.pad(t.reshape(-1).float(), (0, s.dk - s.dim)).to(self.device).contiguous()  # noqa: E731
            self.q_norm, self.k_norm = norm(q_norm), norm(k_norm)
        if vmix is not None:
            self.lam = float(vmix)
        if s.mixed != (mix is not None) or (mix is not None and tuple(mix.shape) != (s.heads, s.heads)):
            raise ValueError(f"grouped attention: mixed scores need a [{s.heads}, {s.heads}] matrix")
        if mix is not None:
            self.mix = mix.to(device=self.device, dtype=torch.float32).contiguous()
        return w, pad_head_columns(o, s.heads, s.vdim, s.dv)

    def load(self, q, k, v, o, k_pad: int, **extra) -> "GroupedAttention":
        """:meth:`pack` with projections of its own; ``k_pad``: padded input width of the rows :meth:`forward` gets."""
        w, o = self.pack(q, k, v, o, **extra)
        put = lambda t: LinearWeight(t.to(device=self.device, dtype=self.dtype).contiguous())  # noqa: E731
        self.w_in, self.w_out = put(torch.nn.functional.pad(w, (0, k_pad - w.shape[1]))), put(o)
        return self

    def nbytes(self) -> int:
        return self.w_in.nbytes() + self.w_out.nbytes()

    def forward(self, x, batch: ForwardBatch, kv, run: int, stage, shared: Optional[dict] = None) -> torch.Tensor:
        """``shared``: what the layers of one forward pass hand on (the first mixing layer's values)."""
        with stage("groupedattention.qkv_projection"):
            p = ops.linear(x, self.w_in)
        a = self.heads(p, batch, kv, run, stage, shared=shared)
        with stage("groupedattention.output_projection"):
            return ops.linear(a, self.w_out)

    def heads(self, p, batch: ForwardBatch, kv, run: int, stage, out=None, shared: Optional[dict] = None) -> torch.Tensor:
        """``p [T, shape.width]``: this mixer's columns of the projection rows -> gated heads ``[T, H * dv]`` (in ``out`` when given)."""
        s = self.shape
        k_cache, v_cache = kv.layer(run)
        with stage("groupedattention.rope"):
            if self.rotate == "pairs":
                gop.rope_pairs_kv(s, p[:, : s.gate_at], batch.positions, batch.slots, self.cos, self.sin, k_cache, v_cache)
            else:
                first = None
                if self.v_mix:
                    v = p[:, s.v_at : s.v_at + s.v_width]
                    first = shared.get("values")
                    if first is None:
                        shared["values"] = v
                    elif first.shape != v.shape:
                        raise ValueError(f"values of {v.shape[1]} columns cannot be mixed with {first.shape[1]}")
                gop.rope_heads_kv(s, p, batch.positions, batch.slots, self.cos, self.sin, k_cache, v_cache, self.q_norm, self.k_norm, self.eps, first, self.lam)
        with stage("groupedattention.score_value"):
            return gop.attention(s, p, batch, k_cache, v_cache, self.scale, self.softcap, self.window, self.keep_first, self.sink, self._splits(batch), self.mult, out, self.mix)

    def _splits(self, batch: ForwardBatch) -> int:
        """Split-KV factor of a decode step: a captured step knows the window but not the contexts it will see."""
        if not batch.is_decode:
            return 1
        span = max(batch.ctx_len_host) if batch.ctx_len_host else self.cos.shape[0]
        if self.window > 0:
            span = min(span, self.window + self.keep_first)
        if self.shape.mixed:  # (a CTA takes all heads)
            return gop.mixed_splits(self.shape, batch.num_seqs, span)
        return ops.decode_splits(batch.num_seqs, self.shape.kv_heads * ((self.shape.heads // self.shape.kv_heads + 15) // 16), span)

    def cache_layout(self) -> dict:
        if self.shape.mixed:  # one wide row per token
            return {"heads": 1, "k": self.shape.k_width, "v": self.shape.v_width, "state": None}
        return {"heads": self.shape.kv_heads, "k": self.shape.dk, "v": self.shape.dv, "state": None}
