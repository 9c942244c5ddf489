"""Latent-attention mixer: weights, rotary tables and the split of a batch between the two evaluation orders of ``ops/latent.py``.

Any decoder can use it: sizes, score scale, window, rotation (halves or neighbouring pairs), a sink per head and the output gate are parameters
of :class:`LatentAttention`; it reads its input rows, keeps its cache in the pair ``kv.layer(i)`` (or, without a down projection, reads the pair
that another layer of the pass has written) and leaves the (gated) heads in a row buffer that an output projection reads: the caller's
(:meth:`heads`) or its own (:meth:`forward`).
"""
from __future__ import annotations

from typing import Optional

import torch

from .. import ops
from ..ops import LinearWeight, latent as lop, ref
from ..ops.latent import LatentShape
from .batch import ForwardBatch

# sequences with at most this many rows in a step go row by row over the latent cache; longer ones expand keys and values first
ROW_BY_ROW = 8


class RotaryTables:
    """cos / sin tables on one device, shared by the layers with the same rotation. ``make``: table builder (frequency scaling rule)."""

    def __init__(self, max_pos: int, device, make=ref.yarn_rope_tables):
        self.max_pos, self.device, self.make = max_pos, device, make
        self._tables: dict = {}

    def get(self, dims: int, base: float, scaling: Optional[dict]):
        key = (dims, base, tuple(sorted(scaling.items())) if scaling else None)
        if key not in self._tables:
            cos, sin = self.make(dims, self.max_pos, base, scaling)
            self._tables[key] = (cos.to(self.device).contiguous(), sin.to(self.device).contiguous())
        return self._tables[key]


class LatentAttention:
    def __init__(self, shape: LatentShape, scale: float, window: int, eps: float, cos, sin, device, dtype, rotate: str = "halves"):
        """``rotate``: the rotated columns turn in pairs (i, i + half), or (2 i, 2 i + 1) with ``pairs``; a score is the same for any order of the rotated
        columns that queries and keys share, so pairs are brought into the order of halves when the weights are packed."""
        self.shape, self.scale, self.window, self.eps = shape, float(scale), int(window), float(eps)
        self.cos, self.sin = cos, sin
        self.device, self.dtype, self.rotate = device, dtype, rotate
        self.sink = self.w_out = None
        if cos.shape[1] * 2 > shape.rot_dim:
            raise ValueError(f"rotation covers {cos.shape[1] * 2} of {shape.rot_dim} rotated columns")

    def _halves_order(self, w, first: int):
        """Rows of ``w [heads, first + rot_dim, K]``: the rotated columns behind the first ones in the order that turns in halves."""
        n = 2 * self.cos.shape[1]
        if self.rotate != "pairs":
            return w
        order = list(range(first)) + [first + i for i in range(0, n, 2)] + [first + i for i in range(1, n, 2)] + list(range(first + n, first + self.shape.rot_dim))
        return w[:, order]

    def load(self, q, dkv, norm, uk, uv, g, k_pad: int, sink=None, o=None) -> "LatentAttention":
        """Weights as stored (``[out, in]``); ``k_pad``: padded input width of the rows :meth:`heads` gets. ``dkv`` and ``norm`` are None for shapes
        without a down projection; ``o``: output projection for :meth:`forward`."""
        s = self.shape
        want = {"q": (q, s.heads * (s.dim + s.rot_dim)), "uk": (uk, s.heads * s.dim), "uv": (uv, s.out_width)}
        if s.down:
            want["dkv"] = (dkv, s.kv_rank + s.rot_dim)
        if s.gate:
            want["g"] = (g, s.out_width)
        for n, (t, rows) in want.items():
            if t.shape[0] != rows:
                raise ValueError(f"latent attention: '{n}' has {t.shape[0]} rows, the configured sizes need {rows}")
        if uk.shape[1] != s.kv_rank or uv.shape[1] != s.kv_rank:
            raise ValueError(f"latent attention: key and value weights read {uk.shape[1]} and {uv.shape[1]} of {s.kv_rank} latent columns")
        dev = lambda t: t.to(device=self.device, dtype=self.dtype).contiguous()  # noqa: E731
        q = self._halves_order(q.reshape(s.heads, s.dim + s.rot_dim, -1), s.dim).reshape(q.shape)
        q, uk, uv = dev(q), dev(uk), dev(uv)
        if s.down:
            dkv = dev(self._halves_order(dkv.unsqueeze(0), s.kv_rank)[0])
        if sink is not None:
            if sink.numel() != s.heads:
                raise ValueError(f"latent attention: {sink.numel()} sinks for {s.heads} heads")
            self.sink = sink.reshape(-1).to(device=self.device, dtype=torch.float32).contiguous()
        if o is not None:
            if o.shape[1] != s.out_width:
                raise ValueError(f"latent attention: 'o' has {o.shape[1]} columns, the configured sizes need {s.out_width}")
            self.w_out = LinearWeight(dev(torch.nn.functional.pad(o, (0, -s.out_width % 8))))
        self.w_in = LinearWeight(lop.pack_input(s, q, dkv, dev(g) if s.gate else None, k_pad))
        self.wuk, self.wuv = lop.pack_absorbed(s, uk, uv)
        self.norm = torch.zeros(s.Rp, dtype=torch.float32, device=self.device)
        if s.down:
            self.norm[: s.kv_rank] = norm.reshape(-1).float().to(self.device)
        self.w_expand, self.dv = None, 0
        if self.device.type == "cuda" and self.dtype == torch.bfloat16:
            self.dv = s.prefill_dv()
            if self.dv:
                self.w_expand = LinearWeight(lop.pack_expand(s, uk, uv, self.dv))
        return self

    def nbytes(self) -> int:
        n = self.w_in.nbytes() + self.norm.numel() * 4 + (self.w_out.nbytes() if self.w_out is not None else 0)
        for t in (self.wuk, self.wuv):
            n += t.numel() * t.element_size()
        return n + (self.w_expand.nbytes() if self.w_expand is not None else 0)

    kind = "latent"

    def forward(self, x, batch: ForwardBatch, kv, run: int, stage) -> torch.Tensor:
        """With the mixer's own output projection (``o`` of :meth:`load`)."""
        n = self.shape.out_width
        row = (torch.zeros if n % 8 else torch.empty)(x.shape[0], self.w_out.K, dtype=x.dtype, device=x.device)
        self.heads(x, batch, kv.layer(run), row, stage)
        with stage("latentattention.output_projection"):
            return ops.linear(row, self.w_out)

    def cache_layout(self) -> dict:
        return {"heads": 1, "k": self.shape.Rp, "v": self.shape.drp, "state": None}

    def heads(self, x, batch: ForwardBatch, kv_pair, out, stage) -> None:
        """``x [T, k_pad]`` (normed) -> gated heads in columns ``[0, H * vdim)`` of ``out [T, .]``. ``stage(name)``: profiler context."""
        s = self.shape
        c_cache, r_cache = kv_pair
        with stage("latentattention.input_projection"):
            p = ops.linear(x, self.w_in)
        write = (batch.positions, batch.slots, self.norm, self.cos, self.sin, c_cache, r_cache, self.eps)
        args = (self.wuk, self.wuv, c_cache, r_cache, batch.block_tables, out, self.scale, self.window)
        if batch.is_decode:
            span = max(batch.ctx_len_host) if batch.ctx_len_host else self.cos.shape[0]
            with stage("latentattention.score_value"):
                lop.rows_attention(s, p, None, None, batch.ctx_len, *args, splits=self._splits(p.shape[0], span), write=write, sink=self.sink)
            return
        with stage("latentattention.rope_norm_cache"):
            lop.prepare(s, p, *write)
        plan = self._plan(batch)
        if plan["rows"] is not None:
            row_idx, row_seq, row_ctx, span = plan["rows"]
            with stage("latentattention.score_value"):
                lop.rows_attention(s, p, row_idx, row_seq, row_ctx, *args, splits=self._splits(row_idx.shape[0], span), sink=self.sink)
        if plan["prompts"] is not None:
            a = plan["prompts"]
            with stage("latentattention.expand"):
                c, kr = lop.gather(s, c_cache, r_cache, batch.block_tables, a["seq"], a["key0"], a["n_keys"], a["row0"], a["max_rows"], a["total"])
                kv = ops.linear(c, self.w_expand)
            with stage("latentattention.score_value"):
                lop.prefill_attention(s, p, kv, kr, a["q_start"], a["q_len"], a["n_keys"], a["row0"], a["tile_seq"], a["tile_q0"], out, self.scale, self.window,
                                      self.sink)

    def _splits(self, rows: int, span: int) -> int:
        return lop.pick_splits(rows, self.shape, min(span, self.window) if self.window > 0 else span)

    def _plan(self, batch: ForwardBatch) -> dict:
        """Which sequences of a mixed batch go row by row and which through expanded keys, with the index arrays of both."""
        tile_rows = lop.prefill_tile_rows(self.dv) if self.w_expand is not None else 0
        key = ("latent", self.window, tile_rows)
        if key in batch.plans:
            return batch.plans[key]
        lens, ctxs = batch.q_len_host, batch.ctx_len_host
        starts = [0]
        for n in lens:
            starts.append(starts[-1] + n)
        dev = batch.q_len.device
        i32 = lambda v: torch.tensor(v, dtype=torch.int32).to(dev, non_blocking=True)  # noqa: E731
        long = [i for i, n in enumerate(lens) if tile_rows and n > ROW_BY_ROW]
        short = [i for i in range(len(lens)) if not (tile_rows and lens[i] > ROW_BY_ROW)]
        plan: dict = {"rows": None, "prompts": None}
        if any(lens[i] for i in short):
            idx = torch.cat([torch.arange(starts[i], starts[i + 1]) for i in short])
            seq = torch.cat([torch.full((lens[i],), i) for i in short])
            ctx = torch.cat([torch.arange(ctxs[i] - lens[i] + 1, ctxs[i] + 1) for i in short])
            put = lambda t: t.to(torch.int32).to(dev, non_blocking=True)  # noqa: E731
            plan["rows"] = (put(idx), put(seq), put(ctx), int(ctx.max()))
        if long:
            first = [max(0, ctxs[i] - lens[i] - self.window + 1) if self.window > 0 else 0 for i in long]
            n_keys = [ctxs[i] - f for i, f in zip(long, first)]
            row0 = [0]
            for n in n_keys:
                row0.append(row0[-1] + n)
            ts, t0 = ops.prefill_tiles([lens[i] for i in long], tile_rows)
            plan["prompts"] = {"seq": i32(long), "key0": i32(first), "n_keys": i32(n_keys), "row0": i32(row0[:-1]), "max_rows": max(n_keys),
                               "total": row0[-1], "q_start": i32([starts[i] for i in long]), "q_len": i32([lens[i] for i in long]),
                               "tile_seq": i32(ts), "tile_q0": i32(t0)}
        batch.plans[key] = plan
        return plan
