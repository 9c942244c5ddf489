"""Gated-delta-rule mixer (``ops/delta.py``): any decoder can use it, alone or beside another mixer. It works on a column range of projection rows, keeps
a ring of convolution inputs and one fp32 state per sequence in the cache manager's state slots and writes its gated heads into a column range of
the rows that the output projection reads. The two low-rank projections (decays, output gate) are one GEMM in decode steps."""
from __future__ import annotations

import torch

from .. import ops
from ..ops import LinearWeight, delta as dop
from ..ops.delta import DeltaShape
from ..ops.grouped import pad_head_columns, pad_head_rows, up8
from ..ops.short_conv import MAX_TAPS
from .batch import ForwardBatch


class GatedDeltaNet:
    def __init__(self, shape: DeltaShape, eps: float, device, dtype, mult: float = 1.0):
        self.shape, self.eps, self.mult = shape, float(eps), float(mult)
        self.q_scale = shape.dim ** -0.5
        self.device, self.dtype = device, dtype
        if device.type == "cuda" and (shape.dk > dop.MAX_DK or shape.taps > MAX_TAPS):
            raise ValueError(f"gated delta rule: {shape.dim} key channels per head, {shape.taps} taps (at most {dop.MAX_DK} and {MAX_TAPS} on CUDA)")

    def pack(self, q, k, v, b, a1, a2, g1, g2, o, convs, A_log, dt_bias, norm) -> tuple:
        """Weights as stored (``[out, in]``; ``convs``: filters of q, k and v) -> (rows of the input projection, columns of the output projection) in the
        padded layout."""
        s, H, G = self.shape, self.shape.heads, self.shape.kv_heads
        pieces = (("q", q, G, s.dim), ("k", k, G, s.dim), ("v", v, H, s.vdim))
        want = [(n, t, h * d) for n, t, h, d in pieces] + [("b", b, H), ("a1", a1, s.rank_a), ("a2", a2, H * s.dim), ("g1", g1, s.rank_g), ("g2", g2, H * s.vdim)]
        want += [(f"{n}.conv", c, h * d) for (n, _, h, d), c in zip(pieces, convs)]
        for n, t, rows in want:
            if t.shape[0] != rows:
                raise ValueError(f"gated delta rule: '{n}' has {t.shape[0]} rows, the configured sizes need {rows}")
        if (o.shape[1] != H * s.vdim or norm.numel() != s.vdim or A_log.numel() != H or dt_bias.numel() != H * s.dim or a2.shape[1] != s.rank_a
                or g2.shape[1] != s.rank_g or any(c.shape[1] != s.taps for c in convs)):
            raise ValueError("gated delta rule: output projection, norm, decays, low-rank factors or filters do not match the configured sizes")
        pad = torch.nn.functional.pad
        heads = lambda t, h, d: pad_head_rows(t, h, d, up8(d))  # noqa: E731
        rows = lambda t: pad(t, (0, 0, 0, up8(t.shape[0]) - t.shape[0]))  # noqa: E731
        w = torch.cat([heads(t, h, d) for _, t, h, d in pieces] + [rows(b), rows(a1), rows(g1)])
        ra, rg = up8(s.rank_a), up8(s.rank_g)
        decay, gate = pad(heads(a2, H, s.dim), (0, ra - s.rank_a + rg)), pad(heads(g2, H, s.vdim), (ra, rg - s.rank_g))
        put = lambda t: LinearWeight(t.to(device=self.device, dtype=self.dtype).contiguous())  # noqa: E731
        self.w_low, self.w_decay, self.w_gate = put(torch.cat([decay, gate])), put(decay[:, :ra]), put(gate[:, ra:])
        dev = lambda t: t.float().to(self.device).contiguous()  # noqa: E731
        self.conv = dev(torch.cat([heads(c.reshape(h * d, s.taps), h, d) for (_, _, h, d), c in zip(pieces, convs)]).t())
        self.dt_bias = dev(heads(dt_bias.reshape(-1, 1), H, s.dim).reshape(-1))
        self.neg_a = dev(-torch.exp(A_log.double()).reshape(-1))
        self.norm = dev(pad(norm.reshape(-1), (0, s.dv - s.vdim)))
        return w, pad_head_columns(o, H, s.vdim, s.dv)

    def nbytes(self) -> int:
        return self.w_low.nbytes() + self.w_decay.nbytes() + self.w_gate.nbytes() + (self.conv.numel() + self.dt_bias.numel() + self.norm.numel()) * 4

    def heads(self, p, batch: ForwardBatch, kv, run: int, out, stage) -> None:
        """``p [T, shape.width]``: this mixer's columns of the projection rows; the heads go to ``out [T, H * dv]``."""
        s = self.shape
        with stage("delta.low_rank_projections"):
            if dop.fused_step(s, batch):  # one launch, block diagonal
                z, gate = ops.linear(p[:, s.low_at :], self.w_low, out_f32=True).split([s.heads * s.dk, s.out_width], dim=1)
            else:
                z = ops.linear(p[:, s.low_at : s.low_at + self.w_decay.K], self.w_decay, out_f32=True)
                gate = ops.linear(p[:, s.low_at + self.w_decay.K : s.width], self.w_gate)
        with stage("delta.recurrence"):
            dop.delta(s, p, z, gate, self.conv, self.dt_bias, self.neg_a, self.norm, kv.state["conv"][run], kv.state["delta"][run], batch, self.q_scale, self.eps, self.mult,
                      out)

    def state_shapes(self) -> dict:
        return self.shape.state_shapes()
