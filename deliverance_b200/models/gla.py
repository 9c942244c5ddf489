"""Gated-linear-attention mixer (``ops/gla.py``): any decoder can use it. It reads its input rows, keeps one fp32 state per sequence in
the cache manager's state slots and returns the output projection."""
from __future__ import annotations

import torch

from .. import ops
from ..ops import LinearWeight, gla as gla_op
from ..ops.gla import GlaShape
from ..ops.grouped import pad_head_columns, pad_head_rows
from .batch import ForwardBatch


class GatedLinearAttention:
    kind = "gla"

    def __init__(self, shape: GlaShape, tau: float, eps: float, device, dtype):
        self.shape, self.tau, self.eps = shape, float(tau), float(eps)
        self.q_scale = shape.dim ** -0.5
        self.device, self.dtype = device, dtype
        if device.type == "cuda" and shape.dk > gla_op.MAX_DK:
            raise ValueError(f"gated linear attention: {shape.dim} key channels per head (at most {gla_op.MAX_DK} on CUDA)")

    def load(self, q, k, v, g, o, a1, a2, a2_bias, norm, k_pad: int) -> "GatedLinearAttention":
        """Weights as stored (``[out, in]``); ``k_pad``: padded input width of the rows :meth:`forward` gets."""
        s, H = self.shape, self.shape.heads
        want = {"q": (q, H * s.dim), "k": (k, H * s.dim), "v": (v, H * s.vdim), "g": (g, H * s.vdim), "a1": (a1, s.rank), "a2": (a2, H * s.dim)}
        for n, (t, rows) in want.items():
            if t.shape[0] != rows:
                raise ValueError(f"gated linear attention: '{n}' has {t.shape[0]} rows, the configured sizes need {rows}")
        if o.shape[1] != H * s.vdim or norm.numel() != s.vdim or a2.shape[1] != s.rank or a2_bias.numel() != H * s.dim:
            raise ValueError("gated linear attention: output projection, norm or decay weights do not match the configured sizes")
        pad = torch.nn.functional.pad
        rows = [pad_head_rows(q, H, s.dim, s.dk), pad_head_rows(k, H, s.dim, s.dk), pad_head_rows(v, H, s.vdim, s.dv), pad_head_rows(g, H, s.vdim, s.dv),
                pad(a1, (0, 0, 0, s.rank8 - s.rank))]
        w = torch.cat(rows)
        dev = lambda t, dt=torch.float32: t.to(device=self.device, dtype=dt).contiguous()  # noqa: E731
        self.w_in = LinearWeight(dev(pad(w, (0, k_pad - w.shape[1])), self.dtype))
        self.w_out = LinearWeight(dev(pad_head_columns(o, H, s.vdim, s.dv), self.dtype))
        self.a2 = dev(pad(pad_head_rows(a2.float(), H, s.dim, s.dk), (0, s.rank8 - s.rank)))
        self.a2_bias = dev(pad_head_rows(a2_bias.float().reshape(-1, 1), H, s.dim, s.dk).reshape(-1))
        self.norm = dev(pad(norm.float().reshape(-1), (0, s.dv - s.vdim)))
        return self

    def nbytes(self) -> int:
        return self.w_in.nbytes() + self.w_out.nbytes() + (self.a2.numel() + self.a2_bias.numel() + self.norm.numel()) * 4

    def forward(self, x, batch: ForwardBatch, kv, run: int, stage) -> torch.Tensor:
        with stage("gla.input_projection"):
            p = ops.linear(x, self.w_in)
        with stage("gla.recurrence"):
            y = gla_op.gla(self.shape, p, self.a2, self.a2_bias, self.norm, kv.state["gla"][run], batch, self.q_scale, self.tau, self.eps)
        with stage("gla.output_projection"):
            return ops.linear(y, self.w_out)

    def cache_layout(self) -> dict:
        return {"heads": 1, "k": 8, "v": 8, "state": {"gla": (self.shape.heads, self.shape.dk, self.shape.dv)}}
