"""Softmax attention and a recurrent mixer (lightning attention, gated delta rule) side by side on the same input rows: ``a * left(h) + b * right(h)``. All
input projections of both are one GEMM; both write their gated heads, already times their constants, into one row buffer, so that the two output
projections, whose results are summed anyway, are one GEMM too. A layer holds pages and a state slot."""
from __future__ import annotations

import torch

from .. import ops
from ..ops import LinearWeight
from .batch import ForwardBatch
from .grouped import GroupedAttention


class SideBySideMixer:
    kind = "attention"

    def __init__(self, left: GroupedAttention, right):
        self.left, self.right = left, right

    def load(self, left: tuple, right: tuple, k_pad: int) -> "SideBySideMixer":
        """``left``, ``right``: (input rows, output columns) of the parts' ``pack``."""
        dev, dt = self.left.device, self.left.dtype
        put = lambda t: LinearWeight(t.to(device=dev, dtype=dt).contiguous())  # noqa: E731
        w = torch.cat([left[0], right[0]])
        self.w_in, self.w_out = put(torch.nn.functional.pad(w, (0, k_pad - w.shape[1]))), put(torch.cat([left[1], right[1]], dim=1))
        return self

    def nbytes(self) -> int:
        return self.w_in.nbytes() + self.w_out.nbytes() + self.right.nbytes()

    def forward(self, x, batch: ForwardBatch, kv, run: int, stage, shared=None) -> torch.Tensor:
        ls, rs = self.left.shape, self.right.shape
        with stage("sidebyside.input_projection"):
            p = ops.linear(x, self.w_in)
        row = torch.empty(x.shape[0], ls.out_width + rs.out_width, dtype=p.dtype, device=p.device)
        self.left.heads(p[:, : ls.width], batch, kv, run, stage, out=row[:, : ls.out_width])
        self.right.heads(p[:, ls.width :], batch, kv, run, row[:, ls.out_width :], stage)
        with stage("sidebyside.output_projection"):
            return ops.linear(row, self.w_out)

    def cache_layout(self) -> dict:
        return dict(self.left.cache_layout(), state=self.right.state_shapes())
