"""Mamba-2 mixer (``ops/mamba.py``): any decoder can use it. It reads its input rows, keeps a ring of convolution inputs and one fp32 state per
sequence in the cache manager's state slots and returns the output projection.

granitemoehybrid's Mamba-2 layers run on the same operator (:func:`mamba_forward`; reference: core/.../model/granitemoehybrid/
GraniteMoeHybridMambaLayer.java:130-252, which walks tokens one by one): ``[gate | x | B | C | dt]`` projection, causal depthwise convolution with a
rolling state + SiLU, recurrence, ``silu(gate)``, RMS norm over the whole intermediate, output projection.
"""
from __future__ import annotations

import torch

from .. import ops
from ..ops import LinearWeight, mamba as mamba_op
from ..ops.grouped import pad_head_columns, up8
from ..ops.mamba import Mamba2Shape, Mamba2Weights
from ..ops.short_conv import MAX_TAPS
from .batch import ForwardBatch


class Mamba2Mixer:
    kind = "mamba"

    def __init__(self, shape: Mamba2Shape, eps: float, device, dtype):
        self.shape, self.eps = shape, float(eps)
        self.device, self.dtype = device, dtype
        if device.type == "cuda" and (shape.dn > mamba_op.MAX_STATE or shape.taps > MAX_TAPS):
            raise ValueError(f"Mamba-2: state size {shape.state}, {shape.taps} taps (at most {mamba_op.MAX_STATE} and {MAX_TAPS} on CUDA)")

    def load(self, w_in, conv, conv_b, dt_bias, A_log, D, norm, o, k_pad: int) -> "Mamba2Mixer":
        """Weights as stored (``[out, in]``); ``k_pad``: padded input width of the rows :meth:`forward` gets."""
        s = self.shape
        rows = 2 * s.heads * s.vdim + 2 * s.groups * s.state + s.heads
        if w_in.shape[0] != rows or o.shape[1] != s.heads * s.vdim:
            raise ValueError(f"Mamba-2: projections of {w_in.shape[0]} rows and {o.shape[1]} columns, the configured sizes need {rows} and {s.heads * s.vdim}")
        w = s.pad_input(w_in)
        w = torch.nn.functional.pad(w, (0, k_pad - w.shape[1], 0, up8(w.shape[0]) - w.shape[0]))
        put = lambda t: LinearWeight(t.to(device=self.device, dtype=self.dtype).contiguous())  # noqa: E731
        self.w_in, self.w_out = put(w), put(pad_head_columns(o, s.heads, s.vdim, s.dv))
        self.w = Mamba2Weights.pack(s, conv, conv_b, dt_bias, A_log, D, norm, self.device)
        return self

    def nbytes(self) -> int:
        return self.w_in.nbytes() + self.w_out.nbytes() + self.w.conv.numel() * 4

    def forward(self, x, batch: ForwardBatch, kv, run: int, stage) -> torch.Tensor:
        with stage("mamba.input_projection"):
            p = ops.linear(x, self.w_in)
        with stage("mamba.recurrence"):
            y = mamba_op.mamba2(self.shape, p, self.w, kv.state["conv"][run], kv.state["ssm"][run], batch, self.eps)
        with stage("mamba.output_projection"):
            return ops.linear(y, self.w_out)

    def cache_layout(self) -> dict:
        return {"heads": 1, "k": 8, "v": 8, "state": self.shape.state_shapes()}


def mamba_forward(model, i: int, lw, x: torch.Tensor, batch, kv) -> torch.Tensor:
    """One granitemoehybrid Mamba-2 layer: the projections are the model's (possibly JQ4) weights."""
    m, s = lw.mamba, lw.mamba["shape"]
    w = m["in_proj"]
    if x.device.type == "cuda" and w.N % 8:  # the kernels read 16-byte pieces of the rows
        p = torch.empty(x.shape[0], up8(w.N), dtype=x.dtype, device=x.device)
        ops.linear(x, w, out=p[:, : w.N])
    else:
        p = ops.linear(x, w)
    y = mamba_op.mamba2(s, p, m["weights"], kv.state["conv"][i], kv.state["ssm"][i], batch, model.cfg.norm_eps)
    return ops.linear(y, m["out_proj"])
