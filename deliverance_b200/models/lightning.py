"""Lightning-attention mixer (``ops/lightning.py``): any decoder can use it, alone or beside another mixer. It works on a column range of
projection rows, keeps one fp32 state per sequence in the cache manager's state slots and writes its gated heads into a column range of the
rows that the output projection reads."""
from __future__ import annotations

import torch

from ..ops import lightning as lop
from ..ops.grouped import pad_head_columns, pad_head_rows
from ..ops.lightning import LightningShape
from .batch import ForwardBatch


class LightningAttention:
    def __init__(self, shape: LightningShape, decay, eps: float, device, dtype, mult: float = 1.0):
        if len(decay) != shape.heads:
            raise ValueError(f"lightning attention: {len(decay)} decays for {shape.heads} heads")
        self.shape, self.eps, self.mult = shape, float(eps), float(mult)
        self.decay = torch.tensor([float(d) for d in decay], dtype=torch.float64)
        self.device, self.dtype = device, dtype
        if device.type == "cuda" and shape.dk > lop.MAX_DK:
            raise ValueError(f"lightning attention: {shape.dim} key channels per head (at most {lop.MAX_DK} on CUDA)")
        self.powers = lop.decay_powers(decay).to(device)

    def pack(self, q, k, v, g, o, norm) -> tuple:
        """Weights as stored (``[out, in]``) -> (rows of the input projection, columns of the output projection) in the padded layout."""
        s, H = self.shape, self.shape.heads
        for n, t, rows in (("q", q, H * s.dim), ("k", k, H * s.dim), ("v", v, H * s.vdim), ("g", g, H * s.vdim)):
            if t.shape[0] != rows:
                raise ValueError(f"lightning attention: '{n}' has {t.shape[0]} rows, the configured sizes need {rows}")
        if o.shape[1] != H * s.vdim or norm.numel() != H * s.vdim:
            raise ValueError("lightning attention: output projection or norm does not match the configured sizes")
        w = torch.cat([pad_head_rows(q, H, s.dim, s.dk), pad_head_rows(k, H, s.dim, s.dk), pad_head_rows(v, H, s.vdim, s.dv), pad_head_rows(g, H, s.vdim, s.dv)])
        self.norm = pad_head_rows(norm.float().reshape(-1, 1), H, s.vdim, s.dv).reshape(-1).to(self.device).contiguous()
        return w, pad_head_columns(o, H, s.vdim, s.dv)

    def nbytes(self) -> int:
        return (self.norm.numel() + self.powers.numel()) * 4

    def heads(self, p, batch: ForwardBatch, kv, run: int, out, stage) -> None:
        """``p [T, shape.width]``: this mixer's columns of the projection rows; the heads go to ``out [T, H * dv]``."""
        with stage("lightning.recurrence"):
            lop.lightning(self.shape, p, self.decay, self.powers, self.norm, kv.state["lightning"][run], batch, self.eps, self.mult, out)

    def state_shapes(self) -> dict:
        return {"lightning": (self.shape.heads, self.shape.dk, self.shape.dv)}
