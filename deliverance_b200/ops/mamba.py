"""Mamba-2 (state-space duality): ``S_t = exp(-exp(A_log) dt_t) S_(t-1) + dt_t B_t x_t^T``, ``y_t = S_t^T C_t + D x_t`` per head, B and C shared by groups
of heads, ``dt = softplus(. + dt_bias)``; x, B and C come through a short convolution (``ops/short_conv.py``); ``y silu(z)`` is RMS-normed in equal
parts of the heads' columns.

One projection row is ``[z (H * dv) | x (H * dv) | B (G * dn) | C (G * dn) | dt (H)]``, head widths and state sizes rounded up to multiples of 8 (zero
weights behind the real columns; ``silu(0) = 0``, so padded channels stay zero). The state is fp32, one slot per sequence, ``[slots, H, dn, dv]``. Two
evaluation orders, the same numbers up to rounding (``csrc/mamba.cu``):

* recurrent (decode, fp32): every token updates the state in registers, decode steps with the convolution in the same launch;
* chunked (bf16 prompts): as in lightning attention, with decays from running sums of ``dt`` inside the chunk instead of powers of a constant.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

import torch

from .. import ops
from . import ref
from .gla import chunk_plan
from .grouped import pad_head_rows, up8
from .lightning import CHUNK
from .short_conv import ring_shape, short_conv

MAX_STATE = 512  # state size per head the CUDA kernels take
MAX_STATE_CHUNKED = 256


@dataclass(frozen=True)
class Mamba2Shape:
    heads: int
    vdim: int
    state: int
    groups: int
    taps: int
    norm_groups: int = 1

    def __post_init__(self):
        if self.heads % self.groups:
            raise ValueError(f"Mamba-2: {self.heads} heads do not divide into {self.groups} groups")
        if (self.heads * self.vdim) % self.norm_groups:
            raise ValueError(f"Mamba-2: {self.heads * self.vdim} columns do not divide into {self.norm_groups} norm groups")
        if self.taps < 1:
            raise ValueError("Mamba-2: the convolution needs at least one tap")

    @property
    def dv(self) -> int:
        return up8(self.vdim)

    @property
    def dn(self) -> int:
        return up8(self.state)

    @property
    def out_width(self) -> int:
        return self.heads * self.dv

    @property
    def conv_width(self) -> int:
        return self.out_width + 2 * self.groups * self.dn

    @property
    def dt_at(self) -> int:
        return self.out_width + self.conv_width

    def state_shapes(self) -> dict:
        return {"conv": ring_shape(self.taps, self.conv_width), "ssm": (self.heads, self.dn, self.dv)}

    def geometry(self) -> list:
        return [self.heads, self.dn, self.dv, self.groups, self.vdim, self.norm_groups, self.dt_at]

    # rows of stored weights -> padded rows of the pieces [z | x | B | C]
    def pad_input(self, w) -> torch.Tensor:
        H, G, I = self.heads, self.groups, self.heads * self.vdim
        z, x, B, C, dt = w.split([I, I, G * self.state, G * self.state, H])
        heads = [pad_head_rows(t, H, self.vdim, self.dv) for t in (z, x)]
        return torch.cat(heads + [pad_head_rows(t, G, self.state, self.dn) for t in (B, C)] + [dt])

    def pad_channels(self, w) -> torch.Tensor:
        """Per-channel rows of the convolution ``[x | B | C]``."""
        I, GN = self.heads * self.vdim, self.groups * self.state
        x, B, C = w.split([I, GN, GN])
        return torch.cat([pad_head_rows(x, self.heads, self.vdim, self.dv)] + [pad_head_rows(t, self.groups, self.state, self.dn) for t in (B, C)])


@dataclass
class Mamba2Weights:
    """fp32 parameters in the padded layout: ``conv [taps, C]``, ``conv_b [C]`` or None, ``dt_bias``, ``neg_a`` = -exp(A_log) and ``D`` ``[H]``, ``norm [H * dv]``."""

    conv: torch.Tensor
    conv_b: Optional[torch.Tensor]
    dt_bias: torch.Tensor
    neg_a: torch.Tensor
    D: torch.Tensor
    norm: torch.Tensor

    @staticmethod
    def pack(s: Mamba2Shape, conv, conv_b, dt_bias, A_log, D, norm, device) -> "Mamba2Weights":
        C = s.heads * s.vdim + 2 * s.groups * s.state
        for n, t, want in (("conv", conv, C * s.taps), ("dt_bias", dt_bias, s.heads), ("A_log", A_log, s.heads), ("D", D, s.heads), ("norm", norm, s.heads * s.vdim)):
            if t.numel() != want:
                raise ValueError(f"Mamba-2: '{n}' has {t.numel()} elements, the configured sizes need {want}")
        dev = lambda t: t.float().to(device).contiguous()  # noqa: E731
        row = lambda t: dev(t.reshape(-1))  # noqa: E731
        b = None if conv_b is None else row(s.pad_channels(conv_b.reshape(-1, 1)))
        return Mamba2Weights(dev(s.pad_channels(conv.reshape(C, s.taps)).t()), b, row(dt_bias), row(-torch.exp(A_log.double())), row(D),
                             row(pad_head_rows(norm.reshape(-1, 1), s.heads, s.vdim, s.dv)))


def mamba2(s: Mamba2Shape, p, w: Mamba2Weights, ring, state, batch, eps: float) -> torch.Tensor:
    """Rows of the input projection -> gated, normed heads ``[T, H * dv]``. ``ring`` and ``state``: the slots' convolution inputs and states, advanced for
    the batch's sequences (one at position 0 starts from zero)."""
    if ops._cuda(p):
        e = ops.require_ext()
        args = (w.conv, w.conv_b, w.dt_bias, w.neg_a, w.D, w.norm, ring, state, batch.state_slots, batch.q_start, batch.q_len, batch.positions, s.geometry(), eps)
        if batch.is_decode:
            ops._count(2)
            return e.mamba2_decode(p, *args)
        xbc = short_conv(p, s.out_width, w.conv, w.conv_b, ring, batch)
        chunked = p.dtype == torch.bfloat16 and s.dn <= MAX_STATE_CHUNKED
        ops._count(5 if chunked else 2)
        return e.mamba2_prompt(p, xbc, *args, CHUNK, list(chunk_plan(batch, CHUNK)) if chunked else [])
    xbc = short_conv(p, s.out_width, w.conv, w.conv_b, ring, batch)
    T, H, G = p.shape[0], s.heads, s.groups
    x, B, C = xbc.split([s.out_width, G * s.dn, G * s.dn], dim=-1)
    x, B, C = x.reshape(T, H, s.dv), B.reshape(T, G, s.dn), C.reshape(T, G, s.dn)
    dt = torch.nn.functional.softplus(p[:, s.dt_at : s.dt_at + H].float() + w.dt_bias)
    y = torch.empty(T, H, s.dv, dtype=torch.float32)
    for slot, lo, n in zip(batch.state_slots.tolist(), batch.q_start.tolist(), batch.q_len.tolist()):
        if n == 0:
            continue
        if int(batch.positions[lo]) == 0:
            state[slot].zero_()
        r = slice(lo, lo + n)
        y[r] = ref.ssd_sequential(x[r], B[r], C[r], dt[r], w.neg_a, w.D, state[slot])
    y = (y * torch.nn.functional.silu(p[:, : s.out_width].float()).reshape(T, H, s.dv))[..., : s.vdim].reshape(T, s.norm_groups, -1)
    y = (y * torch.rsqrt(y.pow(2).mean(dim=-1, keepdim=True) + eps)).reshape(T, H, s.vdim)
    return (torch.nn.functional.pad(y, (0, s.dv - s.vdim)).reshape(T, -1) * w.norm).to(p.dtype)
