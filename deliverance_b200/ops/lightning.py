"""Lightning attention: linear attention with one constant decay per head, ``S_t = decay S_(t-1) + k_t v_t^T``, ``o_t = S_t^T q_t`` on activated rows
(``silu`` of q, k and v); the heads of a row are RMS-normed together and gated with a sigmoid.

One projection row is ``[q (H * dk) | k (H * dk) | v (H * dv) | g (H * dv)]``, head widths rounded up to multiples of 8 (zero weights behind the
real columns; ``silu(0) = 0``, so padded channels stay zero). The state is fp32, one slot per sequence, ``[slots, H, dk, dv]``. Two evaluation
orders, the same numbers up to rounding:

* recurrent (decode, fp32): every token updates the state in registers;
* chunked (bf16 prompts): the rows are activated in place. Because the decay is a constant, what a chunk adds to the state does not depend on the state in front of it. All
  chunks' contributions are computed at once, an elementwise pass turns them into the state in front of every chunk, and all chunks' outputs are
  computed at once. Weighted values, states and weights go through the tensor cores as pairs of bf16 numbers with fp32 accumulation.
"""
from __future__ import annotations

from dataclasses import dataclass

import torch

from .. import ops
from . import ref
from .gla import chunk_plan
from .grouped import up8

CHUNK = 128  # tokens per chunk of the chunked form
MAX_DK = 512  # key channels per head the CUDA kernels take
MAX_DK_CHUNKED = 256


@dataclass(frozen=True)
class LightningShape:
    heads: int
    dim: int
    vdim: int

    @property
    def dk(self) -> int:
        return up8(self.dim)

    @property
    def dv(self) -> int:
        return up8(self.vdim)

    @property
    def offsets(self) -> tuple:
        """First column of k, v and g; total width."""
        k = self.heads * self.dk
        v = 2 * k
        g = v + self.heads * self.dv
        return k, v, g, g + self.heads * self.dv

    @property
    def width(self) -> int:
        return self.offsets[3]

    @property
    def out_width(self) -> int:
        return self.heads * self.dv

    def geometry(self) -> list:
        k, v, g, _ = self.offsets
        return [self.heads, self.dk, self.dv, k, v, g, self.heads * self.vdim]


def decay_powers(decay) -> torch.Tensor:
    """fp32 ``[H, CHUNK + 2]``: decay^0 .. decay^CHUNK, and what fp32 loses of the decay itself."""
    d = torch.tensor([float(x) for x in decay], dtype=torch.float64)
    p = d.unsqueeze(1) ** torch.arange(CHUNK + 1, dtype=torch.float64)
    return torch.cat([p, (d - d.float().double()).unsqueeze(1)], dim=1).float()


def lightning(s: LightningShape, p, decay, powers, norm_w, state, batch, eps: float, mult: float, out) -> None:
    """Rows of the projection -> normed, gated heads times ``mult`` in ``out [T, H * dv]`` (a column range of wider rows). ``decay``: fp64 ``[H]`` on
    the host; ``powers`` of :func:`decay_powers`, ``norm_w [H * dv]`` and ``state [slots, H, dk, dv]`` are fp32; the state slots of the batch's
    sequences are advanced (a sequence at position 0 starts from zero). The q, k and v columns of ``p`` may be overwritten."""
    if ops._cuda(p):
        chunked = not (batch.is_decode or p.dtype == torch.float32 or s.dk > MAX_DK_CHUNKED)
        ops._count(5 if chunked else 2)
        ops.require_ext().lightning(p, powers, CHUNK, norm_w, state, batch.state_slots, batch.q_start, batch.q_len, batch.positions, s.geometry(), eps, mult, out,
                                    list(chunk_plan(batch, CHUNK)) if chunked else [])
        return
    k0, v0, g0, w = s.offsets
    T, H = p.shape[0], s.heads
    q, k, v = (torch.nn.functional.silu(p[:, lo:hi].float()).to(p.dtype).reshape(T, H, -1) for lo, hi in ((0, k0), (k0, v0), (v0, g0)))
    o = torch.empty(T, H, s.dv, dtype=torch.float32)
    for slot, lo, n in zip(batch.state_slots.tolist(), batch.q_start.tolist(), batch.q_len.tolist()):
        if n == 0:
            continue
        if int(batch.positions[lo]) == 0:
            state[slot].zero_()
        o[lo : lo + n] = ref.lightning_sequential(q[lo : lo + n], k[lo : lo + n], v[lo : lo + n], decay, state[slot])
    o = o.reshape(T, -1)
    o = o * torch.rsqrt(o.pow(2).sum(dim=-1, keepdim=True) / (H * s.vdim) + eps) * norm_w
    out.copy_(o * torch.sigmoid(p[:, g0:w].float()) * mult)
