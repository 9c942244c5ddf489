"""Gated linear attention: ``S_t = diag(a_t) S_(t-1) + k_t v_t^T``, ``o_t = S_t^T q_t`` per head, with a decay per key channel
``a = sigmoid(z)^(1/tau)``, ``z`` a low-rank projection; the heads are RMS-normed and gated with ``silu(g)``.

One projection row is ``[q (H * dk) | k (H * dk) | v (H * dv) | g (H * dv) | a (rank)]``, head widths rounded up to multiples of 8 (zero
weights behind the real columns: a padded channel's key is zero, so its state stays zero). The state is fp32, one slot per sequence,
``[slots, H, dk, dv]``. Two evaluation orders, the same numbers up to rounding:

* recurrent (decode, fp32): every token updates the state in registers;
* chunked (bf16 prompts): with cumulative log decays ``b`` inside a chunk, ``q exp(b)``, ``k exp(b_end - b)`` and the causal matrix
  ``A[t, s] = sum_d q_t k_s exp(b_t - b_s)`` are prepared for all chunks at once; one CTA per (sequence, head, 64 value columns) then
  walks the chunks with its part of the state in registers. Everything that enters the recurrence is carried as a pair of bf16 numbers
  (high and low part) through the tensor cores with fp32 accumulation.
"""
from __future__ import annotations

from dataclasses import dataclass

import torch

from .. import ops
from . import ref
from .grouped import up8

MAX_DK = 512  # key channels per head the CUDA kernels take
MAX_DK_CHUNKED = 256
MAX_DV_FUSED = 512  # one cluster of eight CTAs per head norms and gates inside the decode launch


@dataclass(frozen=True)
class GlaShape:
    heads: int
    dim: int
    vdim: int
    rank: int

    @property
    def dk(self) -> int:
        return up8(self.dim)

    @property
    def dv(self) -> int:
        return up8(self.vdim)

    @property
    def rank8(self) -> int:
        return up8(self.rank)

    @property
    def offsets(self) -> tuple:
        """First column of k, v, g and the low-rank decay input; total width."""
        k = self.heads * self.dk
        v = 2 * k
        g = v + self.heads * self.dv
        a = g + self.heads * self.dv
        return k, v, g, a, a + self.rank8

    @property
    def width(self) -> int:
        return self.offsets[4]

    @property
    def out_width(self) -> int:
        return self.heads * self.dv

    @property
    def chunk(self) -> int:
        """Tokens per chunk of the chunked form (shared memory of two stages bounds it)."""
        return 64 if self.dk <= 128 else 32

    def geometry(self) -> list:
        k, v, g, a, w = self.offsets
        return [self.heads, self.dk, self.dv, self.vdim, self.rank8, k, v, g, a, w]


def gla(s: GlaShape, p, a2, a2_bias, norm_w, state, batch, q_scale: float, tau: float, eps: float):
    """Rows of the fused projection -> normed, gated heads ``[T, H * dv]``. ``a2 [H * dk, rank8]``, ``a2_bias [H * dk]``, ``norm_w [dv]`` and
    ``state [slots, H, dk, dv]`` are fp32; the state slots of the batch's sequences are advanced (a sequence at position 0 starts from zero)."""
    if ops._cuda(p):
        e = ops.require_ext()
        args = (a2, a2_bias, norm_w, state, batch.state_slots, batch.q_start, batch.q_len, batch.positions, s.geometry(), q_scale, 1.0 / tau, eps)
        if batch.is_decode or p.dtype == torch.float32 or s.dk > MAX_DK_CHUNKED:
            fused = batch.is_decode and s.dv <= MAX_DV_FUSED
            ops._count(1 if fused else 2)
            return e.gla_recurrent(p, *args, fused)
        ops._count(3)
        return e.gla_chunked(p, *args, s.chunk, *chunk_plan(batch, s.chunk))
    k0, v0, g0, a0, w = s.offsets
    T, H = p.shape[0], s.heads
    q, k, v, g = (p[:, lo:hi].reshape(T, H, -1) for lo, hi in ((0, k0), (k0, v0), (v0, g0), (g0, a0)))
    z = (p[:, a0:w].float() @ a2.T + a2_bias).reshape(T, H, s.dk)
    out = torch.empty(T, H, s.dv, dtype=torch.float32)
    for slot, lo, n in zip(batch.state_slots.tolist(), batch.q_start.tolist(), batch.q_len.tolist()):
        if n == 0:
            continue
        if int(batch.positions[lo]) == 0:
            state[slot].zero_()
        r = slice(lo, lo + n)
        out[r] = ref.gla_sequential(q[r], k[r], v[r], z[r], q_scale, tau, state[slot])
    real = ref.gla_norm_gate(out[..., : s.vdim], g[..., : s.vdim], norm_w[: s.vdim], eps)
    return torch.nn.functional.pad(real, (0, s.dv - s.vdim)).reshape(T, H * s.dv).to(p.dtype)


def chunk_plan(batch, chunk: int):
    """Chunks of every sequence of a batch: int32 device arrays (sequence, first row, length) per chunk and (first chunk, count) per
    sequence, built once per batch and chunk length."""
    key = ("chunks", chunk)
    if key not in batch.plans:
        n = torch.tensor(batch.q_len_host, dtype=torch.int64)
        start = torch.cumsum(n, 0) - n
        count = (n + chunk - 1) // chunk
        first = torch.cumsum(count, 0) - count
        seq = torch.repeat_interleave(torch.arange(len(n)), count)
        at = (torch.arange(len(seq)) - first[seq]) * chunk
        dev = batch.q_len.device
        batch.plans[key] = tuple(t.to(torch.int32).to(dev, non_blocking=True) for t in (seq, start[seq] + at, (n[seq] - at).clamp(max=chunk), first, count))
    return batch.plans[key]
