"""Gated delta rule: linear attention whose write corrects what the state already returns for the key. Per head, with a decay per key channel,
``S <- diag(a_t) S``, ``u_t = beta_t (v_t - S^T k_t)``, ``S <- S + k_t u_t^T``, ``o_t = S^T q_t``; q, k and v come through a short convolution
(``ops/short_conv.py``), q and k are unit vectors; the heads are RMS-normed over the value columns and gated with a sigmoid.

One projection row is ``[q (G * dk) | k (G * dk) | v (H * dv) | beta (H) | a (rank_a) | g (rank_g)]``, every piece rounded up to a multiple of 8 columns
(zero weights behind the real ones: a padded channel's key is zero, so its state stays zero). ``a`` and ``g`` are the inputs of low-rank projections whose
fp32 results ``[H * dk]`` and ``[H * dv]`` are the decay's argument and the output gate's logits. Head h uses the query / key head h // (H / G). The state
is fp32, one slot per sequence, ``[slots, H, dk, dv]``. Two evaluation orders, the same numbers up to rounding (``csrc/delta.cu``):

* recurrent (decode, fp32): every token updates the state in registers; decode steps do convolution, unit vectors, norm and gate in the same launch;
* chunked (bf16 prompts): inside a chunk, with running sums ``b`` of the log decays, the corrected values solve ``(I + M) U = beta (V - K' S_0)`` with
  ``M[t, s] = beta_t sum_d k_t k_s exp(b_t - b_s)`` for s < t and ``K' = k exp(b)``. ``(I + M)^-1 beta``, the causal matrix of the queries and the scaled
  queries and keys of all chunks are prepared at once; one CTA per (sequence, head, 64 value columns) walks the chunks with its part of the state in
  registers. What is fp32 by definition goes through the tensor cores as pairs of bf16 numbers with fp32 accumulation.
"""
from __future__ import annotations

from dataclasses import dataclass

import torch

from .. import ops
from . import ref
from .gla import chunk_plan
from .grouped import up8
from .short_conv import ring_shape, short_conv

MAX_DK = 512  # key channels per head the CUDA kernels take
MAX_DK_CHUNKED = 256
MAX_DK_CHUNK32 = 128  # wider keys: chunks of 16 tokens
MAX_DV_FUSED = 512  # one cluster of eight CTAs per head norms and gates inside the decode launch
UNIT_EPS = 1e-6  # under the root of the unit vectors' length


@dataclass(frozen=True)
class DeltaShape:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    taps: int
    rank_a: int
    rank_g: int

    def __post_init__(self):
        if self.heads % self.kv_heads:
            raise ValueError(f"gated delta rule: {self.heads} heads do not divide into {self.kv_heads} query / key heads")
        if self.taps < 1:
            raise ValueError("gated delta rule: the convolution needs at least one tap")

    @property
    def dk(self) -> int:
        return up8(self.dim)

    @property
    def dv(self) -> int:
        return up8(self.vdim)

    @property
    def conv_width(self) -> int:
        return 2 * self.kv_heads * self.dk + self.heads * self.dv

    @property
    def beta_at(self) -> int:
        return self.conv_width

    @property
    def low_at(self) -> int:
        """First column of the low-rank inputs."""
        return self.beta_at + up8(self.heads)

    @property
    def low_width(self) -> int:
        return up8(self.rank_a) + up8(self.rank_g)

    @property
    def width(self) -> int:
        return self.low_at + self.low_width

    @property
    def out_width(self) -> int:
        return self.heads * self.dv

    def chunk(self, lengths, sms: int = 148) -> int:
        """Tokens per chunk of the chunked form: 32 where shared memory holds two stages of them, unless the walks of the batch's prompts are more than
        the processors; two walks over chunks of 16 fit one processor."""
        walks = sum(n > 32 for n in lengths) * self.heads * ((self.dv + 63) // 64)
        return 32 if self.dk <= MAX_DK_CHUNK32 and walks <= sms else 16

    def state_shapes(self) -> dict:
        return {"conv": ring_shape(self.taps, self.conv_width), "delta": (self.heads, self.dk, self.dv)}

    def geometry(self) -> list:
        return [self.heads, self.kv_heads, self.dk, self.dv, self.vdim, self.beta_at]


def fused_step(s: DeltaShape, batch) -> bool:
    """A decode step of which one launch does everything (its gate logits are fp32)."""
    return batch.is_decode and s.dv <= MAX_DV_FUSED


def delta(s: DeltaShape, p, z, gate, conv_w, dt_bias, neg_a, norm_w, ring, state, batch, q_scale: float, eps: float, mult: float, out) -> None:
    """Rows of the projection -> normed, gated heads times ``mult`` in ``out [T, H * dv]`` (a column range of wider rows). ``z [T, H * dk]``: the decays'
    argument without ``dt_bias``, ``gate [T, H * dv]``: logits of the output gate (results of the low-rank projections). ``z``, ``conv_w [taps, C]``, ``dt_bias [H * dk]``, ``neg_a [H]`` = -exp(A_log),
    ``norm_w [dv]``, ``ring`` and ``state`` are fp32; the slots of the batch's sequences are advanced (one at position 0 starts from zero)."""
    if ops._cuda(p):
        e = ops.require_ext()
        args = (z, gate, conv_w, dt_bias, neg_a, norm_w, ring, state, batch.state_slots, batch.q_start, batch.q_len, batch.positions, s.geometry(), q_scale, UNIT_EPS, eps,
                mult, out)
        if fused_step(s, batch):
            ops._count()
            e.delta_decode(p, *args)
            return
        qkv = short_conv(p, 0, conv_w, None, ring, batch)
        chunked = not batch.is_decode and p.dtype == torch.bfloat16 and s.dk <= MAX_DK_CHUNKED
        ops._count(3 if chunked else 2)
        chunk = s.chunk(batch.q_len_host) if chunked else 0
        e.delta_prompt(p, qkv, *args, chunk, list(chunk_plan(batch, chunk)) if chunked else [])
        return
    qkv = short_conv(p, 0, conv_w, None, ring, batch)
    T, H, G = p.shape[0], s.heads, s.kv_heads
    q, k, v = qkv.float().split([G * s.dk, G * s.dk, H * s.dv], dim=-1)
    unit = lambda x: x * torch.rsqrt(x.pow(2).sum(dim=-1, keepdim=True) + UNIT_EPS)  # noqa: E731
    q, k = (unit(x.reshape(T, G, s.dk)).repeat_interleave(H // G, dim=1) for x in (q, k))
    beta = torch.sigmoid(p[:, s.beta_at : s.beta_at + H].float())
    log_a = neg_a.view(1, H, 1) * torch.nn.functional.softplus(z + dt_bias).reshape(T, H, s.dk)
    o = torch.empty(T, H, s.dv, dtype=torch.float32)
    for slot, lo, n in zip(batch.state_slots.tolist(), batch.q_start.tolist(), batch.q_len.tolist()):
        if n == 0:
            continue
        if int(batch.positions[lo]) == 0:
            state[slot].zero_()
        r = slice(lo, lo + n)
        o[r] = ref.delta_sequential(q[r] * q_scale, k[r], v[r].reshape(n, H, s.dv), log_a[r], beta[r], state[slot])
    o = o * torch.rsqrt(o.pow(2).sum(dim=-1, keepdim=True) / s.vdim + eps) * norm_w
    out.copy_(o.reshape(T, -1) * torch.sigmoid(gate.float()) * mult)
