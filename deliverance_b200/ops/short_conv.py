"""Short causal convolution over time, one filter per channel, followed by silu: the input stage of recurrent mixers. The inputs of a sequence's
last positions live in its state slot as a ring, position ``p`` at row ``p mod taps``: a token's own row is the only one it writes and no other
token of the step reads it, so decode kernels update it in place, and rows in front of position 0 are never read, so a slot needs no clearing."""
from __future__ import annotations

import torch

from .. import ops
from . import ref
from .grouped import row_sequence


MAX_TAPS = 8  # of the CUDA kernels


def ring_shape(taps: int, channels: int) -> tuple:
    return taps, channels


def short_conv(p, at: int, weight, bias, ring, batch) -> torch.Tensor:
    """Columns ``[at, at + C)`` of the projection rows ``p``, convolved and activated, as ``[T, C]`` rows of ``p``'s type. ``weight [taps, C]`` and
    ``bias [C]`` (or None) are fp32; ``ring [slots, taps, C]`` of the batch's sequences is advanced."""
    C = weight.shape[1]
    if ops._cuda(p):
        ops._count(2)
        return ops.require_ext().short_conv(p, at, weight, bias, ring, batch.state_slots, row_sequence(batch), batch.q_start, batch.q_len, batch.positions)
    out = torch.empty(p.shape[0], C, dtype=p.dtype)
    for slot, lo, n in zip(batch.state_slots.tolist(), batch.q_start.tolist(), batch.q_len.tolist()):
        if n:
            out[lo : lo + n] = ref.short_conv(p[lo : lo + n, at : at + C], weight.t(), bias, ring[slot], int(batch.positions[lo])).to(p.dtype)
    return out
