"""Dense feed-forwards without biases: gated ``down(act(gate h) * up h)``, gate and up as one projection, and plain ``down(act(up h))``; the width is
padded to a multiple of 8 with zero rows, the input width to ``k_pad``."""
from __future__ import annotations

import torch

from .. import ops
from ..ops import LinearWeight
from ..ops.grouped import up8


class GatedFeedForward:
    def __init__(self, act: str):
        self.act = act

    def load(self, gate, up, down, ff: int, k_pad: int, device, dtype) -> "GatedFeedForward":
        if gate.shape[0] != ff or up.shape[0] != ff or down.shape[1] != ff:
            raise ValueError(f"feed-forward weights do not have the configured width {ff}")
        pad = torch.nn.functional.pad
        self.ff = up8(ff)
        put = lambda t: LinearWeight(t.to(device=device, dtype=dtype).contiguous())  # noqa: E731
        wide = lambda t: pad(t, (0, k_pad - t.shape[1], 0, self.ff - ff))  # noqa: E731
        self.gate_up, self.down = put(torch.cat([wide(gate), wide(up)])), put(pad(down, (0, self.ff - ff)))
        return self

    def nbytes(self) -> int:
        return self.gate_up.nbytes() + self.down.nbytes()

    def forward(self, x, stage) -> torch.Tensor:
        with stage("mlpblock.gate_up_projection"):
            gu = ops.linear(x, self.gate_up)
        with stage("mlpblock.activation_multiply"):
            h = torch.empty(x.shape[0], self.ff, dtype=x.dtype, device=x.device)
            ops.gated_act_into(gu, self.act, h)
        with stage("mlpblock.down_projection"):
            return ops.linear(h, self.down)


class FeedForward:
    """Without a gate; ``act(0)`` must be 0 (padded columns)."""

    def __init__(self, act: str):
        self.act = act

    def load(self, up, down, ff: int, k_pad: int, device, dtype) -> "FeedForward":
        if up.shape[0] != ff or down.shape[1] != ff:
            raise ValueError(f"feed-forward weights do not have the configured width {ff}")
        pad, self.ff = torch.nn.functional.pad, up8(ff)
        put = lambda t: LinearWeight(t.to(device=device, dtype=dtype).contiguous())  # noqa: E731
        self.up, self.down = put(pad(up, (0, k_pad - up.shape[1], 0, self.ff - ff))), put(pad(down, (0, self.ff - ff)))
        return self

    def nbytes(self) -> int:
        return self.up.nbytes() + self.down.nbytes()

    def forward(self, x, stage) -> torch.Tensor:
        with stage("mlpblock.up_projection"):
            h = ops.linear(x, self.up)
        with stage("mlpblock.activation"):
            h = ops.activation(h, self.act)
        with stage("mlpblock.down_projection"):
            return ops.linear(h, self.down)
