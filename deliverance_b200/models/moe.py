"""Mixture-of-experts feed-forward for mixtral, qwen3_moe and granitemoehybrid, and :class:`RoutedExperts`, the same block with sizes
and routing as parameters, for designs whose layers differ in them.

Routing conventions (reference): Mixtral — softmax over all experts, top-k, renormalise
(core/.../model/MixtureOfExpertsBlock.java:100-112); Qwen3-MoE — softmax over all, top-k, renormalise only with
``norm_topk_prob`` (core/.../model/qwen3/Qwen3MoeFeedForward.java:276-301); Granite — top-k on the logits, softmax over
the k (GraniteMoeHybridMoeFeedForward.java:112-141). Tokens are grouped by expert, each expert runs gate|up -> act*mul ->
down on its rows, and results are scatter-added with the route weight (Qwen3MoeFeedForward.java:107-183).

On CUDA the router (softmax/top-k/renorm + per-expert histogram and row offsets) and the gather / weighted scatter are
single kernels (csrc/moe.cu) and each expert GEMM is a tcgen05 launch on its contiguous row group.
"""
from __future__ import annotations

import os

import torch

from .. import ops
from ..ops import LinearWeight, ref


_SM_COUNT = 148  # B200
_MODES = {"softmax_topk": 0, "topk_softmax": 1, "sigmoid_topk": 2}
_ROUTE_ONE_LAUNCH = [os.environ.get("DLV_MOE_ROUTE", "fused") != "split"]  # decode-size routing in one launch ("split": the separate kernels)


def moe_forward(model, i: int, lw, x: torch.Tensor) -> torch.Tensor:
    """Routed experts of one layer. Under tensor parallelism the experts are split across ranks when their count divides
    (expert parallelism: tokens are replicated after the attention all-reduce, so dispatch is a local selection and the
    combine is a sum over ranks); otherwise every rank holds all experts and no communication is needed."""
    cfg = model.cfg
    E, k = cfg.num_experts, cfg.experts_per_token
    logits = ops.linear(x, lw.router, out_f32=True)
    renorm = True if cfg.model_type == "mixtral" else (cfg.norm_topk_prob if cfg.router_mode == "softmax_topk" else False)
    e0, ne = lw.expert0, lw.n_local_experts or E
    if x.device.type == "cuda":
        y, reduced = _moe_cuda(model, lw, x, logits, E, k, cfg.router_mode, renorm, cfg.hidden_act, e0, ne)
        if reduced:
            return y
    else:
        w, idx = ref.moe_route(logits, k, cfg.router_mode, renorm)
        local = (idx >= e0) & (idx < e0 + ne)
        y = ref.moe_experts(
            x, torch.where(local, w, torch.zeros_like(w)), torch.where(local, idx - e0, torch.full_like(idx, -1)),
            lambda e, rows: ops.linear(rows, lw.experts_gate_up[e]),
            lambda e, h: ops.linear(h, lw.experts_down[e]),
            ne, cfg.hidden_act,
            (lambda e, rows: ops.linear_act(rows, lw.experts_gate_up[e], cfg.hidden_act)) if lw.fused_act_experts else None,
        )
    if ne != E:
        y = model.tp.all_reduce(f"layer.{i}.moe.combine", y)
    return y


def moe_forward_sharded(model, i: int, lw, x_own: torch.Tensor, a2a, total_rows: int) -> torch.Tensor:
    """Routed experts for token rows that are sharded over the ranks (sequence-parallel forward) with expert parallelism: every rank
    routes its own rows, an all-to-all over peer memory carries each (token, slot) row to the rank that owns its expert, the grouped
    expert GEMMs run there, the outputs travel back and are combined with the route weights (``parallel.fused.ExpertAllToAll``).
    ``total_rows``: token rows of the whole batch (bounds what one rank can receive)."""
    cfg = model.cfg
    E, k = cfg.num_experts, cfg.experts_per_token
    e = ops.require_ext()
    ne = lw.n_local_experts
    renorm = True if cfg.model_type == "mixtral" else (cfg.norm_topk_prob if cfg.router_mode == "softmax_topk" else False)
    T = x_own.shape[0]
    logits = ops.linear(x_own, lw.router, out_f32=True) if T else torch.zeros(0, E, device=x_own.device)
    w, idx, counts, offsets, perm, pos = e.moe_route(logits.contiguous(), k, 0 if cfg.router_mode == "softmax_topk" else 1, bool(renorm))
    ops._count(2)
    max_recv = min(total_rows * k, a2a.cap * model.tp.size)
    bn = ops.moe_token_tile(max(1, total_rows * k // model.tp.size), ne, lw.experts_gate_up_grouped.q4)
    if lw.fused_act_experts:
        bn = max(bn, 16)
    max_items = max(1, (max_recv + bn - 1) // bn + ne)
    gu_w, down_w = lw.experts_gate_up_grouped, lw.experts_down_grouped

    def run_experts(xs, local_offsets):
        items = e.moe_items(local_offsets, 0, ne, bn, max_items)
        ops._count()
        if lw.fused_act_experts and bn >= 16:
            hmid = gu_w.run_act(xs, items, bn, 1, cfg.hidden_act)
        else:
            hmid = ops.act_mul(gu_w.run(xs, items, bn, 1), cfg.hidden_act)
        return down_w.run(hmid, items, bn, 1)

    ret = a2a.forward(x_own, perm, offsets, k, run_experts, max_recv)
    a2a.sent_rows += int(T * k)
    if T == 0:
        return x_own
    ops._count()
    return e.moe_combine(ret[: T * k], pos, w, T, k)


def _moe_cuda(model, lw, x, logits, E, k, mode, renorm, act, e0, ne):
    st = model._stage
    T = x.shape[0]
    ys, pos, w, offsets = _experts_cuda(st, lw, x, logits, E, k, mode, renorm, act, e0, ne)
    ep = ne != E
    with st("moe.combine"):
        fused = getattr(model.tp, "fused", None)
        if ep and fused is not None:
            y = fused.moe_combine_all_reduce(ys, pos, w, T, k, offsets, e0, ne)  # combine + sum over ranks in one kernel
            if y is not None:
                return y, True
        ops._count()
        rng = (offsets, e0, ne) if ep else (None, 0, 0)
        return ops.require_ext().moe_combine(ys, pos, w, T, k, *rng), False


def _experts_cuda(st, lw, x, logits, E, k, mode, renorm, act, e0, ne):
    """Routing, expert-grouped gate|up, activation and down projection: ``(ys, pos, w, offsets)`` with the expert outputs ``ys [T * k, H]``
    in grouped order, ``pos [T, k]`` the grouped row of every (token, slot) and its route weight ``w``."""
    e = ops.require_ext()
    T, H = x.shape
    rows = T * k
    ep = ne != E
    gu_w, down_w = lw.experts_gate_up_grouped, lw.experts_down_grouped
    f32 = x.dtype == torch.float32
    bn = 64 if f32 else ops.moe_token_tile(rows if not ep else max(1, rows * ne // E), ne, gu_w.q4)
    if lw.fused_act_experts:
        bn = max(bn, 16)  # interleaved expert rows exist for the tensor-core grouped GEMM's epilogue only
    max_items = min((rows + bn - 1) // bn + ne, rows) if rows >= ne else rows
    max_items = max(1, max_items)
    rng = None
    xs = None
    with st("moe.route"):
        # weights [T, k] fp32, expert ids [T, k], counts [E], offsets [E + 1], perm: grouped row -> (token * k + slot), pos: inverse,
        # items: the grouped GEMM's work list. Decode-size batches get all of it from one launch.
        mode_i = _MODES[mode]
        rules = lw.routing_rules() if hasattr(lw, "routing_rules") else {}
        routed = e.moe_route_items(logits.contiguous(), k, mode_i, bool(renorm), e0, ne, bn, max_items, **rules) if _ROUTE_ONE_LAUNCH[0] else []
        if routed:
            w, idx, counts, offsets, perm, pos, items = routed
            ops._count()
        else:
            w, idx, counts, offsets, perm, pos = e.moe_route(logits.contiguous(), k, mode_i, bool(renorm), **rules)
            items = e.moe_items(offsets, e0, ne, bn, max_items)
            ops._count(3)
        rng = (offsets, e0, ne) if ep else (None, 0, 0)

    def gathered():
        """x rows in expert-grouped order [T * k, H] (only the local experts' rows are filled)."""
        ops._count()
        return e.moe_gather(x, perm, k, *rng)

    if f32:  # 32-bit models: plain FMA projections on the same work list
        h = torch.empty(rows, gu_w.N // 2, dtype=x.dtype, device=x.device)
        ops.gated_act_into(gu_w.run(gathered(), items, bn), act, h)
        return down_w.run(h, items, bn), pos, w, offsets

    small = bn <= 64  # decode-sized groups: split K so that more CTAs stream weights

    def k_splits(wt) -> int:
        """Split K only as far as the grid needs it: every split pays the tile's set-up and a reduction again, so a projection whose
        (local experts x 128-row tiles) already fill two waves of the GPU runs unsplit."""
        if not small:
            return 1
        tiles = max(1, ne) * ((wt.N + 127) // 128)
        want = (2 * _SM_COUNT + tiles - 1) // tiles
        return max(1, min(8, wt.K // 1024, want))

    if lw.fused_act_experts and bn >= 16:
        with st("moe.gate_up"):  # act(gate) * up in the grouped GEMM's epilogue (interleaved expert rows)
            hmid = gu_w.run_act(gathered(), items, bn, k_splits(gu_w), act)
    else:
        if lw.fused_act_experts:
            raise RuntimeError("interleaved expert weights need the tensor-core grouped GEMM (token tile >= 16)")
        hmid = None
        if bn <= 8:
            # a handful of rows per expert: grouped GEMV with the gated activation in its epilogue; it reads the token rows through
            # the permutation, so the copy into expert order is skipped
            with st("moe.gate_up"):
                hmid = gu_w.run_gemv_act(x, items, act, perm, k)
        if hmid is None:
            with st("moe.gate_up"):
                xs = gathered()
                gu = gu_w.run(xs, items, bn, k_splits(gu_w))
            with st("moe.activation_multiply"):
                hmid = ops.act_mul(gu, act)
    with st("moe.down"):
        ys = down_w.run(hmid, items, bn, k_splits(down_w))
    return ys, pos, w, offsets


class RoutedExperts:
    """Routed experts without biases: softmax, top-k first or sigmoid routing (``ref.moe_route``; the last with a correction of the choice,
    ``groups`` of which ``keep`` take part, and a weight ``scale``), ``top`` experts per token, gated activation. The result is left in expert
    order (:class:`ops.Routed`) so that the step behind it can do the weighted sum; ``ops.Routed.dense`` does it alone.

    The expert width is padded to a multiple of 8 with zero rows, the input width to ``k_pad``."""

    expert0, fused_act_experts = 0, False

    def __init__(self, experts: int, top: int, act: str = "silu", mode: str = "softmax_topk", renorm: bool = False, groups: int = 1, keep: int = 1,
                 scale: float = 1.0):
        if not 0 < top <= experts:
            raise ValueError(f"{top} of {experts} experts per token")
        if groups < 1 or experts % groups or not 1 <= keep <= groups or keep * (experts // groups) < top:
            raise ValueError(f"{keep} of {groups} groups of {experts} experts, {top} experts per token")
        self.groups, self.keep, self.scale = int(groups), int(keep), float(scale)
        self.correction = None
        self.experts, self.top, self.act, self.mode, self.renorm = int(experts), int(top), act, mode, bool(renorm)
        self.n_local_experts = self.experts
        self.experts_gate_up: list = []
        self.experts_down: list = []

    def routing_rules(self) -> dict:
        return {"correction": self.correction, "groups": self.groups, "keep": self.keep, "scale": self.scale}

    def load(self, router, experts, ff: int, k_pad: int, device, dtype, correction=None) -> "RoutedExperts":
        """``experts``: (gate, up, down) per expert as stored; ``correction [experts]``: added to the scores where experts are chosen."""
        pad = torch.nn.functional.pad
        ff8 = (ff + 7) // 8 * 8
        put = lambda t: LinearWeight(t.to(device=device, dtype=dtype).contiguous())  # noqa: E731
        if router.shape[0] != self.experts:
            raise ValueError(f"router has {router.shape[0]} rows for {self.experts} experts")
        if correction is not None:
            if correction.numel() != self.experts:
                raise ValueError(f"{correction.numel()} corrections for {self.experts} experts")
            self.correction = correction.reshape(-1).to(device=device, dtype=torch.float32).contiguous()
        self.router = put(pad(router, (0, k_pad - router.shape[1])))
        for gate, up, down in experts:
            if gate.shape[0] != ff or up.shape[0] != ff or down.shape[1] != ff:
                raise ValueError(f"expert weights do not have the configured width {ff}")
            wide = lambda t: pad(t, (0, k_pad - t.shape[1], 0, ff8 - ff))  # noqa: E731
            self.experts_gate_up.append(put(torch.cat([wide(gate), wide(up)])))
            self.experts_down.append(put(pad(down, (0, ff8 - ff, 0, k_pad - down.shape[0]))))
        if torch.device(device).type == "cuda":
            self.experts_gate_up_grouped = ops.GroupedLinearWeight(self.experts_gate_up)
            self.experts_down_grouped = ops.GroupedLinearWeight(self.experts_down)
            self.experts_gate_up, self.experts_down = [], []
        return self

    def nbytes(self) -> int:
        if self.experts_gate_up:
            return self.router.nbytes() + sum(w.nbytes() for w in self.experts_gate_up + self.experts_down)
        return self.router.nbytes() + self.experts_gate_up_grouped.nbytes() + self.experts_down_grouped.nbytes()

    def forward(self, x: torch.Tensor, stage) -> "ops.Routed":
        with stage("moe.router"):
            logits = ops.linear(x, self.router, out_f32=True)
        if x.device.type == "cuda":
            ys, pos, w, _ = _experts_cuda(stage, self, x, logits, self.experts, self.top, self.mode, self.renorm, self.act, 0, self.experts)
            return ops.Routed(ys, pos.reshape(-1, self.top), w)
        w, idx = ref.moe_route(logits, self.top, self.mode, self.renorm, **self.routing_rules())
        y = ref.moe_experts(x, w, idx, lambda e, rows: ops.linear(rows, self.experts_gate_up[e]), lambda e, h: ops.linear(h, self.experts_down[e]),
                            self.experts, self.act)
        return ops.Routed(y, None, None)
