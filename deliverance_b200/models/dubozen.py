"""Dubozen decoder: several fp32 residual streams that every sublayer reads from and writes back to through learned weights
(hyper-connections); grouped attention with a learned sink, a gate per column and values mixed with the first layer's, or grouped attention
with tied values and a gate per head beside lightning attention; dense or routed feed-forwards; LayerNorms without bias; tied embeddings.

How a layer is laid out on the device (decode and prompts alike):

* ONE kernel finishes a sublayer and starts the next: (weighted sum of the experts' rows,) new streams, weighted sum of them for the next
  sublayer, its LayerNorm (``ops.stream_step``); the first one also does the embedding and its norm (``ops.stream_open``);
* all input projections of a mixer are one GEMM, its output projections one, gate and up of a feed-forward one;
* head norms, rotation, value mixing and cache write are one kernel; sink, gate and constants sit in the attention kernels' epilogues.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

import torch

from .. import ops
from ..ckpt.loader import WeightLoader
from ..ops import LinearWeight, ref
from ..ops.grouped import GroupedShape, up8
from ..ops.lightning import LightningShape
from .batch import ForwardBatch
from .feed_forward import GatedFeedForward
from .grouped import GroupedAttention
from .latent import RotaryTables
from .lightning import LightningAttention
from .moe import RoutedExperts
from .side_by_side import SideBySideMixer
from .transformer import DecoderModel


@dataclass
class HyperConnection:
    """How one sublayer reads and writes the streams (fp32): ``read [S]``, ``mix [S, S]`` (from, to), ``write [S]``."""

    read: torch.Tensor
    mix: torch.Tensor
    write: torch.Tensor


@dataclass
class StreamSublayer:
    conn: HyperConnection
    norm: torch.Tensor
    block: object


@dataclass
class StreamLayer:
    mixer: StreamSublayer
    ff: Optional[StreamSublayer] = None


class DubozenModel(DecoderModel):
    def __init__(self, cfg, device="cpu", dtype=None, tp=None):
        from ..parallel.context import SINGLE

        tp = tp or SINGLE
        if tp.enabled:
            raise ValueError("dubozen is not sharded for tensor parallelism")
        super().__init__(cfg, device, dtype, tp)
        if self.device.type == "cuda" and self.dtype not in (torch.bfloat16, torch.float32):
            raise ValueError(f"dubozen runs in bfloat16 or float32 on CUDA, not {self.dtype}")
        self.streams = cfg.extra["streams"]
        self.pitch = up8(cfg.hidden_size)

    def _check_kernels(self) -> None:
        pass  # head sizes are free: every layer's shape checks its own

    # ------------------------------------------------------------------------------------------------ loading
    def load(self, loader: WeightLoader, head_quant: Optional[str] = None, prefix: str = "") -> "DubozenModel":
        if head_quant:
            raise ValueError("output-head quantisation is not available for dubozen")
        cfg, W, S, Kw = self.cfg, self.cfg.hidden_size, self.streams, self.pitch
        get = lambda n: loader.load_dense(prefix + n, self.dtype)  # noqa: E731
        f32 = lambda n: loader.load_dense(prefix + n, torch.float32).reshape(-1).to(self.device).contiguous()  # noqa: E731
        self.embed = self._dev(get("embed"))
        self.embed_norm = f32("embed.norm")
        self.tables = RotaryTables(cfg.max_position_embeddings, self.device, lambda dims, max_pos, base, _: ref.rope_tables(dims, max_pos, base))

        def connection(p: str) -> HyperConnection:
            c = HyperConnection(f32(p + "in"), f32(p + "mix"), f32(p + "out"))
            if c.read.numel() != S or c.write.numel() != S or c.mix.numel() != S * S:
                raise ValueError(f"'{p}*' does not match {S} streams")
            c.mix = c.mix.view(S, S)
            return c

        for i, L in enumerate(cfg.extra["layers"]):
            p, m = f"l{i}.", L["mixer"]
            mixer = self._side_by_side(get, f32, p + "mix.", m) if L["type"] == "parallel" else self._attention(get, f32, p + "mix.", m)
            if mixer.w_out.N != W:
                raise ValueError(f"layer {i}: output projection has {mixer.w_out.N} rows, expected {W}")
            lw = StreamLayer(StreamSublayer(connection(p + "hc1."), f32(p + "norm1"), mixer))
            if L.get("mlp"):
                lw.ff = StreamSublayer(connection(p + "hc2."), f32(p + "norm2"), self._feed_forward(get, f32, p + "mlp.", L["mlp"]))
            self.layers.append(lw)
        self.final_norm = f32("final.norm")
        if Kw == W and self.embed.dtype == self.dtype:
            self.lm_head = LinearWeight(self.embed)  # shares storage with the embedding table
        else:
            self.lm_head = self._lin(torch.nn.functional.pad(self.embed, (0, Kw - W)))
        return self

    def _rotary(self, m: dict):
        return self.tables.get(int(m["rot"]["dims"]), float(m["rot"]["base"]), None)

    def _attention(self, get, f32, p: str, m: dict) -> GroupedAttention:
        shape = GroupedShape(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), gate="columns")
        mix = bool(m.get("v_mix"))
        mixer = GroupedAttention(shape, m["scale"], 0.0, 0, 0, True, *self._rotary(m), self.device, self.dtype, rotate="halves", v_mix=mix)
        return mixer.load(*(get(p + n) for n in ("q", "k", "v", "o")), k_pad=self.pitch, g=get(p + "g"), sink=f32(p + "sink"),
                          vmix=f32(p + "vmix").item() if mix else None)

    def _side_by_side(self, get, f32, p: str, m: dict) -> SideBySideMixer:
        lm, rm, eps = m["left"], m["right"], self.cfg.norm_eps
        shape = GroupedShape(int(lm["heads"]), int(lm["kv_heads"]), int(lm["dim"]), int(lm.get("vdim", lm["dim"])), tied=True, gate="heads")
        left = GroupedAttention(shape, lm["scale"], 0.0, 0, 0, False, *self._rotary(lm), self.device, self.dtype, rotate="halves", eps=eps, mult=m["left_scale"])
        right = LightningAttention(LightningShape(int(rm["heads"]), int(rm["dim"]), int(rm["vdim"])), rm["decay"], eps, self.device, self.dtype, m["right_scale"])
        lp, rp = p + "left.", p + "right."
        packed = left.pack(get(lp + "q"), get(lp + "k"), None, get(lp + "o"), g=get(lp + "g"), q_norm=f32(lp + "q.norm"), k_norm=f32(lp + "k.norm"))
        return SideBySideMixer(left, right).load(packed, right.pack(*(get(rp + n) for n in ("q", "k", "v", "g", "o")), f32(rp + "norm")), self.pitch)

    def _feed_forward(self, get, f32, p: str, m: dict):
        if m["kind"] == "dense":
            return GatedFeedForward("gelu_pytorch_tanh").load(get(p + "gate"), get(p + "up"), get(p + "down"), int(m["ff"]), self.pitch, self.device, self.dtype)
        r, groups = m["router"], m["router"].get("groups") or {"count": 1, "keep": 1}
        ff = RoutedExperts(int(r["experts"]), int(r["top"]), "silu", "sigmoid_topk", groups=int(groups["count"]), keep=int(groups["keep"]), scale=float(r["scale"]))
        experts = (tuple(get(p + f"e{e}.{n}") for n in ("gate", "up", "down")) for e in range(ff.experts))
        return ff.load(get(p + "router"), experts, int(m["expert"]["ff"]), self.pitch, self.device, self.dtype, f32(p + "correction"))

    # ------------------------------------------------------------------------------------------------ forward
    def forward_hidden(self, batch: ForwardBatch, kv) -> torch.Tensor:
        eps, Kw, dt = self.cfg.norm_eps, self.pitch, self.dtype
        shared: dict = {}  # what the layers of this pass hand on
        X = y = conn = None  # streams, output of the last sublayer and how it is written back

        def step(read, w_next, keep=True):
            nonlocal X
            if X is None:
                with self._stage("embedinput"):
                    X, x = ops.stream_open(self.embed, batch.token_ids, self.embed_norm, self.streams, read, w_next, eps, Kw, dt)
                return x
            with self._stage("layernorm"):
                return ops.stream_step(X, y, conn.mix, conn.write, read, w_next, eps, Kw, dt, keep)

        for i, lw in enumerate(self.layers):
            x = step(lw.mixer.conn.read, lw.mixer.norm)
            if i == 0:
                self._trace(-1, "embed", X[:, 0])
            y, conn = lw.mixer.block.forward(x, batch, kv, i, self._stage, shared), lw.mixer.conn
            if lw.ff is not None:
                x = step(lw.ff.conn.read, lw.ff.norm)
                y, conn = lw.ff.block.forward(x, self._stage), lw.ff.conn
            if self.layer_hook is not None:
                self._trace(i, "out", ops.stream_step(X.clone(), y, conn.mix, conn.write, None, None, eps, Kw, dt)[:, : self.cfg.hidden_size])
        return step(None, self.final_norm, keep=False)

    # ------------------------------------------------------------------------------------------------ misc
    def kv_layout(self) -> dict:
        mixers = [lw.mixer.block for lw in self.layers]
        runs = [m.cache_layout() for m in mixers]
        return {"layers": len(runs), "kv_heads": max(r["heads"] for r in runs), "head_dim": max(r["k"] for r in runs),
                "layer_kinds": [m.kind for m in mixers], "kv_heads_per_layer": [r["heads"] for r in runs],
                "head_dim_per_layer": [r["k"] for r in runs], "v_dim_per_layer": [r["v"] for r in runs], "state_shapes": [r["state"] for r in runs],
                "paged": [True] * len(runs)}

    def weight_bytes(self) -> int:
        n = self.embed.numel() * self.embed.element_size()
        if self.lm_head.w is not self.embed:
            n += self.lm_head.nbytes()
        return n + sum(s.block.nbytes() for lw in self.layers for s in (lw.mixer, lw.ff) if s is not None)

    def set_lora(self, adapter=None, prefix: str = "") -> None:
        if adapter is not None:
            raise ValueError("run-time LoRA is not supported for dubozen")
