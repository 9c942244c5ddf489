"""Fopivik decoder: gated-linear-attention and sliding-window softmax-attention layers in any order, each followed by routed experts;
LayerNorms in front of and behind every sublayer; a range of layers that runs several times with the same weights on a learned mix of
the stream and the embedding output.

How a layer run is laid out on the device (decode and prompts alike):

* the residual stream is fp32; ONE kernel finishes a sublayer and starts the next: (weighted sum of the experts' rows,) norm behind the
  sublayer, scaled residual add, norm in front of the next one (``ops.sandwich_norm``);
* all input projections of a mixer are one GEMM, gate and up of all experts one grouped GEMM;
* in front of a pass the same kernel writes the stream beside the embedding output, so that the mix is one GEMM whose bias is the
  pass's own vector and whose fp32 output is the new residual stream.

Every layer run has its own cache or state (a looped layer must not see the keys or the state of another pass).
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

import torch

from .. import ops
from ..ckpt.loader import WeightLoader
from ..ops import LinearWeight, ref
from ..ops.gla import GlaShape
from ..ops.grouped import GroupedShape, up8
from .batch import ForwardBatch
from .gla import GatedLinearAttention
from .grouped import GroupedAttention
from .latent import RotaryTables
from .moe import RoutedExperts
from .transformer import DecoderModel


@dataclass
class SandwichLayer:
    """Weights of one layer; norms in fp32 (``a`` in front of, ``b`` behind the sublayer)."""

    mixer: object
    norm1: torch.Tensor
    norm1b: torch.Tensor
    experts: Optional[RoutedExperts] = None
    norm2: Optional[torch.Tensor] = None
    norm2b: Optional[torch.Tensor] = None


class FopivikModel(DecoderModel):
    def __init__(self, cfg, device="cpu", dtype=None, tp=None):
        from ..parallel.context import SINGLE

        tp = tp or SINGLE
        if tp.enabled:
            raise ValueError("fopivik is not sharded for tensor parallelism")
        super().__init__(cfg, device, dtype, tp)
        if self.device.type == "cuda" and self.dtype not in (torch.bfloat16, torch.float32):
            raise ValueError(f"fopivik runs in bfloat16 or float32 on CUDA, not {self.dtype}")
        self.order, self.passes = cfg.extra["order"], cfg.extra["passes"]
        self.pitch = up8(cfg.hidden_size)
        self.loop_in: list[LinearWeight] = []  # one per pass: the same matrix, the pass's vector as its bias

    def _check_kernels(self) -> None:
        pass  # head sizes are free: every layer's shape checks its own

    # ------------------------------------------------------------------------------------------------ loading
    def load(self, loader: WeightLoader, head_quant: Optional[str] = None, prefix: str = "") -> "FopivikModel":
        if head_quant:
            raise ValueError("output-head quantisation is not available for fopivik")
        cfg, eps, Kw = self.cfg, self.cfg.norm_eps, self.pitch
        W = cfg.hidden_size
        get = lambda n: loader.load_dense(prefix + n, self.dtype)  # noqa: E731
        f32 = lambda n: loader.load_dense(prefix + n, torch.float32).reshape(-1).to(self.device).contiguous()  # noqa: E731
        pad = torch.nn.functional.pad
        self.embed = self._dev(get("embed"))
        tables = RotaryTables(cfg.max_position_embeddings, self.device, ref.banded_rope_tables)
        for i, L in enumerate(cfg.extra["layers"]):
            p, m = f"l{i}.", L["mixer"]
            mix = lambda *names: [get(p + "mix." + n) for n in names]  # noqa: E731, B023
            if L["type"] == "gla":
                shape = GlaShape(int(m["heads"]), int(m["dim"]), int(m["vdim"]), int(get(p + "mix.a1").shape[0]))
                mixer = GatedLinearAttention(shape, m["tau"], eps, self.device, self.dtype)
                mixer.load(*mix("q", "k", "v", "g", "o", "a1", "a2"), f32(p + "mix.a2.b"), f32(p + "mix.norm"), k_pad=Kw)
            else:
                rot, mask = m["rot"], m.get("mask") or {}
                cos, sin = tables.get(int(rot["dims"]), float(rot["base"]), rot.get("scaling"))
                shape = GroupedShape(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]))
                mixer = GroupedAttention(shape, m["scale"], m.get("softcap") or 0.0, mask.get("size") or 0, mask.get("keep_first") or 0, True, cos, sin,
                                         self.device, self.dtype)
                mixer.load(*mix("q", "k", "v", "o"), k_pad=Kw)
            lw = SandwichLayer(mixer, f32(p + "norm1"), f32(p + "norm1b"))
            if mixer.w_out.N != W:
                raise ValueError(f"layer {i}: output projection has {mixer.w_out.N} rows, expected {W}")
            if L.get("mlp"):
                router, ff = L["mlp"]["router"], int(L["mlp"]["expert"]["ff"])
                lw.experts = RoutedExperts(int(router["experts"]), int(router["top"]))
                experts = (tuple(get(p + f"mlp.e{e}.{n}") for n in ("gate", "up", "down")) for e in range(lw.experts.experts))
                lw.experts.load(get(p + "mlp.router"), experts, ff, Kw, self.device, self.dtype)
                lw.norm2, lw.norm2b = f32(p + "norm2"), f32(p + "norm2b")
            self.layers.append(lw)
        if self.passes:
            w, step = get("loop.in"), loader.load_dense(prefix + "loop.step", torch.float32)
            if tuple(w.shape) != (W, 2 * W) or tuple(step.shape) != (len(self.passes), W):
                raise ValueError("loop.in must be [width, 2 width] and loop.step [times, width]")
            halves = self._dev(pad(w.reshape(W, 2, W), (0, Kw - W)).reshape(W, 2 * Kw))
            self.loop_in = [LinearWeight(halves, s.to(self.device).contiguous()) for s in step]
        self.final_norm = f32("final.norm")
        self.lm_head = self._lin(pad(get("head"), (0, Kw - W)))
        return self

    # ------------------------------------------------------------------------------------------------ forward
    def forward_hidden(self, batch: ForwardBatch, kv) -> torch.Tensor:
        cfg, eps, Kw, dt, m = self.cfg, self.cfg.norm_eps, self.pitch, self.dtype, self.cfg.residual_multiplier
        T, W = batch.num_tokens, cfg.hidden_size
        mix = None
        if self.passes:  # rows [stream | embedding output] that the mix in front of every pass reads
            mix = (torch.zeros if Kw != W else torch.empty)(T, 2 * Kw, dtype=dt, device=self.device)
        with self._stage("embedinput"):
            residual = ops.bigram_embedding(self.embed, None, batch.token_ids, None, 0, 0, 1.0, mix[:, Kw : Kw + W] if mix is not None else None)
        self._trace(-1, "embed", residual)
        sub = w_sub = None  # output of the last sublayer and the norm behind it

        def add(w_next, out=None):
            with self._stage("layernorm"):
                return ops.sandwich_norm(residual, sub, w_sub, m, w_next, eps, Kw, dt, out)

        for run, i in enumerate(self.order):
            lw = self.layers[i]
            if run in self.passes:
                add(None, mix[:, :W])
                with self._stage("loop.input_mix"):
                    residual = ops.linear(mix, self.loop_in[self.passes[run]], out_f32=True)
                sub = w_sub = None
            x = add(lw.norm1)
            sub, w_sub = lw.mixer.forward(x, batch, kv, run, self._stage), lw.norm1b
            if lw.experts is not None:
                x = add(lw.norm2)
                sub, w_sub = lw.experts.forward(x, self._stage), lw.norm2b
            if self.layer_hook is not None:
                after = residual.clone()
                ops.sandwich_norm(after, sub, w_sub, m, None, eps, Kw, torch.float32)
                self._trace(run, "out", after)
        return add(self.final_norm)

    # ------------------------------------------------------------------------------------------------ misc
    def kv_layout(self) -> dict:
        runs = [self.layers[i].mixer.cache_layout() for i in self.order]
        return {"layers": len(runs), "kv_heads": max(r["heads"] for r in runs), "head_dim": max(r["k"] for r in runs),
                "layer_kinds": [self.layers[i].mixer.kind for i in self.order], "kv_heads_per_layer": [r["heads"] for r in runs],
                "head_dim_per_layer": [r["k"] for r in runs], "v_dim_per_layer": [r["v"] for r in runs], "state_shapes": [r["state"] for r in runs]}

    def weight_bytes(self) -> int:
        n = self.embed.numel() * self.embed.element_size() + self.lm_head.nbytes() + (self.loop_in[0].nbytes() if self.loop_in else 0)
        for lw in self.layers:
            n += lw.mixer.nbytes() + (lw.experts.nbytes() if lw.experts is not None else 0)
        return n

    def set_lora(self, adapter=None, prefix: str = "") -> None:
        if adapter is not None:
            raise ValueError("run-time LoRA is not supported for fopivik")
