"""Gevovik decoder: Mamba-2, windowed grouped attention with mixed scores beside a gated delta rule, and latent attention (whose cache a later layer may
share) in any order, each followed by a dense feed-forward or nothing. Nothing is normed in front of a sublayer; its output is RMS-normed with a
single gain and added. The embedding adds a hashed-bigram row.

How a layer is laid out on the device (decode and prompts alike):

* the residual stream is fp32; ONE kernel finishes a sublayer and starts the next: norm of the output, add, the row in the projections' type
  (``ops.sandwich_norm``); the last one applies the final norm as well;
* all input projections of a mixer are one GEMM, its output projections one (for the two halves of a parallel mixer together);
* convolution, unit vectors, decays, recurrence, norm and gate of a decode step are one kernel (Mamba-2: two).
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

import torch

from .. import ops
from ..ckpt.loader import WeightLoader
from ..ops.delta import DeltaShape
from ..ops.grouped import GroupedShape, up8
from ..ops.latent import LatentShape
from ..ops.mamba import Mamba2Shape
from .batch import ForwardBatch
from .delta import GatedDeltaNet
from .feed_forward import FeedForward
from .grouped import GroupedAttention
from .latent import LatentAttention, RotaryTables
from .mamba import Mamba2Mixer
from .side_by_side import SideBySideMixer
from .transformer import DecoderModel


@dataclass
class PostNormLayer:
    """A mixer and a feed-forward, each with the gain (fp32, one element) of the norm behind it."""

    mixer: object
    norm1: torch.Tensor
    ff: Optional[FeedForward] = None
    norm2: Optional[torch.Tensor] = None


class GevovikModel(DecoderModel):
    reads_previous_token = True

    def __init__(self, cfg, device="cpu", dtype=None, tp=None):
        from ..parallel.context import SINGLE

        tp = tp or SINGLE
        if tp.enabled:
            raise ValueError("gevovik is not sharded for tensor parallelism")
        super().__init__(cfg, device, dtype, tp)
        if self.device.type == "cuda" and self.dtype not in (torch.bfloat16, torch.float32):
            raise ValueError(f"gevovik runs in bfloat16 or float32 on CUDA, not {self.dtype}")
        self.pitch = up8(cfg.hidden_size)
        self.bigram: Optional[torch.Tensor] = None

    def _check_kernels(self) -> None:
        pass  # head sizes are free: every layer's shape checks its own

    # ------------------------------------------------------------------------------------------------ loading
    def load(self, loader: WeightLoader, head_quant: Optional[str] = None, prefix: str = "") -> "GevovikModel":
        if head_quant:
            raise ValueError("output-head quantisation is not available for gevovik")
        cfg, W, Kw = self.cfg, self.cfg.hidden_size, self.pitch
        get = lambda n: loader.load_dense(prefix + n, self.dtype)  # noqa: E731
        f32 = lambda n: loader.load_dense(prefix + n, torch.float32)  # noqa: E731

        def gain(n):
            t = f32(n).reshape(-1).to(self.device).contiguous()
            if t.numel() != 1:
                raise ValueError(f"'{n}' has {t.numel()} elements, a norm's gain is one number")
            return t

        self.embed = self._dev(get("embed"))
        if cfg.extra["bigram"]:
            b = int(cfg.extra["bigram"]["buckets"])
            self.bigram = self._dev(get("bigram"))
            if self.bigram.shape[0] != b + 1:
                raise ValueError(f"bigram table has {self.bigram.shape[0]} rows, expected {b + 1}")
        self.tables = RotaryTables(cfg.max_position_embeddings, self.device)
        make = {"mamba2": self._mamba2, "parallel": self._parallel, "latent_attention": self._latent}
        for i, L in enumerate(cfg.extra["layers"]):
            p = f"l{i}."
            mixer = make[L["type"]](get, f32, p + "mix.", L["mixer"])
            if mixer.w_out.N != W:
                raise ValueError(f"layer {i}: output projection has {mixer.w_out.N} rows, expected {W}")
            lw = PostNormLayer(mixer, gain(p + "norm1"))
            if L.get("mlp"):
                lw.ff = FeedForward("relu2").load(get(p + "mlp.up"), get(p + "mlp.down"), int(L["mlp"]["ff"]), Kw, self.device, self.dtype)
                lw.norm2 = gain(p + "norm2")
            self.layers.append(lw)
        self.final_norm = gain("final.norm")
        self.lm_head = self._lin(torch.nn.functional.pad(get("head"), (0, Kw - W)))
        return self

    def _rotary(self, m: dict):
        rot = m["rot"]
        return self.tables.get(int(rot["dims"]), float(rot["base"]), rot.get("scaling"))

    def _mamba2(self, get, f32, p: str, m: dict) -> Mamba2Mixer:
        shape = Mamba2Shape(*(int(m[k]) for k in ("heads", "vdim", "state", "groups", "conv", "norm_groups")))
        mixer = Mamba2Mixer(shape, self.cfg.norm_eps, self.device, self.dtype)
        return mixer.load(get(p + "in"), *(f32(p + n) for n in ("conv", "conv.b", "dt_bias", "A_log", "D", "norm")), get(p + "o"), k_pad=self.pitch)

    def _parallel(self, get, f32, p: str, m: dict) -> SideBySideMixer:
        lm, rm, eps, lp, rp = m["left"], m["right"], self.cfg.norm_eps, p + "left.", p + "right."
        shape = GroupedShape(*(int(lm[k]) for k in ("heads", "kv_heads", "dim", "vdim")), gate="heads", mixed=True)
        left = GroupedAttention(shape, lm["scale"], 0.0, (lm.get("mask") or {}).get("size") or 0, 0, False, *self._rotary(lm), self.device, self.dtype,
                                rotate="halves", eps=eps, mult=m["left_scale"])
        mix = f32(lp + "talk") * f32(lp + "temp").reshape(1, -1)  # a head's own factor applies to its score ahead of the mixing
        packed = left.pack(*(get(lp + n) for n in ("q", "k", "v", "o")), g=get(lp + "g"), q_norm=f32(lp + "q.norm"), k_norm=f32(lp + "k.norm"), mix=mix)
        low = {n: get(rp + n) for n in ("a1", "a2", "g1", "g2")}
        shape = DeltaShape(*(int(rm[k]) for k in ("heads", "kv_heads", "dim", "vdim", "conv")), int(low["a1"].shape[0]), int(low["g1"].shape[0]))
        right = GatedDeltaNet(shape, eps, self.device, self.dtype, m["right_scale"])
        convs = [f32(rp + n + ".conv") for n in ("q", "k", "v")]
        return SideBySideMixer(left, right).load(packed, right.pack(*(get(rp + n) for n in ("q", "k", "v", "b")), *low.values(), get(rp + "o"), convs,
                                                                    *(f32(rp + n) for n in ("A_log", "dt_bias", "norm"))), self.pitch)

    def _latent(self, get, f32, p: str, m: dict) -> LatentAttention:
        own = m.get("kv_from") is None
        shape = LatentShape(*(int(m[k]) for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank")), gate=False, down=own)
        mixer = LatentAttention(shape, m["scale"], 0, self.cfg.norm_eps, *self._rotary(m), self.device, self.dtype, rotate="pairs")
        dkv, norm = (get(p + "dkv"), f32(p + "dkv.norm")) if own else (None, None)
        return mixer.load(get(p + "q"), dkv, norm, get(p + "uk"), get(p + "uv"), None, k_pad=self.pitch, sink=f32(p + "sink"), o=get(p + "o"))

    # ------------------------------------------------------------------------------------------------ forward
    def forward_hidden(self, batch: ForwardBatch, kv) -> torch.Tensor:
        cfg, eps, Kw, dt = self.cfg, self.cfg.norm_eps, self.pitch, self.dtype
        bg, T, W = cfg.extra["bigram"] or {}, batch.num_tokens, cfg.hidden_size
        x = (torch.zeros if Kw != W else torch.empty)(T, Kw, dtype=dt, device=self.device)
        with self._stage("embedinput"):
            residual = ops.bigram_embedding(self.embed, self.bigram, batch.token_ids, batch.prev_ids, int(bg.get("mul_prev", 0)), int(bg.get("mul_cur", 0)),
                                            cfg.embedding_multiplier, x[:, :W])
        self._trace(-1, "embed", residual)

        def add(y, gain, w_next=None):
            with self._stage("layernorm"):
                return ops.sandwich_norm(residual, y, gain, 1.0, w_next, eps, Kw, dt, rms=True)

        for i, lw in enumerate(self.layers):
            last = self.final_norm if i + 1 == len(self.layers) else None
            x = add(lw.mixer.forward(x, batch, kv, i, self._stage), lw.norm1, last if lw.ff is None else None)
            if lw.ff is not None:
                x = add(lw.ff.forward(x, self._stage), lw.norm2, last)
            self._trace(i, "out", residual)
        return x

    # ------------------------------------------------------------------------------------------------ misc
    def kv_layout(self) -> dict:
        runs = [lw.mixer.cache_layout() for lw in self.layers]
        layers = self.cfg.extra["layers"]
        src = [L["mixer"].get("kv_from") for L in layers]
        return {"layers": len(runs), "kv_heads": max(r["heads"] for r in runs), "head_dim": max(r["k"] for r in runs),
                "layer_kinds": [lw.mixer.kind for lw in self.layers], "kv_heads_per_layer": [r["heads"] for r in runs],
                "head_dim_per_layer": [r["k"] for r in runs], "v_dim_per_layer": [r["v"] for r in runs], "state_shapes": [r["state"] for r in runs],
                "shared_from": [-1 if j is None else int(j) for j in src], "paged": [L["type"] != "mamba2" for L in layers]}

    def weight_bytes(self) -> int:
        n = self.embed.numel() * self.embed.element_size() + self.lm_head.nbytes()
        if self.bigram is not None:
            n += self.bigram.numel() * self.bigram.element_size()
        return n + sum(lw.mixer.nbytes() + (lw.ff.nbytes() if lw.ff is not None else 0) for lw in self.layers)

    def set_lora(self, adapter=None, prefix: str = "") -> None:
        if adapter is not None:
            raise ValueError("run-time LoRA is not supported for gevovik")
