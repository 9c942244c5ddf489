"""Fatotar decoder: per layer a latent-attention mixer and a dense gated feed-forward read two LayerNorms of the same residual row and
are added to it together; a range of layers runs several times with the same weights; the embedding adds a hashed-bigram row.

How a layer run is laid out on the device (decode and prompts alike):

* the residual stream is fp32; one kernel adds the previous run's output and writes both LayerNorms (one set of statistics);
* query, latent-down and gate projections are one GEMM, gate and up another;
* the mixer writes its gated heads and the feed-forward its activations into one row buffer ``[heads | ff]``, so that the output and the
  down projection, whose results are summed anyway, are ONE GEMM with fp32 output.

Every layer run has its own cache entry (a looped layer must not see the keys of another pass).
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

import torch

from .. import ops
from ..ckpt.loader import WeightLoader
from ..ops import LinearWeight
from ..ops.latent import LatentShape
from .batch import ForwardBatch
from .latent import LatentAttention, RotaryTables
from .transformer import DecoderModel


def _up8(n: int) -> int:
    return (n + 7) // 8 * 8


@dataclass
class ParallelLayer:
    """Weights of one layer: norms as fp32 (weight, bias) pairs, ``out`` = output | down projection over the joint row buffer."""

    norm1: tuple
    mixer: LatentAttention
    norm2: Optional[tuple] = None
    gate_up: Optional[LinearWeight] = None
    ff: int = 0  # padded feed-forward width (0: the layer has none)
    ff_at: int = 0  # first feed-forward column of the row buffer
    row: int = 0  # width of the row buffer
    padded: bool = False  # the row buffer has columns nobody writes
    out: Optional[LinearWeight] = None


class FatotarModel(DecoderModel):
    reads_previous_token = True

    def __init__(self, cfg, device="cpu", dtype=None, tp=None):
        from ..parallel.context import SINGLE

        tp = tp or SINGLE
        if tp.enabled:
            raise ValueError("fatotar is not sharded for tensor parallelism")
        super().__init__(cfg, device, dtype, tp)
        if self.device.type == "cuda" and self.dtype not in (torch.bfloat16, torch.float32):
            raise ValueError(f"fatotar runs in bfloat16 or float32 on CUDA, not {self.dtype}")
        self.order = cfg.extra["order"]
        self.pitch = _up8(cfg.hidden_size)
        self.n_kv = 1
        self.bigram: Optional[torch.Tensor] = None

    def _check_kernels(self) -> None:
        pass  # head sizes are free: every layer's LatentShape checks its own

    # ------------------------------------------------------------------------------------------------ loading
    def load(self, loader: WeightLoader, head_quant: Optional[str] = None, prefix: str = "") -> "FatotarModel":
        if head_quant:
            raise ValueError("output-head quantisation is not available for fatotar")
        cfg = self.cfg
        W, Kw = cfg.hidden_size, self.pitch
        get = lambda n: loader.load_dense(prefix + n, self.dtype)  # noqa: E731
        f32 = lambda n: loader.load_dense(prefix + n, torch.float32).reshape(-1).to(self.device).contiguous()  # noqa: E731
        norm = lambda n: (f32(n), f32(n + ".b"))  # noqa: E731

        def lin(w, bias=None):
            if w.shape[1] % 8:
                w = torch.nn.functional.pad(w, (0, _up8(w.shape[1]) - w.shape[1]))
            return self._lin(w, bias)

        self.embed = self._dev(get("embed"))
        if cfg.extra["bigram"]:
            b = int(cfg.extra["bigram"]["buckets"])
            self.bigram = self._dev(get("bigram"))
            if self.bigram.shape[0] != b + 1:
                raise ValueError(f"bigram table has {self.bigram.shape[0]} rows, expected {b + 1}")
        tables = RotaryTables(cfg.max_position_embeddings, self.device)
        for i, L in enumerate(cfg.extra["layers"]):
            p, m = f"l{i}.", L["mixer"]
            shape = LatentShape(int(m["heads"]), int(m["dim"]), int(m["rot_dim"]), int(m["vdim"]), int(m["kv_rank"]), gate=True)
            rot = m["rot"]
            cos, sin = tables.get(int(rot["dims"]), float(rot["base"]), rot.get("scaling"))
            mixer = LatentAttention(shape, m["scale"], m["mask"]["size"], cfg.norm_eps, cos, sin, self.device, self.dtype)
            mixer.load(*(get(p + "mix." + n) for n in ("q", "dkv", "dkv.norm", "uk", "uv", "g")), k_pad=Kw)
            lw = ParallelLayer(norm(p + "norm1"), mixer)
            lw.ff_at = _up8(shape.out_width)
            w_o = get(p + "mix.o")
            parts, bias = [torch.nn.functional.pad(w_o, (0, lw.ff_at - shape.out_width))], None
            lw.row = lw.ff_at
            ff = int(L["mlp"]["ff"]) if L.get("mlp") else 0
            if ff:
                lw.norm2 = norm(p + "norm2")
                lw.ff = _up8(ff)
                lw.row += lw.ff
                pad = lw.ff - ff
                rows = lambda n: torch.nn.functional.pad(get(p + f"mlp.{n}"), (0, 0, 0, pad))  # noqa: E731
                rb = lambda n: torch.nn.functional.pad(get(p + f"mlp.{n}.b").reshape(-1).float(), (0, pad))  # noqa: E731
                lw.gate_up = lin(torch.cat([rows("gate"), rows("up")]), torch.cat([rb("gate"), rb("up")]))
                parts.append(torch.nn.functional.pad(get(p + "mlp.down"), (0, pad)))
                bias = get(p + "mlp.down.b").reshape(-1)
            lw.padded = lw.ff_at != shape.out_width
            lw.out = lin(torch.cat(parts, dim=1), bias)
            if lw.out.N != W:
                raise ValueError(f"layer {i}: output projection has {lw.out.N} rows, expected {W}")
            self.layers.append(lw)
        self.final_norm = norm("final.norm")
        self.lm_head = lin(get("head"))
        return self

    # ------------------------------------------------------------------------------------------------ forward
    def forward_hidden(self, batch: ForwardBatch, kv) -> torch.Tensor:
        cfg = self.cfg
        bg = cfg.extra["bigram"] or {}
        eps, pitch, dt = cfg.norm_eps, self.pitch, self.dtype
        with self._stage("embedinput"):
            residual = ops.bigram_embedding(self.embed, self.bigram, batch.token_ids, batch.prev_ids, int(bg.get("mul_prev", 0)), int(bg.get("mul_cur", 0)),
                                            cfg.embedding_multiplier)
        self._trace(-1, "embed", residual)
        T, delta = residual.shape[0], None
        for run, i in enumerate(self.order):
            lw = self.layers[i]
            with self._stage("layernorm"):
                x1, x2 = ops.add_layernorm(residual, delta, lw.norm1, lw.norm2, eps, pitch, dt)
            row = (torch.zeros if lw.padded else torch.empty)(T, lw.row, dtype=dt, device=self.device)
            lw.mixer.heads(x1, batch, kv.layer(run), row, self._stage)
            if lw.ff:
                with self._stage("mlpblock.gate_up_projection"):
                    gu = ops.linear(x2, lw.gate_up)
                with self._stage("mlpblock.activation_multiply"):
                    ops.gated_act_into(gu, cfg.hidden_act, row[:, lw.ff_at :])
            with self._stage("mlpblock.down_projection"):
                delta = ops.linear(row, lw.out, out_f32=True)
            if self.layer_hook is not None:
                self._trace(run, "out", residual + delta)
        return ops.add_layernorm(residual, delta, self.final_norm, None, eps, pitch, dt)[0]

    # ------------------------------------------------------------------------------------------------ misc
    def kv_layout(self) -> dict:
        shapes = [LatentShape(*(int(m[k]) for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank"))) for m in
                  (self.cfg.extra["layers"][i]["mixer"] for i in self.order)]
        return {"layers": len(shapes), "kv_heads": 1, "head_dim": max(s.Rp for s in shapes), "layer_kinds": ["latent"] * len(shapes),
                "head_dim_per_layer": [s.Rp for s in shapes], "v_dim_per_layer": [s.drp for s in shapes]}

    def weight_bytes(self) -> int:
        n = self.embed.numel() * self.embed.element_size() + self.lm_head.nbytes()
        if self.bigram is not None:
            n += self.bigram.numel() * self.bigram.element_size()
        for lw in self.layers:
            n += lw.mixer.nbytes() + lw.out.nbytes() + (lw.gate_up.nbytes() if lw.gate_up is not None else 0)
        return n

    def set_lora(self, adapter=None, prefix: str = "") -> None:
        if adapter is not None:
            raise ValueError("run-time LoRA is not supported for fatotar")
