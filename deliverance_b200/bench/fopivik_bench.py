"""Throughput and kernel times of the Fopivik decoder beside the framework's closest models, all bf16 with random weights.

    python bench.py --design fopivik [--sizes small,1b,3b] [--steps K] [--warmup W]

The model beside it is a GQA decoder with routed experts (qwen3_moe family): same width, layer runs, vocabulary, experts, query and KV
heads, full attention in the end-to-end rows (its attention kernels are timed with the same sliding window). Gated linear attention is
held against the Mamba2 kernels of granitemoehybrid with a state of the same size. Fractions are of the measured copy bandwidth and
cuBLAS bf16 burst rate; the L2 is flushed before every timed launch, medians.
"""
from __future__ import annotations

import json

import torch

from .design_bench import Timer, _batch, _engine_splits, throughput

# layers: 2 gated-linear-attention layers per softmax-attention layer, the middle three run twice
SIZES = {
    "small": dict(width=1024, ff=1024, experts=8, top=2, heads=16, kv=4, dim=64, gla_heads=4, gla_dim=128, gla_vdim=256, window=1024, keep=64, vocab=32000),
    "1b": dict(width=2048, ff=1536, experts=16, top=2, heads=16, kv=4, dim=128, gla_heads=4, gla_dim=256, gla_vdim=512, window=1024, keep=64, vocab=32000),
    "3b": dict(width=3072, ff=1536, experts=16, top=4, heads=24, kv=6, dim=128, gla_heads=6, gla_dim=256, gla_vdim=512, window=1024, keep=64, vocab=32000),
}
KINDS = ("attention", "gla", "gla", "attention", "gla")
LOOP = {"start": 1, "stop": 4, "times": 2}
RUNS = 8  # 5 layers, three of them twice


def fopivik_shape(z: dict) -> dict:
    from ..ckpt.tiny import fopivik_config

    moe = {k: z[k] for k in ("experts", "top", "ff")}
    soft = dict(moe, heads=z["heads"], kv_heads=z["kv"], dim=z["dim"], vdim=z["dim"], window=z["window"], keep_first=z["keep"], rot_dims=z["dim"] // 2,
                base=500000.0, scaling={"factor": 8.0, "low": 1.0, "high": 4.0, "original": 4096}, softcap=50.0)
    lin = dict(moe, heads=z["gla_heads"], dim=z["gla_dim"], vdim=z["gla_vdim"], tau=16.0, rank=16)
    return fopivik_config(z["width"], z["vocab"], [soft if k == "attention" else lin for k in KINDS], loop=LOOP, residual_mult=0.3, logit_softcap=15.0,
                          max_position_embeddings=8192)


def moe_shape(z: dict) -> dict:
    return dict(model_type="qwen3_moe", vocab_size=z["vocab"], hidden_size=z["width"], intermediate_size=z["ff"], num_hidden_layers=RUNS,
                num_attention_heads=z["heads"], num_key_value_heads=z["kv"], head_dim=z["dim"], max_position_embeddings=8192, rms_norm_eps=1e-5,
                rope_theta=500000.0, tie_word_embeddings=False, hidden_act="silu", bos_token_id=1, eos_token_id=2, num_experts=z["experts"],
                num_experts_per_tok=z["top"], moe_intermediate_size=z["ff"], norm_topk_prob=False, decoder_sparse_step=1, mlp_only_layers=[])


class Mamba:
    """The Mamba-2 mixer core (convolution, recurrence, gated norm) with a state as large as the linear-attention layer's."""

    def __init__(self, z: dict, dev):
        from ..ops.mamba import Mamba2Shape, Mamba2Weights

        self.S, self.dh = 128, 64
        self.H = z["gla_heads"] * z["gla_dim"] * z["gla_vdim"] // (self.S * self.dh)
        self.I = self.H * self.dh
        self.shape = Mamba2Shape(self.H, self.dh, self.S, 1, 4)
        r = lambda *s: torch.randn(*s)  # noqa: E731
        C = self.shape.conv_width
        self.w = Mamba2Weights.pack(self.shape, r(C, 4) * 0.3, None, r(self.H), r(self.H) * 0.3, r(self.H), 1 + 0.1 * r(self.I), dev)
        self.width = self.shape.dt_at + self.H

    def states(self, slots, dev):
        return tuple(torch.zeros((slots,) + s, device=dev) for s in self.shape.state_shapes().values())

    def run(self, zx, st, b):
        from ..ops.mamba import mamba2

        return mamba2(self.shape, zx, self.w, *st, b, 1e-5)


def kernel_times(fop, moe, z: dict, t: Timer, peaks: dict) -> list:
    """One row per pair of like kernels: microseconds and roofline fraction of both designs."""
    from .. import ops
    from ..kv.paged import KvCacheSettings, PagedKVCache
    from ..ops import gla as gla_op, grouped as gop

    dev = fop.device
    hbm, tf = peaks["hbm_gbs"] * 1e9, peaks["bf16_tflops"] * 1e12
    soft, lin, ml = fop.layers[0], fop.layers[1], moe.layers[0]
    sx, gx, s, g = soft.mixer, lin.mixer, soft.mixer.shape, lin.mixer.shape
    W, H, KV, D = z["width"], z["heads"], z["kv"], z["dim"]
    rows: list = []
    roof = lambda b, f: max(b / hbm, f / tf) * 1e6  # noqa: E731
    rnd = lambda *shape: torch.randn(*shape, device=dev).to(torch.bfloat16)  # noqa: E731

    def add(name, fn_f, cost_f, fn_g, cost_g):
        uf, ug = t.us(fn_f), t.us(fn_g)
        ff, fg = roof(*cost_f) / uf, roof(*cost_g) / ug
        rows.append({"kernel": name, "us": round(uf, 2), "roofline_us": round(roof(*cost_f), 2), "fraction": round(ff, 3), "like_us": round(ug, 2),
                     "like_roofline_us": round(roof(*cost_g), 2), "like_fraction": round(fg, 3), "distance_ratio": round(fg / ff, 2)})

    def gemm(name, M, wf, wg, out_f32=False):
        xf, xg = rnd(M, wf.K), rnd(M, wg.K)
        cost = lambda w, ob: (w.N * w.K * 2 + M * w.K * 2 + M * w.N * ob, 2.0 * M * w.N * w.K)  # noqa: E731
        add(f"{name} M={M}", lambda: ops.linear(xf, wf, out_f32=out_f32), cost(wf, 4 if out_f32 else 2), lambda: ops.linear(xg, wg), cost(wg, 2))

    stage = lambda _: _NULL  # noqa: E731
    for M in (64, 8192):
        gemm("q|k|v projection", M, sx.w_in, ml.qkv)
        gemm("linear attention input projection (against q|k|v)", M, gx.w_in, ml.qkv)
        gemm("output projection", M, sx.w_out, ml.o)
        gemm("pass input mix (against o)", M, fop.loop_in[0], ml.o, out_f32=True)
        x = rnd(M, W)
        per = min(z["experts"], M * z["top"]) * 3 * z["ff"] * W * 2 + M * W * 4 * z["top"]
        flops = 2.0 * M * z["top"] * 3 * z["ff"] * W
        add(f"routed experts M={M}", lambda: soft.experts.forward(x, stage), (per, flops), lambda: moe.moe(0, ml, x), (per + M * W * 2 * (z["top"] + 1), flops))
        res, sub, rb, xb = torch.randn(M, W, device=dev), rnd(M, W), rnd(M, W), rnd(M, W)
        add(f"norm, add, norm M={M}", lambda: ops.sandwich_norm(res, sub, soft.norm1b, 0.3, soft.norm2, 1e-5, fop.pitch, torch.bfloat16), (M * W * 12, 0),
            lambda: ops.add_rmsnorm(xb, rb, ml.pre_ff_norm, 1e-5), (M * W * 8, 0))
        k = z["top"]
        pos = torch.randperm(M * k, device=dev).to(torch.int32).reshape(M, k)
        ys, w = rnd(M * k, W), torch.rand(M, k, device=dev)
        routed = ops.Routed(ys, pos, w)
        e = ops.require_ext()

        def combine_add():
            ops.add_rmsnorm(e.moe_combine(ys, pos.reshape(-1), w, M, k), rb, ml.pre_ff_norm, 1e-5)

        add(f"expert sum, norm, add, norm M={M}", lambda: ops.sandwich_norm(res, routed, soft.norm2b, 0.3, soft.norm1, 1e-5, fop.pitch, torch.bfloat16),
            (M * W * (10 + 2 * k), 0), combine_add, (M * W * (2 * k + 10), 0))

    mam = Mamba(z, dev)
    for B, start, n in ((1, 2047, 1), (8, 2047, 1), (64, 2047, 1), (4, 0, 2048)):
        b, pages = _batch(B, start, n, dev)
        b.state_slots = torch.arange(1, B + 1, device=dev)
        T = B * n
        tag = f"B={B} context 2048" if n == 1 else f"{B} x {n} tokens"
        kf = PagedKVCache({"layers": 1, "kv_heads": KV, "head_dim": s.dk, "layer_kinds": ["sliding"]}, pages, dev, torch.bfloat16, KvCacheSettings(enabled=False))
        kf.k[0].normal_(), kf.v[0].normal_()
        kc, vc = kf.layer(0)
        qkv = rnd(T, s.width)
        q = qkv[:, : H * D]
        add(f"rotation + cache write {tag}", lambda: gop.rope_pairs_kv(s, qkv, b.positions, b.slots, sx.cos, sx.sin, kc, vc),
            (T * (H * (z["dim"] // 2) + 2 * KV * D) * 4, 0),
            lambda: ops.rope_kv(qkv, b.positions, b.slots, None, None, moe.cos, moe.sin, kc, vc, H, KV, D, 1e-5), (T * (H + 2 * KV) * D * 4, 0))
        win, keep = z["window"], z["keep"]
        att = (sx.scale, sx.softcap, win, keep, sx.sink)
        if n == 1:
            span = min(2048, win + keep)
            sp = ops.decode_splits(B, KV, span)
            add(f"decode attention {tag}", lambda: gop.attention(s, qkv, b, kc, vc, *att, sp), (B * span * 2 * KV * D * 2 + T * H * D * 4, 0),
                lambda: ops.decode_attention(q, kc, vc, b.block_tables, b.ctx_len, H, D ** -0.5, 50.0, win, _engine_splits(B, KV)),
                (B * min(2048, win) * 2 * KV * D * 2 + T * H * D * 4, 0))
        else:
            pairs = lambda w: B * (n * (n + 1) / 2 if w >= n else w * (n - w) + w * (w + 1) / 2)  # noqa: E731
            for cap in (50.0, 0.0):
                tail = " soft-capped" if cap else " no cap"
                add(f"prompt attention {tag}{tail}", lambda: gop.attention(s, qkv, b, kc, vc, sx.scale, cap, win, keep, sx.sink, 1),
                    (0, 4.0 * (pairs(win) + B * keep * max(0, n - win - keep)) * H * D),
                    lambda: ops.prefill_attention(q, kc, vc, b.block_tables, b.q_start, b.q_len, b.ctx_len, H, D ** -0.5, cap, win, True, b.tile_seq, b.tile_q0,
                                                  tiles_for=b.tiles), (0, 4.0 * pairs(win) * H * D))
        st = torch.zeros(B + 1, g.heads, g.dk, g.dv, device=dev)
        p, zx = rnd(T, g.width), rnd(T, mam.width)
        cst = mam.states(B + 1, dev)
        state = B * g.heads * g.dk * g.dv * 8
        fl = lambda h, a, c: 6.0 * T * h * a * c  # noqa: E731  (state update and read per token)
        add(f"linear attention {tag} (against Mamba2)", lambda: gla_op.gla(g, p, gx.a2, gx.a2_bias, gx.norm, st, b, gx.q_scale, gx.tau, 1e-5),
            (state + T * (g.width + g.out_width) * 2, fl(g.heads, g.dk, g.dv)), lambda: mam.run(zx, cst, b),
            (B * mam.H * mam.dh * mam.S * 8 + T * (mam.width + mam.I) * 2, fl(mam.H, mam.dh, mam.S)))
        del kf, st, cst
    return rows


class _Null:
    def __enter__(self):
        return self

    def __exit__(self, *a):
        return False


_NULL = _Null()


def run(sizes, steps: int, warmup: int, kernels: bool = True) -> dict:
    from .. import ops
    from ..ckpt.synthetic import SyntheticLoader
    from ..config import parse_config
    from ..models.fopivik import FopivikModel
    from ..models.transformer import DecoderModel
    from .roofline import load_peaks

    torch.set_grad_enabled(False)
    dev = torch.device("cuda", torch.cuda.current_device())
    ops.require_ext()
    peaks, kind = load_peaks()
    out = {"metric": "design_tokens_per_s", "dtype": "bf16", "data": "synthetic (uniform random prompts, random weights)", "denominators": kind, "sizes": {}}
    t = Timer(dev, max(10, min(steps, 40)), warmup)
    for name in sizes:
        z = SIZES[name]
        fs, ms = fopivik_shape(z), moe_shape(z)
        fop = FopivikModel(parse_config(fs), dev, torch.bfloat16).load(SyntheticLoader(fs, 0, False, dev))
        moe = DecoderModel(parse_config(ms), dev, torch.bfloat16).load(SyntheticLoader(ms, 0, False, dev))
        r = {"shape": z, "weight_bytes": {"fopivik": fop.weight_bytes(), "gqa_moe": moe.weight_bytes()}}
        if kernels:
            r["kernels"] = kernel_times(fop, moe, z, t, peaks)
        r["fopivik"] = {k: round(v, 1) for k, v in throughput(fop, z["vocab"], steps, warmup).items()}
        r["gqa_moe"] = {k: round(v, 1) for k, v in throughput(moe, z["vocab"], steps, warmup).items()}
        ops.check_status()
        out["sizes"][name] = r
        del fop, moe
        torch.cuda.empty_cache()
    return out


def main(args) -> int:
    print(json.dumps(run(args.sizes.split(","), args.steps, args.warmup, not args.no_kernels)))
    return 0
