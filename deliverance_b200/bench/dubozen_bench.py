"""Throughput and kernel times of the Dubozen decoder beside the framework's closest models, all bf16 with random weights.

    python bench.py --design dubozen [--sizes small,1b,3b] [--steps K] [--warmup W]

The model beside it is a GQA decoder with per-head q/k norms and routed experts in every other layer (qwen3_moe family): same width, layers,
vocabulary, feed-forwards, experts, query and KV heads. Lightning attention has no counterpart in it; its kernels are held against gated
linear attention (fopivik) with as many heads of the same widths. Fractions are of the measured copy bandwidth and cuBLAS bf16 burst
rate; the L2 is flushed before every timed launch, medians.
"""
from __future__ import annotations

import json

import torch

from .design_bench import Timer, _batch, _engine_splits, throughput

# layers alternate between grouped attention with a dense feed-forward and attention beside lightning attention with routed experts
SIZES = {
    "small": dict(width=1024, dense=2816, ff=1024, experts=8, top=2, heads=16, kv=4, dim=64, ln_heads=4, ln_dim=128, streams=2, vocab=32000),
    "1b": dict(width=2048, dense=5632, ff=1536, experts=16, top=2, heads=16, kv=4, dim=128, ln_heads=8, ln_dim=128, streams=2, vocab=32000),
    "3b": dict(width=3072, dense=8192, ff=1536, experts=16, top=4, heads=24, kv=6, dim=128, ln_heads=12, ln_dim=128, streams=2, vocab=32000),
}
LAYERS = 8


def dubozen_shape(z: dict) -> dict:
    from ..ckpt.tiny import dubozen_config

    soft = dict(heads=z["heads"], kv_heads=z["kv"], dim=z["dim"], rot_dims=z["dim"] // 2, base=500000.0)
    decay = [1.0 - 2.0 ** -(2 + 8 * i / max(1, z["ln_heads"] - 1)) for i in range(z["ln_heads"])]
    both = dict(soft, right=(z["ln_heads"], z["ln_dim"], z["ln_dim"], decay), ff=z["ff"], experts=z["experts"], top=z["top"], groups=4, keep=2)
    return dubozen_config(z["width"], z["vocab"], [dict(soft, ff=z["dense"]), both] * (LAYERS // 2), streams=z["streams"], max_position_embeddings=8192)


def moe_shape(z: dict) -> dict:
    return dict(model_type="qwen3_moe", vocab_size=z["vocab"], hidden_size=z["width"], intermediate_size=z["dense"], num_hidden_layers=LAYERS,
                num_attention_heads=z["heads"], num_key_value_heads=z["kv"], head_dim=z["dim"], max_position_embeddings=8192, rms_norm_eps=1e-5,
                rope_theta=500000.0, tie_word_embeddings=True, hidden_act="silu", bos_token_id=1, eos_token_id=2, num_experts=z["experts"],
                num_experts_per_tok=z["top"], moe_intermediate_size=z["ff"], norm_topk_prob=True, decoder_sparse_step=2, mlp_only_layers=[])


def kernel_times(dub, moe, z: dict, t: Timer, peaks: dict) -> list:
    """One row per pair of like kernels: microseconds and roofline fraction of both designs."""
    from .. import ops
    from ..kv.paged import KvCacheSettings, PagedKVCache
    from ..ops import gla as gla_op, grouped as gop, lightning as lop
    from ..ops.gla import GlaShape

    dev = dub.device
    hbm, tf = peaks["hbm_gbs"] * 1e9, peaks["bf16_tflops"] * 1e12
    la, lb, ma, mb = dub.layers[0], dub.layers[1], moe.layers[0], moe.layers[1]
    ax, px = la.mixer.block, lb.mixer.block
    left, right, s, ls = px.left, px.right, ax.shape, px.left.shape
    W, H, KV, D, S = z["width"], z["heads"], z["kv"], z["dim"], z["streams"]
    rows: list = []
    roof = lambda b, f: max(b / hbm, f / tf) * 1e6  # noqa: E731
    rnd = lambda *shape: torch.randn(*shape, device=dev).to(torch.bfloat16)  # noqa: E731

    def add(name, fn_f, cost_f, fn_g, cost_g):
        uf, ug = t.us(fn_f), t.us(fn_g)
        ff, fg = roof(*cost_f) / uf, roof(*cost_g) / ug
        rows.append({"kernel": name, "us": round(uf, 2), "roofline_us": round(roof(*cost_f), 2), "fraction": round(ff, 3), "like_us": round(ug, 2),
                     "like_roofline_us": round(roof(*cost_g), 2), "like_fraction": round(fg, 3), "distance_ratio": round(fg / ff, 2)})

    def gemm(name, M, wf, wg):
        xf, xg = rnd(M, wf.K), rnd(M, wg.K)
        cost = lambda w: (w.N * w.K * 2 + M * w.K * 2 + M * w.N * 2, 2.0 * M * w.N * w.K)  # noqa: E731
        add(f"{name} M={M}", lambda: ops.linear(xf, wf), cost(wf), lambda: ops.linear(xg, wg), cost(wg))

    stage = lambda _: _NULL  # noqa: E731
    for M in (1, 64, 8192):
        gemm("q|k|v|g projection", M, ax.w_in, ma.qkv)
        gemm("side-by-side input projection (against q|k|v)", M, px.w_in, ma.qkv)
        gemm("output projection", M, ax.w_out, ma.o)
        gemm("side-by-side output projection (against o)", M, px.w_out, ma.o)
        gemm("gate|up projection", M, la.ff.block.gate_up, ma.gate_up)
        gemm("down projection", M, la.ff.block.down, ma.down)
        x = rnd(M, W)
        gu, gg = rnd(M, 2 * z["dense"]), rnd(M, 2 * z["dense"])
        h = torch.empty(M, z["dense"], dtype=torch.bfloat16, device=dev)
        add(f"gelu(gate) * up (against silu) M={M}", lambda: ops.gated_act_into(gu, "gelu_pytorch_tanh", h), (M * z["dense"] * 6, 0), lambda: ops.act_mul(gg, "silu"),
            (M * z["dense"] * 6, 0))
        per = min(z["experts"], M * z["top"]) * 3 * z["ff"] * W * 2 + M * W * 4 * z["top"]
        flops = 2.0 * M * z["top"] * 3 * z["ff"] * W
        add(f"routed experts M={M}", lambda: lb.ff.block.forward(x, stage), (per, flops), lambda: moe.moe(1, mb, x), (per + M * W * 2 * (z["top"] + 1), flops))
        X, sub, rb, xb = torch.randn(M, S, W, device=dev), rnd(M, W), rnd(M, W), rnd(M, W)
        c, w2 = la.mixer.conn, la.ff.norm
        step = lambda y, k: ops.stream_step(X, y, c.mix, c.write, c.read, w2, 1e-5, dub.pitch, torch.bfloat16, k)  # noqa: E731
        add(f"streams: write, read, norm (against add, norm) M={M}", lambda: step(sub, True), (M * W * (8 * S + 4), 0),
            lambda: ops.add_rmsnorm(xb, rb, ma.pre_ff_norm, 1e-5), (M * W * 8, 0))
        k = z["top"]
        pos = torch.randperm(M * k, device=dev).to(torch.int32).reshape(M, k)
        ys, w = rnd(M * k, W), torch.rand(M, k, device=dev)
        routed, e = ops.Routed(ys, pos, w), ops.require_ext()

        def combine_add():
            ops.add_rmsnorm(e.moe_combine(ys, pos.reshape(-1), w, M, k), rb, ma.pre_ff_norm, 1e-5)

        add(f"streams: expert sum, write, read, norm (against combine, add, norm) M={M}", lambda: step(routed, True), (M * W * (8 * S + 2 + 2 * k), 0), combine_add,
            (M * W * (2 * k + 10), 0))
        ids = torch.randint(0, z["vocab"], (M,), device=dev).to(torch.int32)
        add(f"embedding, norm, streams, norm (against embedding, norm) M={M}",
            lambda: ops.stream_open(dub.embed, ids, dub.embed_norm, S, c.read, la.mixer.norm, 1e-5, dub.pitch, torch.bfloat16), (M * W * (4 * S + 4), 0),
            lambda: ops.rmsnorm(ops.embedding(moe.embed, ids), ma.input_norm, 1e-5), (M * W * 8, 0))

    gs = GlaShape(z["ln_heads"], z["ln_dim"], z["ln_dim"], 16)
    a2, a2b, gn = torch.randn(gs.heads * gs.dk, gs.rank8, device=dev), torch.randn(gs.heads * gs.dk, device=dev) + 2, torch.ones(gs.dv, device=dev)
    rs = right.shape
    for B, start, n in ((1, 2047, 1), (8, 2047, 1), (64, 2047, 1), (4, 0, 2048)):
        b, pages = _batch(B, start, n, dev)
        b.state_slots = torch.arange(1, B + 1, device=dev)
        T = B * n
        tag = f"B={B} context 2048" if n == 1 else f"{B} x {n} tokens"
        kf = PagedKVCache({"layers": 1, "kv_heads": KV, "head_dim": D, "layer_kinds": ["attention"]}, pages, dev, torch.bfloat16, KvCacheSettings(enabled=False))
        kf.k[0].normal_(), kf.v[0].normal_()
        kc, vc = kf.layer(0)
        pa, pl, qkv, first = rnd(T, s.width), rnd(T, px.w_in.N), rnd(T, (H + 2 * KV) * D), rnd(T, KV * D)
        q, rot = qkv[:, : H * D], z["dim"] // 2
        like_rope = lambda: ops.rope_kv(qkv, b.positions, b.slots, ma.q_norm, ma.k_norm, moe.cos, moe.sin, kc, vc, H, KV, D, 1e-5)  # noqa: E731
        add(f"rotation, value mixing, cache write {tag}", lambda: gop.rope_heads_kv(s, pa, b.positions, b.slots, ax.cos, ax.sin, kc, vc, v_first=first, lam=0.4),
            (T * (H * rot * 4 + KV * D * 10), 0), like_rope, (T * (H + 2 * KV) * D * 4, 0))
        add(f"head norms, rotation, tied cache write {tag}",
            lambda: gop.rope_heads_kv(ls, pl[:, : ls.width], b.positions, b.slots, left.cos, left.sin, kc, vc, left.q_norm, left.k_norm, 1e-5),
            (T * (H * D * 4 + KV * D * 6), 0), like_rope, (T * (H + 2 * KV) * D * 4, 0))
        row = torch.empty(T, ls.out_width + rs.out_width, dtype=torch.bfloat16, device=dev)
        if n == 1:
            sp, sl = ops.decode_splits(B, KV, 2048), _engine_splits(B, KV)
            kvb = B * 2048 * 2 * KV * D * 2 + T * H * D * 4
            like = lambda: ops.decode_attention(q, kc, vc, b.block_tables, b.ctx_len, H, D ** -0.5, 0.0, 0, sl)  # noqa: E731
            add(f"decode attention, sink, column gate {tag}", lambda: gop.attention(s, pa, b, kc, vc, ax.scale, 0.0, 0, 0, ax.sink, sp), (kvb + T * H * D * 2, 0), like, (kvb, 0))
            add(f"decode attention, head gate {tag}", lambda: gop.attention(ls, pl[:, : ls.width], b, kc, vc, left.scale, 0.0, 0, 0, None, sp, 0.6, row[:, : ls.out_width]),
                (kvb, 0), like, (kvb, 0))
        else:
            fl = (0, 4.0 * B * n * (n + 1) / 2 * H * D)
            like = lambda: ops.prefill_attention(q, kc, vc, b.block_tables, b.q_start, b.q_len, b.ctx_len, H, D ** -0.5, 0.0, 0, True, b.tile_seq, b.tile_q0,  # noqa: E731
                                                 tiles_for=b.tiles)
            add(f"prompt attention, sink, column gate {tag}", lambda: gop.attention(s, pa, b, kc, vc, ax.scale, 0.0, 0, 0, ax.sink, 1), fl, like, fl)
            add(f"prompt attention, head gate {tag}", lambda: gop.attention(ls, pl[:, : ls.width], b, kc, vc, left.scale, 0.0, 0, 0, None, 1, 0.6, row[:, : ls.out_width]),
                fl, like, fl)
        st, sg, pg = torch.zeros(B + 1, rs.heads, rs.dk, rs.dv, device=dev), torch.zeros(B + 1, gs.heads, gs.dk, gs.dv, device=dev), rnd(T, gs.width)
        state = B * rs.heads * rs.dk * rs.dv * 8
        fl = 6.0 * T * rs.heads * rs.dk * rs.dv  # (state update and read per token)
        add(f"lightning attention, norm, gate {tag} (against gated linear attention)",
            lambda: lop.lightning(rs, pl[:, ls.width :], right.decay, right.powers, right.norm, st, b, 1e-5, 0.4, row[:, ls.out_width :]),
            (state + T * (rs.width + rs.out_width) * 2, fl), lambda: gla_op.gla(gs, pg, a2, a2b, gn, sg, b, gs.dim ** -0.5, 16.0, 1e-5),
            (state + T * (gs.width + gs.out_width) * 2, fl))
        del kf, st, sg
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
    from ..models.dubozen import DubozenModel
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
        ds, ms = dubozen_shape(z), moe_shape(z)
        dub = DubozenModel(parse_config(ds), dev, torch.bfloat16).load(SyntheticLoader(ds, 0, False, dev))
        moe = DecoderModel(parse_config(ms), dev, torch.bfloat16).load(SyntheticLoader(ms, 0, False, dev))
        r = {"shape": z, "weight_bytes": {"dubozen": dub.weight_bytes(), "gqa_moe": moe.weight_bytes()}}
        if kernels:
            r["kernels"] = kernel_times(dub, moe, z, t, peaks)
        r["dubozen"] = {k: round(v, 1) for k, v in throughput(dub, z["vocab"], steps, warmup).items()}
        r["gqa_moe"] = {k: round(v, 1) for k, v in throughput(moe, z["vocab"], steps, warmup).items()}
        ops.check_status()
        out["sizes"][name] = r
        del dub, moe
        torch.cuda.empty_cache()
    return out


def main(args) -> int:
    print(json.dumps(run(args.sizes.split(","), args.steps, args.warmup, not args.no_kernels)))
    return 0
