"""Throughput and kernel times of the Gevovik decoder beside the framework's closest models, all bf16 with random weights.

    python bench.py --design gevovik [--sizes small,1b,3b] [--steps K] [--warmup W]

The model beside it is a granitemoehybrid decoder without routed experts: same width, vocabulary and Mamba-2 layers, grouped attention (same query and KV
heads, full) in the place of the other layers, gated feed-forwards with as many weights. Kernels are held against the like kernels of the closest family:
projections, norms and softmax attention (same window) against granitemoehybrid's, Mamba-2 against lightning attention (dubozen) and the gated delta rule
against gated linear attention (fopivik) with heads of the same sizes, latent attention with a sink against latent attention with an output gate
(fatotar). Fractions are of the measured copy bandwidth and cuBLAS bf16 burst rate; the L2 is flushed before every timed launch, medians.
"""
from __future__ import annotations

import json

import torch

from .design_bench import Timer, _batch, _engine_splits, throughput

SIZES = {
    "small": dict(width=1024, ff=4096, heads=16, kv=4, dim=64, window=1024, ssd_heads=32, state=64, delta_heads=8, delta_dim=128, rank=64, lat_dim=64, lat_rot=32, kv_rank=256,
                  vocab=32000),
    "1b": dict(width=2048, ff=8192, heads=16, kv=4, dim=128, window=1024, ssd_heads=64, state=128, delta_heads=16, delta_dim=128, rank=128, lat_dim=128, lat_rot=64, kv_rank=512,
               vocab=32000),
    "3b": dict(width=3072, ff=12288, heads=24, kv=4, dim=128, window=1024, ssd_heads=96, state=128, delta_heads=24, delta_dim=128, rank=128, lat_dim=128, lat_rot=64, kv_rank=512,
               vocab=32000),
}
SSD_DIM = 64
KINDS = ("mamba", "parallel", "latent", "mamba", "parallel", "latent", "mamba", "parallel")
YARN = {"factor": 4.0, "original": 4096, "fast": 32.0, "slow": 1.0}


def gevovik_shape(z: dict) -> dict:
    from ..ckpt.tiny import gevovik_config

    ssd = dict(heads=z["ssd_heads"], vdim=SSD_DIM, state=z["state"], groups=1, conv=4, norm_groups=1, ff=z["ff"])
    both = dict(heads=z["heads"], kv_heads=z["kv"], dim=z["dim"], window=z["window"], base=500000.0, scaling=YARN, ff=z["ff"],
                right=(z["delta_heads"], z["delta_heads"], z["delta_dim"], z["delta_dim"], 4), ranks=(z["rank"], z["rank"]))
    lat = dict(heads=z["heads"], dim=z["lat_dim"], rot_dim=z["lat_rot"], vdim=z["dim"], kv_rank=z["kv_rank"], base=500000.0, ff=z["ff"])
    layers = [dict({"mamba": ssd, "parallel": both, "latent": lat}[k]) for k in KINDS]
    layers[5]["kv_from"] = 2
    return gevovik_config(z["width"], z["vocab"], layers, buckets=65521, mul=(8191, 131), max_position_embeddings=8192)


def hybrid_shape(z: dict) -> dict:
    return dict(model_type="granitemoehybrid", vocab_size=z["vocab"], hidden_size=z["width"], intermediate_size=z["ff"] * 2 // 3 // 64 * 64, num_hidden_layers=len(KINDS),
                num_attention_heads=z["heads"], num_key_value_heads=z["kv"], max_position_embeddings=8192, rms_norm_eps=1e-5, rope_theta=500000.0, bos_token_id=1,
                eos_token_id=2, hidden_act="silu", tie_word_embeddings=False, layer_types=["mamba" if k == "mamba" else "attention" for k in KINDS],
                embedding_multiplier=1.0, attention_multiplier=z["dim"] ** -0.5, residual_multiplier=1.0, logits_scaling=1.0, num_local_experts=0, num_experts_per_tok=0,
                shared_intermediate_size=z["ff"] * 2 // 3 // 64 * 64, position_embedding_type="rope", mamba_n_heads=z["ssd_heads"], mamba_n_groups=1,
                mamba_d_state=z["state"], mamba_d_head=SSD_DIM, mamba_d_conv=4, mamba_expand=z["ssd_heads"] * SSD_DIM // z["width"], mamba_conv_bias=True, mamba_proj_bias=False)


def kernel_times(gev, hyb, z: dict, t: Timer, peaks: dict) -> list:
    """One row per pair of like kernels: microseconds and roofline fraction of both designs."""
    from types import SimpleNamespace

    from .. import ops
    from ..kv.paged import KvCacheSettings, PagedKVCache
    from ..models.latent import LatentAttention
    from ..ops import gla as gla_op, grouped as gop, lightning as lop
    from ..ops.gla import GlaShape
    from ..ops.latent import LatentShape
    from ..ops.lightning import LightningShape, decay_powers
    from ..ops.mamba import mamba2

    dev = gev.device
    hbm, tf = peaks["hbm_gbs"] * 1e9, peaks["bf16_tflops"] * 1e12
    lm, lp, ll, ls = gev.layers[0], gev.layers[1], gev.layers[2], gev.layers[5]
    hm, ha = hyb.layers[0], hyb.layers[1]
    ssd, px, lat = lm.mixer.shape, lp.mixer, ll.mixer
    left, right = px.left, px.right
    s, d = left.shape, right.shape
    W, H, KV, D, win = z["width"], z["heads"], z["kv"], z["dim"], z["window"]
    rows: list = []
    roof = lambda b, f: max(b / hbm, f / tf) * 1e6  # noqa: E731
    rnd = lambda *shape: torch.randn(*shape, device=dev).to(torch.bfloat16)  # noqa: E731
    stage = lambda _: _NULL  # noqa: E731

    def add(name, fn_f, cost_f, fn_g, cost_g):
        uf, ug = t.us(fn_f), t.us(fn_g)
        ff, fg = roof(*cost_f) / uf, roof(*cost_g) / ug
        rows.append({"kernel": name, "us": round(uf, 2), "roofline_us": round(roof(*cost_f), 2), "fraction": round(ff, 3), "like_us": round(ug, 2),
                     "like_roofline_us": round(roof(*cost_g), 2), "like_fraction": round(fg, 3), "distance_ratio": round(fg / ff, 2)})

    def gemm(name, M, wf, wg, out_f32=False):
        xf, xg = rnd(M, wf.K), rnd(M, wg.K)
        cost = lambda w, ob: (w.N * w.K * 2 + M * w.K * 2 + M * w.N * ob, 2.0 * M * w.N * w.K)  # noqa: E731
        add(f"{name} M={M}", lambda: ops.linear(xf, wf, out_f32=out_f32), cost(wf, 4 if out_f32 else 2), lambda: ops.linear(xg, wg), cost(wg, 2))

    for M in (1, 64, 8192):
        gemm("Mamba-2 input projection", M, lm.mixer.w_in, hm.mamba["in_proj"])
        gemm("Mamba-2 output projection", M, lm.mixer.w_out, hm.mamba["out_proj"])
        gemm("side-by-side input projection (against q|k|v)", M, px.w_in, ha.qkv)
        gemm("side-by-side output projection (against o)", M, px.w_out, ha.o)
        gemm("low-rank projection(s) (against o)", M, right.w_low if M < 8192 else right.w_decay, ha.o, out_f32=True)
        gemm("latent input projection (against q|k|v)", M, lat.w_in, ha.qkv)
        gemm("queries on a shared cache (against q|k|v)", M, ls.mixer.w_in, ha.qkv)
        gemm("latent output projection", M, lat.w_out, ha.o)
        ff, fg = lm.ff, hm.shared_gate_up.N // 2
        x, xg = rnd(M, ff.up.K), rnd(M, hm.shared_gate_up.K)

        def gated_ff():
            ops.linear(ops.act_mul(ops.linear(xg, hm.shared_gate_up), "silu"), hm.shared_down)

        add(f"feed-forward (against gated) M={M}", lambda: ff.forward(x, stage), (2 * ff.ff * W * 2 + M * W * 4, 4.0 * M * W * ff.ff), gated_ff,
            (3 * fg * W * 2 + M * W * 4, 6.0 * M * W * fg))
        res, sub, rb, xb = torch.randn(M, W, device=dev), rnd(M, W), rnd(M, W), rnd(M, W)
        add(f"norm, add, next input M={M}", lambda: ops.sandwich_norm(res, sub, lm.norm1, 1.0, None, 1e-5, gev.pitch, torch.bfloat16, rms=True), (M * W * 12, 0),
            lambda: ops.add_rmsnorm(xb, rb, hm.pre_ff_norm, 1e-5), (M * W * 8, 0))
        ids = torch.randint(0, z["vocab"], (M,), device=dev).to(torch.int32)
        add(f"bigram embedding (against embedding, norm) M={M}", lambda: ops.bigram_embedding(gev.embed, gev.bigram, ids, ids, 8191, 131, 4.0, xb), (M * W * 10, 0),
            lambda: ops.rmsnorm(ops.embedding(hyb.embed, ids), hm.input_norm, 1e-5), (M * W * 8, 0))

    lns = LightningShape(ssd.heads, ssd.state, ssd.vdim)
    decay = [1.0 - 2.0 ** -(2 + 8 * i / max(1, ssd.heads - 1)) for i in range(ssd.heads)]
    ln_pow, ln_norm = decay_powers(decay).to(dev), torch.ones(lns.out_width, device=dev)
    ln_decay = torch.tensor(decay, dtype=torch.float64)
    gs = GlaShape(d.heads, d.dim, d.vdim, 16)
    a2, a2b, gn = torch.randn(gs.heads * gs.dk, gs.rank8, device=dev), torch.randn(gs.heads * gs.dk, device=dev) + 2, torch.ones(gs.dv, device=dev)
    gated = LatentAttention(LatentShape(H, z["lat_dim"], z["lat_rot"], D, z["kv_rank"], gate=True), lat.scale, 0, 1e-5, lat.cos, lat.sin, dev, torch.bfloat16)
    r_ = lambda *shape: rnd(*shape) * 0.02  # noqa: E731
    gated.load(r_(H * (z["lat_dim"] + z["lat_rot"]), W), r_(z["kv_rank"] + z["lat_rot"], W), torch.ones(z["kv_rank"]), r_(H * z["lat_dim"], z["kv_rank"]),
               r_(H * D, z["kv_rank"]), r_(H * D, W), k_pad=W)
    for B, start, n in ((1, 2047, 1), (8, 2047, 1), (64, 2047, 1), (4, 0, 2048)):
        b, pages = _batch(B, start, n, dev)
        b.state_slots = torch.arange(1, B + 1, device=dev)
        T = B * n
        tag = f"B={B} context 2048" if n == 1 else f"{B} x {n} tokens"
        off = KvCacheSettings(enabled=False)
        # ---- recurrences
        p, pl = rnd(T, lm.mixer.w_in.N), rnd(T, lns.width)
        ring, st = torch.zeros(B + 1, ssd.taps, ssd.conv_width, device=dev), torch.zeros(B + 1, ssd.heads, ssd.dn, ssd.dv, device=dev)
        sl, out = torch.zeros(B + 1, lns.heads, lns.dk, lns.dv, device=dev), torch.empty(T, lns.out_width, dtype=torch.bfloat16, device=dev)
        state, fl = B * ssd.heads * ssd.dn * ssd.dv * 8, 6.0 * T * ssd.heads * ssd.dn * ssd.dv
        add(f"Mamba-2: convolution, recurrence, gate, norm {tag} (against lightning attention)", lambda: mamba2(ssd, p, lm.mixer.w, ring, st, b, 1e-5),
            (state + T * (p.shape[1] + ssd.out_width) * 2, fl), lambda: lop.lightning(lns, pl, ln_decay, ln_pow, ln_norm, sl, b, 1e-5, 1.0, out),
            (state + T * (lns.width + lns.out_width) * 2, fl))
        del st, sl
        pd, pg = rnd(T, px.w_in.N), rnd(T, gs.width)
        ring, st = torch.zeros(B + 1, d.taps, d.conv_width, device=dev), torch.zeros(B + 1, d.heads, d.dk, d.dv, device=dev)
        sg, row = torch.zeros(B + 1, gs.heads, gs.dk, gs.dv, device=dev), torch.empty(T, s.out_width + d.out_width, dtype=torch.bfloat16, device=dev)
        kv = SimpleNamespace(state={"conv": {0: ring}, "delta": {0: st}})
        state, fl = B * d.heads * d.dk * d.dv * 8, 6.0 * T * d.heads * d.dk * d.dv
        add(f"gated delta rule: low-rank projections, convolution, recurrence, norm, gate {tag} (against gated linear attention)",
            lambda: right.heads(pd[:, s.width :], b, kv, 0, row[:, s.out_width :], stage), (state + (right.w_decay.nbytes() + right.w_gate.nbytes()) + T * (d.width + d.out_width) * 2, fl * 4 / 3),
            lambda: gla_op.gla(gs, pg, a2, a2b, gn, sg, b, gs.dim ** -0.5, 16.0, 1e-5), (state + a2.numel() * 4 + T * (gs.width + gs.out_width) * 2, fl))
        del st, sg
        # ---- attention with mixed scores
        kf = PagedKVCache({"layers": 2, "kv_heads": KV, "head_dim": D, "layer_kinds": ["attention"] * 2, "kv_heads_per_layer": [1, KV], "head_dim_per_layer": [s.k_width, D],
                           "v_dim_per_layer": [s.v_width, D]}, pages, dev, torch.bfloat16, off)
        for i in range(2):
            kf.k[i].normal_(), kf.v[i].normal_()
        kc, vc = kf.layer(0)
        kg, vg = kf.layer(1)
        qkv = rnd(T, (H + 2 * KV) * D)
        q = qkv[:, : H * D]
        nw = torch.ones(D, device=dev, dtype=torch.bfloat16)
        pm = pd[:, : s.width]
        add(f"head norms, rotation, cache write {tag}",
            lambda: gop.rope_heads_kv(s, pm, b.positions, b.slots, left.cos, left.sin, kc, vc, left.q_norm, left.k_norm, 1e-5), (T * (H + 2 * KV) * D * 4, 0),
            lambda: ops.rope_kv(qkv, b.positions, b.slots, nw, nw, hyb.cos, hyb.sin, kg, vg, H, KV, D, 1e-5), (T * (H + 2 * KV) * D * 4, 0))
        att = lambda: gop.attention(s, pm, b, kc, vc, left.scale, 0.0, win, 0, None, left._splits(b), 0.6, row[:, : s.out_width], left.mix)  # noqa: E731
        if n == 1:
            span = min(2048, win)
            kvb = B * span * 2 * KV * D * 2 + T * H * D * 4
            add(f"decode attention, mixed scores, head gate {tag}", att, (kvb, 0),
                lambda: ops.decode_attention(q, kg, vg, b.block_tables, b.ctx_len, H, D ** -0.5, 0.0, win, _engine_splits(B, KV)), (kvb, 0))
        else:
            pairs = B * (n * (n + 1) / 2 if win >= n else win * (n - win) + win * (win + 1) / 2)
            add(f"prompt attention, mixed scores, head gate {tag}", att, (0, pairs * H * (4.0 * D + 2.0 * H)),
                lambda: ops.prefill_attention(q, kg, vg, b.block_tables, b.q_start, b.q_len, b.ctx_len, H, D ** -0.5, 0.0, win, True, b.tile_seq, b.tile_q0,
                                              tiles_for=b.tiles), (0, 4.0 * pairs * H * D))
        del kf
        # ---- latent attention (input projection, everything up to the heads)
        kl = PagedKVCache({"layers": 1, "kv_heads": 1, "head_dim": lat.shape.Rp, "layer_kinds": ["latent"], "v_dim_per_layer": [lat.shape.drp]}, pages, dev, torch.bfloat16, off)
        kl.k[0].normal_(), kl.v[0].normal_()
        x, row = rnd(T, W), torch.empty(T, H * D, dtype=torch.bfloat16, device=dev)
        keys = B * 2048 * (z["kv_rank"] + z["lat_rot"]) * 2
        io = lambda m: m.w_in.nbytes() + 2 * H * z["kv_rank"] * (z["lat_dim"] + D) * 2 + T * (W + H * D) * 2  # noqa: E731
        pairs = B * 2048 if n == 1 else B * n * (n + 1) / 2
        work = lambda m: 2.0 * T * m.w_in.N * W + 2.0 * pairs * H * (z["lat_dim"] + z["lat_rot"] + D) + (0 if n == 1 else 2.0 * T * H * z["kv_rank"] * (z["lat_dim"] + D))  # noqa: E731
        for name, m in (("latent attention with a sink", lat), ("latent attention on a shared cache", ls.mixer)):
            add(f"{name} {tag} (against one with a gate)", lambda m=m: m.heads(x, b, kl.layer(0), row, stage), (keys + io(m), work(m)),
                lambda: gated.heads(x, b, kl.layer(0), row, stage), (keys + io(gated), work(gated)))
        del kl
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
    from ..models.gevovik import GevovikModel
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
        gshape, hshape = gevovik_shape(z), hybrid_shape(z)
        gev = GevovikModel(parse_config(gshape), dev, torch.bfloat16).load(SyntheticLoader(gshape, 0, False, dev))
        hyb = DecoderModel(parse_config(hshape), dev, torch.bfloat16).load(SyntheticLoader(hshape, 0, False, dev))
        r = {"shape": z, "weight_bytes": {"gevovik": gev.weight_bytes(), "hybrid": hyb.weight_bytes()}}
        if kernels:
            r["kernels"] = kernel_times(gev, hyb, z, t, peaks)
        r["gevovik"] = {k: round(v, 1) for k, v in throughput(gev, z["vocab"], steps, warmup).items()}
        r["hybrid"] = {k: round(v, 1) for k, v in throughput(hyb, z["vocab"], steps, warmup).items()}
        ops.check_status()
        out["sizes"][name] = r
        del gev, hyb
        torch.cuda.empty_cache()
    return out


def main(args) -> int:
    print(json.dumps(run(args.sizes.split(","), args.steps, args.warmup, not args.no_kernels)))
    return 0
