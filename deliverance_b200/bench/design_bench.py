"""Throughput and kernel times of a latent-attention decoder (Fatotar) beside a GQA decoder of equal size, both bf16 with random weights.

    python bench.py --design fatotar [--sizes small,1b,3b] [--steps K] [--warmup W]

Per size: prefill tokens/s (4 prompts of 2048), decode tokens/s at 1, 8 and 64 sequences (captured step replayed on the device, context
2048), and device times of the kernels of one layer with their roofline fractions (L2 flushed before every timed launch; medians).
The GQA decoder (llama family) has the same width, feed-forward, layer runs, vocabulary and query heads; its head_dim is 128 (64 for the
small size) with one KV head per four query heads; its attention kernels are timed with the same sliding window. Fractions are of the measured copy bandwidth and cuBLAS bf16 burst rate.
"""
from __future__ import annotations

import json
import statistics

import torch

SIZES = {
    "small": dict(width=1024, ff=4096, heads=16, dim=64, rot_dim=32, vdim=64, kv_rank=256, window=1024, layers=8, vocab=32000, gqa_dim=64),
    "1b": dict(width=2048, ff=6144, heads=16, dim=128, rot_dim=64, vdim=128, kv_rank=512, window=4096, layers=8, vocab=32000, gqa_dim=128),
    "3b": dict(width=3072, ff=8192, heads=24, dim=128, rot_dim=64, vdim=128, kv_rank=512, window=1024, layers=8, vocab=32000, gqa_dim=128),
}
YARN = {"factor": 4.0, "original": 4096, "fast": 32.0, "slow": 1.0}


def fatotar_shape(z: dict) -> dict:
    from ..ckpt.tiny import fatotar_config

    layer = {k: z[k] for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank", "window", "ff")}
    layer.update(base=500000.0, scaling=YARN)
    return fatotar_config(z["width"], z["vocab"], [layer] * z["layers"], scale=4.0, bigram={"buckets": 65521, "mul_prev": 8191, "mul_cur": 131},
                          max_position_embeddings=8192)


def gqa_shape(z: dict) -> dict:
    return dict(model_type="llama", vocab_size=z["vocab"], hidden_size=z["width"], intermediate_size=z["ff"], num_hidden_layers=z["layers"],
                num_attention_heads=z["heads"], num_key_value_heads=z["heads"] // 4, head_dim=z["gqa_dim"], max_position_embeddings=8192, rms_norm_eps=1e-5,
                rope_theta=500000.0, tie_word_embeddings=False, hidden_act="silu", bos_token_id=1, eos_token_id=2)


class Timer:
    def __init__(self, dev, steps: int, warmup: int):
        self.flush = torch.empty(256 << 20, dtype=torch.uint8, device=dev)
        self.steps, self.warmup = steps, warmup

    def us(self, fn) -> float:
        for _ in range(self.warmup):
            fn()
        torch.cuda.synchronize()
        times = []
        for _ in range(self.steps):
            self.flush.zero_()
            a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            a.record()
            fn()
            b.record()
            torch.cuda.synchronize()
            times.append(a.elapsed_time(b) * 1e3)
        return statistics.median(times)


def throughput(model, vocab: int, steps: int, warmup: int) -> dict:
    """Prefill and decode tokens/s through the engine."""
    from ..engine.engine import Engine, EngineConfig
    from ..params import GeneratorParameters

    P, out = 2048, {}
    for B in (1, 8, 64):
        econf = EngineConfig(max_batch_tokens=8192, max_seqs=B, num_pages=B * ((P + 3 * (steps + warmup) + 96) // 32) + 8)
        econf.kv.enabled = False
        eng = Engine(model, econf, eos_ids=(-1,))
        g = torch.Generator().manual_seed(B)
        prompts = torch.randint(0, vocab, (B, P), generator=g).tolist()

        def prefill(n):
            reqs = [eng.add_request(p, GeneratorParameters(temperature=0.0)) for p in prompts[:n]]
            torch.cuda.synchronize()
            a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            a.record()
            while any(not r.output for r in reqs):
                eng.step()
            b.record()
            torch.cuda.synchronize()
            return reqs, a.elapsed_time(b)

        if B == 8:  # 4 prompts = one full prefill step; warmed up, then timed on a fresh set
            for _ in range(3):
                reqs, ms = prefill(4)
                for r in reqs:
                    eng.abort(r)
                while eng.has_work():
                    eng.step()
            out["prefill_tok_s"] = 4 * P / ms * 1e3
        prefill(B)
        for _ in range(warmup):
            eng.step()
        torch.cuda.synchronize()
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        a.record()
        for _ in range(steps):
            eng.step()
        b.record()
        torch.cuda.synchronize()
        out[f"decode_tok_s_b{B}_e2e"] = B * steps / a.elapsed_time(b) * 1e3
        gr = eng._graphs[B]
        a.record()
        for _ in range(steps):
            gr["graph"].replay()
            eng._greedy(gr["logits"])
        b.record()
        torch.cuda.synchronize()
        out[f"decode_tok_s_b{B}"] = B * steps / a.elapsed_time(b) * 1e3
        eng._drain()
        eng._graphs.clear()
        del eng
        torch.cuda.empty_cache()
    return out


def _batch(B: int, start: int, n: int, dev):
    from ..models.batch import make_batch

    per = (start + n + 31) // 32
    return make_batch([{"tokens": [1] * n, "start": start, "pages": list(range(1 + i * per, 1 + (i + 1) * per)), "prev": 1} for i in range(B)], 32, dev), B * per + 1


def kernel_times(fat, gqa, z: dict, t: Timer, peaks: dict) -> list:
    """One row per pair of like kernels: microseconds and roofline fraction of both designs."""
    from .. import ops
    from ..kv.paged import KvCacheSettings, PagedKVCache
    from ..ops import latent as lop

    dev = fat.device
    hbm, tf = peaks["hbm_gbs"] * 1e9, peaks["bf16_tflops"] * 1e12
    lw, gl = fat.layers[0], gqa.layers[0]
    mx, s = lw.mixer, lw.mixer.shape
    W, H, D, KV = z["width"], z["heads"], z["gqa_dim"], z["heads"] // 4
    rows = []

    def roof(bytes_, flops):
        return max(bytes_ / hbm, flops / tf) * 1e6

    def add(name, fn_f, cost_f, fn_g, cost_g):
        uf, ug = t.us(fn_f), t.us(fn_g)
        ff, fg = roof(*cost_f) / uf, roof(*cost_g) / ug
        rows.append({"kernel": name, "us": round(uf, 2), "roofline_us": round(roof(*cost_f), 2), "fraction": round(ff, 3), "gqa_us": round(ug, 2),
                     "gqa_roofline_us": round(roof(*cost_g), 2), "gqa_fraction": round(fg, 3), "distance_ratio": round(fg / ff, 2)})

    def gemm(name, M, wf, wg, out_f32=False):
        xf = torch.randn(M, wf.K, device=dev).to(torch.bfloat16)
        xg = torch.randn(M, wg.K, device=dev).to(torch.bfloat16)
        cost = lambda w, ob: (w.N * w.K * 2 + M * w.K * 2 + M * w.N * ob, 2.0 * M * w.N * w.K)  # noqa: E731
        add(f"{name} M={M}", lambda: ops.linear(xf, wf, out_f32=out_f32), cost(wf, 4 if out_f32 else 2), lambda: ops.linear(xg, wg), cost(wg, 2))

    for M in (64, 8192):
        gemm("input projection", M, mx.w_in, gl.qkv)
        gemm("gate|up projection", M, lw.gate_up, gl.gate_up)
        gemm("output projection(s)", M, lw.out, gl.down, out_f32=True)
        res, dl = torch.randn(M, W, device=dev), torch.randn(M, W, device=dev)
        rb, xb = res.to(torch.bfloat16), dl.to(torch.bfloat16)
        add(f"residual + norm(s) M={M}", lambda: ops.add_layernorm(res, dl, lw.norm1, lw.norm2, 1e-5, fat.pitch, torch.bfloat16), (M * W * 16, 0),
            lambda: ops.add_rmsnorm(xb, rb, gl.pre_ff_norm, 1e-5), (M * W * 8, 0))
        gf = torch.randn(M, 2 * lw.ff, device=dev).to(torch.bfloat16)
        gg = torch.randn(M, 2 * z["ff"], device=dev).to(torch.bfloat16)
        of = torch.empty(M, lw.row, dtype=torch.bfloat16, device=dev)
        add(f"activation M={M}", lambda: ops.gated_act_into(gf, "relu", of[:, lw.ff_at :]), (M * lw.ff * 6, 0), lambda: ops.act_mul(gg, "silu"), (M * z["ff"] * 6, 0))

    def caches(model, pages):
        return PagedKVCache(model.kv_layout(), pages, dev, torch.bfloat16, KvCacheSettings(enabled=False))

    for B, start, n in ((1, 2047, 1), (64, 2047, 1), (4, 0, 2048)):
        b, pages = _batch(B, start, n, dev)
        T = B * n
        kf, kg = caches(fat, pages), caches(gqa, pages)
        for i in range(1):
            kf.k[i].normal_(), kf.v[i].normal_(), kg.k[i].normal_(), kg.v[i].normal_()
        p = torch.randn(T, s.width, device=dev).to(torch.bfloat16)
        qkv = torch.randn(T, (H + 2 * KV) * D, device=dev).to(torch.bfloat16)
        row = torch.empty(T, lw.row, dtype=torch.bfloat16, device=dev)
        tag = f"B={B} context 2048" if n == 1 else f"{B} x {n} tokens"
        cf, rf = kf.layer(0)
        cg, vg = kg.layer(0)
        wbytes = s.heads * s.kv_rank * (s.dim + s.vdim) * 2
        q = qkv[:, : H * D]
        if n == 1:
            span = min(2048, z["window"])
            sp = mx._splits(B, 2048)
            gsp = _engine_splits(B, KV)
            args = (mx.wuk, mx.wuv, cf, rf, b.block_tables, row, mx.scale, mx.window, sp, (b.positions, b.slots, mx.norm, mx.cos, mx.sin, cf, rf, 1e-5))
            keyb = B * span * (s.kv_rank + s.rot_dim) * 2
            # absorbed query + rotation, norm and cache write + attention + value expansion and gate (three launches) against attention + merge
            add(f"decode attention {tag}", lambda: lop.rows_attention(s, p, None, None, b.ctx_len, *args),
                (keyb + wbytes + T * H * (s.dim + s.rot_dim + 2 * s.vdim) * 2, 2.0 * B * H * (span * (2 * s.kv_rank + s.rot_dim) + s.kv_rank * (s.dim + s.vdim))),
                lambda: ops.decode_attention(q, cg, vg, b.block_tables, b.ctx_len, H, D ** -0.5, 0.0, z["window"], gsp),
                (B * span * 2 * KV * D * 2 + T * H * D * 4, 0))
        else:
            add(f"rotation, norm, cache write {tag}", lambda: lop.prepare(s, p, b.positions, b.slots, mx.norm, mx.cos, mx.sin, cf, rf, 1e-5),
                (T * (s.kv_rank + s.rot_dim + H * s.rot_dim) * 4, 0),
                lambda: ops.rope_kv(qkv, b.positions, b.slots, None, None, gqa.cos, gqa.sin, cg, vg, H, KV, D, 1e-5), (T * (H + 2 * KV) * D * 4, 0))
            a = mx._plan(b)["prompts"]
            win = z["window"]
            pairs = B * (n * (n + 1) / 2 if win >= n else win * (n - win) + win * (win + 1) / 2)
            c, kr = lop.gather(s, cf, rf, b.block_tables, a["seq"], a["key0"], a["n_keys"], a["row0"], a["max_rows"], a["total"])
            kvx = ops.linear(c, mx.w_expand)
            add(f"prompt attention {tag}", lambda: lop.prefill_attention(s, p, kvx, kr, a["q_start"], a["q_len"], a["n_keys"], a["row0"], a["tile_seq"],
                                                                         a["tile_q0"], row, mx.scale, mx.window),
                (0, 2.0 * pairs * H * (s.dim + s.rot_dim + s.vdim)),
                lambda: ops.prefill_attention(q, cg, vg, b.block_tables, b.q_start, b.q_len, b.ctx_len, H, D ** -0.5, 0.0, win, True, b.tile_seq, b.tile_q0,
                                              tiles_for=b.tiles), (0, 4.0 * pairs * H * D))
            xg = torch.randn(T, W, device=dev).to(torch.bfloat16)
            add(f"key / value expansion {tag} (against the gate|up GEMM)", lambda: ops.linear(c, mx.w_expand),
                (mx.w_expand.N * mx.w_expand.K * 2 + T * (mx.w_expand.N + mx.w_expand.K) * 2, 2.0 * T * s.kv_rank * s.heads * (s.dim + s.vdim)),
                lambda: ops.linear(xg, gl.gate_up), (gl.gate_up.N * W * 2 + T * (gl.gate_up.N + W) * 2, 2.0 * T * gl.gate_up.N * W))
            add(f"gather of cached rows {tag} (against the cache write)",
                lambda: lop.gather(s, cf, rf, b.block_tables, a["seq"], a["key0"], a["n_keys"], a["row0"], a["max_rows"], a["total"]),
                (T * (s.kv_rank + s.rot_dim) * 4, 0),
                lambda: ops.rope_kv(qkv, b.positions, b.slots, None, None, gqa.cos, gqa.sin, cg, vg, H, KV, D, 1e-5), (T * (H + 2 * KV) * D * 4, 0))
    return rows


def _engine_splits(B: int, kv_heads: int) -> int:
    """The engine's split-KV rule (:meth:`Engine._splits`)."""
    from types import SimpleNamespace

    from ..engine.engine import Engine

    return Engine._splits(SimpleNamespace(model=SimpleNamespace(n_kv=kv_heads)), B)


def run(sizes, steps: int, warmup: int, kernels: bool = True) -> dict:
    from .. import ops
    from ..ckpt.synthetic import SyntheticLoader
    from ..config import parse_config
    from ..models.fatotar import FatotarModel
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
        fs, gs = fatotar_shape(z), gqa_shape(z)
        fat = FatotarModel(parse_config(fs), dev, torch.bfloat16).load(SyntheticLoader(fs, 0, False, dev))
        gqa = DecoderModel(parse_config(gs), dev, torch.bfloat16).load(SyntheticLoader(gs, 0, False, dev))
        r = {"shape": z, "weight_bytes": {"fatotar": fat.weight_bytes(), "gqa": gqa.weight_bytes()}}
        if kernels:
            r["kernels"] = kernel_times(fat, gqa, z, t, peaks)
        r["fatotar"] = {k: round(v, 1) for k, v in throughput(fat, z["vocab"], steps, warmup).items()}
        r["gqa"] = {k: round(v, 1) for k, v in throughput(gqa, z["vocab"], steps, warmup).items()}
        ops.check_status()
        out["sizes"][name] = r
        del fat, gqa
        torch.cuda.empty_cache()
    return out


def main(args) -> int:
    print(json.dumps(run(args.sizes.split(","), args.steps, args.warmup, not args.no_kernels)))
    return 0
