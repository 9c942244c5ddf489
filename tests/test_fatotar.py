"""Fatotar decoder against a plain float64 statement of its equations (``fatotar_plain.py``), mechanism by mechanism and through the
engine. Every test runs on the CPU operator set in fp32 and, on a GPU box, on the CUDA kernels in fp32 and in bf16."""
import io
import json
import os

import pytest
import torch

import fatotar_plain as plain
from design_helpers import RUNS, Dict2Loader, _Stage, engine_for, gpu, rel, replay, tokens_of, tol
from deliverance_b200 import ops
from deliverance_b200.ckpt.loader import WeightLoader
from deliverance_b200.ckpt.tiny import build_tensors, fatotar_config, tiny_config, write_tiny_model
from deliverance_b200.config import layer_run_order, load_config, parse_config
from deliverance_b200.kv.paged import KvCacheSettings, PagedKVCache
from deliverance_b200.models.batch import make_batch
from deliverance_b200.models.fatotar import FatotarModel
from deliverance_b200.models.latent import LatentAttention
from deliverance_b200.ops import latent as lop, ref
from deliverance_b200.ops.latent import LatentShape
from deliverance_b200.params import GeneratorParameters

def build(cfg, run, seed=0, tensors=None):
    """(model, weights as the plain statement reads them); bf16 runs get weights that are exact in bf16."""
    device, dtype = run
    W = tensors or build_tensors(cfg, seed, torch.bfloat16)
    return FatotarModel(parse_config(cfg), device, dtype).load(Dict2Loader(W)), W


# --------------------------------------------------------------------------------------------------- single mechanisms
@pytest.mark.parametrize("run", RUNS)
@pytest.mark.parametrize("W,mp,mc,buckets", [(40, 139, 23, 61), (33, 1, 1, 7), (64, 4093, 9001, 1000)])
def test_bigram_embedding(run, W, mp, mc, buckets):
    device, dtype = run
    V, toks = 50000, [49999, 0, 0, 3, 49998, 49999, 49999, 1]
    g = torch.Generator().manual_seed(W)
    table, bigram = torch.randn(V, W, generator=g).to(torch.bfloat16), torch.randn(buckets + 1, W, generator=g).to(torch.bfloat16)
    cfg = {"embedding": {"scale": 1.75, "bigram": {"buckets": buckets, "mul_prev": mp, "mul_cur": mc}}}
    want = plain.embed({"embed": table, "bigram": bigram}, cfg, toks)
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=device)  # noqa: E731
    got = ops.bigram_embedding(table.to(device, dtype), bigram.to(device, dtype), i32(toks), i32([-1] + toks[:-1]), mp, mc, 1.75)
    assert got.dtype == torch.float32 and rel(got, want) < 1e-6  # the residual stream starts in fp32
    # a second sequence that starts with the same token takes the start row again, not the hash of a neighbour in the batch
    got = ops.bigram_embedding(table.to(device, dtype), bigram.to(device, dtype), i32([7, 9, 7]), i32([-1, 7, -1]), mp, mc, 1.0)
    assert torch.equal(got[0], got[2]) and torch.allclose(got[0].cpu(), table[7].float() + bigram[buckets].float())


@pytest.mark.parametrize("run", RUNS)
@pytest.mark.parametrize("W", [8, 92, 257, 1024])
def test_add_layernorm_pair(run, W):
    device, dtype = run
    g = torch.Generator().manual_seed(W)
    r = lambda *s: torch.randn(*s, generator=g)  # noqa: E731
    x, d = r(5, W) * 3 + 40, r(5, W)  # a large common offset: the variance must be the mean of squared deviations
    w1, b1, w2, b2 = r(W), r(W), r(W), r(W)
    pitch = (W + 7) // 8 * 8
    res = x.clone().to(device)
    c = lambda *t: tuple(v.to(device) for v in t)  # noqa: E731
    y1, y2 = ops.add_layernorm(res, d.to(device), c(w1, b1), c(w2, b2), 1e-3, pitch, dtype)
    s = (x + d).double()
    assert torch.allclose(res.cpu(), x + d)
    t = 5e-5 if dtype == torch.float32 else 6e-3
    assert rel(y1[:, :W], plain.layer_norm(s, w1, b1, 1e-3)) < t and rel(y2[:, :W], plain.layer_norm(s, w2, b2, 1e-3)) < t
    assert y1.shape == (5, pitch) and (y1[:, W:] == 0).all()
    y, none = ops.add_layernorm(res, None, c(w1, b1), None, 1e-3, pitch, dtype)
    assert none is None and torch.equal(y, y1) and torch.allclose(res.cpu(), x + d)


@pytest.mark.parametrize("dims,base,scaling", [
    (16, 10000.0, None), (6, 500.0, {"factor": 8.0, "original": 64, "fast": 16.0, "slow": 2.0}), (64, 1e6, {"factor": 40.0, "original": 4096, "fast": 32.0, "slow": 1.0}),
    (10, 100.0, {"factor": 1.0, "original": 128, "fast": 8.0, "slow": 1.0}), (8, 10000.0, {"factor": 2.0, "original": 4, "fast": 64.0, "slow": 32.0})])
def test_yarn_tables(dims, base, scaling):
    freqs, mult = plain.yarn_frequencies(dims, base, scaling)
    cos, sin = ref.yarn_rope_tables(dims, 3000, base, scaling)
    for p in (0, 1, 37, 2999):
        a = torch.tensor([p * f for f in freqs], dtype=torch.float64)
        assert torch.allclose(cos[p].double(), torch.cos(a) * mult, atol=1e-6) and torch.allclose(sin[p].double(), torch.sin(a) * mult, atol=1e-6)
    v = torch.randn(dims + 3, dtype=torch.float64, generator=torch.Generator().manual_seed(1))
    got = ref.apply_rope(v.view(1, 1, -1), torch.tensor([37]), cos, sin)[0, 0]
    assert torch.allclose(got.double(), plain.rotate(v, 37, freqs, mult), atol=1e-5) and torch.equal(got[dims:], v[dims:].float())


def mixer_case(run, H, dn, dr, dv, R, window, width=48, scaling=None, scale=None, seed=0):
    """A latent mixer, its plain-statement arguments and a paged cache with shuffled pages."""
    device, dtype = run
    g = torch.Generator().manual_seed(seed * 7919 + H * 31 + R)
    r = lambda *s, k=1.0: (torch.randn(*s, generator=g) * k).to(torch.bfloat16)  # noqa: E731
    m = {"heads": H, "dim": dn, "rot_dim": dr, "vdim": dv, "kv_rank": R, "mask": {"size": window}, "scale": scale or (dn + dr) ** -0.5,
         "rot": {"base": 700.0, "dims": dr, "scaling": scaling}}
    W = {"q": r(H * (dn + dr), width, k=2 * width ** -0.5), "dkv": r(R + dr, width, k=width ** -0.5), "dkv.norm": 1 + r(R, k=0.2), "uk": r(H * dn, R, k=R ** -0.5),
         "uv": r(H * dv, R, k=R ** -0.5), "g": r(H * dv, width, k=2 * width ** -0.5), "o": torch.eye(H * dv).to(torch.bfloat16)}
    shape = LatentShape(H, dn, dr, dv, R)
    cos, sin = ref.yarn_rope_tables(dr, 4096, 700.0, scaling)
    mixer = LatentAttention(shape, m["scale"], window, 1e-5, cos.to(device), sin.to(device), torch.device(device), dtype)
    mixer.load(*(W[n] for n in ("q", "dkv", "dkv.norm", "uk", "uv", "g")), k_pad=(width + 7) // 8 * 8)
    layout = {"layers": 1, "kv_heads": 1, "head_dim": shape.Rp, "layer_kinds": ["latent"], "head_dim_per_layer": [shape.Rp], "v_dim_per_layer": [shape.drp]}
    kv = PagedKVCache(layout, 96, device, dtype, KvCacheSettings(enabled=False))
    for t in (kv.k[0], kv.v[0]):
        t.uniform_(-3, 3)  # stale rows of earlier owners
    pages = (torch.randperm(95, generator=g) + 1).tolist()
    return mixer, m, W, kv, pages


def run_mixer(mixer, kv, h, portions, pages, run):
    """Feed rows of ``h`` in the given portion sizes; returns the mixer's gated heads."""
    device, dtype = run
    out, at, width = [], 0, h.shape[1]
    pad = (width + 7) // 8 * 8 - width
    for n in portions:
        b = make_batch([{"tokens": [0] * n, "start": at, "pages": pages}], kv.page_size, device)
        y = torch.zeros(n, (mixer.shape.out_width + 7) // 8 * 8, dtype=dtype, device=device)
        mixer.heads(torch.nn.functional.pad(h[at : at + n], (0, pad)).to(device, dtype), b, kv.layer(0), y, lambda _: _Stage())
        out.append(y[:, : mixer.shape.out_width].float().cpu())
        at += n
    return torch.cat(out)


YARN = {"factor": 6.0, "original": 48, "fast": 12.0, "slow": 1.5}
# heads, dim, rot_dim, vdim, kv_rank, window: single heads, odd sizes, more heads than one head group, wide latents, every tensor-core
# width of the prompt kernel (128 / 192 / 256 query columns x 64 / 128 / 256 value columns) and head sizes beyond it
SIZES = [(1, 1, 2, 1, 1, 1), (2, 8, 4, 8, 16, 9), (3, 20, 6, 12, 40, 24), (5, 64, 64, 64, 136, 33), (16, 32, 16, 48, 128, 64), (17, 24, 8, 33, 264, 50),
         (33, 16, 8, 16, 64, 70), (4, 96, 40, 128, 512, 65), (2, 128, 64, 100, 72, 500), (2, 160, 64, 130, 96, 64), (3, 192, 64, 256, 200, 31), (2, 192, 64, 128, 80, 100),
         (2, 260, 20, 24, 48, 40), (2, 40, 12, 300, 56, 40), (1, 16, 16, 16, 1000, 48), (20, 8, 64, 8, 480, 90)]


@pytest.mark.parametrize("run", RUNS)
@pytest.mark.parametrize("H,dn,dr,dv,R,window", SIZES)
def test_latent_attention_sizes(run, H, dn, dr, dv, R, window):
    """Whole prompt, ragged portions and token by token: the same numbers, and those of the plain statement."""
    T = 101
    mixer, m, W, kv, pages = mixer_case(run, H, dn, dr, dv, R, window, scaling=YARN if H % 2 else None)
    h = torch.randn(T, 48, generator=torch.Generator().manual_seed(5)).to(torch.bfloat16)
    want = plain.latent_attention(W, m, "", h.double(), 1e-5)
    for portions in ([T], [2, 3, 37, 2, 30, 27], [90] + [1] * 11):
        assert rel(run_mixer(mixer, kv, h, portions, pages, run), want) < tol(run[1]), portions
        kv.k[0].uniform_(-3, 3), kv.v[0].uniform_(-3, 3)
        pages = pages[::-1]


@pytest.mark.parametrize("run", RUNS)
@pytest.mark.parametrize("window", [1, 2, 31, 32, 33, 64, 96, 130])
def test_window_edges(run, window):
    """One key per query stands out; it sits exactly inside or just outside the window. A window that is one token off moves the output
    by the order of the output itself."""
    T, n = 270, 44
    mixer, m, W, kv, pages = mixer_case(run, 2, 16, 4, 16, 24, window, width=n, scale=0.6)
    g = torch.Generator().manual_seed(window)
    h = torch.randn(T, n, generator=g)
    wq = W["q"].double().reshape(2, 20, n)[0, :16]
    c = plain.rms_norm(h.to(torch.bfloat16).double() @ W["dkv"][:24].double().T, W["dkv.norm"], 1e-5)
    k = c @ W["uk"][:16].double().T
    probes = [t for t in range(window, T, 13)]
    for j, t in enumerate(probes):  # query t points at key t - window + 1 (the last one it sees) or t - window (the first it does not)
        far = t - window + (1 if j % 2 == 0 else 0)
        if window > 1 and far not in probes:
            h[t] += 6.0 * torch.linalg.lstsq(wq, k[far].unsqueeze(1)).solution.squeeze(1).float() / k[far].norm().float()
    h = h.to(torch.bfloat16)
    want = plain.latent_attention(W, m, "", h.double(), 1e-5)
    off = plain.latent_attention(W, dict(m, mask={"size": window + 1}), "", h.double(), 1e-5)
    assert rel(off[probes], want[probes]) > 0.3  # the probes see an edge that is one off
    for portions in ([T], [100, 2, 29, 64, 75], [window + 3] + [1] * (T - window - 3)):
        # (scores in the tens: bf16 rounding of one score moves its weight by several per cent)
        assert rel(run_mixer(mixer, kv, h, portions, pages, run), want) < tol(run[1], bf16=0.1), portions


@pytest.mark.parametrize("run", RUNS)
def test_far_key_at_page_borders(run):
    """A single far key outweighs hundreds of others: keys around page borders, in the first page and at position 0, from prompts and
    from decoded tokens."""
    T, n = 300, 40
    mixer, m, W, kv, pages = mixer_case(run, 1, 24, 4, 24, 32, 1000, width=n, scale=1.0)
    h = torch.randn(T, n, generator=torch.Generator().manual_seed(3))
    wq = W["q"].double()[:24]
    c = plain.rms_norm(h.to(torch.bfloat16).double() @ W["dkv"][:32].double().T, W["dkv.norm"], 1e-5)
    k = c @ W["uk"].double().T
    for j, far in enumerate([0, 1, 31, 32, 33, 63, 64, 95, 127, 128, 150]):
        h[270 + 2 * j] += 10.0 * torch.linalg.lstsq(wq, k[far].unsqueeze(1)).solution.squeeze(1).float() / k[far].norm().float()
    h = h.to(torch.bfloat16)
    want = plain.latent_attention(W, m, "", h.double(), 1e-5)
    for portions in ([T], [260] + [1] * 40, [33, 31, 32, 64, 96, 2, 42]):
        got = run_mixer(mixer, kv, h, portions, pages, run)
        assert rel(got, want) < tol(run[1], 5e-5, 0.1), portions


@pytest.mark.parametrize("run", RUNS)
def test_mixed_rows_and_prompts_in_one_batch(run):
    """Unequal sequences in one batch, short ones row by row and long ones through expanded keys, each as if it were alone."""
    device, dtype = run
    mixer, m, W, kv, pages = mixer_case(run, 3, 20, 6, 12, 40, 24)
    lens, starts = [1, 50, 3, 9, 1, 140, 8], [0, 0, 0, 0, 17, 0, 70]
    hs = [torch.randn(s + n, 48, generator=torch.Generator().manual_seed(100 + i)).to(torch.bfloat16) for i, (s, n) in enumerate(zip(starts, lens))]
    own, at = [], 0
    for s, n in zip(starts, lens):
        k = (s + n + 31) // 32
        own.append(pages[at : at + k])
        at += k
    for h, s, pg in zip(hs, starts, own):
        if s:
            run_mixer(mixer, kv, h, [s], pg, run)
    b = make_batch([{"tokens": [0] * n, "start": s, "pages": pg} for n, s, pg in zip(lens, starts, own)], kv.page_size, device)
    x = torch.cat([h[s:] for h, s in zip(hs, starts)]).to(device, dtype)
    y = torch.zeros(sum(lens), 40, dtype=dtype, device=device)
    mixer.heads(x, b, kv.layer(0), y, lambda _: _Stage())
    row = 0
    for h, s, n in zip(hs, starts, lens):
        want = plain.latent_attention(W, m, "", h.double(), 1e-5)[s:]
        assert rel(y[row : row + n, :36].float(), want) < tol(dtype)
        row += n


@pytest.mark.parametrize("run", RUNS)
def test_relu_feed_forward(run):
    device, dtype = run
    g = torch.Generator().manual_seed(2)
    W = {"gate": torch.randn(52, 32, generator=g) * 0.2, "up": torch.randn(52, 32, generator=g) * 0.2, "down": torch.randn(24, 52, generator=g) * 0.2,
         "gate.b": torch.randn(52, generator=g), "up.b": torch.randn(52, generator=g), "down.b": torch.randn(24, generator=g)}
    W = {k: v.to(torch.bfloat16) for k, v in W.items()}
    x = torch.randn(7, 32, generator=g).to(torch.bfloat16)
    pad = lambda t: torch.nn.functional.pad(t, (0, 0, 0, 4) if t.dim() == 2 else (0, 4))  # noqa: E731
    gu = ops.LinearWeight(torch.cat([pad(W["gate"]), pad(W["up"])]).to(device, dtype), torch.cat([pad(W["gate.b"]), pad(W["up.b"])]).float().to(device))
    row = torch.full((7, 72), float("nan"), dtype=dtype, device=device)
    ops.gated_act_into(ops.linear(x.to(device, dtype), gu), "relu", row[:, 16:])
    assert torch.isnan(row[:, :16]).all() and (row[:, 16 + 52 :] == 0).all()
    down = ops.LinearWeight(torch.nn.functional.pad(W["down"], (0, 4)).to(device, dtype), W["down.b"].float().to(device))
    got = ops.linear(row[:, 16:], down, out_f32=True)
    assert got.dtype == torch.float32 and rel(got, plain.feed_forward(W, "", x.double())) < tol(dtype, 1e-5, 1e-2)


@gpu
@pytest.mark.parametrize("M,N,K", [(1, 1, 8), (3, 70, 33), (130, 257, 96), (64, 64, 16)])
def test_linear_f32_is_true_fp32(M, N, K):
    g = torch.Generator().manual_seed(M)
    x, w, b = torch.randn(M, K, generator=g), torch.randn(N, K, generator=g), torch.randn(N, generator=g)
    got = ops.linear(x.cuda(), ops.LinearWeight(w.cuda(), b.cuda()))
    want = x.double() @ w.double().T + b.double()
    assert (got.cpu().double() - want).abs().max().item() < 1e-6 * K ** 0.5 * 8


def test_layer_order_and_config_errors():
    assert layer_run_order(4, None) == (0, 1, 2, 3)
    assert layer_run_order(5, {"start": 1, "stop": 3, "times": 3}) == (0, 1, 2, 1, 2, 1, 2, 3, 4) == tuple(
        plain.layer_order({"layers": [0] * 5, "loop": {"start": 1, "stop": 3, "times": 3}}))
    assert layer_run_order(2, {"start": 0, "stop": 2, "times": 1}) == (0, 1)
    with pytest.raises(ValueError, match="loop"):
        layer_run_order(2, {"start": 1, "stop": 3, "times": 2})
    cfg = tiny_config("fatotar")
    bad = json.loads(json.dumps(cfg))
    bad["layers"][0]["type"] = "something_else"
    with pytest.raises(ValueError, match="unknown mixer"):
        parse_config(bad)
    bad = json.loads(json.dumps(cfg))
    bad["layers"][0]["mlp"]["kind"] = "sparse"
    with pytest.raises(ValueError, match="unknown feed-forward"):
        parse_config(bad)
    with pytest.raises(ValueError, match="unsupported"):
        parse_config({"architecture": "nobody"})
    from deliverance_b200.parallel.context import TensorParallelContext

    with pytest.raises(ValueError, match="tensor parallelism"):
        FatotarModel(parse_config(cfg), "cpu", None, TensorParallelContext(0, 2, object()))
    t = build_tensors(cfg)
    with pytest.raises(ValueError, match="rows"):
        build(cfg, ("cpu", torch.float32), tensors=dict(t, **{"l0.mix.uk": t["l0.mix.uk"][:-1]}))


# --------------------------------------------------------------------------------------------------- whole models
def variety():
    """Configurations that differ in every size, in layer order and loop, in the presence of feed-forwards and of YaRN."""
    a = dict(heads=3, dim=20, rot_dim=6, vdim=12, kv_rank=40, window=24, ff=52)
    yarn = {"factor": 8.0, "original": 64, "fast": 16.0, "slow": 2.0}
    return {
        "tiny": tiny_config("fatotar"),
        "one-layer": fatotar_config(40, 97, [dict(a, heads=1, vdim=8, ff=24)], scale=1.0, bigram={"buckets": 1, "mul_prev": 1, "mul_cur": 1}),
        "looped-middle": fatotar_config(72, 333, [dict(a), dict(a, heads=2, window=7, scaling=yarn, base=3000.0, ff=16), dict(a, ff=0, dim=64, rot_dim=8),
                                                 dict(a, kv_rank=24, window=200)], loop={"start": 1, "stop": 3, "times": 3}, eps=1e-3,
                                        bigram={"buckets": 97, "mul_prev": 1009, "mul_cur": 3}),
        "wide-heads": fatotar_config(128, 512, [dict(heads=4, dim=64, rot_dim=32, vdim=72, kv_rank=96, window=33, ff=192, scaling=yarn)] * 2),
    }


@pytest.mark.parametrize("run", RUNS)
@pytest.mark.parametrize("name", list(variety()))
def test_model_portions_batches_and_reused_pages(run, name):
    """Whole prompts, decoding, portions down to two tokens and mixed batches in a pool so small that pages are used again; logits of every
    position against the plain statement, and the residual stream after every layer run for one prompt."""
    cfg = variety()[name]
    model, W = build(cfg, run, seed=3)
    V = cfg["vocab"]
    req = {f"r{i}": tokens_of(n, V, 10 + i) for i, n in enumerate((150, 97, 34, 1, 66, 23))}
    want = {k: plain.forward(W, cfg, t) for k, t in req.items()}
    t = tol(run[1], 5e-5, 4e-2)
    stream = []
    model.layer_hook = lambda i, stage, x: stream.append(x.float().cpu()) if stage == "out" else None
    eng = engine_for(model, 192, max_seqs=4)
    got = replay(eng, [[(k, len(v))] for k, v in req.items()], req)
    model.layer_hook = None
    for k in req:
        assert rel(got[k], want[k]) < t, k
    _, layers = plain.forward(W, cfg, req["r0"], want_layers=True)
    for i, w in enumerate(layers):
        assert rel(stream[i], w) < t, i
    decode = [[(k, max(1, len(v) - 20))] for k, v in req.items()]
    plan = []
    for (step,), k in zip(decode, req):
        plan += [[step]] + [[(k, 1)]] * (len(req[k]) - step[1])
    for k, v in replay(eng, plan, req).items():
        assert rel(v, want[k]) < t, k
    # portions of changing size, several requests live at once, places and pages handed on
    sizes, at, live, plan, n = [2, 17, 2, 31, 1, 33, 5, 2, 64, 3], dict.fromkeys(req, 0), [], [], 0
    waiting = list(req)
    while waiting or live:
        while waiting and len(live) < 3 and sum(-(-len(req[k]) // 32) for k in live + waiting[:1]) <= 6:
            live.append(waiting.pop(0))
        step = []
        for k in live:
            n += 1
            c = min(sizes[n % len(sizes)], len(req[k]) - at[k])
            at[k] += c
            step.append((k, c))
        plan.append(step)
        live = [k for k in live if at[k] < len(req[k])]
    for k, v in replay(eng, plan, req).items():
        assert rel(v, want[k]) < t, k
    assert eng.kv.allocator.available() == eng.kv.num_pages - 1
    eng.kv.audit([])


@pytest.mark.parametrize("run", RUNS)
def test_long_decoding(run):
    """Several hundred decoded tokens, far beyond every window and the YaRN context."""
    cfg = fatotar_config(32, 64, [dict(heads=2, dim=8, rot_dim=4, vdim=8, kv_rank=16, window=40, ff=16, scaling=YARN)], loop={"start": 0, "stop": 1, "times": 2})
    model, W = build(cfg, run, seed=9)
    req = {"a": tokens_of(330, 64, 1)}
    got = replay(engine_for(model, 384), [[("a", 3)]] + [[("a", 1)]] * 327, req)["a"]
    assert rel(got, plain.forward(W, cfg, req["a"])) < tol(run[1], 5e-5, 4e-2)


def check_greedy(W, cfg, prompt, produced, dtype):
    """Every produced token is the plain statement's best continuation of what came before it (bf16: the best or a near-tie)."""
    lo = plain.forward(W, cfg, prompt + produced[:-1])[len(prompt) - 1 :]
    if dtype == torch.float32:
        assert produced == lo.argmax(-1).tolist()
    else:
        picked = lo[torch.arange(len(produced)), torch.tensor(produced)]
        assert ((lo.max(-1).values - picked) < 0.1 * lo.std()).all()


@pytest.mark.parametrize("run", RUNS)
@pytest.mark.parametrize("how", ["plain", "small-chunks", "preempted", "no-lookahead", "interleaved"])
def test_greedy_generation_through_the_scheduler(run, how):
    """Unequal prompts generated together: the tokens of the plain statement, whatever the scheduler does with them."""
    cfg = tiny_config("fatotar", width=48)
    model, W = build(cfg, run, seed=4)
    prompts = [tokens_of(n, cfg["vocab"], 40 + n) for n in ((31, 1, 63, 30) if how == "preempted" else (37, 1, 70, 12))]
    kw = {"plain": {}, "small-chunks": {"max_batch_tokens": 16}, "preempted": {}, "no-lookahead": {"lookahead": False, "cuda_graphs": False},
          "interleaved": {"max_batch_tokens": 24, "decode_interleave": 1}}[how]
    if run[0] == "cpu" and how == "plain":
        kw["lookahead"] = "force"
    eng = engine_for(model, 192 if how == "preempted" else 1024, kv=KvCacheSettings(), **kw)
    outs = eng.generate_batch(prompts, GeneratorParameters(max_tokens=14, temperature=0.0))
    if how == "preempted":
        assert eng.metrics.get("preemptions", 0) > 0
    for p, r in zip(prompts, outs):
        check_greedy(W, cfg, p, r.token_ids, run[1])
    # prefix cache: the same prompt again continues from cached pages (its last token or the tail replayed), same tokens
    hit = eng.generate(prompts[2], GeneratorParameters(max_tokens=14, temperature=0.0))
    assert (hit.prefix_hit_tokens > 0 or how == "preempted") and (run[1] != torch.float32 or hit.token_ids == outs[2].token_ids)


def test_generation_through_the_public_loader_and_server_registry(tmp_path):
    """``config.json`` + safetensors in a directory, loaded and generated from the way every other family is."""
    from deliverance_b200.api import AutoModelForCausalLM
    from deliverance_b200.model_support import detect_model, load_model

    d = str(tmp_path / "m")
    cfg = write_tiny_model(d, "fatotar", seed=6, dtype=torch.bfloat16, sharded=True)
    assert detect_model(d) == "fatotar" and load_config(d).model_type == "fatotar"
    W = {n: WeightLoader(d).load(n) for n in WeightLoader(d).names()}
    prompt = tokens_of(20, 256, 8)
    clm = AutoModelForCausalLM.new_builder(d).with_device("cpu").build()
    p = GeneratorParameters(max_tokens=8, temperature=0.0)
    check_greedy(W, cfg, prompt, clm.generate(prompt, p).token_ids, torch.float32)
    seeded = GeneratorParameters(max_tokens=8, temperature=0.8, top_k=20, top_p=0.9, seed=3)
    a = clm.generate(prompt, seeded)
    assert load_model(d, device="cpu").generate(prompt, GeneratorParameters(max_tokens=8, temperature=0.8, top_k=20, top_p=0.9, seed=3)).token_ids == a.token_ids
    with pytest.raises(ValueError, match="LoRA"):
        clm.model.set_lora(object())


def test_latent_cache_snapshots(tmp_path):
    """Disk tier and snapshot codecs of a cache whose two halves differ in width."""
    from deliverance_b200.kv.turboquant import restore_pages, snapshot_pages

    model, _ = build(tiny_config("fatotar"), ("cpu", torch.float32))
    kv = engine_for(model).kv
    for i in range(len(kv.k)):
        kv.k[i].normal_(), kv.v[i].normal_()
    for comp, t in (("NONE", 0), ("LZ4", 0), ("MSE_TURBOQUANT", 0.2)):
        before = [(kv.k[i][[3, 5]].clone(), kv.v[i][[3, 5]].clone()) for i in range(len(kv.k))]
        snap = snapshot_pages(kv, [3, 5], 64, comp, 4)
        restore_pages(kv, snap, [7, 9])
        for i, (k, v) in enumerate(before):
            assert rel(kv.k[i][[7, 9]].flatten(0, 2), k.flatten(0, 2)) <= t and rel(kv.v[i][[7, 9]].flatten(0, 2), v.flatten(0, 2)) <= max(t, 2 * t)
    assert PagedKVCache.bytes_per_page(kv.layout, 32, torch.float32) == sum(4 * 32 * (k.shape[-1] + v.shape[-1]) for k, v in zip(kv.k, kv.v))


def test_disk_prefix_tier_keeps_the_output(tmp_path):
    cfg = tiny_config("fatotar", width=48)
    model, _ = build(cfg, ("cpu", torch.float32), seed=2)
    eng = engine_for(model, 1024, kv=KvCacheSettings(max_entries=1))
    eng.kv.attach_disk(str(tmp_path), "LZ4")
    p = [tokens_of(80, cfg["vocab"], s) for s in (1, 2)]
    par = lambda: GeneratorParameters(max_tokens=6, temperature=0.0)  # noqa: E731
    first = eng.generate(p[0], par()).token_ids
    eng.generate(p[1], par())
    again = eng.generate(p[0], par())
    assert again.token_ids == first and again.prefix_hit_tokens > 0 and eng.kv.prefix.disk.metrics["disk_hits"] > 0


# --------------------------------------------------------------------------------------------------- trace replay program
@pytest.mark.parametrize("run", RUNS)
def test_trace_replay_program(run, tmp_path, monkeypatch, capsys):
    """Steps on standard input, logits files and ``done`` lines out; a finished request's pages serve the next one."""
    from deliverance_b200.engine import replay as prog

    device, dtype = run
    d, out = str(tmp_path / "m"), str(tmp_path / "out")
    cfg = write_tiny_model(d, "fatotar", seed=1, dtype=torch.bfloat16)
    W = {n: WeightLoader(d).load(n) for n in WeightLoader(d).names()}
    a, b, c = (tokens_of(n, cfg["vocab"], n) for n in (60, 40, 61))
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:57], "want": [0, 56]}, {"id": "b", "tokens": b[:2], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": b[2:39], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "b", "tokens": b[39:], "want": [0]}, {"id": "a", "tokens": a[57:58], "want": []}], "end": ["b"]},
             {"step": 5, "entries": [{"id": "a", "tokens": a[58:], "want": [1, 0]}], "end": ["a"]},
             {"step": 6, "entries": [{"id": "c", "tokens": c, "want": [60]}], "end": ["c"]}]
    monkeypatch.setattr("sys.stdin", io.StringIO("".join(json.dumps(s) + "\n" for s in steps)))
    name = "float32" if dtype == torch.float32 else "bfloat16"
    assert prog.main(["--model", d, "--dtype", name, "--out", out, "--max-tokens", "128", "--device", device]) == 0
    lines = [ln for ln in capsys.readouterr().out.splitlines() if ln.startswith("done")]
    assert lines == ["done 0", "done 1", "done 2", "done 5", "done 6"]
    assert sorted(os.listdir(out)) == ["0.f32", "2.f32", "5.f32", "6.f32"]
    wa, wb, wc = (plain.forward(W, cfg, t) for t in (a, b, c))
    load = lambda s: torch.frombuffer(bytearray(open(os.path.join(out, f"{s}.f32"), "rb").read()), dtype=torch.float32).view(-1, cfg["vocab"])  # noqa: E731
    for s, want in ((0, wa[[0, 56]]), (2, wb[[39]]), (5, wa[[59, 58]]), (6, wc[[60]])):
        assert load(s).shape == want.shape and rel(load(s), want) < tol(dtype, 5e-5, 4e-2)


def test_replay_and_generation_do_not_mix():
    model, _ = build(tiny_config("fatotar"), ("cpu", torch.float32))
    eng = engine_for(model, 256, max_seqs=1)
    r = eng.open_replay()
    with pytest.raises(MemoryError):
        eng.open_replay()
    with pytest.raises(RuntimeError, match="replay"):
        eng.add_request([1, 2, 3])
    for bad in ([(r, [], [])], [(r, [10 ** 6], [])], [(r, [1, 2], [2])]):
        with pytest.raises(ValueError):
            eng.replay_step(bad)
    assert eng.replay_step([(r, [1, 2], [])]) is None
    eng.close_replay(r)
    eng.add_request([1, 2, 3], GeneratorParameters(max_tokens=2))
    with pytest.raises(RuntimeError, match="replay"):
        eng.open_replay()
    eng.run()


@gpu
def test_the_row_form_and_the_expanded_form_agree_on_cuda():
    """The same prompt through the tensor-core prompt kernel and, with its weights withheld, row by row: two evaluation orders, one result;
    no kernel writes outside its outputs."""
    run = ("cuda", torch.bfloat16)
    ops.set_bounds_check(True)
    try:
        for H, dn, dr, dv, R, window in ((16, 128, 64, 128, 512, 300), (4, 40, 16, 72, 112, 90), (2, 192, 64, 256, 256, 64)):
            mixer, m, W, kv, pages = mixer_case(run, H, dn, dr, dv, R, window)
            assert mixer.w_expand is not None
            h = torch.randn(700, 48, generator=torch.Generator().manual_seed(5)).to(torch.bfloat16)
            a = run_mixer(mixer, kv, h, [256, 444], pages, run)
            mixer.w_expand = None
            b = run_mixer(mixer, kv, h, [256, 444], pages[::-1], run)
            assert rel(a, b) < 2e-2
            ops.check_guards()
            ops.check_status()
    finally:
        ops.set_bounds_check(False)


@gpu
def test_groups_of_16_heads_give_the_same_decode_result():
    """More than 16 heads per CTA (the default) and groups of 16, with one cluster per row and with several."""
    run = ("cuda", torch.bfloat16)
    mixer, m, W, kv, pages = mixer_case(run, 24, 32, 16, 24, 320, 900)
    h = torch.randn(700, 48, generator=torch.Generator().manual_seed(6)).to(torch.bfloat16)
    want = plain.latent_attention(W, m, "", h.double(), 1e-5)[697:]
    s, ext = mixer.shape, ops.require_ext()
    run_mixer(mixer, kv, h[:697], [697], pages, run)
    for groups in (0, 1):
        ext.latent_head_groups(groups)
        try:
            for splits in (1, 2, 8, 32):
                mixer._splits = lambda rows, span: splits  # noqa: B023
                out = []
                for t in range(697, 700):
                    b = make_batch([{"tokens": [0], "start": t, "pages": pages}], kv.page_size, "cuda")
                    y = torch.zeros(1, s.out_width, dtype=torch.bfloat16, device="cuda")
                    mixer.heads(h[t : t + 1].cuda(), b, kv.layer(0), y, lambda _: _Stage())
                    out.append(y.float().cpu())
                assert rel(torch.cat(out), want) < tol(torch.bfloat16), (groups, splits)
        finally:
            ext.latent_head_groups(0)
