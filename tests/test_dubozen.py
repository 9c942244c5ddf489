"""Dubozen decoder against a plain float64 statement of its equations (``dubozen_plain.py``), mechanism by mechanism and through the
engine. Every test runs on the CPU operator set in fp32 and, on a GPU box, on the CUDA kernels in fp32 and in bf16."""
import copy
import io
import json
import os

import pytest
import torch

import dubozen_plain as plain
from design_helpers import RUNS, Dict2Loader, _Stage, engine_for, gpu, rel, replay, tokens_of, tol
from deliverance_b200 import ops
from deliverance_b200.ckpt.loader import WeightLoader
from deliverance_b200.ckpt.tiny import build_tensors, dubozen_config, tiny_config, write_tiny_model
from deliverance_b200.config import load_config, parse_config
from deliverance_b200.kv.paged import KvCacheSettings, PagedKVCache
from deliverance_b200.models.batch import make_batch
from deliverance_b200.models.dubozen import DubozenModel
from deliverance_b200.models.feed_forward import GatedFeedForward
from deliverance_b200.models.grouped import GroupedAttention
from deliverance_b200.models.lightning import LightningAttention
from deliverance_b200.models.moe import RoutedExperts
from deliverance_b200.models.side_by_side import SideBySideMixer
from deliverance_b200.ops import ref
from deliverance_b200.ops.grouped import GroupedShape, up8
from deliverance_b200.ops.lightning import CHUNK, LightningShape, decay_powers
from deliverance_b200.params import GeneratorParameters

F32, BF16 = torch.float32, torch.bfloat16
EPS = 1e-5


def gen(seed):
    return torch.Generator().manual_seed(seed)


def randn(g, *s, k=1.0):
    return (torch.randn(*s, generator=g) * k).to(BF16)


def rows_rel(got, want):
    """Per-row RMS error over the RMS of the expected values."""
    got, want = got.detach().double().cpu(), want.double()
    return (got - want).pow(2).mean(-1).sqrt() / want.pow(2).mean().sqrt().clamp_min(1e-12)


def close_model(got, want, dtype, what=None):
    """Every row in fp32. In bf16 a token whose expert scores are within rounding of each other may take another expert: nine rows of ten
    must be close, and no row may be of another order."""
    e = rows_rel(got, want)
    if dtype == F32:
        assert e.max() < 1e-4, (what, e.max())
    else:
        assert e.quantile(0.9) < 6e-2 and e.max() < 0.6, (what, e.quantile(0.9), e.max())


def build(cfg, run, seed=0, tensors=None):
    device, dtype = run
    W = tensors or build_tensors(cfg, seed, BF16)
    return DubozenModel(parse_config(cfg), device, dtype).load(Dict2Loader(W)), W


# --------------------------------------------------------------------------------------------------- streams
@pytest.mark.parametrize("run", RUNS)
@pytest.mark.parametrize("W,S", [(8, 1), (76, 2), (257, 3), (1024, 4), (1600, 2), (600, 7), (5000, 2), (40, 16)])
def test_stream_steps(run, W, S):
    """Open, write back + read, with one row per token and with expert rows; the streams all come from the old ones."""
    device, dtype = run
    g = gen(W + S)
    T, pitch, V, eps = 5, up8(W), 11, 1e-3
    r = lambda *s: torch.randn(*s, generator=g)  # noqa: E731
    dev = lambda t: t.to(device)  # noqa: E731
    t = tol(dtype, 2e-5, 6e-3)
    table, ids = (r(V, W) + 20).to(BF16), torch.randint(0, V, (T,), generator=g)  # a large common offset: variances are means of squared deviations
    w0, w1 = 1 + 0.3 * r(W), 1 + 0.3 * r(W)
    read, write, mix = r(S), r(S), torch.eye(S) + 0.3 * r(S, S)  # (not symmetric: from and to must not be exchanged)
    x0 = plain.layer_norm(table[ids].double(), w0, eps)
    X, y = ops.stream_open(table.to(device, dtype), dev(ids.int()), dev(w0), S, dev(read), dev(w1), eps, pitch, dtype)
    want = torch.stack([x0] * S, dim=1)
    assert rel(X.flatten(1), want.flatten(1)) < 2e-5
    assert rel(y[:, :W], plain.layer_norm(plain.read_streams(want, read.double()), w1, eps)) < 10 * t and (y[:, W:] == 0).all()  # (read sums may nearly cancel)
    start = r(T, S, W) * 3
    sub = r(T, pitch).to(BF16)
    new = plain.write_streams(start.double(), sub[:, :W].double(), mix.double(), write.double())
    X = dev(start.clone())
    y = ops.stream_step(X, sub.to(device, dtype), dev(mix), dev(write), dev(read), dev(w1), eps, pitch, dtype)
    assert rel(X.flatten(1), new.flatten(1)) < 1e-5 and rel(y[:, :W], plain.layer_norm(plain.read_streams(new, read), w1, eps)) < t and y.shape == (T, pitch)
    assert (y[:, W:] == 0).all()
    # nothing reads the streams again: they need not be written; the sum of the streams, with and without a norm; nothing to write back
    X = dev(start.clone())
    y = ops.stream_step(X, sub.to(device, dtype), dev(mix), dev(write), None, dev(w1), eps, pitch, dtype, keep=False)
    assert rel(y[:, :W], plain.layer_norm(new.sum(1), w1, eps)) < t
    y = ops.stream_step(dev(start.clone()), sub.to(device, dtype), dev(mix), dev(write), None, None, eps, pitch, dtype)
    assert rel(y[:, :W], new.sum(1)) < t
    y = ops.stream_step(dev(start.clone()), None, None, None, dev(read), dev(w1), eps, pitch, dtype)
    assert rel(y[:, :W], plain.layer_norm(plain.read_streams(start.double(), read), w1, eps)) < t
    # expert rows: the weighted sum is part of the step
    k = 3
    ys, pos, w = r(T * k, pitch).to(BF16), torch.randperm(T * k, generator=g).to(torch.int32).reshape(T, k), r(T, k).abs()
    f = (ys[pos.long()].double() * w.double().unsqueeze(-1)).sum(1)[:, :W]
    new = plain.write_streams(start.double(), f, mix.double(), write.double())
    X = dev(start.clone())
    y = ops.stream_step(X, ops.Routed(ys.to(device, dtype), dev(pos), dev(w)), dev(mix), dev(write), dev(read), dev(w1), eps, pitch, dtype)
    assert rel(X.flatten(1), new.flatten(1)) < 2e-5 and rel(y[:, :W], plain.layer_norm(plain.read_streams(new, read), w1, eps)) < t


# --------------------------------------------------------------------------------------------------- rotation, feed-forwards
@pytest.mark.parametrize("dims,base,extra", [(16, 10000.0, 0), (6, 300.0, 5), (64, 5e5, 32), (2, 100.0, 1), (24, 5e4, 0)])
def test_half_rotation(dims, base, extra):
    cos, sin = ref.rope_tables(dims, 3000, base)
    v = torch.randn(dims + extra, dtype=torch.float64, generator=gen(1))
    for p in (0, 1, 37, 2999):
        got = ref.apply_rope(v.view(1, 1, -1), torch.tensor([p]), cos, sin)[0, 0]
        assert torch.allclose(got.double(), plain.rotate_halves(v, p, dims, base), atol=1e-5) and torch.allclose(got[dims:].double(), v[dims:])


@pytest.mark.parametrize("run", RUNS)
@pytest.mark.parametrize("ff,width,T", [(64, 48, 33), (1, 40, 7), (36, 76, 150), (20, 257, 1)])
def test_dense_feed_forward(run, ff, width, T):
    device, dtype = run
    g = gen(ff)
    W = {"gate": randn(g, ff, width, k=2 * width ** -0.5), "up": randn(g, ff, width, k=width ** -0.5), "down": randn(g, width, ff, k=ff ** -0.5)}
    h = randn(g, T, width)
    block = GatedFeedForward("gelu_pytorch_tanh").load(*(W[n].to(dtype) for n in ("gate", "up", "down")), ff, up8(width), torch.device(device), dtype)
    got = block.forward(torch.nn.functional.pad(h, (0, up8(width) - width)).to(device, dtype), lambda _: _Stage())
    assert rel(got, plain.dense(W, "", h.double())) < tol(dtype, 1e-5, 3e-2)


ROUTES = [(8, 3, 2, 1, 33), (16, 4, 4, 2, 150), (5, 5, 1, 1, 7), (12, 1, 6, 3, 40), (6, 2, 6, 4, 20), (128, 8, 8, 3, 60), (64, 2, 64, 40, 9), (3, 1, 1, 1, 1), (10, 2, 5, 5, 700)]


@pytest.mark.parametrize("run", RUNS)
@pytest.mark.parametrize("E,top,groups,keep,T", ROUTES)
def test_group_limited_sigmoid_routing(run, E, top, groups, keep, T):
    """Choice and weights alone: corrections that overturn the order, negative choice scores, groups of one expert, all groups kept."""
    device, _ = run
    g = gen(E * 100 + T)
    z = torch.randn(T, E, generator=g) * 2
    corr = torch.randn(E, generator=g) * 0.6 - 1.5
    rt = {"top": top, "groups": {"count": groups, "keep": keep}, "scale": 2.5}
    want = [plain.route(row, corr.double(), rt) for row in z.double()]
    w_all = torch.zeros(T, E, dtype=torch.float64)
    for t, (idx, w) in enumerate(want):
        w_all[t, idx] = w
    if device == "cpu":
        w, idx = ref.moe_route(z, top, "sigmoid_topk", False, corr, groups, keep, 2.5)
        outs = [(w, idx)]
    else:
        e = ops.require_ext()
        rules = {"correction": corr.to(device), "groups": groups, "keep": keep, "scale": 2.5}
        many = e.moe_route(z.to(device), top, 2, False, **rules)
        outs = [(many[0], many[1])]
        one = e.moe_route_items(z.to(device), top, 2, False, 0, E, 16, T * top, **rules)
        if one:
            outs.append((one[0], one[1]))
    for w, idx in outs:
        got = torch.zeros(T, E, dtype=torch.float64).scatter_(1, idx.long().cpu(), w.double().cpu())
        assert (got - w_all).abs().max() < 1e-5
    assert torch.allclose(w_all.sum(1), torch.full((T,), 2.5, dtype=torch.float64))
    if E == 16:
        flat = [plain.route(row, corr.double(), dict(rt, groups=None))[0] for row in z.double()]
        plainly = [plain.route(row, torch.zeros(E, dtype=torch.float64), rt)[0] for row in z.double()]
        assert sum(set(a) != set(b[0]) for a, b in zip(flat, want)) > T // 4 and sum(set(a) != set(b[0]) for a, b in zip(plainly, want)) > T // 4


@pytest.mark.parametrize("run", RUNS)
@pytest.mark.parametrize("E,top,groups,keep,ff,width,T", [(8, 3, 2, 1, 64, 48, 33), (5, 2, 1, 1, 20, 40, 7), (12, 4, 4, 2, 36, 76, 150), (128, 4, 8, 4, 8, 32, 40), (4, 2, 2, 2, 1, 24, 1)])
def test_routed_experts(run, E, top, groups, keep, ff, width, T):
    device, dtype = run
    g = gen(E * 100 + T)
    W = {"router": randn(g, E, width, k=2.0 * width ** -0.5), "correction": randn(g, E, k=0.4) - 1.5}
    for e in range(E):
        W.update({f"e{e}.gate": randn(g, ff, width, k=width ** -0.5), f"e{e}.up": randn(g, ff, width, k=width ** -0.5), f"e{e}.down": randn(g, width, ff, k=ff ** -0.5)})
    h = randn(g, T, width)
    moe = RoutedExperts(E, top, mode="sigmoid_topk", groups=groups, keep=keep, scale=1.7)
    moe.load(W["router"].to(dtype), (tuple(W[f"e{e}.{n}"].to(dtype) for n in ("gate", "up", "down")) for e in range(E)), ff, up8(width), torch.device(device), dtype,
             W["correction"].float())
    got = moe.forward(torch.nn.functional.pad(h, (0, up8(width) - width)).to(device, dtype), lambda _: _Stage()).dense()[:, :width]
    want = plain.moe(W, {"router": {"top": top, "groups": {"count": groups, "keep": keep}, "scale": 1.7}}, "", h.double())
    assert rel(got, want) < tol(dtype, 1e-5, 3e-2)  # (the router reads the same bf16 rows in both: no close call differs)


# --------------------------------------------------------------------------------------------------- mixers
def cache_for(mixer, run, slots=3, pages=96, seed=0):
    device, dtype = run
    c = mixer.cache_layout()
    layout = {"layers": 1, "kv_heads": c["heads"], "head_dim": c["k"], "layer_kinds": [mixer.kind], "v_dim_per_layer": [c["v"]], "state_shapes": [c["state"]], "paged": [True]}
    kv = PagedKVCache(layout, pages, device, dtype, KvCacheSettings(enabled=False), slots)
    for t in (kv.k[0], kv.v[0]):
        t.uniform_(-3, 3)  # stale rows and states of earlier owners
    for layers in kv.state.values():
        layers[0].uniform_(-3, 3)
    return kv, (torch.randperm(pages - 1, generator=gen(seed)) + 1).tolist()


def attention_case(run, H, G, dk, dv, rot=None, scale=None, width=48, seed=0, v_mix=False, base=700.0):
    device, dtype = run
    g = gen(seed * 7919 + H * 31 + dk)
    rot = dk // 2 * 2 if rot is None else rot
    m = {"heads": H, "kv_heads": G, "dim": dk, "vdim": dv, "scale": scale or dk ** -0.5, "rot": {"base": base, "dims": rot}, "v_mix": v_mix}
    W = {"q": randn(g, H * dk, width, k=2 * width ** -0.5), "k": randn(g, G * dk, width, k=width ** -0.5), "v": randn(g, G * dv, width, k=width ** -0.5),
         "g": randn(g, H * dv, width, k=2 * width ** -0.5), "sink": torch.linspace(-2, 4, H).to(BF16), "o": torch.eye(H * dv).to(BF16), "vmix": torch.tensor(0.625).to(BF16)}
    cos, sin = ref.rope_tables(rot, 4096, base)
    mixer = GroupedAttention(GroupedShape(H, G, dk, dv, gate="columns"), m["scale"], 0.0, 0, 0, True, cos.to(device), sin.to(device), torch.device(device), dtype,
                             rotate="halves", v_mix=v_mix)
    mixer.load(*(W[n] for n in ("q", "k", "v", "o")), k_pad=up8(width), g=W["g"], sink=W["sink"], vmix=W["vmix"].item())
    return (mixer, m, W) + cache_for(mixer, run)


def parallel_case(run, H, G, dim, R, rk, rv, decay, rot=None, scale=None, width=48, seed=0, ls=0.75, rs=0.5, base=700.0):
    device, dtype = run
    g = gen(seed * 7919 + H * 31 + dim)
    rot = dim // 2 * 2 if rot is None else rot
    m = {"left": {"heads": H, "kv_heads": G, "dim": dim, "vdim": dim, "scale": scale or dim ** -0.5, "rot": {"base": base, "dims": rot}}, "left_scale": ls,
         "right": {"heads": R, "dim": rk, "vdim": rv, "decay": list(decay)}, "right_scale": rs}
    n = H * dim + R * rv
    eye = torch.eye(n).to(BF16)  # both outputs side by side: neither hides the other
    W = {"left.q": randn(g, H * dim, width), "left.k": randn(g, G * dim, width, k=width ** -0.5), "left.g": randn(g, H, width, k=2 * width ** -0.5), "left.o": eye[:, : H * dim],
         "left.q.norm": 1 + randn(g, dim, k=0.3), "left.k.norm": 1 + randn(g, dim, k=0.3), "right.o": eye[:, H * dim :], "right.norm": 1 + randn(g, R * rv, k=0.2)}
    W.update({"right." + a: randn(g, R * b, width, k=width ** -0.5) for a, b in (("q", rk), ("k", rk), ("v", rv), ("g", rv))})
    cos, sin = ref.rope_tables(rot, 4096, base)
    left = GroupedAttention(GroupedShape(H, G, dim, dim, tied=True, gate="heads"), m["left"]["scale"], 0.0, 0, 0, False, cos.to(device), sin.to(device),
                            torch.device(device), dtype, rotate="halves", eps=EPS, mult=ls)
    right = LightningAttention(LightningShape(R, rk, rv), decay, EPS, torch.device(device), dtype, rs)
    mixer = SideBySideMixer(left, right)
    mixer.load(left.pack(W["left.q"], W["left.k"], None, W["left.o"], g=W["left.g"], q_norm=W["left.q.norm"], k_norm=W["left.k.norm"]),
               right.pack(*(W["right." + n] for n in ("q", "k", "v", "g", "o", "norm"))), up8(width))
    return (mixer, m, W) + cache_for(mixer, run)


def run_mixer(mixer, kv, h, portions, pages, run, slot=1, shared=None):
    """Feed rows of ``h`` in the given portion sizes; returns the mixer's output rows."""
    device, dtype = run
    out, at, pad = [], 0, up8(h.shape[1]) - h.shape[1]
    for n in portions:
        b = make_batch([{"tokens": [0] * n, "start": at, "pages": pages, "state_slot": slot}], kv.page_size, device)
        s = {} if shared is None else {"values": shared[at : at + n]}
        out.append(mixer.forward(torch.nn.functional.pad(h[at : at + n], (0, pad)).to(device, dtype), b, kv, 0, lambda _: _Stage(), s).float().cpu())
        at += n
    return torch.cat(out)


# heads, kv heads, dim, vdim, rotated: odd widths, more than 16 heads per group, values wider and narrower than keys, every tile width of the
# tensor-core kernels (64 / 128 / 256; keys of 128 with values of 64) and heads beyond them, rotations of all, some and two columns
SOFT = [(1, 1, 2, 1, 2), (4, 2, 20, 12, 6), (6, 2, 64, 64, 64), (3, 3, 24, 72, 10), (20, 1, 16, 16, 16), (36, 2, 40, 8, 8), (4, 1, 128, 128, 32), (2, 1, 72, 40, 72),
        (4, 2, 130, 200, 64), (2, 2, 256, 64, 14), (2, 1, 264, 24, 16), (2, 1, 24, 300, 24)]


@pytest.mark.parametrize("run", RUNS)
@pytest.mark.parametrize("H,G,dk,dv,rot", SOFT)
def test_attention_sizes(run, H, G, dk, dv, rot):
    """Whole prompt, ragged portions and token by token: the same numbers, and those of the plain statement."""
    T = 141
    mixer, m, W, kv, pages = attention_case(run, H, G, dk, dv, rot)
    h = torch.randn(T, 48, generator=gen(5)).to(BF16)
    want, _ = plain.attention(W, m, "", h.double())
    for portions in ([T], [2, 3, 37, 2, 70, 27], [129] + [1] * 12):
        assert rel(run_mixer(mixer, kv, h, portions, pages, run), want) < tol(run[1], bf16=2.5e-2 if H * dv > 1 else 6e-2), portions
        kv.k[0].uniform_(-3, 3), kv.v[0].uniform_(-3, 3)
        pages = pages[::-1]


@pytest.mark.parametrize("run", RUNS)
@pytest.mark.parametrize("lam", [0.0, 0.625, 1.0, -0.5])
def test_mixed_values(run, lam):
    """Values blended with another layer's; the blend is what later tokens see in the cache."""
    T = 70
    mixer, m, W, kv, pages = attention_case(run, 4, 2, 12, 20, 8, v_mix=True)
    W["vmix"] = torch.tensor(lam)
    mixer.lam = lam
    h, first = torch.randn(T, 48, generator=gen(5)).to(BF16), torch.randn(T, 2 * 20, generator=gen(6)).to(BF16)
    want, v = plain.attention(W, m, "", h.double(), first.double().reshape(T, 2, 20))
    padded = torch.nn.functional.pad(first.reshape(T, 2, 20), (0, 4)).reshape(T, -1).to(*run)
    for portions in ([T], [40, 2, 28], [50] + [1] * 20):
        assert rel(run_mixer(mixer, kv, h, portions, pages, run, shared=padded), want) < tol(run[1]), portions
    assert rel(kv.gather_rows(0, pages, T)[1].permute(1, 0, 2)[..., :20].flatten(1).float(), v.flatten(1)) < tol(run[1], 1e-5, 1e-2)
    # the first mixing layer of a pass leaves its own values to the others and mixes nothing
    shared = {}
    b = make_batch([{"tokens": [0] * T, "start": 0, "pages": pages, "state_slot": 1}], kv.page_size, run[0])
    y = mixer.forward(h.to(*run), b, kv, 0, lambda _: _Stage(), shared)
    alone, v0 = plain.attention(W, m, "", h.double())
    assert rel(y.float(), alone) < tol(run[1]) and rel(shared["values"].float().reshape(T, 2, 24)[..., :20].flatten(1), v0.flatten(1)) < tol(run[1], 1e-5, 1e-2)
    if lam not in (0.0,):
        assert rel(want, alone) > 0.1


def point_at(h, t, far, wq, wk, dim, rot, base, strength):
    """Move row t of the input so that its query (head 0) points at the key of row ``far``, rotation undone."""
    h[t] *= 0.1
    k = plain.rotate_halves(wk[:dim].double() @ h[far].to(BF16).double(), far - t, rot, base)
    h[t] += strength * torch.linalg.lstsq(wq[:dim].double(), k.unsqueeze(1)).solution.squeeze(1).float() / k.norm().float()


@pytest.mark.parametrize("run", RUNS)
def test_far_keys_at_page_borders(run):
    """One key per query stands out among hundreds: the first tokens, both sides of page and tile borders, far back."""
    T, n = 300, 40
    mixer, m, W, kv, pages = attention_case(run, 1, 1, 24, 24, 8, scale=2.0, width=n)
    h = torch.randn(T, n, generator=gen(3))
    far = [0, 1, 31, 32, 33, 63, 64, 95, 127, 128, 150]
    for j, f in enumerate(far):
        point_at(h, 270 + 2 * j, f, W["q"], W["k"], 24, 8, 700.0, 6.0)
    h = h.to(BF16)
    want, v = plain.attention(W, m, "", h.double())
    gate = torch.sigmoid(h.double() @ W["g"].double().T)
    for j, f in enumerate(far):  # the far key decides the output
        assert rel((want / gate)[270 + 2 * j].unsqueeze(0), v[f].reshape(1, -1)) < 0.1, f
    for portions in ([T], [260] + [1] * 40, [33, 31, 32, 64, 96, 2, 42]):
        assert rel(run_mixer(mixer, kv, h, portions, pages, run), want) < tol(run[1], 5e-5, 0.1), portions


@pytest.mark.parametrize("run", RUNS)
@pytest.mark.parametrize("scale,level", [(0.05, 0.0), (1.5, 6.0), (1.0, -8.0), (0.3, 30.0)])
def test_sink(run, scale, level):
    """Sinks far above, around and far below the scores, one per head, from the first token on; they are not scaled."""
    T, n = 90, 40
    mixer, m, W, kv, pages = attention_case(run, 3, 1, 16, 24, 6, scale=scale, width=n)
    W["sink"] = (torch.tensor([0.0, 1.0, -2.0]) + level).to(BF16)
    mixer.load(*(W[x] for x in ("q", "k", "v", "o")), k_pad=up8(n), g=W["g"], sink=W["sink"])
    h = torch.randn(T, n, generator=gen(8)).to(BF16)
    want, v = plain.attention(W, m, "", h.double())
    for portions in ([T], [1] * T, [2, 40, 2, 46]):
        assert rel(run_mixer(mixer, kv, h, portions, pages, run), want) < tol(run[1], 5e-5, 0.05), portions
    scaled = dict(W, sink=W["sink"] * scale)
    if level:
        assert rel(plain.attention(scaled, m, "", h.double())[0], want) > 1e-3 or level < 0


# heads, kv heads, dim, lightning heads, dim, vdim, decays: widths that are no multiple of 8 or 16, several value slices, key widths of every
# kernel form, decays of 1, hardly below 1, and so small that a chunk forgets everything
PAR = [(1, 1, 2, 1, 1, 1, (0.5,)), (4, 2, 20, 2, 12, 20, (0.9, 0.999)), (6, 2, 64, 3, 24, 72, (1.0, 0.6, 0.05)), (20, 1, 16, 1, 32, 130, (0.97,)), (3, 3, 40, 2, 64, 64, (0.99, 0.8)),
       (4, 1, 128, 2, 100, 40, (0.3, 0.9999)), (2, 2, 72, 1, 128, 200, (0.95,)), (1, 1, 136, 1, 136, 24, (0.999,)), (2, 1, 256, 2, 256, 64, (0.7, 0.995)), (2, 1, 264, 1, 300, 40, (0.98,)),
       (2, 1, 8, 5, 8, 16, (0.1, 0.5, 0.9, 0.99, 0.999))]


def state_after(W, m, h):
    r = m["right"]
    S = torch.zeros(r["heads"], r["dim"], r["vdim"], dtype=torch.float64)
    plain.lightning(W, r, "right.", h.double(), EPS, S)
    return S


def close_rows(got, want, dtype, what=None):
    """(Lightning rows of weak heads: where the activated rows nearly cancel, the norm behind them magnifies their bf16 rounding.)"""
    e = rows_rel(got, want)
    assert e.max() < 5e-5 if dtype == F32 else (e.quantile(0.9) < 3e-2 and e.max() < 0.2), (what, e.max())


@pytest.mark.parametrize("run", RUNS)
@pytest.mark.parametrize("H,G,dim,R,rk,rv,decay", PAR)
def test_side_by_side_sizes(run, H, G, dim, R, rk, rv, decay):
    """Whole prompt, ragged portions (across, inside and at the edges of chunks) and token by token, from stale pages and slots; each half on
    its own columns; the state that is left behind."""
    T = 280
    mixer, m, W, kv, pages = parallel_case(run, H, G, dim, R, rk, rv, decay, rot=max(2, dim // 4 * 2))
    h = torch.randn(T, 48, generator=gen(5)).to(BF16)
    want = plain.parallel(W, m, "", h.double(), EPS)
    cut = H * dim
    S = state_after(W, m, h)
    for slot, portions in ((1, [T]), (2, [2, 3, CHUNK, 2, 97, 48]), (3, [250] + [1] * 30), (1, [CHUNK - 1, 2, 151]), (2, [1] * 40 + [240])):
        got = run_mixer(mixer, kv, h, portions, pages, run, slot)
        assert rel(got[:, :cut], want[:, :cut]) < tol(run[1], 5e-5, 3e-2), portions
        close_rows(got[:, cut:], want[:, cut:], run[1], portions)
        st = kv.state["lightning"][0][slot]
        assert rel(st[:, :rk, :rv].flatten(1), S.flatten(1)) < tol(run[1], 5e-5, 2e-2)
        assert (st[:, rk:] == 0).all() and (st[:, :, rv:] == 0).all()
        pages = pages[::-1]
    lost = plain.parallel(W, m, "", h[140:].double(), EPS)
    if max(decay) > 0.9:
        assert rel(lost[:20, cut:], want[140:160, cut:]) > 0.1  # a state that is dropped on the way shows


@pytest.mark.parametrize("run", RUNS)
def test_tokens_at_chunk_edges_stay_in_the_state(run):
    """One token's key and value stand out by far, just in front of or behind the edge of a chunk or portion; later queries still see it, with
    the weight its distance gives it."""
    T, n = 300, 40
    mixer, m, W, kv, pages = parallel_case(run, 1, 1, 8, 2, 16, 24, (0.995, 1.0), width=n)
    for spot in (0, 1, CHUNK - 1, CHUNK, CHUNK + 1, 2 * CHUNK - 1, 2 * CHUNK):
        h = torch.randn(T, n, generator=gen(spot)) * 0.3
        h[spot] *= 40.0
        h = h.to(BF16)
        want = plain.parallel(W, m, "", h.double(), EPS)[:, 8:]
        gone = h.clone()
        gone[spot] = 0
        after = slice(min(spot + 2, T - 5), T)
        assert rel(plain.parallel(W, m, "", gone.double(), EPS)[after, 8:], want[after]) > 0.3
        for portions in ([T], [CHUNK, CHUNK, T - 2 * CHUNK], [max(1, spot), T - max(1, spot)], [spot + 1, T - spot - 1], [270] + [1] * 30):
            close_rows(run_mixer(mixer, kv, h, portions, pages, run)[:, 8:], want, run[1], (spot, portions))


def test_powers_of_decays():
    p = decay_powers([0.999, 0.25, 1.0, 0.0]).double()
    assert p.shape == (4, CHUNK + 2) and (p[:, 0] == 1).all()
    d = p[:, 1] + p[:, -1]
    assert (d - torch.tensor([0.999, 0.25, 1.0, 0.0], dtype=torch.float64)).abs().max() < 1e-14
    assert abs(p[0, CHUNK] - 0.999 ** CHUNK) < 1e-7 and p[3, 1] == 0 and p[2, CHUNK] == 1


@pytest.mark.parametrize("run", RUNS)
@pytest.mark.parametrize("kind", ["attention", "parallel"])
def test_unequal_sequences_in_one_batch(run, kind):
    """Each sequence as if it were alone: single tokens beside portions that start and end inside pages and chunks."""
    device, dtype = run
    if kind == "attention":
        mixer, m, W, _, _ = attention_case(run, 6, 2, 20, 12, 10)
        fn = lambda h: plain.attention(W, m, "", h)[0]  # noqa: E731
    else:
        mixer, m, W, _, _ = parallel_case(run, 4, 2, 20, 3, 20, 36, (0.9, 0.99, 0.999))
        fn = lambda h: plain.parallel(W, m, "", h, EPS)  # noqa: E731
    kv, pages = cache_for(mixer, run, slots=9)
    lens, starts = [1, 50, 3, 9, 1, 140, 8, 2], [0, 0, 0, 0, 17, 0, 70, 131]
    hs = [torch.randn(s + n, 48, generator=gen(100 + i)).to(BF16) for i, (s, n) in enumerate(zip(starts, lens))]
    own, at = [], 0
    for s, n in zip(starts, lens):
        k = (s + n + 31) // 32
        own.append(pages[at : at + k])
        at += k
    for i, (h, s, pg) in enumerate(zip(hs, starts, own)):
        if s:
            run_mixer(mixer, kv, h[:s], [s], pg, run, i + 1)
    b = make_batch([{"tokens": [0] * n, "start": s, "pages": pg, "state_slot": i + 1} for i, (n, s, pg) in enumerate(zip(lens, starts, own))], kv.page_size, device)
    y = mixer.forward(torch.cat([h[s:] for h, s in zip(hs, starts)]).to(device, dtype), b, kv, 0, lambda _: _Stage(), {})
    row = 0
    for h, s, n in zip(hs, starts, lens):
        assert rel(y[row : row + n].float(), fn(h.double())[s:]) < tol(dtype, 5e-5, 5e-2)
        row += n


# --------------------------------------------------------------------------------------------------- configuration, cache
def test_config_and_weight_errors():
    cfg = tiny_config("dubozen")
    c = parse_config(cfg)
    assert c.model_type == "dubozen" and c.extra["streams"] == 3 and c.num_layers == 4 and c.tie_word_embeddings and c.num_experts == 6
    for path, value, msg in ((("layers", 0, "type"), "mamba", "unknown mixer"), (("layers", 1, "mlp", "kind"), "wide", "unknown feed-forward"), (("streams",), 17, "streams"),
                             (("layers",), [], "no layers")):
        bad = copy.deepcopy(cfg)
        d = bad
        for k in path[:-1]:
            d = d[k]
        d[path[-1]] = value
        with pytest.raises(ValueError, match=msg):
            parse_config(bad)
    t = build_tensors(cfg)
    for name, msg in (("l0.mix.k", "rows"), ("l0.mix.sink", "sinks"), ("l0.mix.g", "rows"), ("l1.mix.left.q.norm", "norms"), ("l1.mix.right.v", "rows"), ("l1.mix.right.norm", "norm"),
                      ("l1.mlp.correction", "corrections"), ("l1.mlp.router", "router"), ("l0.mlp.up", "width"), ("l2.hc2.in", "streams")):
        with pytest.raises(ValueError, match=msg):
            build(cfg, ("cpu", F32), tensors=dict(t, **{name: t[name][:-1]}))
    bad = copy.deepcopy(cfg)
    bad["layers"][1]["mixer"]["right"]["decay"].pop()
    with pytest.raises(ValueError, match="decays"):
        build(bad, ("cpu", F32), tensors=t)
    for kw, msg in ((dict(groups=4, keep=1), "groups"), (dict(groups=3, keep=4), "groups"), (dict(groups=3, keep=1), "groups")):
        with pytest.raises(ValueError, match=msg):
            RoutedExperts(6, 3, mode="sigmoid_topk", **kw)
    with pytest.raises(ValueError, match="values"):
        GroupedShape(2, 1, 8, 16, tied=True)
    with pytest.raises(ValueError, match="mixed"):  # layers that mix values have to agree on their size
        cfg2 = dubozen_config(32, 64, [dict(heads=2, kv_heads=1, dim=8, vdim=8, ff=0), dict(heads=2, kv_heads=1, dim=8, vdim=16, ff=0)])
        engine_for(build(cfg2, ("cpu", F32))[0], 64).generate([1, 2], GeneratorParameters(max_tokens=1))
    from deliverance_b200.parallel.context import TensorParallelContext

    with pytest.raises(ValueError, match="tensor parallelism"):
        DubozenModel(c, "cpu", None, TensorParallelContext(0, 2, object()))


def test_layers_with_pages_and_a_state():
    layout = {"layers": 2, "kv_heads": 2, "head_dim": 16, "layer_kinds": ["attention", "attention"], "state_shapes": [None, {"s": (2, 3, 8)}], "paged": [True, True]}
    kv = PagedKVCache(layout, 8, "cpu", F32, KvCacheSettings(), 2)
    assert kv.k[1] is not None and kv.state["s"][1].shape == (3, 2, 3, 8)
    assert PagedKVCache.bytes_per_page(layout, 32, F32) == 2 * 2 * 32 * 32 * 4 and PagedKVCache.bytes_per_state_slot(layout) == 4 * 48
    del layout["paged"]  # without the flag a layer with a state has no pages
    assert PagedKVCache(layout, 8, "cpu", F32, KvCacheSettings(), 2).k[1] is None and PagedKVCache.bytes_per_page(layout, 32, F32) == 2 * 32 * 32 * 4


# --------------------------------------------------------------------------------------------------- whole models
def variety():
    soft = dict(heads=6, kv_heads=2, dim=20, vdim=28, rot_dims=12, ff=52)
    both = dict(heads=4, kv_heads=1, dim=18, rot_dims=10, base=500.0, right=(3, 12, 20, (0.4, 0.97, 0.999)))
    return {
        "tiny": tiny_config("dubozen"),
        "attention-only": dubozen_config(40, 97, [dict(soft, heads=1, kv_heads=1, ff=8, v_mix=False), dict(soft, heads=1, kv_heads=1, ff=0, v_mix=True)], streams=1, eps=1e-3),
        "parallel-only": dubozen_config(56, 120, [dict(both, heads=1, right=(1, 8, 1, (0.5,)), ff=20), dict(both, ff=16, experts=4, top=1, groups=4, keep=2, left_scale=1.0,
                                                                                                                   right_scale=-1.5)], streams=4),
        "mixed-late": dubozen_config(72, 333, [dict(both, ff=24, experts=9, top=4, groups=3, keep=2, route_scale=0.5), dict(soft, v_mix=False, ff=0), dict(soft, heads=4, scale=0.5),
                                               dict(both, heads=2, kv_heads=2, dim=64, rot_dims=64, ff=0), dict(soft, heads=2, ff=30, experts=3, top=3)], streams=5),
        "wide-heads": dubozen_config(128, 512, [dict(soft, heads=4, kv_heads=1, dim=128, vdim=64, ff=192), dict(both, dim=128, heads=2, right=(2, 64, 96, (0.9, 0.995)), ff=64)]),
    }


@pytest.mark.parametrize("run", RUNS)
@pytest.mark.parametrize("name", list(variety()))
def test_model_portions_batches_reused_pages_and_slots(run, name):
    """Whole prompts, decoding, portions down to two tokens and mixed batches in a pool so small that pages and slots are used again; logits
    of every position against the plain statement, and the sum of the streams after every layer for one prompt."""
    cfg = variety()[name]
    model, W = build(cfg, run, seed=3)
    V = cfg["vocab"]
    req = {f"r{i}": tokens_of(n, V, 10 + i) for i, n in enumerate((150, 97, 34, 1, 66, 23))}
    want = {k: plain.forward(W, cfg, t) for k, t in req.items()}
    stream = []
    model.layer_hook = lambda i, stage, x: stream.append(x.float().cpu()) if stage == "out" else None
    eng = engine_for(model, 192, max_seqs=4)
    got = replay(eng, [[(k, len(v))] for k, v in req.items()], req)
    model.layer_hook = None
    for k in req:
        close_model(got[k], want[k], run[1], k)
    _, layers = plain.forward(W, cfg, req["r0"], want_layers=True)
    for i, w in enumerate(layers):
        close_model(stream[i], w, run[1], i)
    plan = []
    for k, v in req.items():
        n = max(1, len(v) - 20)
        plan += [[(k, n)]] + [[(k, 1)]] * (len(v) - n)
    for k, v in replay(eng, plan, req).items():
        close_model(v, want[k], run[1], k)
    # portions of changing size, three requests live at once (a captured step of three pads to four rows), places, pages, slots handed on
    sizes, at, live, plan, n = [2, 17, 2, 31, 1, 33, 1, 1, 1, 5, 2, 64, 3], dict.fromkeys(req, 0), [], [], 0
    waiting = list(req)
    while waiting or live:
        while waiting and len(live) < 3 and sum(-(-len(req[k]) // 32) for k in live + waiting[:1]) <= 6:
            live.append(waiting.pop(0))
        step = []
        n += 1
        for j, k in enumerate(live):
            c = min(1 if n % 3 == 0 else sizes[(n + j) % len(sizes)], len(req[k]) - at[k])
            at[k] += c
            step.append((k, c))
        plan.append(step)
        live = [k for k in live if at[k] < len(req[k])]
    for k, v in replay(eng, plan, req).items():
        close_model(v, want[k], run[1], k)
    assert eng.kv.allocator.available() == eng.kv.num_pages - 1 and (not eng.hybrid or len(eng.kv.free_slots) == 4)
    eng.kv.audit([])


def test_every_mechanism_of_the_model_shows():
    """The plain statement without one mechanism at a time: the logits move, so the comparisons above would see it missing."""
    cfg = tiny_config("dubozen")
    W = build_tensors(cfg, 3, BF16)
    toks = tokens_of(60, cfg["vocab"], 1)
    want = plain.forward(W, cfg, toks)
    for change in ({"l2.mix.vmix": torch.tensor(0.0)}, {"l0.mix.sink": W["l0.mix.sink"] * 0 - 50}, {"l0.mix.g": W["l0.mix.g"] * 0}, {"l1.mlp.correction": W["l1.mlp.correction"] * 0},
                   {"l1.mix.left.q.norm": W["l1.mix.left.q.norm"] * 0 + 1}, {"l1.mix.right.norm": W["l1.mix.right.norm"] * 0 + 1}, {"l3.hc1.mix": W["l3.hc1.mix"].T},
                   {"l1.mix.left.g": W["l1.mix.left.g"] * 0}, {"embed.norm": W["embed.norm"] * 0 + 1}):
        assert rel(plain.forward(dict(W, **change), cfg, toks), want) > 1e-3, list(change)
    assert torch.equal(plain.forward(dict(W, **{"l0.mix.vmix": torch.tensor(0.0)}), cfg, toks), want)  # the first mixing layer's is unused


@pytest.mark.parametrize("run", RUNS)
def test_paused_request_keeps_its_state(run):
    """A request that is left out of several steps goes on where it was, whatever ran in between."""
    cfg = tiny_config("dubozen", width=48)
    model, W = build(cfg, run, seed=8)
    req = {"a": tokens_of(60, 261, 1), "b": tokens_of(50, 261, 2), "c": tokens_of(40, 261, 3)}
    plan = [[("a", 33)], [("b", 20)], [("b", 1), ("c", 10)], [("b", 1), ("c", 1)], [("b", 1), ("c", 1)], [("c", 28), ("b", 27)], [("a", 1)], [("a", 26)]]
    for k, v in replay(engine_for(model, 320, max_seqs=3), plan, req).items():
        close_model(v, plain.forward(W, cfg, req[k]), run[1], k)


@pytest.mark.parametrize("run", RUNS)
def test_long_decoding(run):
    """Several hundred decoded tokens, over many pages and several chunks of the state."""
    cfg = dubozen_config(32, 64, [dict(heads=2, kv_heads=1, dim=8, vdim=12, rot_dims=4, ff=16), dict(heads=2, kv_heads=2, dim=10, right=(2, 8, 8, (0.9, 0.9995)), ff=8)])
    model, W = build(cfg, run, seed=9)
    req = {"a": tokens_of(330, 64, 1)}
    got = replay(engine_for(model, 384), [[("a", 3)]] + [[("a", 1)]] * 327, req)["a"]
    close_model(got, plain.forward(W, cfg, req["a"]), run[1])


def check_greedy(W, cfg, prompt, produced, dtype):
    """Every produced token is the plain statement's best continuation of what came before it (bf16: the best or a near-tie)."""
    lo = plain.forward(W, cfg, prompt + produced[:-1])[len(prompt) - 1 :]
    if dtype == F32:
        assert produced == lo.argmax(-1).tolist()
    else:
        picked = lo[torch.arange(len(produced)), torch.tensor(produced)]
        gap = (lo.max(-1).values - picked) / lo.std()
        assert (gap < 0.15).float().mean() > 0.9 and gap.max() < 1.0  # (a close call of the router may move a token)


@pytest.mark.parametrize("run", RUNS)
@pytest.mark.parametrize("how", ["plain", "small-chunks", "preempted", "no-lookahead", "interleaved"])
def test_greedy_generation_through_the_scheduler(run, how):
    """Unequal prompts generated together: the tokens of the plain statement, whatever the scheduler does with them."""
    cfg = tiny_config("dubozen", width=48)
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
    # prefix cache: the same prompt again continues from cached pages and a state snapshot, same tokens
    hit = eng.generate(prompts[2], GeneratorParameters(max_tokens=14, temperature=0.0))
    assert (hit.prefix_hit_tokens > 0 or how == "preempted") and (run[1] != F32 or hit.token_ids == outs[2].token_ids)


def test_generation_through_the_public_loader_and_server_registry(tmp_path):
    """``config.json`` + safetensors in a directory, loaded and generated from the way every other family is."""
    from deliverance_b200.api import AutoModelForCausalLM
    from deliverance_b200.model_support import detect_model, load_model

    d = str(tmp_path / "m")
    cfg = write_tiny_model(d, "dubozen", seed=6, dtype=BF16, sharded=True)
    assert detect_model(d) == "dubozen" and load_config(d).model_type == "dubozen"
    W = {n: WeightLoader(d).load(n) for n in WeightLoader(d).names()}
    prompt = tokens_of(20, 256, 8)
    clm = AutoModelForCausalLM.new_builder(d).with_device("cpu").build()
    p = GeneratorParameters(max_tokens=8, temperature=0.0)
    check_greedy(W, cfg, prompt, clm.generate(prompt, p).token_ids, F32)
    seeded = lambda: GeneratorParameters(max_tokens=8, temperature=0.8, top_k=20, top_p=0.9, seed=3)  # noqa: E731
    assert load_model(d, device="cpu").generate(prompt, seeded()).token_ids == clm.generate(prompt, seeded()).token_ids
    with pytest.raises(ValueError, match="LoRA"):
        clm.model.set_lora(object())


# --------------------------------------------------------------------------------------------------- trace replay program
@pytest.mark.parametrize("run", RUNS)
def test_trace_replay_program(run, tmp_path, monkeypatch, capsys):
    """Steps on standard input, logits and ``done`` lines out; a finished request's pages and slot serve the next one."""
    from deliverance_b200.engine import replay as prog

    device, dtype = run
    d, out = str(tmp_path / "m"), str(tmp_path / "out")
    cfg = write_tiny_model(d, "dubozen", seed=1, dtype=BF16)
    W = {n: WeightLoader(d).load(n) for n in WeightLoader(d).names()}
    a, b, c = (tokens_of(n, cfg["vocab"], n) for n in (60, 40, 61))
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:57], "want": [0, 56]}, {"id": "b", "tokens": b[:2], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": b[2:39], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "b", "tokens": b[39:], "want": [0]}, {"id": "a", "tokens": a[57:58], "want": []}], "end": ["b"]},
             {"step": 5, "entries": [{"id": "a", "tokens": a[58:], "want": [1, 0]}], "end": ["a"]},
             {"step": 6, "entries": [{"id": "c", "tokens": c, "want": [60]}], "end": ["c"]}]
    monkeypatch.setattr("sys.stdin", io.StringIO("".join(json.dumps(s) + "\n" for s in steps)))
    name = "float32" if dtype == F32 else "bfloat16"
    assert prog.main(["--model", d, "--dtype", name, "--out", out, "--max-tokens", "128", "--device", device]) == 0
    assert [ln for ln in capsys.readouterr().out.splitlines() if ln.startswith("done")] == ["done 0", "done 1", "done 2", "done 5", "done 6"]
    assert sorted(os.listdir(out)) == ["0.f32", "2.f32", "5.f32", "6.f32"]
    wa, wb, wc = (plain.forward(W, cfg, t) for t in (a, b, c))
    load = lambda s: torch.frombuffer(bytearray(open(os.path.join(out, f"{s}.f32"), "rb").read()), dtype=F32).view(-1, cfg["vocab"])  # noqa: E731
    got = torch.cat([load(s) for s in (0, 2, 5, 6)])
    close_model(got, torch.cat([wa[[0, 56]], wb[[39]], wa[[59, 58]], wc[[60]]]), dtype)


# --------------------------------------------------------------------------------------------------- CUDA only
@gpu
def test_prompt_kernels_agree_with_the_row_forms_on_cuda():
    """Tensor-core prompt and decode attention with gates and sinks against the CUDA-core rows form, chunked against recurrent lightning
    attention, on inputs of several tiles and chunks; no kernel writes outside its outputs."""
    import deliverance_b200.ops.grouped as gop
    import deliverance_b200.ops.lightning as lop

    run = ("cuda", BF16)
    h = torch.randn(700, 48, generator=gen(5)).to(BF16)

    def without_tensor_cores(fn):
        old, gop.GroupedShape.tensor_core = gop.GroupedShape.tensor_core, property(lambda self: False)
        old_dk, lop.MAX_DK_CHUNKED = lop.MAX_DK_CHUNKED, 0
        try:
            return fn()
        finally:
            gop.GroupedShape.tensor_core, lop.MAX_DK_CHUNKED = old, old_dk

    ops.set_bounds_check(True)
    try:
        cases = [attention_case(run, *a) for a in ((8, 2, 64, 64), (4, 4, 72, 128), (20, 1, 128, 40), (2, 1, 200, 256), (4, 1, 128, 128))]
        cases += [parallel_case(run, *a) for a in ((4, 2, 64, 2, 64, 128, (0.9, 0.999)), (2, 1, 128, 1, 256, 192, (0.99,)), (24, 1, 40, 3, 40, 24, (0.2, 0.95, 1.0)),
                                                   (2, 2, 256, 2, 128, 64, (0.8, 0.9995)))]
        for mixer, m, W, kv, pages in cases:
            soft = getattr(mixer, "left", mixer)
            a = run_mixer(mixer, kv, h, [256, 424] + [1] * 20, pages, run)
            b = without_tensor_cores(lambda: run_mixer(mixer, kv, h, [256, 444], pages[::-1], run, 2))  # noqa: B023
            assert rel(a, b) < 3e-2
            if kv.state:
                st = kv.state["lightning"][0]
                assert rel(st[1].flatten(1), st[2].flatten(1).cpu()) < 1e-3  # fp32-grade state on the tensor cores
            for splits in (2, 5, 16):
                soft._splits = lambda batch: splits if batch.is_decode else 1  # noqa: B023
                assert rel(run_mixer(mixer, kv, h, [690] + [1] * 10, pages, run)[690:], b[690:]) < 3e-2
            ops.check_guards()
        ops.check_status()
    finally:
        ops.set_bounds_check(False)
