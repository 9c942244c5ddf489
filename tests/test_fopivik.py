"""Fopivik decoder against a plain float64 statement of its equations (``fopivik_plain.py``), mechanism by mechanism and through the
engine. Every test runs on the CPU operator set in fp32 and, on a GPU box, on the CUDA kernels in fp32 and in bf16."""
import copy
import io
import json
import os

import pytest
import torch

import fopivik_plain as plain
from design_helpers import RUNS, Dict2Loader, _Stage, engine_for, gpu, rel, replay, tokens_of, tol
from deliverance_b200 import ops
from deliverance_b200.ckpt.loader import WeightLoader
from deliverance_b200.ckpt.tiny import build_tensors, fopivik_config, tiny_config, write_tiny_model
from deliverance_b200.config import layer_run_order, load_config, loop_pass_starts, parse_config
from deliverance_b200.kv.paged import KvCacheSettings, PagedKVCache
from deliverance_b200.models.batch import make_batch
from deliverance_b200.models.fopivik import FopivikModel
from deliverance_b200.models.gla import GatedLinearAttention
from deliverance_b200.models.grouped import GroupedAttention
from deliverance_b200.models.moe import RoutedExperts
from deliverance_b200.ops import ref
from deliverance_b200.ops.gla import GlaShape
from deliverance_b200.ops.grouped import GroupedShape
from deliverance_b200.params import GeneratorParameters

F32, BF16 = torch.float32, torch.bfloat16
BANDS = {"factor": 6.0, "low": 1.0, "high": 4.0, "original": 96}


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
        assert e.quantile(0.9) < 5e-2 and e.max() < 0.6, (what, e.quantile(0.9), e.max())


def build(cfg, run, seed=0, tensors=None):
    device, dtype = run
    W = tensors or build_tensors(cfg, seed, BF16)
    return FopivikModel(parse_config(cfg), device, dtype).load(Dict2Loader(W)), W


def randn(g, *s, k=1.0):
    return (torch.randn(*s, generator=g) * k).to(BF16)


def gen(seed):
    return torch.Generator().manual_seed(seed)


# --------------------------------------------------------------------------------------------------- norms, tables, experts
@pytest.mark.parametrize("run", RUNS)
@pytest.mark.parametrize("W", [8, 76, 257, 1024, 1600, 5000])
def test_sandwich_norm(run, W):
    device, dtype = run
    g = gen(W)
    T, pitch, eps, m = 5, (W + 7) // 8 * 8, 1e-3, 0.37
    r = lambda *s: torch.randn(*s, generator=g)  # noqa: E731
    x, sub = r(T, W) * 3, (r(T, pitch) + 20).to(BF16)  # a large common offset: variances must be means of squared deviations
    wb, wn = 1 + 0.3 * r(W), 1 + 0.3 * r(W)
    dev = lambda t: t.to(device)  # noqa: E731
    want_r = x.double() + m * plain.layer_norm(sub[:, :W].double(), wb, eps)
    want_y = plain.layer_norm(want_r, wn, eps)
    t = 2e-5 if dtype == F32 else 6e-3
    res = dev(x.clone())
    y = ops.sandwich_norm(res, sub.to(device, dtype), dev(wb), m, dev(wn), eps, pitch, dtype)
    assert rel(res, want_r) < 1e-5 and rel(y[:, :W], want_y) < t and y.shape == (T, pitch) and (y[:, W:] == 0).all()
    # nothing to add: the norm alone; nothing in front of the next step: the stream itself, beside what is in the rows already
    again = ops.sandwich_norm(res, None, None, m, dev(wn), eps, pitch, dtype)
    assert rel(again[:, :W], want_y) < t
    wide = torch.full((T, 2 * pitch), 7.0, dtype=dtype, device=device)
    res2 = dev(x.clone())
    ops.sandwich_norm(res2, sub.to(device, dtype), dev(wb), m, None, eps, pitch, dtype, wide[:, :W])
    assert rel(res2, want_r) < 1e-5 and rel(wide[:, :W], want_r) < t and (wide[:, W:] == 7).all()
    # expert rows: the weighted sum is part of the step
    k = 3
    ys, pos, w = (r(T * k, pitch) + 5).to(BF16), torch.randperm(T * k, generator=g).to(torch.int32).reshape(T, k), r(T, k).abs()
    f = (ys[pos.long()].double() * w.double().unsqueeze(-1)).sum(1)[:, :W]
    want_r = x.double() + m * plain.layer_norm(f, wb, eps)
    routed = ops.Routed(ys.to(device, dtype), dev(pos), dev(w))
    res = dev(x.clone())
    y = ops.sandwich_norm(res, routed, dev(wb), m, dev(wn), eps, pitch, dtype)
    assert rel(res, want_r) < 2e-5 and rel(y[:, :W], plain.layer_norm(want_r, wn, eps)) < t
    assert rel(routed.dense()[:, :W], f) < 1e-5


@pytest.mark.parametrize("dims,base,scaling", [
    (16, 10000.0, None), (6, 300.0, {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 64}), (64, 5e5, {"factor": 32.0, "low": 1.0, "high": 4.0, "original": 8192}),
    (10, 100.0, {"factor": 1.0, "low": 1.0, "high": 2.0, "original": 128}), (20, 1e4, {"factor": 3.0, "low": 0.5, "high": 30.0, "original": 200})])
def test_banded_tables_and_pair_rotation(dims, base, scaling):
    freqs = plain.banded_frequencies(dims, base, scaling)
    cos, sin = ref.banded_rope_tables(dims, 3000, base, scaling)
    for p in (0, 1, 37, 2999):
        a = torch.tensor([p * f for f in freqs], dtype=torch.float64)
        assert torch.allclose(cos[p].double(), torch.cos(a), atol=1e-6) and torch.allclose(sin[p].double(), torch.sin(a), atol=1e-6)
    v = torch.randn(dims + 3, dtype=torch.float64, generator=gen(1))
    got = ref.apply_rope_pairs(v.view(1, 1, -1), torch.tensor([37]), cos, sin)[0, 0]
    assert torch.allclose(got.double(), plain.rotate_pairs(v, 37, freqs), atol=1e-5) and torch.equal(got[dims:], v[dims:].float())
    if scaling and scaling["factor"] != 1.0:
        unscaled = plain.banded_frequencies(dims, base, None)
        changed = [abs(a - b) > 1e-9 for a, b in zip(freqs, unscaled)]
        assert any(changed) and (not all(changed) or dims == 6 or dims == 20)


@pytest.mark.parametrize("run", RUNS)
@pytest.mark.parametrize("E,top,ff,width,T", [(8, 3, 64, 48, 33), (5, 5, 20, 40, 7), (3, 1, 36, 76, 150), (130, 4, 8, 32, 40), (4, 2, 16, 24, 1), (6, 2, 48, 64, 700)])
def test_routed_experts(run, E, top, ff, width, T):
    device, dtype = run
    g = gen(E * 100 + T)
    W = {"router": randn(g, E, width, k=1.5 * width ** -0.5)}
    for e in range(E):
        W.update({f"e{e}.gate": randn(g, ff, width, k=width ** -0.5), f"e{e}.up": randn(g, ff, width, k=width ** -0.5), f"e{e}.down": randn(g, width, ff, k=ff ** -0.5)})
    h = randn(g, T, width)
    pad = (width + 7) // 8 * 8
    moe = RoutedExperts(E, top).load(W["router"].to(dtype), (tuple(W[f"e{e}.{n}"].to(dtype) for n in ("gate", "up", "down")) for e in range(E)), ff, pad,
                                     torch.device(device), dtype)
    got = moe.forward(torch.nn.functional.pad(h, (0, pad - width)).to(device, dtype), lambda _: _Stage()).dense()[:, :width]
    want = plain.moe(W, {"router": {"top": top}}, "", h.double())
    assert rel(got, want) < tol(dtype, 1e-5, 3e-2)  # (the router reads the same bf16 rows in both: no close call differs)
    idx, w = plain.route(W["router"].double() @ h[0].double(), top)
    assert top == E or w.sum() < 0.99  # the weights are not renormalised


# --------------------------------------------------------------------------------------------------- softmax attention
def soft_case(run, H, G, dk, dv, window, keep=0, rot=None, softcap=20.0, scale=None, width=48, scaling=None, seed=0):
    device, dtype = run
    g = gen(seed * 7919 + H * 31 + dk)
    rot = rot or (dk // 2 * 2 if dk > 1 else 0)
    m = {"heads": H, "kv_heads": G, "dim": dk, "vdim": dv, "mask": {"size": window, "keep_first": keep}, "softcap": softcap, "scale": scale or dk ** -0.5,
         "rot": {"base": 700.0, "dims": rot, "scaling": scaling}}
    W = {"q": randn(g, H * dk, width, k=2 * width ** -0.5), "k": randn(g, G * dk, width, k=width ** -0.5), "v": randn(g, G * dv, width, k=width ** -0.5),
         "o": torch.eye(H * dv).to(BF16)}
    cos, sin = ref.banded_rope_tables(rot, 4096, 700.0, scaling)
    shape = GroupedShape(H, G, dk, dv)
    mixer = GroupedAttention(shape, m["scale"], softcap, window, keep, True, cos.to(device), sin.to(device), torch.device(device), dtype)
    mixer.load(*(W[n] for n in ("q", "k", "v", "o")), k_pad=(width + 7) // 8 * 8)
    layout = {"layers": 1, "kv_heads": G, "head_dim": shape.dk, "layer_kinds": ["sliding"], "v_dim_per_layer": [shape.dv]}
    kv = PagedKVCache(layout, 96, device, dtype, KvCacheSettings(enabled=False))
    for t in (kv.k[0], kv.v[0]):
        t.uniform_(-3, 3)  # stale rows of earlier owners
    return mixer, m, W, kv, (torch.randperm(95, generator=g) + 1).tolist()


def gla_case(run, H, dk, dv, rank=8, tau=4.0, bias=1.0, width=48, seed=0):
    device, dtype = run
    g = gen(seed * 7919 + H * 31 + dk)
    m = {"heads": H, "dim": dk, "vdim": dv, "tau": tau}
    W = {n: randn(g, rows, width, k=width ** -0.5) for n, rows in (("q", H * dk), ("k", H * dk), ("v", H * dv), ("g", H * dv), ("a1", rank))}
    W.update({"a2": randn(g, H * dk, rank, k=rank ** -0.5), "a2.b": randn(g, H * dk) + bias, "norm": 1 + randn(g, dv, k=0.2), "o": torch.eye(H * dv).to(BF16)})
    W["a2.b"] = W["a2.b"].to(BF16)
    shape = GlaShape(H, dk, dv, rank)
    mixer = GatedLinearAttention(shape, tau, 1e-5, torch.device(device), dtype)
    mixer.load(*(W[n] for n in ("q", "k", "v", "g", "o", "a1", "a2", "a2.b", "norm")), k_pad=(width + 7) // 8 * 8)
    layout = {"layers": 1, "kv_heads": 1, "head_dim": 8, "layer_kinds": ["gla"], "state_shapes": [mixer.cache_layout()["state"]]}
    kv = PagedKVCache(layout, 96, device, dtype, KvCacheSettings(enabled=False), 3)
    kv.state["gla"][0].uniform_(-3, 3)  # stale states of earlier owners
    return mixer, m, W, kv, list(range(1, 96))


def run_mixer(mixer, kv, h, portions, pages, run, slot=1):
    """Feed rows of ``h`` in the given portion sizes; returns the mixer's output rows."""
    device, dtype = run
    out, at, width = [], 0, h.shape[1]
    pad = (width + 7) // 8 * 8 - width
    for n in portions:
        b = make_batch([{"tokens": [0] * n, "start": at, "pages": pages, "state_slot": slot}], kv.page_size, device)
        out.append(mixer.forward(torch.nn.functional.pad(h[at : at + n], (0, pad)).to(device, dtype), b, kv, 0, lambda _: _Stage()).float().cpu())
        at += n
    return torch.cat(out)


# heads, kv heads, dim, vdim, window, kept, rotated: odd widths, more than 16 heads per group, values wider and narrower than keys, every tile
# width of the tensor-core kernels (64 / 128 / 256) and heads beyond them, kept tokens that fill several key tiles, windows of one key
SOFT = [(1, 1, 2, 1, 1, 0, 2), (4, 2, 20, 12, 9, 3, 6), (6, 2, 64, 64, 33, 40, 64), (3, 3, 24, 72, 70, 20, 10), (20, 1, 16, 16, 64, 5, 16), (36, 2, 40, 8, 50, 66, 8),
        (4, 1, 128, 128, 65, 17, 32), (2, 1, 96, 40, 500, 10, 96), (4, 2, 130, 200, 31, 31, 64), (2, 2, 256, 64, 40, 70, 16), (2, 1, 264, 24, 40, 9, 16), (2, 1, 24, 300, 24, 65, 24)]


@pytest.mark.parametrize("run", RUNS)
@pytest.mark.parametrize("H,G,dk,dv,window,keep,rot", SOFT)
def test_grouped_attention_sizes(run, H, G, dk, dv, window, keep, rot):
    """Whole prompt, ragged portions and token by token: the same numbers, and those of the plain statement."""
    T = 141
    mixer, m, W, kv, pages = soft_case(run, H, G, dk, dv, window, keep, rot, scaling=BANDS if H % 2 else None)
    h = torch.randn(T, 48, generator=gen(5)).to(BF16)
    want = plain.attention(W, m, "", h.double())
    for portions in ([T], [2, 3, 37, 2, 70, 27], [129] + [1] * 12):
        assert rel(run_mixer(mixer, kv, h, portions, pages, run), want) < tol(run[1]), portions
        kv.k[0].uniform_(-3, 3), kv.v[0].uniform_(-3, 3)
        pages = pages[::-1]


def point_at(h, t, far, m, W, width, strength):
    """Move row t of the input so that its query points at the key of row ``far`` (head 0, rotation undone)."""
    dk = m["dim"]
    freqs = plain.banded_frequencies(m["rot"]["dims"], m["rot"]["base"], m["rot"].get("scaling"))
    k = plain.rotate_pairs(W["k"][:dk].double() @ h[far].to(BF16).double(), far - t, freqs)
    h[t] += strength * torch.linalg.lstsq(W["q"][:dk].double(), k.unsqueeze(1)).solution.squeeze(1).float() / k.norm().float()


@pytest.mark.parametrize("run", RUNS)
@pytest.mark.parametrize("window,keep", [(1, 0), (2, 1), (32, 5), (33, 32), (64, 20), (96, 64), (130, 33)])
def test_window_and_kept_token_edges(run, window, keep):
    """One key per query stands out; it sits just inside or just outside the window, or is the last kept token or the one behind it. A
    window or a count of kept tokens that is one off moves the output by the order of the output itself."""
    T, n = 330, 44
    mixer, m, W, kv, pages = soft_case(run, 2, 1, 16, 16, window, keep, rot=4, softcap=40.0, scale=0.6, width=n)
    h = torch.randn(T, n, generator=gen(window))
    start = window + keep + 2
    probes = list(range(start, T, 7))
    for j, t in enumerate(probes):
        far = [t - window + 1, t - window, max(0, keep - 1), keep][j % 4]
        if far not in probes and far < t:
            point_at(h, t, far, m, W, n, 10.0)
    h = h.to(BF16)
    want = plain.attention(W, m, "", h.double())
    for mask in ({"size": window + 1, "keep_first": keep}, {"size": window, "keep_first": keep + 1}, {"size": max(1, window - 1), "keep_first": keep}):
        if mask != m["mask"]:
            assert rel(plain.attention(W, dict(m, mask=mask), "", h.double())[probes], want[probes]) > 0.3  # the probes see an edge that is one off
    for portions in ([T], [100, 2, 29, 64, 135], [start] + [1] * (T - start)):
        assert rel(run_mixer(mixer, kv, h, portions, pages, run), want) < tol(run[1], 5e-5, 0.1), portions


@pytest.mark.parametrize("run", RUNS)
def test_far_key_at_page_borders(run):
    T, n = 300, 40
    mixer, m, W, kv, pages = soft_case(run, 1, 1, 24, 24, 1000, 0, rot=8, softcap=30.0, scale=1.0, width=n)
    h = torch.randn(T, n, generator=gen(3))
    for j, far in enumerate([0, 1, 31, 32, 33, 63, 64, 95, 127, 128, 150]):
        point_at(h, 270 + 2 * j, far, m, W, n, 10.0)
    h = h.to(BF16)
    want = plain.attention(W, m, "", h.double())
    for portions in ([T], [260] + [1] * 40, [33, 31, 32, 64, 96, 2, 42]):
        assert rel(run_mixer(mixer, kv, h, portions, pages, run), want) < tol(run[1], 5e-5, 0.1), portions


@pytest.mark.parametrize("run", RUNS)
@pytest.mark.parametrize("scale,softcap", [(0.05, 50.0), (1.5, 4.0), (8.0, 60.0), (3.0, 1.0)])
def test_sink_and_softcap(run, scale, softcap):
    """Scores around and far below 0 (the sink takes most of the weight), far inside and far beyond the cap, from the first token on."""
    T, n = 90, 40
    mixer, m, W, kv, pages = soft_case(run, 2, 1, 16, 24, 50, 4, rot=6, softcap=softcap, scale=scale, width=n)
    h = torch.randn(T, n, generator=gen(8))
    for t in range(30, T, 3):
        point_at(h, t, t - 20, m, W, n, -8.0)  # every visible key a low score, one of them very low
    h = h.to(BF16)
    want = plain.attention(W, m, "", h.double())
    for portions in ([T], [1] * T, [2, 40, 2, 46]):
        assert rel(run_mixer(mixer, kv, h, portions, pages, run), want) < tol(run[1], 5e-5, 0.12 if scale > 5 else 0.05), portions
    v = (h[:1].double() @ W["v"].double().T)[0]
    assert (want[0, :24] / v).abs().max() < 0.99  # a single visible key does not get the whole weight


# --------------------------------------------------------------------------------------------------- gated linear attention
# heads, dim, vdim, rank, tau, bias of the decay: widths that are no multiple of 8 or 16, several value slices, key widths of every kernel
# form, decays from nearly none to beyond what one exponent per chunk can hold (strong: the causal matrix is formed term by term)
GLA = [(1, 1, 1, 1, 1.0, 0.0), (2, 12, 20, 8, 4.0, 1.0), (3, 24, 72, 5, 16.0, 0.0), (1, 32, 130, 16, 1.0, -6.0), (2, 64, 64, 16, 16.0, 3.0), (2, 100, 40, 24, 2.0, -3.0),
       (1, 128, 200, 16, 8.0, 1.0), (1, 136, 24, 9, 1.0, -4.0), (2, 256, 64, 16, 16.0, 2.0), (1, 300, 40, 8, 4.0, 0.0), (1, 16, 520, 8, 4.0, 1.0)]


@pytest.mark.parametrize("run", RUNS)
@pytest.mark.parametrize("H,dk,dv,rank,tau,bias", GLA)
def test_gla_sizes(run, H, dk, dv, rank, tau, bias):
    """Whole prompt, ragged portions (across and inside chunks) and token by token, from a stale slot."""
    T = 150
    mixer, m, W, kv, pages = gla_case(run, H, dk, dv, rank, tau, bias)
    h = torch.randn(T, 48, generator=gen(5)).to(BF16)
    want = plain.gla(W, m, "", h.double(), 1e-5)
    for slot, portions in ((1, [T]), (2, [2, 3, 64, 2, 31, 48]), (3, [130] + [1] * 20), (1, [1] * 40 + [110])):
        e = rows_rel(run_mixer(mixer, kv, h, portions, pages, run, slot), want)
        # (with strong decays a head is hardly more than (q . k) v: where bf16 rows make q . k almost vanish, the norm behind it magnifies
        # their rounding)
        assert (e.max() < 5e-5) if run[1] == F32 else (e.quantile(0.9) < 3e-2 and e.max() < (3e-2 if bias >= 0 else 0.5)), portions
    # the state that is left behind
    S = torch.zeros(H, dk, dv, dtype=torch.float64)
    plain.gla(W, m, "", h.double(), 1e-5, S)
    for slot in (1, 2, 3):
        assert rel(kv.state["gla"][0][slot, :, :dk, :dv].flatten(1), S.flatten(1)) < tol(run[1], 5e-5, 2e-2)
    lost = plain.gla(W, m, "", h[75:].double(), 1e-5)
    if bias >= 0 and tau >= 4:
        assert rel(lost[:20], want[75:95]) > 0.3  # a state that is dropped on the way shows


@pytest.mark.parametrize("run", RUNS)
def test_gla_mixed_decays_in_one_chunk(run):
    """Channels that hardly decay beside channels that forget everything within a token, and zero decay logits."""
    mixer, m, W, kv, pages = gla_case(run, 2, 48, 32, 8, 1.0, 0.0)
    b = torch.linspace(-40, 40, 96).to(BF16)
    W["a2.b"] = b[torch.randperm(96, generator=gen(1))]
    mixer.load(*(W[n] for n in ("q", "k", "v", "g", "o", "a1", "a2", "a2.b", "norm")), k_pad=48)
    h = torch.randn(200, 48, generator=gen(2)).to(BF16)
    want = plain.gla(W, m, "", h.double(), 1e-5)
    for portions in ([200], [100, 2, 98], [150] + [1] * 50):
        assert rel(run_mixer(mixer, kv, h, portions, pages, run), want) < tol(run[1], 5e-5, 3e-2), portions


@pytest.mark.parametrize("run", RUNS)
@pytest.mark.parametrize("kind", ["soft", "gla"])
def test_unequal_sequences_in_one_batch(run, kind):
    """Each sequence as if it were alone: single tokens beside portions that start and end inside pages, windows and chunks."""
    device, dtype = run
    mixer, m, W, kv, pages = soft_case(run, 6, 2, 20, 12, 24, 7) if kind == "soft" else gla_case(run, 3, 20, 36, 8, 6.0, 1.0)
    if kind == "gla":
        kv.state["gla"][0] = torch.randn(9, *kv.state["gla"][0].shape[1:], device=device)
    fn = (lambda h: plain.attention(W, m, "", h)) if kind == "soft" else (lambda h: plain.gla(W, m, "", h, 1e-5))
    lens, starts = [1, 50, 3, 9, 1, 140, 8], [0, 0, 0, 0, 17, 0, 70]
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
    y = mixer.forward(torch.cat([h[s:] for h, s in zip(hs, starts)]).to(device, dtype), b, kv, 0, lambda _: _Stage())
    row = 0
    for h, s, n in zip(hs, starts, lens):
        assert rel(y[row : row + n].float(), fn(h.double())[s:]) < tol(dtype, 5e-5, 3e-2)
        row += n


# --------------------------------------------------------------------------------------------------- configuration, loop
def test_pass_starts_and_config_errors():
    loop = {"start": 1, "stop": 3, "times": 3}
    assert layer_run_order(5, loop) == (0, 1, 2, 1, 2, 1, 2, 3, 4) and loop_pass_starts(5, loop) == {1: 0, 3: 1, 5: 2} and loop_pass_starts(4, None) == {}
    assert loop_pass_starts(2, {"start": 0, "stop": 2, "times": 1}) == {0: 0}
    cfg = tiny_config("fopivik")
    c = parse_config(cfg)
    assert c.model_type == "fopivik" and c.extra["order"] == (0, 1, 0, 1, 2) and c.layer_types == ("gla", "sliding", "gla", "sliding", "gla")
    for path, value, msg in ((("layers", 0, "type"), "mamba", "unknown mixer"), (("layers", 1, "mlp", "kind"), "dense", "unknown feed-forward"),
                             (("loop", "stop"), 9, "loop")):
        bad = copy.deepcopy(cfg)
        d = bad
        for k in path[:-1]:
            d = d[k]
        d[path[-1]] = value
        with pytest.raises(ValueError, match=msg):
            parse_config(bad)
    t = build_tensors(cfg)
    for name, msg in (("l1.mix.k", "rows"), ("l0.mix.a2", "rows"), ("l0.mlp.router", "router"), ("loop.step", "loop")):
        with pytest.raises(ValueError, match=msg):
            build(cfg, ("cpu", F32), tensors=dict(t, **{name: t[name][:-1]}))
    from deliverance_b200.parallel.context import TensorParallelContext

    with pytest.raises(ValueError, match="tensor parallelism"):
        FopivikModel(c, "cpu", None, TensorParallelContext(0, 2, object()))


def test_state_slots_of_the_cache_manager():
    shapes = [{"a": (2, 3), "b": (4,)}, None, {"a": (1, 5)}]
    layout = {"layers": 3, "kv_heads": 1, "head_dim": 16, "layer_kinds": ["gla", "attention", "gla"], "state_shapes": shapes}
    kv = PagedKVCache(layout, 8, "cpu", F32, KvCacheSettings(), 2)
    assert kv.k[0] is None and kv.k[1] is not None and kv.state["a"][0].shape == (3, 2, 3) and kv.state["b"][0].shape == (3, 4) and 1 not in kv.state["a"]
    assert PagedKVCache.bytes_per_state_slot(layout) == 4 * (6 + 4 + 5) and PagedKVCache.bytes_per_page(layout, 32, F32) == 32 * 32 * 4
    s1, s2 = kv.alloc_state_slot(), kv.alloc_state_slot()
    assert {s1, s2} == {1, 2}  # 0 is scratch
    with pytest.raises(MemoryError):
        kv.alloc_state_slot()
    kv.state["a"][0][s1] = 5.0
    snap = kv.snapshot_state(s1)
    kv.restore_state(s2, snap)
    assert (kv.state["a"][0][s2] == 5).all()
    kv.free_state_slot(s1)
    with pytest.raises(RuntimeError):
        kv.free_state_slot(s1)
    with pytest.raises(RuntimeError):
        kv.free_state_slot(0)
    assert kv.alloc_state_slot() == s1 and (kv.state["a"][0][s1] == 0).all()


# --------------------------------------------------------------------------------------------------- whole models
def variety():
    soft = dict(heads=6, kv_heads=2, dim=20, vdim=28, rot_dims=12, window=24, keep_first=5, experts=5, top=2, ff=36)
    lin = dict(heads=3, dim=12, vdim=20, tau=4.0, rank=6, experts=4, top=1, ff=24)
    return {
        "tiny": tiny_config("fopivik"),
        "soft-only": fopivik_config(40, 97, [dict(soft, heads=1, kv_heads=1, experts=1, top=1, ff=8, softcap=3.0)], residual_mult=1.0, logit_softcap=2.0),
        "linear-only": fopivik_config(56, 120, [dict(lin, heads=1, dim=8, vdim=1, tau=1.0), dict(lin, experts=0)], loop={"start": 1, "stop": 2, "times": 1}, eps=1e-3),
        "looped-end": fopivik_config(72, 333, [dict(soft, window=7, keep_first=0, base=3000.0, scaling=BANDS), dict(lin, heads=2, dim=40, tau=32.0, experts=9, top=4),
                                               dict(soft, dim=64, vdim=16, rot_dims=8, window=300, keep_first=40, experts=0)], loop={"start": 0, "stop": 3, "times": 3},
                                     residual_mult=0.2),
        "wide-heads": fopivik_config(128, 512, [dict(soft, heads=4, kv_heads=1, dim=128, vdim=64, window=33, experts=3, top=3, ff=192), dict(lin, dim=64, vdim=96)]),
    }


@pytest.mark.parametrize("run", RUNS)
@pytest.mark.parametrize("name", list(variety()))
def test_model_portions_batches_reused_pages_and_slots(run, name):
    """Whole prompts, decoding, portions down to two tokens and mixed batches in a pool so small that pages and slots are used again; logits
    of every position against the plain statement, and the residual stream after every layer run for one prompt."""
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


@pytest.mark.parametrize("run", RUNS)
def test_paused_request_keeps_its_state(run):
    """A request that is left out of several steps goes on where it was, whatever ran in between."""
    cfg = tiny_config("fopivik", width=48)
    model, W = build(cfg, run, seed=8)
    req = {"a": tokens_of(60, 261, 1), "b": tokens_of(50, 261, 2), "c": tokens_of(40, 261, 3)}
    plan = [[("a", 33)], [("b", 20)], [("b", 1), ("c", 10)], [("b", 1), ("c", 1)], [("b", 1), ("c", 1)], [("c", 28), ("b", 27)], [("a", 1)], [("a", 26)]]
    for k, v in replay(engine_for(model, 320, max_seqs=3), plan, req).items():
        close_model(v, plain.forward(W, cfg, req[k]), run[1], k)


@pytest.mark.parametrize("run", RUNS)
def test_long_decoding(run):
    """Several hundred decoded tokens, far beyond every window and the context the rotation was made for."""
    cfg = fopivik_config(32, 64, [dict(heads=2, kv_heads=1, dim=8, vdim=12, rot_dims=4, window=40, keep_first=3, scaling=BANDS, experts=2, top=1, ff=16),
                                  dict(heads=2, dim=8, vdim=8, tau=8.0, experts=0)], loop={"start": 0, "stop": 2, "times": 2})
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
    cfg = tiny_config("fopivik", width=48)
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
    cfg = write_tiny_model(d, "fopivik", seed=6, dtype=BF16, sharded=True)
    assert detect_model(d) == "fopivik" and load_config(d).model_type == "fopivik"
    W = {n: WeightLoader(d).load(n) for n in WeightLoader(d).names()}
    prompt = tokens_of(20, 256, 8)
    clm = AutoModelForCausalLM.new_builder(d).with_device("cpu").build()
    p = GeneratorParameters(max_tokens=8, temperature=0.0)
    check_greedy(W, cfg, prompt, clm.generate(prompt, p).token_ids, F32)
    seeded = lambda: GeneratorParameters(max_tokens=8, temperature=0.8, top_k=20, top_p=0.9, seed=3)  # noqa: E731
    assert load_model(d, device="cpu").generate(prompt, seeded()).token_ids == clm.generate(prompt, seeded()).token_ids
    # log-probabilities are those of the soft-capped logits
    r = clm.generate(prompt, GeneratorParameters(max_tokens=1, temperature=0.0, logprobs=True))
    lp = torch.log_softmax(plain.forward(W, cfg, prompt)[-1], dim=-1)
    assert abs(r.sampler_returns[0].logprob - lp.max().item()) < 1e-3
    with pytest.raises(ValueError, match="LoRA"):
        clm.model.set_lora(object())


# --------------------------------------------------------------------------------------------------- trace replay program
@pytest.mark.parametrize("run", RUNS)
def test_trace_replay_program(run, tmp_path, monkeypatch, capsys):
    """Steps on standard input, soft-capped logits and ``done`` lines out; a finished request's pages and slot serve the next one."""
    from deliverance_b200.engine import replay as prog

    device, dtype = run
    d, out = str(tmp_path / "m"), str(tmp_path / "out")
    cfg = write_tiny_model(d, "fopivik", seed=1, dtype=BF16)
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
    assert got.abs().max() <= cfg["logit_softcap"]


# --------------------------------------------------------------------------------------------------- CUDA only
@gpu
def test_prompt_kernels_agree_with_the_row_forms_on_cuda():
    """Tensor-core prompt and decode attention against the CUDA-core rows form, chunked against recurrent linear attention, on inputs of
    several tiles and chunks; no kernel writes outside its outputs."""
    import deliverance_b200.ops.gla as gla_op
    import deliverance_b200.ops.grouped as gop

    run = ("cuda", BF16)
    h = torch.randn(700, 48, generator=gen(5)).to(BF16)
    ops.set_bounds_check(True)
    try:
        for H, G, dk, dv, window, keep in ((8, 2, 64, 64, 300, 100), (4, 4, 72, 128, 90, 3), (20, 1, 128, 40, 129, 200), (2, 1, 200, 256, 256, 64)):
            mixer, m, W, kv, pages = soft_case(run, H, G, dk, dv, window, keep)
            a = run_mixer(mixer, kv, h, [256, 424] + [1] * 20, pages, run)
            old, gop.GroupedShape.tensor_core = gop.GroupedShape.tensor_core, property(lambda self: False)
            try:
                b = run_mixer(mixer, kv, h, [256, 444], pages[::-1], run)
            finally:
                gop.GroupedShape.tensor_core = old
            assert rel(a, b) < 2e-2
            for splits in (2, 5, 16):
                mixer._splits = lambda batch: splits if batch.is_decode else 1  # noqa: B023
                assert rel(run_mixer(mixer, kv, h, [690] + [1] * 10, pages, run)[690:], b[690:]) < 2e-2
            ops.check_guards()
        for H, dk, dv, bias in ((2, 64, 128, 2.0), (1, 256, 192, 0.0), (3, 40, 24, -5.0)):
            mixer, m, W, kv, pages = gla_case(run, H, dk, dv, 16, 2.0, bias)
            a = run_mixer(mixer, kv, h, [256, 444], pages, run)
            old, gla_op.MAX_DK_CHUNKED = gla_op.MAX_DK_CHUNKED, 0
            try:
                b = run_mixer(mixer, kv, h, [300, 400], pages, run, 2)
            finally:
                gla_op.MAX_DK_CHUNKED = old
            assert rel(a, b) < 1e-2
            st = kv.state["gla"][0]
            assert rel(st[1].flatten(1), st[2].flatten(1).cpu()) < 1e-3  # fp32-grade state on the tensor cores
            ops.check_guards()
        ops.check_status()
    finally:
        ops.set_bounds_check(False)
