"""Gevovik decoder against a plain float64 statement of its equations (``gevovik_plain.py``), mechanism by mechanism and through the
engine. Every test runs on the CPU operator set in fp32 and, on a GPU box, on the CUDA kernels in fp32 and in bf16."""
import copy
import io
import json
import os

import pytest
import torch

import gevovik_plain as plain
from design_helpers import RUNS, Dict2Loader, _Stage, engine_for, gpu, rel, replay, tokens_of, tol
from deliverance_b200 import ops
from deliverance_b200.ckpt.loader import WeightLoader
from deliverance_b200.ckpt.tiny import build_tensors, gevovik_config, tiny_config, write_tiny_model
from deliverance_b200.config import load_config, parse_config
from deliverance_b200.kv.paged import KvCacheSettings, PagedKVCache
from deliverance_b200.models.batch import make_batch
from deliverance_b200.models.delta import GatedDeltaNet
from deliverance_b200.models.feed_forward import FeedForward
from deliverance_b200.models.gevovik import GevovikModel
from deliverance_b200.models.grouped import GroupedAttention
from deliverance_b200.models.latent import LatentAttention
from deliverance_b200.models.mamba import Mamba2Mixer
from deliverance_b200.models.side_by_side import SideBySideMixer
from deliverance_b200.ops import ref
from deliverance_b200.ops.delta import DeltaShape
from deliverance_b200.ops.grouped import GroupedShape, up8
from deliverance_b200.ops.latent import LatentShape
from deliverance_b200.ops.lightning import CHUNK
from deliverance_b200.ops.mamba import Mamba2Shape
from deliverance_b200.ops.short_conv import short_conv
from deliverance_b200.params import GeneratorParameters

F32, BF16 = torch.float32, torch.bfloat16
EPS = 1e-5
WIDTH = 48


def gen(seed):
    return torch.Generator().manual_seed(seed)


def randn(g, *s, k=1.0):
    return (torch.randn(*s, generator=g) * k).to(BF16)


def rows_rel(got, want):
    """Per-row RMS error over the RMS of the expected values."""
    got, want = got.detach().double().cpu(), want.double()
    return (got - want).pow(2).mean(-1).sqrt() / want.pow(2).mean().sqrt().clamp_min(1e-12)


def close(got, want, dtype, what=None, f32=5e-5, bf16=(2.5e-2, 8e-2)):
    """Every row in fp32; in bf16 nine rows of ten within the first bound and all within the second (rows whose heads nearly cancel in front of a norm
    carry their rounding magnified)."""
    e = rows_rel(got, want)
    assert e.max() < f32 if dtype == F32 else (e.quantile(0.9) < bf16[0] and e.max() < bf16[1]), (what, e.quantile(0.9), e.max())


def close_model(got, want, dtype, what=None):
    close(got, want, dtype, what, 2e-4, (6e-2, 0.25))


def build(cfg, run, seed=0, tensors=None):
    device, dtype = run
    W = tensors or build_tensors(cfg, seed, BF16)
    return GevovikModel(parse_config(cfg), device, dtype).load(Dict2Loader(W)), W


def pad_to(x, n):
    return torch.nn.functional.pad(x, (0, n - x.shape[-1]))


# --------------------------------------------------------------------------------------------------- embedding, norm, feed-forward, rotations
@pytest.mark.parametrize("run", RUNS)
@pytest.mark.parametrize("W", [8, 76, 257, 1024, 1600, 5000])
def test_norm_behind_a_sublayer(run, W):
    """One gain for all columns (and a vector): normed output added to the stream, the stream itself or its own norm handed on."""
    device, dtype = run
    g = gen(W)
    T, pitch, eps = 5, up8(W), 1e-3
    x, sub = torch.randn(T, W, generator=g) * 3 + 1, (torch.randn(T, pitch, generator=g) * 7 + 2).to(BF16)
    gain, last, vec = torch.tensor([0.6]), torch.tensor([-1.3]), torch.randn(W, generator=g)
    new = plain.add_normed(x.double(), sub[:, :W].double(), gain, eps)
    dev = lambda t: t.to(device)  # noqa: E731
    res = dev(x.clone())
    y = ops.sandwich_norm(res, sub.to(device, dtype), dev(gain), 1.0, None, eps, pitch, dtype, rms=True)
    assert rel(res, new) < 1e-5 and rel(y[:, :W], new) < tol(dtype, 1e-5, 6e-3) and (y[:, W:] == 0).all() and y.shape == (T, pitch)
    res = dev(x.clone())
    y = ops.sandwich_norm(res, sub.to(device, dtype), dev(gain), 1.0, dev(last), eps, pitch, dtype, rms=True)
    assert rel(y[:, :W], plain.rms(new, eps) * last.double()) < tol(dtype, 1e-5, 6e-3) and (y[:, W:] == 0).all()
    res = dev(x.clone())
    y = ops.sandwich_norm(res, sub.to(device, dtype), dev(vec), 0.5, dev(vec), eps, pitch, dtype, rms=True)
    new = x.double() + 0.5 * plain.rms(sub[:, :W].double(), eps) * vec.double()
    assert rel(res, new) < 1e-5 and rel(y[:, :W], plain.rms(new, eps) * vec.double()) < tol(dtype, 1e-5, 6e-3)


@pytest.mark.parametrize("run", RUNS)
@pytest.mark.parametrize("ff,width,T", [(64, 48, 33), (1, 40, 7), (36, 76, 150), (20, 257, 1)])
def test_squared_relu_feed_forward(run, ff, width, T):
    device, dtype = run
    g = gen(ff)
    W = {"up": randn(g, ff, width, k=2 * width ** -0.5), "down": randn(g, width, ff, k=ff ** -0.5)}
    h = randn(g, T, width)
    block = FeedForward("relu2").load(W["up"].to(dtype), W["down"].to(dtype), ff, up8(width), torch.device(device), dtype)
    got = block.forward(pad_to(h, up8(width)).to(device, dtype), lambda _: _Stage())
    assert rel(got, plain.dense(W, "", h.double())) < tol(dtype, 1e-5, 3e-2)


YARN = {"factor": 8.0, "original": 64, "fast": 16.0, "slow": 2.0}


@pytest.mark.parametrize("dims,base,scaling", [(16, 10000.0, None), (12, 500.0, YARN), (64, 3e5, dict(YARN, original=700, fast=24.0, slow=1.0)), (2, 100.0, YARN),
                                               (24, 700.0, dict(YARN, fast=1.0, slow=1.0, factor=3.0))])
def test_rotations(dims, base, scaling):
    rot, extra = {"dims": dims, "base": base, "scaling": scaling}, 3
    cos, sin = ref.yarn_rope_tables(dims, 200, base, scaling)
    x = torch.randn(200, 2, dims + extra, dtype=torch.float64, generator=gen(1))
    pos = torch.arange(200)
    got = ref.apply_rope(x, pos, cos, sin).double()
    assert torch.allclose(got, plain.rotate(x, rot, False), atol=2e-5) and torch.equal(got[..., dims:], x[..., dims:].float().double())
    assert torch.allclose(ref.apply_rope_pairs(x, pos, cos, sin).double(), plain.rotate(x, rot, True), atol=2e-5)


@pytest.mark.parametrize("run", RUNS)
def test_bigram_embedding(run):
    device, dtype = run
    g = gen(3)
    W = {"embed": randn(g, 50, 20), "bigram": randn(g, 12, 20)}
    cfg = {"embedding": {"scale": 2.5, "bigram": {"buckets": 11, "mul_prev": 13, "mul_cur": 5}}}
    toks = tokens_of(40, 50, 1)
    prev = torch.tensor([-1] + toks[:-1], dtype=torch.int32)
    row = torch.zeros(40, 24, dtype=dtype, device=device)
    got = ops.bigram_embedding(W["embed"].to(device, dtype), W["bigram"].to(device, dtype), torch.tensor(toks, dtype=torch.int32, device=device), prev.to(device), 13, 5,
                               2.5, row[:, :20])
    want = plain.embed(W, cfg, toks)
    assert rel(got, want) < 1e-6 and rel(row[:, :20], want) < tol(dtype, 1e-6, 5e-3) and (row[:, 20:] == 0).all()


# --------------------------------------------------------------------------------------------------- mixers
def cache_for(mixer, run, slots=3, pages=96, seed=0, paged=True):
    device, dtype = run
    c = mixer.cache_layout()
    layout = {"layers": 1, "kv_heads": c["heads"], "head_dim": c["k"], "layer_kinds": [mixer.kind], "v_dim_per_layer": [c["v"]], "state_shapes": [c["state"]],
              "paged": [paged]}
    kv = PagedKVCache(layout, pages, device, dtype, KvCacheSettings(enabled=False), slots)
    for t in (kv.k[0], kv.v[0]):
        if t is not None:
            t.uniform_(-3, 3)  # stale rows and states of earlier owners
    for layers in kv.state.values():
        layers[0].uniform_(-3, 3)
    return kv, (torch.randperm(pages - 1, generator=gen(seed)) + 1).tolist()


def run_mixer(mixer, kv, h, portions, pages, run, slot=1):
    """Feed rows of ``h`` in the given portion sizes; returns the mixer's output rows."""
    device, dtype = run
    out, at = [], 0
    for n in portions:
        b = make_batch([{"tokens": [0] * n, "start": at, "pages": pages, "state_slot": slot}], kv.page_size, device)
        out.append(mixer.forward(pad_to(h[at : at + n], up8(h.shape[1])).to(device, dtype), b, kv, 0, lambda _: _Stage()).float().cpu())
        at += n
    return torch.cat(out)


@pytest.mark.parametrize("run", RUNS)
@pytest.mark.parametrize("taps", [1, 2, 3, 4, 5, 7, 8])
def test_short_convolution(run, taps):
    """Portions shorter and longer than the filter, from a stale ring, several sequences at once: the inputs in front of a portion come from the ring."""
    device, dtype = run
    g = gen(taps)
    T, C, at = 61, 24, 8
    x, w, bias = randn(g, T, C), torch.randn(taps, C, generator=g), torch.randn(C, generator=g)
    for b in (None, bias):
        want = plain.silu(plain.causal_conv(x.double(), w.T.double(), b))
        for portions in ([T], [1] * T, [2, 3, 2, 1, 20, 1, 1, 31], [taps] * (T // taps) + [T % taps] * (T % taps > 0)):
            ring, got, lo = torch.full((4, taps, C), 9.0, device=device), [], 0
            ring[3] = -9.0
            for n in portions:
                batch = make_batch([{"tokens": [0], "start": 0, "pages": [2], "state_slot": 2}, {"tokens": [0] * n, "start": lo, "pages": [3, 4, 5], "state_slot": 3}], 32, device)
                rows = torch.cat([torch.ones(1, C), x[lo : lo + n].float()])
                p = torch.nn.functional.pad(rows, (at, 8)).to(device, dtype)
                got.append(short_conv(p, at, w.to(device), None if b is None else b.to(device), ring, batch)[1:].float().cpu())
                lo += n
            assert rel(torch.cat(got), want) < tol(dtype, 1e-5, 1e-2), portions
            last = torch.stack([x[T - 1 - (T - 1 - j) % taps] for j in range(taps)]).float()  # position p at row p mod taps
            assert torch.equal(ring[3].cpu(), last) and (ring[2][0] == 1).all() and (ring[2][1:] == 9).all() and (ring[1] == 9).all()


def mamba_case(run, H, dv, N, G, taps, ng, width=WIDTH, seed=0, slow=False):
    device, dtype = run
    g = gen(seed * 7919 + H * 31 + N)
    m = {"heads": H, "vdim": dv, "state": N, "groups": G, "conv": taps, "norm_groups": ng}
    I, GN = H * dv, G * N
    W = {"in": randn(g, 2 * I + 2 * GN + H, width, k=width ** -0.5), "conv": randn(g, I + 2 * GN, taps, k=0.5), "conv.b": randn(g, I + 2 * GN, k=0.3),
         "dt_bias": randn(g, H) - (6.0 if slow else 1.0), "A_log": torch.linspace(-4, 2.5, H).to(BF16), "D": randn(g, H), "norm": 1 + randn(g, I, k=0.3), "o": torch.eye(I).to(BF16)}
    mixer = Mamba2Mixer(Mamba2Shape(H, dv, N, G, taps, ng), EPS, torch.device(device), dtype)
    mixer.load(*(W[n] for n in ("in", "conv", "conv.b", "dt_bias", "A_log", "D", "norm", "o")), k_pad=up8(width))
    return (mixer, m, W) + cache_for(mixer, run, paged=False)


# heads, value columns, state, groups, taps, norm groups: sizes of one, widths that are no multiple of 8 or 16, several value slices, one and as many
# groups as heads, norm groups that cut heads, state sizes of every kernel form (32 / 64 / 128 / 256, beyond them)
SSD = [(1, 1, 1, 1, 1, 1), (4, 20, 12, 2, 4, 2), (6, 10, 20, 3, 3, 4), (3, 72, 64, 1, 2, 1), (8, 16, 128, 8, 4, 8), (2, 130, 40, 1, 5, 5), (5, 8, 200, 1, 4, 1), (2, 24, 264, 2, 8, 1),
       (4, 64, 128, 2, 4, 1)]


@pytest.mark.parametrize("run", RUNS)
@pytest.mark.parametrize("H,dv,N,G,taps,ng", SSD)
def test_mamba2_sizes(run, H, dv, N, G, taps, ng):
    """Whole prompt, ragged portions (across, inside and at the edges of chunks) and token by token, from stale slots."""
    T = 280
    mixer, m, W, kv, pages = mamba_case(run, H, dv, N, G, taps, ng)
    h = torch.randn(T, WIDTH, generator=gen(5)).to(BF16)
    want = plain.mamba2(W, m, "", h.double(), EPS)
    states = []
    for slot, portions in ((1, [T]), (2, [2, 3, CHUNK, 2, 97, 48]), (3, [250] + [1] * 30), (1, [CHUNK - 1, 2, 151]), (2, [1] * 40 + [240])):
        close(run_mixer(mixer, kv, h, portions, pages, run, slot), want, run[1], portions, bf16=(3e-2, 0.25))
        states.append(kv.state["ssm"][0][slot].float().cpu().flatten(1).clone())
    for st in states[1:]:
        assert rel(st, states[0]) < tol(run[1], 5e-5, 2e-2)
    st = kv.state["ssm"][0][1]
    assert (st[:, N:] == 0).all() and (st[:, :, dv:] == 0).all()
    lost = plain.mamba2(W, m, "", h[140:].double(), EPS)
    assert H * dv == 1 or rel(lost[:20], want[140:160]) > 0.02  # a state that is dropped on the way shows


def delta_case(run, H, G, dk, dv, taps, ra, rg, width=WIDTH, seed=0, a_log=None, mult=0.8):
    """The mixer alone: projections of its own around :meth:`GatedDeltaNet.heads`."""
    device, dtype = run
    g = gen(seed * 7919 + H * 31 + dk)
    m = {"heads": H, "kv_heads": G, "dim": dk, "vdim": dv, "conv": taps}
    W = {n: randn(g, r, width, k=width ** -0.5) for n, r in (("q", G * dk), ("k", G * dk), ("v", H * dv), ("b", H), ("a1", ra), ("g1", rg))}
    W.update({n + ".conv": randn(g, r, taps, k=0.5) for n, r in (("q", G * dk), ("k", G * dk), ("v", H * dv))})
    W.update({"a2": randn(g, H * dk, ra, k=ra ** -0.5), "g2": randn(g, H * dv, rg, k=rg ** -0.5), "A_log": (torch.linspace(-5, 0.5, H) if a_log is None else a_log).to(BF16),
              "dt_bias": randn(g, H * dk) - 2.0, "norm": 1 + randn(g, dv, k=0.3), "o": torch.eye(H * dv).to(BF16)})
    net = GatedDeltaNet(DeltaShape(H, G, dk, dv, taps, ra, rg), EPS, torch.device(device), dtype, mult)
    w_in, w_out = net.pack(*(W[n] for n in ("q", "k", "v", "b", "a1", "a2", "g1", "g2", "o")), [W[n + ".conv"] for n in ("q", "k", "v")], W["A_log"], W["dt_bias"], W["norm"])

    class Alone:
        kind = "attention"
        w_in_, w_out_ = (ops.LinearWeight(t.to(device, dtype).contiguous()) for t in (pad_to(w_in, up8(width)), w_out))

        def cache_layout(self):
            return {"heads": 1, "k": 8, "v": 8, "state": net.state_shapes()}

        def forward(self, x, batch, kv, run_, stage):
            p = ops.linear(x, self.w_in_)
            y = torch.empty(x.shape[0], net.shape.out_width, dtype=p.dtype, device=p.device)
            net.heads(p, batch, kv, run_, y, stage)
            return ops.linear(y, self.w_out_)

    mixer = Alone()
    return (mixer, m, W) + cache_for(mixer, run, paged=False) + (lambda h: mult * plain.gated_delta(W, m, "", h.double(), EPS),)


# heads, query / key heads, dim, vdim, taps, ranks: sizes of one, widths that are no multiple of 8 or 16, several value slices, shared query / key
# heads, key widths of every kernel form (32 / 64 / 128 / 256, beyond them), values beyond the fused decode step
DELTA = [(1, 1, 1, 1, 1, 1, 1), (4, 2, 20, 12, 3, 10, 6), (3, 3, 24, 72, 4, 8, 24), (6, 2, 64, 64, 4, 16, 16), (2, 1, 100, 40, 2, 5, 7), (2, 2, 128, 130, 4, 24, 8), (1, 1, 136, 24, 5, 8, 8),
         (2, 2, 256, 64, 4, 8, 8), (1, 1, 300, 20, 8, 8, 8), (1, 1, 16, 520, 4, 8, 8)]


@pytest.mark.parametrize("run", RUNS)
@pytest.mark.parametrize("H,G,dk,dv,taps,ra,rg", DELTA)
def test_gated_delta_sizes(run, H, G, dk, dv, taps, ra, rg):
    T = 180
    mixer, m, W, kv, pages, fn = delta_case(run, H, G, dk, dv, taps, ra, rg)
    h = torch.randn(T, WIDTH, generator=gen(5)).to(BF16)
    want = fn(h)
    states = []
    for slot, portions in ((1, [T]), (2, [2, 3, 32, 2, 93, 48]), (3, [150] + [1] * 30), (1, [31, 2, 147]), (2, [1] * 40 + [16, 15, 109])):
        close(run_mixer(mixer, kv, h, portions, pages, run, slot), want, run[1], portions, bf16=(3e-2, 0.25))
        states.append(kv.state["delta"][0][slot].float().cpu().flatten(1).clone())
    for st in states[1:]:
        assert rel(st, states[0]) < tol(run[1], 5e-5, 2e-2)
    st = kv.state["delta"][0][1]
    assert (st[:, dk:] == 0).all() and (st[:, :, dv:] == 0).all()
    assert H * dv == 1 or rel(fn(h[90:])[:10], want[90:100]) > 0.02  # a state that is dropped on the way shows


@pytest.mark.parametrize("run", RUNS)
@pytest.mark.parametrize("kind", ["mamba2", "delta"])
@pytest.mark.parametrize("pace", ["slow", "fast"])
def test_decays_from_none_to_all(run, kind, pace):
    """States that hardly decay over hundreds of tokens, and decays that leave nothing of a chunk (beyond the fp32 range of its running sums)."""
    T = 300
    if kind == "mamba2":
        mixer, m, W, kv, pages = mamba_case(run, 4, 16, 24, 1, 4, 1, slow=pace == "slow")
        W["A_log"] = (torch.linspace(-8, -4, 4) if pace == "slow" else torch.linspace(2, 5, 4)).to(BF16)
        mixer.load(*(W[n] for n in ("in", "conv", "conv.b", "dt_bias", "A_log", "D", "norm", "o")), k_pad=WIDTH)
        fn = lambda h: plain.mamba2(W, m, "", h.double(), EPS)  # noqa: E731
    else:
        mixer, m, W, kv, pages, fn = delta_case(run, 4, 2, 24, 16, 4, 8, 8, a_log=torch.linspace(-9, -5, 4) if pace == "slow" else torch.linspace(2, 5, 4))
    h = torch.randn(T, WIDTH, generator=gen(15)).to(BF16)
    want = fn(h)
    for portions in ([T], [270] + [1] * 30, [33, 31, 2, 130, 104]):
        close(run_mixer(mixer, kv, h, portions, pages, run), want, run[1], portions, f32=2e-4, bf16=(4e-2, 0.3))


@pytest.mark.parametrize("run", RUNS)
@pytest.mark.parametrize("kind", ["mamba2", "delta"])
def test_tokens_at_chunk_edges_stay_in_the_state(run, kind):
    """One token's input stands out by far, just in front of or behind the edge of a chunk or portion; later rows still see it."""
    T, edge = 300, CHUNK if kind == "mamba2" else 32
    if kind == "mamba2":
        mixer, m, W, kv, pages = mamba_case(run, 2, 24, 16, 1, 3, 1, slow=True)
        W["A_log"] = torch.tensor([-4.0, -6.0]).to(BF16)
        W["dt_bias"] = torch.tensor([-1.0, -2.0]).to(BF16)
        mixer.load(*(W[n] for n in ("in", "conv", "conv.b", "dt_bias", "A_log", "D", "norm", "o")), k_pad=WIDTH)
        fn = lambda h: plain.mamba2(W, m, "", h.double(), EPS)  # noqa: E731
    else:
        mixer, m, W, kv, pages, fn = delta_case(run, 2, 1, 24, 24, 3, 8, 8, a_log=torch.tensor([-5.0, -7.0]))
    for spot in (0, 1, edge - 1, edge, edge + 1, 2 * edge - 1, 2 * edge):
        h = torch.randn(T, WIDTH, generator=gen(spot)) * 0.3
        h[spot] *= 40.0
        h = h.to(BF16)
        want = fn(h)
        gone = h.clone()
        gone[spot] = 0
        after = slice(min(spot + 4, T - 5), min(spot + 60, T))
        assert rel(fn(gone)[after], want[after]) > 0.1
        for portions in ([T], [edge, edge, T - 2 * edge], [max(1, spot), T - max(1, spot)], [spot + 1, T - spot - 1], [270] + [1] * 30):
            close(run_mixer(mixer, kv, h, portions, pages, run), want, run[1], (spot, portions), f32=2e-4, bf16=(4e-2, 0.4))


def attention_case(run, H, G, dk, dv, window, rot=None, scale=None, width=WIDTH, seed=0, base=700.0, scaling=None, talk=None):
    device, dtype = run
    g = gen(seed * 7919 + H * 31 + dk)
    rot = dk // 2 * 2 if rot is None else rot
    m = {"heads": H, "kv_heads": G, "dim": dk, "vdim": dv, "scale": scale or dk ** -0.5, "rot": {"base": base, "dims": rot, "scaling": scaling}, "mask": {"size": window}}
    W = {"q": randn(g, H * dk, width, k=width ** -0.5), "k": randn(g, G * dk, width, k=width ** -0.5), "v": randn(g, G * dv, width, k=width ** -0.5),
         "g": randn(g, H, width, k=2 * width ** -0.5), "o": torch.eye(H * dv).to(BF16), "q.norm": 1 + randn(g, dk, k=0.3), "k.norm": 1 + randn(g, dk, k=0.3),
         "temp": 1.3 + randn(g, H, k=0.4), "talk": randn(g, H, H, k=H ** -0.5) + 0.5 * torch.eye(H).to(BF16) if talk is None else talk}
    cos, sin = ref.yarn_rope_tables(rot, 4096, base, scaling)
    mixer = GroupedAttention(GroupedShape(H, G, dk, dv, gate="heads", mixed=True), m["scale"], 0.0, window, 0, False, cos.to(device), sin.to(device), torch.device(device),
                             dtype, rotate="halves", eps=EPS)
    mixer.load(*(W[n] for n in ("q", "k", "v", "o")), k_pad=up8(width), g=W["g"], q_norm=W["q.norm"], k_norm=W["k.norm"],
               mix=W["talk"].float() * W["temp"].float().reshape(1, -1))
    return (mixer, m, W) + cache_for(mixer, run)


# heads, kv heads, dim, vdim, window, rotated: odd widths, one head, more than 16 heads per KV head, as many KV heads as heads, cache rows of every form of the
# prompt kernel (64 / 128 / 256 columns, pieces of rows up to 512 and beyond), values narrower and wider than keys, sizes outside the decode kernel
MIXED = [(1, 1, 2, 1, 5, 2), (6, 2, 20, 12, 40, 6), (4, 1, 64, 64, 33, 64), (6, 3, 72, 64, 64, 32), (20, 1, 16, 24, 50, 16), (36, 2, 24, 40, 100, 8), (8, 8, 40, 40, 32, 20),
         (4, 4, 128, 128, 70, 128), (5, 5, 104, 72, 45, 24), (6, 6, 128, 64, 96, 64), (10, 10, 64, 200, 31, 64), (2, 2, 264, 24, 20, 16), (3, 1, 24, 300, 60, 24), (66, 2, 8, 8, 40, 8)]


@pytest.mark.parametrize("run", RUNS)
@pytest.mark.parametrize("H,G,dk,dv,window,rot", MIXED)
def test_mixed_score_attention_sizes(run, H, G, dk, dv, window, rot):
    """Whole prompt, ragged portions and token by token: the same numbers, and those of the plain statement."""
    T = 141
    mixer, m, W, kv, pages = attention_case(run, H, G, dk, dv, window, rot, scaling=YARN if H % 4 == 0 else None)
    h = torch.randn(T, WIDTH, generator=gen(5)).to(BF16)
    want = plain.attention(W, m, "", h.double(), EPS)
    for portions in ([T], [2, 3, 37, 2, 70, 27], [129] + [1] * 12):
        close(run_mixer(mixer, kv, h, portions, pages, run), want, run[1], portions, bf16=(3e-2, 0.1))
        kv.k[0].uniform_(-3, 3), kv.v[0].uniform_(-3, 3)
        pages = pages[::-1]
    if H > 1:  # the mixing, its direction and the heads' own factors show
        for change in ({"talk": torch.eye(H)}, {"talk": W["talk"].T}, {"temp": W["temp"] * 0 + 1}):
            assert rel(plain.attention(dict(W, **change), m, "", h.double(), EPS), want) > 0.05


def point_at(h, t, far, W, m, strength):
    """Move row t of the input so that its query (one head) points at the key of row ``far``, norms and rotation undone."""
    d, key = m["dim"], plain.rms(W["k"].double() @ h[far].to(BF16).double(), EPS) * W["k.norm"].double()
    rows = torch.zeros(t + 1, 1, d, dtype=torch.float64)
    rows[far] = key
    key = plain.rotate(rows, m["rot"], False)[far, 0]
    turn = lambda v: plain.rotate(torch.cat([torch.zeros(t, 1, d, dtype=torch.float64), v.reshape(1, 1, d)]), m["rot"], False)[t, 0]  # noqa: E731
    back = torch.stack([turn(e) for e in torch.eye(d, dtype=torch.float64)])  # rows: rotated unit vectors (an orthogonal matrix times a constant)
    q = (back @ key) / W["q.norm"].double()
    h[t] = (strength * torch.linalg.lstsq(W["q"].double(), q.unsqueeze(1)).solution.squeeze(1) / q.norm()).float()


@pytest.mark.parametrize("run", RUNS)
@pytest.mark.parametrize("window", [0, 96])
def test_far_keys_and_window_edges(run, window):
    """One key per query stands out among hundreds: at page and tile borders, the first tokens, just inside and just outside the window."""
    T, n = 300, 40
    mixer, m, W, kv, pages = attention_case(run, 1, 1, 24, 24, window, 8, scale=2.0, width=n, talk=torch.tensor([[1.5]]).to(BF16))
    m["mask"]["size"] = window
    h = torch.randn(T, n, generator=gen(3))
    at = [270 + 2 * j for j in range(11)]
    far = [0, 1, 31, 32, 33, 63, 64, 95, 127, 128, 150] if not window else [t - back for t, back in zip(at, (95, 96, 94, 97, 95, 96, 64, 32, 31, 95, 1))]
    for t, f in zip(at, far):
        point_at(h, t, f, W, m, 6.0)
    h = h.to(BF16)
    want = plain.attention(W, m, "", h.double(), EPS)
    gate = torch.sigmoid(h.double() @ W["g"].double().T)
    v = h.double() @ W["v"].double().T
    for t, f in zip(at, far):
        decided = rel((want / gate)[t].unsqueeze(0), v[f].reshape(1, -1)) < 0.2
        assert decided == (not window or t - f < window), (t, f)
    for portions in ([T], [260] + [1] * 40, [33, 31, 32, 64, 96, 2, 42]):
        assert rel(run_mixer(mixer, kv, h, portions, pages, run), want) < tol(run[1], 5e-5, 0.1), portions


def latent_case(run, H, d, dr, dv, R, width=WIDTH, seed=0, scale=None, base=700.0, share=False):
    """One layer, or two (``share``), the second reading the first one's cache."""
    device, dtype = run
    g = gen(seed * 7919 + H * 31 + R)
    m = {"heads": H, "dim": d, "rot_dim": dr, "vdim": dv, "kv_rank": R, "rot": {"dims": dr, "base": base}, "scale": scale or (d + dr) ** -0.5}
    W = {"dkv": randn(g, R + dr, width, k=width ** -0.5), "dkv.norm": 1 + randn(g, R, k=0.3)}
    cos, sin = ref.rope_tables(dr, 4096, base)
    mixers = []
    for a in ("a.", "b.") if share else ("a.",):
        W.update({a + "q": randn(g, H * (d + dr), width, k=2 * width ** -0.5), a + "uk": randn(g, H * d, R, k=R ** -0.5), a + "uv": randn(g, H * dv, R, k=R ** -0.5),
                  a + "sink": torch.linspace(-1, 4, H).to(BF16), a + "o": torch.eye(H * dv).to(BF16)})
        own = a == "a."
        mixer = LatentAttention(LatentShape(H, d, dr, dv, R, gate=False, down=own), m["scale"], 0, EPS, cos.to(device), sin.to(device), torch.device(device), dtype, rotate="pairs")
        mixers.append(mixer.load(W[a + "q"], W["dkv"] if own else None, W["dkv.norm"] if own else None, W[a + "uk"], W[a + "uv"], None, k_pad=up8(width), sink=W[a + "sink"],
                                 o=W[a + "o"]))

    def fn(h, a="a."):
        return plain.latent_attention({n.removeprefix(a): t for n, t in W.items()}, m, "", h.double(), *plain.latent_rows(W, m, "", h.double(), EPS))

    return (mixers, m, W) + cache_for(mixers[0], run) + (fn,)


# heads, dim, rotated, vdim, latent: sizes of one, odd widths, more than 16 and 32 heads, latent sizes of every decode form, value widths of every
# prompt form and beyond them
LATENT = [(1, 1, 2, 1, 1), (3, 20, 6, 12, 40), (4, 32, 16, 32, 72), (20, 16, 8, 24, 130), (34, 8, 4, 8, 24), (2, 128, 64, 128, 256), (2, 72, 10, 200, 300), (2, 192, 64, 256, 512),
          (1, 300, 32, 20, 520)]


@pytest.mark.parametrize("run", RUNS)
@pytest.mark.parametrize("H,d,dr,dv,R", LATENT)
def test_latent_attention_with_sinks(run, H, d, dr, dv, R):
    T = 141
    (mixer,), m, W, kv, pages, fn = latent_case(run, H, d, dr, dv, R)
    h = torch.randn(T, WIDTH, generator=gen(5)).to(BF16)
    want = fn(h)
    for portions in ([T], [2, 3, 37, 2, 70, 27], [129] + [1] * 12):
        close(run_mixer(mixer, kv, h, portions, pages, run), want, run[1], portions, bf16=(3e-2, 0.1))
        kv.k[0].uniform_(-3, 3), kv.v[0].uniform_(-3, 3)
        pages = pages[::-1]
    W["a.sink"] = W["a.sink"] * 0 - 60
    assert rel(fn(h), want) > 0.01


@pytest.mark.parametrize("run", RUNS)
@pytest.mark.parametrize("scale,level", [(0.05, 0.0), (1.5, 6.0), (1.0, -8.0), (0.3, 30.0)])
def test_sink_levels(run, scale, level):
    """Sinks far above, around and far below the scores, one per head, from the first token on; they are not scaled. Many splits as well."""
    T = 90
    (mixer,), m, W, kv, pages, fn = latent_case(run, 3, 16, 6, 24, 32, scale=scale)
    W["a.sink"] = (torch.tensor([0.0, 1.0, -2.0]) + level).to(BF16)
    mixer.sink = W["a.sink"].float().to(run[0])
    h = torch.randn(T, WIDTH, generator=gen(8)).to(BF16)
    want = fn(h)
    for splits, portions in ((None, [T]), (None, [1] * T), (None, [2, 40, 2, 46]), (4, [80] + [1] * 10), (32, [80] + [1] * 10)):
        if splits:
            mixer._splits = lambda rows, span: splits  # noqa: B023
        # (below a sink that outweighs everything, an output's relative error is the scores' absolute one)
        assert rel(run_mixer(mixer, kv, h, portions, pages, run), want) < tol(run[1], 5e-5, 0.1 if level > 20 else 0.05), (splits, portions)


@pytest.mark.parametrize("run", RUNS)
def test_layer_on_another_layers_cache(run):
    """Queries, key and value weights of its own on the rows that the first layer wrote, in prompts, portions and decoding; nothing of the cache changes."""
    T = 100
    (first, second), m, W, kv, pages, fn = latent_case(run, 4, 24, 10, 20, 56, share=True)
    h, h2 = (torch.randn(T, WIDTH, generator=gen(5 + i)).to(BF16) for i in range(2))
    c, r = plain.latent_rows(W, m, "", h.double(), EPS)
    want = plain.latent_attention({n.removeprefix("b."): t for n, t in W.items()}, m, "", h2.double(), c, r)
    for portions in ([T], [60, 2, 38], [70] + [1] * 30):
        got, at = [], 0
        for n in portions:
            b = make_batch([{"tokens": [0] * n, "start": at, "pages": pages, "state_slot": 1}], kv.page_size, run[0])
            rows = lambda x: pad_to(x[at : at + n], WIDTH).to(*run)  # noqa: B023, E731
            first.forward(rows(h), b, kv, 0, lambda _: _Stage())
            before = kv.k[0].clone(), kv.v[0].clone()
            got.append(second.forward(rows(h2), b, kv, 0, lambda _: _Stage()).float().cpu())
            assert torch.equal(before[0], kv.k[0]) and torch.equal(before[1], kv.v[0])
            at += n
        close(torch.cat(got), want, run[1], portions, bf16=(3e-2, 0.1))


def parallel_case(run, width=WIDTH):
    left, lm, lw, _, _ = attention_case(run, 6, 2, 20, 12, 24, 10, width=width)
    g, (device, dtype) = gen(11), run
    _, rm, rw, _, _, _ = delta_case(run, 4, 2, 12, 20, 3, 10, 6, width=width)
    m = {"left": lm, "left_scale": 0.75, "right": rm, "right_scale": -0.5}
    eye = torch.eye(6 * 12 + 4 * 20).to(BF16)  # both outputs side by side: neither hides the other
    lw["o"], rw["o"] = eye[:, : 6 * 12], eye[:, 6 * 12 :]
    W = {**{"left." + n: t for n, t in lw.items()}, **{"right." + n: t for n, t in rw.items()}}
    left.mult = m["left_scale"]
    net = GatedDeltaNet(DeltaShape(4, 2, 12, 20, 3, 10, 6), EPS, torch.device(device), dtype, m["right_scale"])
    mixer = SideBySideMixer(left, net)
    mixer.load(left.pack(*(lw[n] for n in ("q", "k", "v", "o")), g=lw["g"], q_norm=lw["q.norm"], k_norm=lw["k.norm"], mix=lw["talk"].float() * lw["temp"].float().reshape(1, -1)),
               net.pack(*(rw[n] for n in ("q", "k", "v", "b", "a1", "a2", "g1", "g2", "o")), [rw[n + ".conv"] for n in ("q", "k", "v")], rw["A_log"], rw["dt_bias"], rw["norm"]),
               up8(width))
    return mixer, m, W


@pytest.mark.parametrize("run", RUNS)
@pytest.mark.parametrize("kind", ["mamba2", "parallel", "latent"])
def test_unequal_sequences_in_one_batch(run, kind):
    """Each sequence as if it were alone: single tokens beside portions that start and end inside pages and chunks."""
    device, dtype = run
    if kind == "mamba2":
        mixer, m, W, _, _ = mamba_case(run, 4, 20, 12, 2, 4, 2)
        fn = lambda h: plain.mamba2(W, m, "", h.double(), EPS)  # noqa: E731
    elif kind == "parallel":
        mixer, m, W = parallel_case(run)
        fn = lambda h: plain.parallel(W, m, "", h.double(), EPS)  # noqa: E731
    else:
        (mixer,), m, W, _, _, fn = latent_case(run, 3, 20, 6, 12, 40)
    kv, pages = cache_for(mixer, run, slots=9, paged=kind != "mamba2")
    lens, starts = [1, 50, 3, 9, 1, 140, 8, 2], [0, 0, 0, 0, 17, 0, 70, 131]
    hs = [torch.randn(s + n, WIDTH, generator=gen(100 + i)).to(BF16) for i, (s, n) in enumerate(zip(starts, lens))]
    own, at = [], 0
    for s, n in zip(starts, lens):
        k = (s + n + 31) // 32
        own.append(pages[at : at + k])
        at += k
    for i, (h, s, pg) in enumerate(zip(hs, starts, own)):
        if s:
            run_mixer(mixer, kv, h[:s], [s], pg, run, i + 1)
    for step in range(2):  # a mixed step, then a decode step of all of them
        take = lens if step == 0 else [1] * 8
        if step:
            starts = [s + n for s, n in zip(starts, lens)]
            hs = [torch.cat([h, torch.randn(1, WIDTH, generator=gen(200 + i)).to(BF16)]) for i, h in enumerate(hs)]
            own = [pg + ([pages[at + i]] if (s + 1 + 31) // 32 > len(pg) else []) for i, (pg, s) in enumerate(zip(own, starts))]
        b = make_batch([{"tokens": [0] * n, "start": s, "pages": pg, "state_slot": i + 1} for i, (n, s, pg) in enumerate(zip(take, starts, own))], kv.page_size, device)
        y = mixer.forward(torch.cat([h[s : s + n] for h, s, n in zip(hs, starts, take)]).to(device, dtype), b, kv, 0, lambda _: _Stage())
        row = 0
        for h, s, n in zip(hs, starts, take):
            want = fn(h)
            got = torch.cat([want[:s].float(), y[row : row + n].float().cpu()])
            close(got, want, dtype, (step, s, n), f32=1e-4, bf16=(6e-2, 0.3))
            row += n


# --------------------------------------------------------------------------------------------------- configuration, cache
def test_config_and_weight_errors():
    cfg = tiny_config("gevovik")
    c = parse_config(cfg)
    assert c.model_type == "gevovik" and c.num_layers == 6 and c.embedding_multiplier == 4.0 and not c.tie_word_embeddings
    for path, value, msg in ((("layers", 0, "type"), "gla", "unknown mixer"), (("layers", 1, "mlp", "kind"), "moe", "unknown feed-forward"), (("layers",), [], "no layers"),
                             (("layers", 3, "mixer", "kv_from"), 1, "kv_from"), (("layers", 3, "mixer", "kv_from"), 4, "kv_from"), (("layers", 3, "mixer", "kv_rank"), 48, "latent size"),
                             (("layers", 3, "mixer", "rot"), {"dims": 6, "base": 5.0}, "rotation")):
        bad = copy.deepcopy(cfg)
        d = bad
        for k in path[:-1]:
            d = d[k]
        d[path[-1]] = value
        with pytest.raises(ValueError, match=msg):
            parse_config(bad)
    t = build_tensors(cfg)
    for name, msg in (("l0.mix.q", "rows"), ("l0.mix.sink", "sinks"), ("l0.mix.dkv", "rows"), ("l1.mix.in", "projections"), ("l1.mix.conv", "conv"), ("l1.mix.norm", "norm"),
                      ("l1.mix.dt_bias", "dt_bias"), ("l2.mix.left.k", "rows"), ("l2.mix.left.q.norm", "norms"), ("l2.mix.right.v", "rows"), ("l2.mix.right.q.conv", "rows"),
                      ("l2.mix.right.norm", "norm"), ("l2.mix.right.g2", "rows"), ("l0.mlp.up", "width"), ("bigram", "bigram"), ("l2.mix.o", "output")):
        tensor = t.get(name, t["l0.mix.o"])
        with pytest.raises(ValueError, match=msg):
            build(cfg, ("cpu", F32), tensors=dict(t, **{name if name in t else "l0.mix.o": tensor[:-1]}))
    with pytest.raises(ValueError, match="one number"):
        build(cfg, ("cpu", F32), tensors=dict(t, **{"l0.norm1": torch.ones(3)}))
    with pytest.raises(ValueError, match="mixed scores"):
        build(cfg, ("cpu", F32), tensors=dict(t, **{"l2.mix.left.talk": torch.ones(5, 6)}))
    for make in (lambda: Mamba2Shape(4, 8, 8, 3, 4), lambda: Mamba2Shape(4, 8, 8, 2, 4, 5), lambda: Mamba2Shape(4, 8, 8, 2, 0), lambda: DeltaShape(4, 3, 8, 8, 4, 8, 8),
                 lambda: DeltaShape(4, 2, 8, 8, 0, 8, 8), lambda: GroupedShape(4, 2, 8, 8, tied=True, mixed=True)):
        with pytest.raises(ValueError):
            make()
    from deliverance_b200.parallel.context import TensorParallelContext

    with pytest.raises(ValueError, match="tensor parallelism"):
        GevovikModel(c, "cpu", None, TensorParallelContext(0, 2, object()))


def test_cache_layout_of_shared_and_stateful_layers():
    model, _ = build(tiny_config("gevovik"), ("cpu", F32))
    layout = model.kv_layout()
    kv = PagedKVCache(layout, 8, "cpu", F32, KvCacheSettings(), 2)
    assert kv.k[3] is kv.k[0] and kv.v[3] is kv.v[0] and kv.k[1] is None and kv.k[2].shape[1:] == (1, 32, 2 * 24)
    assert set(kv.state["conv"]) == {1, 2, 4, 5} and set(kv.state["ssm"]) == {1, 5} and set(kv.state["delta"]) == {2, 4}
    rows = 48 + 16 + 2 * 24 + 2 * 32 + 6 * 24 + 6 * 32  # latent 40 + 6 (padded to 16), wide rows of two and of six heads
    assert PagedKVCache.bytes_per_page(layout, 32, F32) == rows * 32 * 4


# --------------------------------------------------------------------------------------------------- whole models
def variety():
    ssd = dict(heads=6, vdim=12, state=20, groups=3, conv=4, norm_groups=2)
    both = dict(heads=6, kv_heads=2, dim=20, vdim=28, rot_dims=12, window=24, right=(4, 2, 12, 20, 3), ranks=(10, 6))
    lat = dict(heads=3, dim=20, rot_dim=6, vdim=12, kv_rank=40)
    return {
        "tiny": tiny_config("gevovik"),
        "mamba-only": gevovik_config(40, 97, [dict(ssd, heads=1, vdim=8, state=8, groups=1, conv=1, norm_groups=1, ff=8), dict(ssd, heads=2, groups=2, norm_groups=1, ff=0)], eps=1e-3,
                                     scale=1.0),
        "latent-only": gevovik_config(56, 120, [dict(lat, ff=20), dict(lat, heads=5, dim=8, vdim=24, kv_from=0, ff=16, base=10000.0), dict(lat, kv_rank=16, rot_dim=10, ff=0),
                                                dict(lat, kv_rank=16, rot_dim=10, heads=2, kv_from=2, ff=12), dict(lat, heads=1, kv_from=0, ff=0)], buckets=7, mul=(3, 1)),
        "parallel-only": gevovik_config(72, 333, [dict(both, heads=4, kv_heads=4, window=2, left_scale=1.0, right_scale=-1.5, right=(2, 1, 8, 24, 2), ff=24),
                                                  dict(both, heads=2, kv_heads=1, dim=64, rot_dims=64, window=1000, right=(3, 3, 33, 7, 5), ranks=(3, 30), ff=0)]),
        "wide-heads": gevovik_config(128, 512, [dict(ssd, heads=4, vdim=64, state=128, groups=1, norm_groups=1, ff=192),
                                                dict(both, heads=4, kv_heads=4, dim=128, vdim=64, window=64, right=(2, 2, 64, 96, 4), ranks=(24, 24), ff=64),
                                                dict(lat, heads=4, dim=64, rot_dim=32, vdim=64, kv_rank=192, ff=0)]),
    }


@pytest.mark.parametrize("run", RUNS)
@pytest.mark.parametrize("name", list(variety()))
def test_model_portions_batches_reused_pages_and_slots(run, name):
    """Whole prompts, decoding, portions down to two tokens and mixed batches in a pool so small that pages and slots are used again; logits
    of every position against the plain statement, and the residual stream after every layer for one prompt."""
    cfg = variety()[name]
    model, W = build(cfg, run, seed=3)
    V = cfg["vocab"]
    req = {f"r{i}": tokens_of(n, V, 10 + i) for i, n in enumerate((150, 97, 34, 1, 66, 23))}
    want, layers = {}, None
    for k, t in req.items():
        want[k], after = plain.forward(W, cfg, t, want_layers=True)
        layers = layers or after
    stream = []
    model.layer_hook = lambda i, stage, x: stream.append(x.float().cpu().clone()) if stage == "out" else None
    eng = engine_for(model, 192, max_seqs=4)
    got = replay(eng, [[(k, len(v))] for k, v in req.items()], req)
    model.layer_hook = None
    for k in req:
        close_model(got[k], want[k], run[1], k)
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
    cfg = tiny_config("gevovik")
    W = build_tensors(cfg, 3, BF16)
    toks = tokens_of(60, cfg["vocab"], 1)
    want = plain.forward(W, cfg, toks)
    zero, one = (lambda n: {n: W[n] * 0}), (lambda n: {n: W[n] * 0 + 1})  # noqa: E731
    for change in (zero("bigram"), one("l1.norm1"), one("final.norm"), zero("l1.mix.conv.b"), zero("l1.mix.D"), one("l1.mix.norm"), zero("l1.mix.dt_bias"), zero("l2.mix.left.g"),
                   one("l2.mix.left.q.norm"), one("l2.mix.left.temp"), {"l2.mix.left.talk": W["l2.mix.left.talk"].T}, zero("l2.mix.right.b"), zero("l2.mix.right.a2"),
                   zero("l2.mix.right.g2"), one("l2.mix.right.norm"), one("l0.mix.dkv.norm"), {"l0.mix.sink": W["l0.mix.sink"] * 0 - 50}, zero("l0.mlp.up")):
        assert rel(plain.forward(dict(W, **change), cfg, toks), want) > 1e-3, list(change)
    for path, value in ((("layers", 2, "mixer", "left", "mask", "size"), 23), (("layers", 2, "mixer", "left", "mask", "size"), 25), (("layers", 2, "mixer", "left_scale"), 0.9),
                        (("layers", 2, "mixer", "left", "rot", "scaling"), None), (("layers", 0, "mixer", "rot", "base"), 100.0), (("embedding", "scale"), 1.0),
                        (("embedding", "bigram", "mul_prev"), 14), (("layers", 1, "mixer", "norm_groups"), 1)):
        other = copy.deepcopy(cfg)
        d = other
        for k in path[:-1]:
            d = d[k]
        d[path[-1]] = value
        assert rel(plain.forward(W, other, toks), want) > 1e-4, path


@pytest.mark.parametrize("run", RUNS)
def test_paused_request_keeps_its_state(run):
    """A request that is left out of several steps goes on where it was, whatever ran in between."""
    cfg = tiny_config("gevovik", width=48)
    model, W = build(cfg, run, seed=8)
    req = {"a": tokens_of(60, 261, 1), "b": tokens_of(50, 261, 2), "c": tokens_of(40, 261, 3)}
    plan = [[("a", 33)], [("b", 20)], [("b", 1), ("c", 10)], [("b", 1), ("c", 1)], [("b", 1), ("c", 1)], [("c", 28), ("b", 27)], [("a", 1)], [("a", 26)]]
    for k, v in replay(engine_for(model, 320, max_seqs=3), plan, req).items():
        close_model(v, plain.forward(W, cfg, req[k]), run[1], k)


@pytest.mark.parametrize("run", RUNS)
def test_long_decoding(run):
    """Several hundred decoded tokens, over many pages, a window that moves along and many chunks of the states."""
    cfg = gevovik_config(32, 64, [dict(heads=2, vdim=8, state=8, groups=1, conv=4, ff=16), dict(heads=2, kv_heads=2, dim=10, window=40, right=(2, 1, 8, 8, 4), ff=8),
                                  dict(heads=2, dim=8, rot_dim=4, vdim=8, kv_rank=12, ff=0)])
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
        assert (gap < 0.15).float().mean() > 0.9 and gap.max() < 0.5


@pytest.mark.parametrize("run", RUNS)
@pytest.mark.parametrize("how", ["plain", "small-chunks", "preempted", "no-lookahead", "interleaved"])
def test_greedy_generation_through_the_scheduler(run, how):
    """Unequal prompts generated together: the tokens of the plain statement, whatever the scheduler does with them."""
    cfg = tiny_config("gevovik", width=48)
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
    cfg = write_tiny_model(d, "gevovik", seed=6, dtype=BF16, sharded=True)
    assert detect_model(d) == "gevovik" and load_config(d).model_type == "gevovik"
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
    cfg = write_tiny_model(d, "gevovik", seed=1, dtype=BF16)
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
    """Tensor-core prompt and decode attention with mixed scores against the CUDA-core rows form, chunked against recurrent Mamba-2 and gated delta
    rule, on inputs of several tiles and chunks; no kernel writes outside its outputs."""
    import deliverance_b200.ops.delta as dop
    import deliverance_b200.ops.grouped as gop
    import deliverance_b200.ops.mamba as mop

    run = ("cuda", BF16)
    h = torch.randn(700, WIDTH, generator=gen(5)).to(BF16)

    def row_forms(fn):
        """The rows kernel for attention, token by token for the recurrences."""
        e = ops.require_ext()

        class Rows:
            def __getattr__(self, n):
                return {"prefill_wide_tile_rows": lambda *a: 0, "mixed_decode_ok": lambda *a: False}.get(n) or getattr(e, n)

        old = ops.require_ext, mop.MAX_STATE_CHUNKED, dop.MAX_DK_CHUNKED
        gop.ops.require_ext, mop.MAX_STATE_CHUNKED, dop.MAX_DK_CHUNKED = (lambda: Rows()), 0, 0
        try:
            return fn()
        finally:
            gop.ops.require_ext, mop.MAX_STATE_CHUNKED, dop.MAX_DK_CHUNKED = old

    wide = dop.MAX_DK_CHUNK32
    ops.set_bounds_check(True)
    try:
        cases = [("attention",) + attention_case(run, *a) for a in ((8, 2, 64, 64, 100), (16, 4, 128, 128, 256), (24, 4, 128, 128, 0), (16, 8, 128, 64, 300), (8, 1, 40, 256, 77))]
        cases += [("ssm",) + mamba_case(run, *a) for a in ((8, 64, 128, 1, 4, 1), (4, 96, 64, 2, 4, 2), (2, 40, 200, 1, 3, 1))]
        cases += [("delta",) + delta_case(run, *a)[:5] for a in ((4, 2, 128, 128, 4, 16, 16), (2, 2, 64, 192, 4, 8, 8), (2, 1, 256, 64, 3, 8, 8))]
        cases += [("delta 16",) + delta_case(run, *a)[:5] for a in ((4, 2, 128, 128, 4, 16, 16), (2, 2, 24, 48, 4, 8, 8), (2, 1, 56, 64, 3, 8, 8))]
        for name, mixer, m, W, kv, pages in cases:
            name, _, short = name.partition(" ")  # chunks of 16 tokens where the batch would get 32
            dop.MAX_DK_CHUNK32 = 0 if short else wide
            a = run_mixer(mixer, kv, h, [256, 424] + [1] * 20, pages, run)
            b = row_forms(lambda: run_mixer(mixer, kv, h, [256, 444], pages[::-1], run, 2))  # noqa: B023
            e = rows_rel(a, b)
            assert e.quantile(0.9) < 3e-2 and e.max() < 0.2, (name, e.max())
            if name != "attention":
                st = kv.state[name][0]
                assert rel(st[1].flatten(1), st[2].flatten(1).cpu()) < 5e-3  # fp32-grade state on the tensor cores
            else:
                for splits in (2, 5, 16):
                    mixer._splits = lambda batch: splits if batch.is_decode else 1  # noqa: B023
                    assert rel(run_mixer(mixer, kv, h, [690] + [1] * 10, pages, run)[690:], b[690:]) < 3e-2
            ops.check_guards()
        ops.check_status()
    finally:
        dop.MAX_DK_CHUNK32 = wide
        ops.set_bounds_check(False)
