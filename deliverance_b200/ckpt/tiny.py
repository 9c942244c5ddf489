"""Random-weight checkpoints with the real tensor names and shape formulas of every supported family.

Used by the tests (tiny shapes) and by the benchmarks (full benchmark shapes, random-init N(0, 0.02)), mirroring the
reference's "HF-ported" test suites that write a synthetic model directory and load it through the normal loader
(core/src/test/.../model/qwen3/Qwen3HfTextModelPortedTest.java:86-93).
"""
from __future__ import annotations

import json
import os
from typing import Optional

import torch

from ..config import config_model_type
from .safetensors_io import write_safetensors, write_sharded


def _rand(gen, *shape, std=0.02, dtype=torch.float32):
    return (torch.randn(*shape, generator=gen, dtype=torch.float32) * std).to(dtype)


def fatotar_config(width: int, vocab: int, layers: list, loop: Optional[dict] = None, eps: float = 1e-5, scale: float = 2.0,
                   bigram: Optional[dict] = None, **extra) -> dict:
    """``config.json`` of a Fatotar model. ``layers``: one dict of sizes per layer (``heads, dim, rot_dim, vdim, kv_rank, window, base,
    scaling, ff``, score ``scale``; ``ff`` 0 = no feed-forward)."""
    out = []
    for L in layers:
        rot = {"base": L.get("base", 10000.0), "dims": L["rot_dim"]}
        if L.get("scaling"):
            rot["scaling"] = L["scaling"]
        out.append({"type": "latent_attention", "mlp": {"kind": "dense", "ff": L["ff"]} if L.get("ff") else None,
                    "mixer": {"heads": L["heads"], "dim": L["dim"], "rot_dim": L["rot_dim"], "vdim": L["vdim"], "kv_rank": L["kv_rank"],
                              "mask": {"size": L["window"]}, "rot": rot, "scale": L.get("scale", (L["dim"] + L["rot_dim"]) ** -0.5)}})
    cfg = {"architecture": "Fatotar", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": out,
           "embedding": {"scale": scale, "bigram": bigram or {"buckets": 211, "mul_prev": 31, "mul_cur": 7}}}
    if loop:
        cfg["loop"] = loop
    cfg.update(extra)
    return cfg


def fatotar_shapes(cfg: dict) -> dict:
    """Tensor name -> shape of a Fatotar checkpoint."""
    W, V = cfg["width"], cfg["vocab"]
    s = {"embed": (V, W), "head": (V, W), "final.norm": (W,), "final.norm.b": (W,), "bigram": (cfg["embedding"]["bigram"]["buckets"] + 1, W)}
    for i, L in enumerate(cfg["layers"]):
        m, p = L["mixer"], f"l{i}."
        H, dn, dr, dv, R = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
        s.update({p + "norm1": (W,), p + "norm1.b": (W,), p + "mix.q": (H * (dn + dr), W), p + "mix.dkv": (R + dr, W), p + "mix.dkv.norm": (R,),
                  p + "mix.uk": (H * dn, R), p + "mix.uv": (H * dv, R), p + "mix.g": (H * dv, W), p + "mix.o": (W, H * dv)})
        if L.get("mlp"):
            F = L["mlp"]["ff"]
            s.update({p + "norm2": (W,), p + "norm2.b": (W,), p + "mlp.gate": (F, W), p + "mlp.gate.b": (F,), p + "mlp.up": (F, W), p + "mlp.up.b": (F,),
                      p + "mlp.down": (W, F), p + "mlp.down.b": (W,)})
    return s


def fatotar_is_norm(name: str) -> bool:
    return name.rsplit(".", 1)[-1].startswith("norm")


def _fatotar_tensors(cfg: dict, seed: int, dtype) -> dict:
    """Random weights with projections scaled by their fan-in, so that every mechanism moves the output."""
    g = torch.Generator().manual_seed(seed)
    t = {}
    for name, shape in fatotar_shapes(cfg).items():
        r = torch.randn(*shape, generator=g, dtype=torch.float32)
        if fatotar_is_norm(name):
            r = 1.0 + 0.2 * r
        elif len(shape) == 1:
            r = 0.2 * r
        elif name not in ("embed", "bigram"):
            r = r * shape[1] ** -0.5
        t[name] = r.to(dtype)
    return t


def fopivik_config(width: int, vocab: int, layers: list, loop: Optional[dict] = None, eps: float = 1e-5, residual_mult: float = 0.5,
                   logit_softcap: float = 12.0, **extra) -> dict:
    """``config.json`` of a Fopivik model. ``layers``: one dict of sizes per layer; softmax attention has ``heads, kv_heads, dim, vdim, window,
    keep_first`` (and ``rot_dims, base, scaling, softcap, scale``), gated linear attention ``heads, dim, vdim, tau`` (``rank`` columns of the
    decay projection); ``experts, top, ff`` for the routed experts (``experts`` 0 = no feed-forward)."""
    out, ranks = [], {}
    for i, L in enumerate(layers):
        mlp = {"kind": "moe", "expert": {"ff": L["ff"]}, "router": {"experts": L["experts"], "top": L["top"]}} if L.get("experts") else None
        if "tau" in L:
            mixer = {k: L[k] for k in ("heads", "dim", "vdim", "tau")}
            ranks[i] = L.get("rank", 8)
            out.append({"type": "gla", "mixer": mixer, "mlp": mlp})
            continue
        rot = {"base": L.get("base", 10000.0), "dims": L.get("rot_dims", L["dim"])}
        if L.get("scaling"):
            rot["scaling"] = L["scaling"]
        mixer = {k: L[k] for k in ("heads", "kv_heads", "dim", "vdim")}
        mixer.update(mask={"size": L["window"], "keep_first": L.get("keep_first", 0)}, rot=rot, scale=L.get("scale", L["dim"] ** -0.5),
                     softcap=L.get("softcap", 30.0))
        out.append({"type": "attention", "mixer": mixer, "mlp": mlp})
    cfg = {"architecture": "Fopivik", "vocab": vocab, "width": width, "norm": {"eps": eps}, "residual_mult": residual_mult,
           "logit_softcap": logit_softcap, "layers": out}
    if loop:
        cfg["loop"] = loop
    cfg.update(extra)
    cfg["_decay_ranks"] = ranks  # (shapes of random checkpoints only; a model reads the rank off its tensors)
    return cfg


def fopivik_shapes(cfg: dict) -> dict:
    """Tensor name -> shape of a Fopivik checkpoint."""
    W, V = cfg["width"], cfg["vocab"]
    s = {"embed": (V, W), "head": (V, W), "final.norm": (W,)}
    if cfg.get("loop"):
        s.update({"loop.in": (W, 2 * W), "loop.step": (cfg["loop"]["times"], W)})
    ranks = {int(k): v for k, v in (cfg.get("_decay_ranks") or {}).items()}
    for i, L in enumerate(cfg["layers"]):
        m, p = L["mixer"], f"l{i}."
        H, dk, dv = m["heads"], m["dim"], m["vdim"]
        G = m.get("kv_heads", H)
        s.update({p + "norm1": (W,), p + "norm1b": (W,), p + "mix.q": (H * dk, W), p + "mix.k": (G * dk, W), p + "mix.v": (G * dv, W), p + "mix.o": (W, H * dv)})
        if L["type"] == "gla":
            R = ranks.get(i, 8)
            s.update({p + "mix.g": (H * dv, W), p + "mix.norm": (dv,), p + "mix.a1": (R, W), p + "mix.a2": (H * dk, R), p + "mix.a2.b": (H * dk,)})
        if L.get("mlp"):
            F, E = L["mlp"]["expert"]["ff"], L["mlp"]["router"]["experts"]
            s.update({p + "norm2": (W,), p + "norm2b": (W,), p + "mlp.router": (E, W)})
            for e in range(E):
                s.update({f"{p}mlp.e{e}.gate": (F, W), f"{p}mlp.e{e}.up": (F, W), f"{p}mlp.e{e}.down": (W, F)})
    return s


def fopivik_is_norm(name: str) -> bool:
    return name.rsplit(".", 1)[-1].startswith("norm")


def _fopivik_tensors(cfg: dict, seed: int, dtype) -> dict:
    """Random weights with projections scaled by their fan-in, wide router logits and decays spread over fast and slow channels."""
    g = torch.Generator().manual_seed(seed)
    t = {}
    for name, shape in fopivik_shapes(cfg).items():
        r = torch.randn(*shape, generator=g, dtype=torch.float32)
        if fopivik_is_norm(name):
            r = 1.0 + 0.2 * r
        elif name.endswith(".a2.b"):
            r = 2.0 * r + 1.0
        elif len(shape) == 2 and name not in ("embed", "loop.step"):
            r = r * shape[1] ** -0.5 * (2.0 if name.endswith("router") else 1.0)
        t[name] = r.to(dtype)
    return t


def dubozen_config(width: int, vocab: int, layers: list, streams: int = 2, eps: float = 1e-5, **extra) -> dict:
    """``config.json`` of a Dubozen model. ``layers``: one dict of sizes per layer: ``heads, kv_heads, dim`` of the softmax attention with ``vdim``
    (and ``v_mix``), or with ``right`` = ``(heads, dim, vdim, decays)`` of the lightning attention beside it (and ``left_scale, right_scale``);
    ``rot_dims, base, scale``; ``ff`` alone for a dense feed-forward, with ``experts, top`` (and ``groups, keep, route_scale``) for routed experts,
    ``ff`` 0 = none."""
    out = []
    for L in layers:
        mlp = None
        if L.get("ff") and L.get("experts"):
            mlp = {"kind": "moe", "expert": {"ff": L["ff"]}, "router": {"experts": L["experts"], "top": L["top"], "scale": L.get("route_scale", 1.5),
                                                                        "groups": {"count": L.get("groups", 1), "keep": L.get("keep", 1)}}}
        elif L.get("ff"):
            mlp = {"kind": "dense", "ff": L["ff"]}
        soft = {k: L[k] for k in ("heads", "kv_heads", "dim")}
        soft.update(vdim=L.get("vdim", L["dim"]), rot={"base": L.get("base", 10000.0), "dims": L.get("rot_dims", L["dim"] // 2 * 2)},
                    scale=L.get("scale", L["dim"] ** -0.5))
        if L.get("right"):
            h, dk, dv, decay = L["right"]
            mixer = {"left": soft, "left_scale": L.get("left_scale", 0.7), "right": {"heads": h, "dim": dk, "vdim": dv, "decay": list(decay)},
                     "right_scale": L.get("right_scale", 0.4)}
            out.append({"type": "parallel", "mixer": mixer, "mlp": mlp})
        else:
            out.append({"type": "attention", "mixer": dict(soft, v_mix=L.get("v_mix", True)), "mlp": mlp})
    cfg = {"architecture": "Dubozen", "vocab": vocab, "width": width, "streams": streams, "norm": {"eps": eps}, "layers": out}
    cfg.update(extra)
    return cfg


def dubozen_shapes(cfg: dict) -> dict:
    """Tensor name -> shape of a Dubozen checkpoint."""
    W, V, S = cfg["width"], cfg["vocab"], cfg["streams"]
    s = {"embed": (V, W), "embed.norm": (W,), "final.norm": (W,)}
    for i, L in enumerate(cfg["layers"]):
        m, p = L["mixer"], f"l{i}."
        for q in (1, 2) if L.get("mlp") else (1,):
            s.update({f"{p}norm{q}": (W,), f"{p}hc{q}.in": (S,), f"{p}hc{q}.out": (S,), f"{p}hc{q}.mix": (S, S)})
        soft = m["left"] if L["type"] == "parallel" else m
        H, G, dk, dv = soft["heads"], soft["kv_heads"], soft["dim"], soft["vdim"]
        if L["type"] == "parallel":
            a, b, r = p + "mix.left.", p + "mix.right.", m["right"]
            R, rk, rv = r["heads"], r["dim"], r["vdim"]
            s.update({a + "q": (H * dk, W), a + "k": (G * dk, W), a + "q.norm": (dk,), a + "k.norm": (dk,), a + "g": (H, W), a + "o": (W, H * dk),
                      b + "q": (R * rk, W), b + "k": (R * rk, W), b + "v": (R * rv, W), b + "g": (R * rv, W), b + "o": (W, R * rv), b + "norm": (R * rv,)})
        else:
            a = p + "mix."
            s.update({a + "q": (H * dk, W), a + "k": (G * dk, W), a + "v": (G * dv, W), a + "g": (H * dv, W), a + "o": (W, H * dv), a + "sink": (H,)})
            if m.get("v_mix"):
                s[a + "vmix"] = ()
        if L.get("mlp") and L["mlp"]["kind"] == "dense":
            F = L["mlp"]["ff"]
            s.update({p + "mlp.gate": (F, W), p + "mlp.up": (F, W), p + "mlp.down": (W, F)})
        elif L.get("mlp"):
            F, E = L["mlp"]["expert"]["ff"], L["mlp"]["router"]["experts"]
            s.update({p + "mlp.router": (E, W), p + "mlp.correction": (E,)})
            for e in range(E):
                s.update({f"{p}mlp.e{e}.gate": (F, W), f"{p}mlp.e{e}.up": (F, W), f"{p}mlp.e{e}.down": (W, F)})
    return s


def dubozen_value(name: str, r, cfg: dict):
    """Weight ``name`` from standard normal numbers ``r`` of its shape: projections scaled by their fan-in, mixes near the identity, every
    mechanism moving the output."""
    last = name.rsplit(".", 1)[-1]
    if "norm" in last:
        return 1.0 + 0.2 * r
    if last == "vmix":
        return 0.4 + 0.1 * r
    if last == "sink":
        return 1.0 + r
    if last == "correction":
        return 0.3 * r - 1.0  # (negative choice scores)
    if ".hc" in name:
        if last == "mix":
            return 0.9 * torch.eye(r.shape[0], dtype=r.dtype, device=r.device) + 0.15 * r
        return (0.7 + 0.3 * r) / (cfg["streams"] ** 0.5 if last == "in" else 1.0)
    if len(r.shape) == 2 and name != "embed":
        return r * r.shape[1] ** -0.5 * (2.0 if last == "router" else 1.0)
    return r


def _dubozen_tensors(cfg: dict, seed: int, dtype) -> dict:
    g = torch.Generator().manual_seed(seed)
    return {n: dubozen_value(n, torch.randn(shape, generator=g, dtype=torch.float32), cfg).to(dtype) for n, shape in dubozen_shapes(cfg).items()}


def gevovik_config(width: int, vocab: int, layers: list, eps: float = 1e-5, scale: float = 4.0, buckets: int = 61, mul: tuple = (13, 5), **extra) -> dict:
    """``config.json`` of a Gevovik model. ``layers``: one dict of sizes per layer, told apart by their keys: ``state`` (Mamba-2: ``heads, vdim, state,
    groups, conv, norm_groups``), ``right`` = ``(heads, kv_heads, dim, vdim, conv)`` of the gated delta rule beside attention (``heads, kv_heads, dim,
    vdim, window, rot_dims, base, scaling, scale, left_scale, right_scale``; ``ranks`` = sizes of the two low-rank projections, kept in the weights
    only), else latent attention (``heads, dim, rot_dim, vdim, kv_rank, base, scale, kv_from``). ``ff`` 0 = no feed-forward."""
    out, ranks = [], {}
    for i, L in enumerate(layers):
        mlp = {"kind": "dense", "ff": L["ff"]} if L.get("ff") else None
        if "state" in L:
            kind, m = "mamba2", {k: L[k] for k in ("heads", "vdim", "state", "groups", "conv")}
            m["norm_groups"] = L.get("norm_groups", 1)
        elif "right" in L:
            kind = "parallel"
            left = {k: L[k] for k in ("heads", "kv_heads", "dim")}
            rot = {"dims": L.get("rot_dims", L["dim"] // 2 * 2), "base": L.get("base", 10000.0)}
            if L.get("scaling"):
                rot["scaling"] = L["scaling"]
            left.update(vdim=L.get("vdim", L["dim"]), rot=rot, scale=L.get("scale", L["dim"] ** -0.5), mask={"size": L["window"]})
            m = {"left": left, "left_scale": L.get("left_scale", 0.7), "right": dict(zip(("heads", "kv_heads", "dim", "vdim", "conv"), L["right"])),
                 "right_scale": L.get("right_scale", 0.8)}
            ranks[str(i)] = list(L.get("ranks", (8, 8)))
        else:
            kind, m = "latent_attention", {k: L[k] for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank")}
            m.update(rot={"dims": L["rot_dim"], "base": L.get("base", 10000.0)}, scale=L.get("scale", (L["dim"] + L["rot_dim"]) ** -0.5))
            if L.get("kv_from") is not None:
                m["kv_from"] = L["kv_from"]
        out.append({"type": kind, "mixer": m, "mlp": mlp})
    cfg = {"architecture": "Gevovik", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": out, "_ranks": ranks,
           "embedding": {"scale": scale, "bigram": {"buckets": buckets, "mul_prev": mul[0], "mul_cur": mul[1]}}}
    cfg.update(extra)
    return cfg


def gevovik_shapes(cfg: dict) -> dict:
    """Tensor name -> shape of a Gevovik checkpoint."""
    W, V = cfg["width"], cfg["vocab"]
    s = {"embed": (V, W), "final.norm": (), "head": (V, W)}
    if cfg["embedding"].get("bigram"):
        s["bigram"] = (cfg["embedding"]["bigram"]["buckets"] + 1, W)
    for i, L in enumerate(cfg["layers"]):
        m, p = L["mixer"], f"l{i}."
        a = p + "mix."
        s[p + "norm1"] = ()
        if L["type"] == "mamba2":
            H, I, GN = m["heads"], m["heads"] * m["vdim"], m["groups"] * m["state"]
            s.update({a + "in": (2 * I + 2 * GN + H, W), a + "conv": (I + 2 * GN, m["conv"]), a + "conv.b": (I + 2 * GN,), a + "dt_bias": (H,), a + "A_log": (H,),
                      a + "D": (H,), a + "norm": (I,), a + "o": (W, I)})
        elif L["type"] == "parallel":
            l, r = m["left"], m["right"]
            H, G, dk, dv, b = l["heads"], l["kv_heads"], l["dim"], l["vdim"], a + "left."
            s.update({b + "q": (H * dk, W), b + "k": (G * dk, W), b + "v": (G * dv, W), b + "q.norm": (dk,), b + "k.norm": (dk,), b + "talk": (H, H), b + "temp": (H,),
                      b + "g": (H, W), b + "o": (W, H * dv)})
            H, G, dk, dv, b = r["heads"], r["kv_heads"], r["dim"], r["vdim"], a + "right."
            ra, rg = cfg["_ranks"][str(i)]
            for n, rows in (("q", G * dk), ("k", G * dk), ("v", H * dv)):
                s.update({b + n: (rows, W), f"{b}{n}.conv": (rows, r["conv"])})
            s.update({b + "b": (H, W), b + "A_log": (H,), b + "norm": (dv,), b + "a1": (ra, W), b + "a2": (H * dk, ra), b + "dt_bias": (H * dk,), b + "g1": (rg, W),
                      b + "g2": (H * dv, rg), b + "o": (W, H * dv)})
        else:
            H, d, dr, dv, R = (m[k] for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank"))
            s.update({a + "q": (H * (d + dr), W), a + "uk": (H * d, R), a + "uv": (H * dv, R), a + "sink": (H,), a + "o": (W, H * dv)})
            if m.get("kv_from") is None:
                s.update({a + "dkv": (R + dr, W), a + "dkv.norm": (R,)})
        if L.get("mlp"):
            F = L["mlp"]["ff"]
            s.update({p + "norm2": (), p + "mlp.up": (F, W), p + "mlp.down": (W, F)})
    return s


def gevovik_value(name: str, r, cfg: dict):
    """Weight ``name`` from standard normal numbers ``r`` of its shape: projections scaled by their fan-in, decays from slow to fast, every mechanism
    moving the output."""
    last = name.rsplit(".", 1)[-1]
    if "norm" in last or last == "D":
        return 1.0 + 0.2 * r
    if last == "A_log":
        return 1.2 * r - 1.5
    if last == "dt_bias":
        return r - 2.0
    if last == "sink":
        return 1.5 + r
    if last == "temp":
        return 1.2 + 0.3 * r
    if last == "talk":
        return 0.7 * torch.eye(r.shape[0], dtype=r.dtype, device=r.device) + 0.3 * r
    if last == "conv":
        return 0.5 * r + 0.3
    if name.endswith("conv.b"):
        return 0.3 * r
    if len(r.shape) == 2 and name not in ("embed", "bigram"):
        return r * r.shape[1] ** -0.5 * (2.0 if name.endswith("mix.q") else 1.0)
    return r


def _gevovik_tensors(cfg: dict, seed: int, dtype) -> dict:
    g = torch.Generator().manual_seed(seed)
    return {n: gevovik_value(n, torch.randn(shape, generator=g, dtype=torch.float32), cfg).to(dtype) for n, shape in gevovik_shapes(cfg).items()}


def tiny_config(model_type: str, **over) -> dict:
    if model_type == "gevovik":
        ssd = dict(heads=6, vdim=12, state=20, groups=3, conv=4, norm_groups=2, ff=52)
        both = dict(heads=6, kv_heads=2, dim=20, vdim=28, rot_dims=12, window=24, right=(4, 2, 12, 20, 3), ranks=(10, 6), ff=36)
        lat = dict(heads=3, dim=20, rot_dim=6, vdim=12, kv_rank=40, ff=24)
        yarn = {"factor": 8.0, "original": 64, "fast": 16.0, "slow": 2.0}
        kw = dict(width=76, vocab=261, layers=[dict(lat), dict(ssd), dict(both, scaling=yarn, base=500.0), dict(lat, heads=2, vdim=20, kv_from=0, ff=0), dict(both, kv_heads=6),
                                               dict(ssd, heads=4, groups=1, conv=2, norm_groups=1, ff=0)])
        kw.update(over)
        return gevovik_config(**kw)
    if model_type == "dubozen":
        soft = dict(heads=6, kv_heads=2, dim=20, vdim=28, rot_dims=12, ff=52)
        both = dict(heads=4, kv_heads=1, dim=18, rot_dims=10, base=500.0, right=(3, 12, 20, (0.4, 0.97, 0.999)), ff=36, experts=6, top=2, groups=3, keep=2)
        kw = dict(width=76, vocab=261, layers=[dict(soft), dict(both), dict(soft, heads=2, scale=0.4, ff=24, experts=5, top=2), dict(both, ff=0)], streams=3)
        kw.update(over)
        return dubozen_config(**kw)
    if model_type == "fopivik":
        soft = dict(heads=6, kv_heads=2, dim=20, vdim=28, rot_dims=12, window=24, keep_first=5, experts=5, top=2, ff=36)
        lin = dict(heads=3, dim=12, vdim=20, tau=4.0, experts=4, top=1, ff=24)
        kw = dict(width=76, vocab=261, layers=[dict(lin), dict(soft, scaling={"factor": 4.0, "low": 1.0, "high": 4.0, "original": 64}), dict(lin, vdim=8, experts=0)],
                  loop={"start": 0, "stop": 2, "times": 2})
        kw.update(over)
        return fopivik_config(**kw)
    if model_type == "fatotar":
        size = dict(heads=3, dim=20, rot_dim=6, vdim=12, kv_rank=40, window=24, ff=52)
        yarn = {"factor": 8.0, "original": 64, "fast": 16.0, "slow": 2.0}
        kw = dict(width=92, vocab=261, layers=[dict(size), dict(size, window=40, base=500.0, scaling=yarn), dict(size, heads=2, vdim=24, ff=0)],
                  loop={"start": 0, "stop": 2, "times": 2})
        kw.update(over)
        return fatotar_config(**kw)
    base = dict(
        model_type=model_type, vocab_size=256, hidden_size=64, intermediate_size=128, num_hidden_layers=2,
        num_attention_heads=4, num_key_value_heads=2, max_position_embeddings=256, rms_norm_eps=1e-5, rope_theta=10000.0,
        bos_token_id=1, eos_token_id=2, hidden_act="silu", tie_word_embeddings=False,
    )
    if model_type in ("qwen3", "qwen3_moe"):
        base.update(head_dim=64 if "head_dim" not in over else over["head_dim"], rope_theta=1e6, tie_word_embeddings=True)
    if model_type == "qwen3_moe":
        base.update(num_experts=4, num_experts_per_tok=2, moe_intermediate_size=64, norm_topk_prob=True, decoder_sparse_step=1,
                    mlp_only_layers=[])
    if model_type == "mixtral":
        base.update(num_local_experts=4, num_experts_per_tok=2, rope_theta=1e6)
    if model_type == "gemma2":
        base.update(head_dim=64, attn_logit_softcapping=50.0, final_logit_softcapping=30.0, hidden_activation="gelu_pytorch_tanh",
                    sliding_window=64, query_pre_attn_scalar=64, tie_word_embeddings=True)
    if model_type == "gemma3_text":
        base.update(head_dim=64, hidden_activation="gelu_pytorch_tanh", sliding_window=8, query_pre_attn_scalar=64, tie_word_embeddings=True,
                    num_hidden_layers=3, layer_types=["sliding_attention", "sliding_attention", "full_attention"], rms_norm_eps=1e-6,
                    rope_parameters={"sliding_attention": {"rope_type": "default", "rope_theta": 10000.0},
                                     "full_attention": {"rope_type": "default", "rope_theta": 1000000.0}})
        base.pop("rope_theta")
    if model_type == "gpt2":
        base = dict(model_type="gpt2", vocab_size=256, n_embd=64, n_head=4, n_layer=2, n_ctx=256, n_positions=256,
                    layer_norm_epsilon=1e-5, bos_token_id=1, eos_token_id=2, activation_function="gelu_new")
    if model_type == "bert":
        base = dict(model_type="bert", vocab_size=256, hidden_size=64, intermediate_size=128, num_hidden_layers=2,
                    num_attention_heads=4, max_position_embeddings=128, layer_norm_eps=1e-12, hidden_act="gelu", type_vocab_size=2,
                    pad_token_id=0)
    if model_type == "granitemoehybrid":
        base.update(
            layer_types=["mamba", "attention"], embedding_multiplier=12.0, attention_multiplier=0.0156, residual_multiplier=0.22,
            logits_scaling=8.0, shared_intermediate_size=64, num_local_experts=0, num_experts_per_tok=0, position_embedding_type="rope",
            mamba_n_heads=4, mamba_n_groups=1, mamba_d_state=16, mamba_d_head=32, mamba_d_conv=4, mamba_expand=2, mamba_chunk_size=32,
            mamba_conv_bias=True, mamba_proj_bias=False, tie_word_embeddings=True,
        )
    base.update(over)
    return base


def build_tensors(cfg: dict, seed: int = 0, dtype=torch.float32, std: float = 0.02) -> dict:
    g = torch.Generator().manual_seed(seed)
    mt = config_model_type(cfg)
    if mt == "fatotar":
        return _fatotar_tensors(cfg, seed, dtype)
    if mt == "fopivik":
        return _fopivik_tensors(cfg, seed, dtype)
    if mt == "dubozen":
        return _dubozen_tensors(cfg, seed, dtype)
    if mt == "gevovik":
        return _gevovik_tensors(cfg, seed, dtype)
    R = lambda *s: _rand(g, *s, std=std, dtype=dtype)  # noqa: E731
    ones = lambda n: (torch.ones(n) + torch.randn(n, generator=g) * 0.05).to(dtype)  # noqa: E731
    t: dict = {}
    if mt == "gpt2":
        h, L, V, P = cfg["n_embd"], cfg["n_layer"], cfg["vocab_size"], cfg["n_positions"]
        t["wte.weight"] = R(V, h)
        t["wpe.weight"] = R(P, h)
        for i in range(L):
            p = f"h.{i}."
            t[p + "ln_1.weight"], t[p + "ln_1.bias"] = ones(h), R(h)
            t[p + "attn.c_attn.weight"], t[p + "attn.c_attn.bias"] = R(h, 3 * h), R(3 * h)
            t[p + "attn.c_proj.weight"], t[p + "attn.c_proj.bias"] = R(h, h), R(h)
            t[p + "ln_2.weight"], t[p + "ln_2.bias"] = ones(h), R(h)
            t[p + "mlp.c_fc.weight"], t[p + "mlp.c_fc.bias"] = R(h, 4 * h), R(4 * h)
            t[p + "mlp.c_proj.weight"], t[p + "mlp.c_proj.bias"] = R(4 * h, h), R(h)
        t["ln_f.weight"], t["ln_f.bias"] = ones(h), R(h)
        return t
    if mt == "bert":
        h, L, V, I = cfg["hidden_size"], cfg["num_hidden_layers"], cfg["vocab_size"], cfg["intermediate_size"]
        t["embeddings.word_embeddings.weight"] = R(V, h)
        t["embeddings.position_embeddings.weight"] = R(cfg["max_position_embeddings"], h)
        t["embeddings.token_type_embeddings.weight"] = R(cfg["type_vocab_size"], h)
        t["embeddings.LayerNorm.weight"], t["embeddings.LayerNorm.bias"] = ones(h), R(h)
        for i in range(L):
            p = f"encoder.layer.{i}."
            for n in ("query", "key", "value"):
                t[p + f"attention.self.{n}.weight"], t[p + f"attention.self.{n}.bias"] = R(h, h), R(h)
            t[p + "attention.output.dense.weight"], t[p + "attention.output.dense.bias"] = R(h, h), R(h)
            t[p + "attention.output.LayerNorm.weight"], t[p + "attention.output.LayerNorm.bias"] = ones(h), R(h)
            t[p + "intermediate.dense.weight"], t[p + "intermediate.dense.bias"] = R(I, h), R(I)
            t[p + "output.dense.weight"], t[p + "output.dense.bias"] = R(h, I), R(h)
            t[p + "output.LayerNorm.weight"], t[p + "output.LayerNorm.bias"] = ones(h), R(h)
        t["pooler.dense.weight"], t["pooler.dense.bias"] = R(h, h), R(h)
        nl = len(cfg.get("label2id") or {})
        if nl:
            t["classifier.weight"], t["classifier.bias"] = R(nl, h), R(nl)
        return t
    h, L, V = cfg["hidden_size"], cfg["num_hidden_layers"], cfg["vocab_size"]
    nh, nkv = cfg["num_attention_heads"], cfg.get("num_key_value_heads") or cfg["num_attention_heads"]
    hd = cfg.get("head_dim") or h // nh
    I = cfg.get("intermediate_size", 0)
    t["model.embed_tokens.weight"] = R(V, h)
    for i in range(L):
        p = f"model.layers.{i}."
        t[p + "input_layernorm.weight"] = ones(h) if mt not in ("gemma2", "gemma3_text") else R(h)
        is_mamba = mt == "granitemoehybrid" and cfg["layer_types"][i] == "mamba"
        if is_mamba:
            H, G, S, dh, K = cfg["mamba_n_heads"], cfg["mamba_n_groups"], cfg["mamba_d_state"], cfg["mamba_d_head"], cfg["mamba_d_conv"]
            inter = cfg["mamba_expand"] * h
            assert inter == H * dh, "mamba_expand * hidden must equal mamba_n_heads * mamba_d_head"
            conv_dim = inter + 2 * G * S
            t[p + "mamba.in_proj.weight"] = R(inter + conv_dim + H, h)
            t[p + "mamba.conv1d.weight"] = _rand(g, conv_dim, 1, K, std=0.2, dtype=dtype)
            t[p + "mamba.conv1d.bias"] = R(conv_dim)
            t[p + "mamba.dt_bias"] = _rand(g, H, std=0.5, dtype=dtype)
            t[p + "mamba.A_log"] = torch.log(torch.rand(H, generator=g) * 3 + 0.5).to(dtype)
            t[p + "mamba.D"] = ones(H)
            t[p + "mamba.norm.weight"] = ones(inter)
            t[p + "mamba.out_proj.weight"] = R(h, inter)
        else:
            t[p + "self_attn.q_proj.weight"] = R(nh * hd, h)
            t[p + "self_attn.k_proj.weight"] = R(nkv * hd, h)
            t[p + "self_attn.v_proj.weight"] = R(nkv * hd, h)
            t[p + "self_attn.o_proj.weight"] = R(h, nh * hd)
            if mt == "qwen2":
                for n, w in (("q", nh * hd), ("k", nkv * hd), ("v", nkv * hd)):
                    t[p + f"self_attn.{n}_proj.bias"] = R(w)
            if mt in ("qwen3", "qwen3_moe"):
                t[p + "self_attn.q_norm.weight"] = ones(hd)
                t[p + "self_attn.k_norm.weight"] = ones(hd)
            if mt == "gemma3_text":  # stored as w - 1
                t[p + "self_attn.q_norm.weight"] = R(hd)
                t[p + "self_attn.k_norm.weight"] = R(hd)
        t[p + "post_attention_layernorm.weight"] = ones(h) if mt not in ("gemma2", "gemma3_text") else R(h)
        if mt in ("gemma2", "gemma3_text"):
            t[p + "pre_feedforward_layernorm.weight"] = R(h)
            t[p + "post_feedforward_layernorm.weight"] = R(h)
        if mt == "mixtral":
            E = cfg["num_local_experts"]
            t[p + "block_sparse_moe.gate.weight"] = _rand(g, E, h, std=0.5, dtype=dtype)
            for e in range(E):
                ep = p + f"block_sparse_moe.experts.{e}."
                t[ep + "w1.weight"], t[ep + "w3.weight"], t[ep + "w2.weight"] = R(I, h), R(I, h), R(h, I)
        elif mt == "qwen3_moe" and (i not in cfg.get("mlp_only_layers", []) and (i + 1) % cfg.get("decoder_sparse_step", 1) == 0):
            E, MI = cfg["num_experts"], cfg["moe_intermediate_size"]
            t[p + "mlp.gate.weight"] = _rand(g, E, h, std=0.5, dtype=dtype)
            for e in range(E):
                ep = p + f"mlp.experts.{e}."
                t[ep + "gate_proj.weight"], t[ep + "up_proj.weight"], t[ep + "down_proj.weight"] = R(MI, h), R(MI, h), R(h, MI)
        elif mt == "granitemoehybrid":
            S = cfg["shared_intermediate_size"]
            t[p + "shared_mlp.input_linear.weight"] = R(2 * S, h)
            t[p + "shared_mlp.output_linear.weight"] = R(h, S)
            E = cfg.get("num_local_experts", 0)
            if E:
                t[p + "block_sparse_moe.router.layer.weight"] = _rand(g, E, h, std=0.5, dtype=dtype)
                t[p + "block_sparse_moe.input_linear.weight"] = R(E, 2 * I, h)
                t[p + "block_sparse_moe.output_linear.weight"] = R(E, h, I)
        else:
            t[p + "mlp.gate_proj.weight"], t[p + "mlp.up_proj.weight"], t[p + "mlp.down_proj.weight"] = R(I, h), R(I, h), R(h, I)
    t["model.norm.weight"] = ones(h) if mt not in ("gemma2", "gemma3_text") else R(h)
    if not cfg.get("tie_word_embeddings", False):
        t["lm_head.weight"] = R(V, h)
    return t


def write_tiny_model(out_dir: str, model_type: str = "llama", seed: int = 0, dtype=torch.float32, quantize: bool = False,
                     sharded: bool = False, config: Optional[dict] = None, std: float = 0.02, **over) -> dict:
    """Write ``config.json`` + safetensors (optionally JQ4-quantised with the default policy) into ``out_dir``."""
    os.makedirs(out_dir, exist_ok=True)
    cfg = config or tiny_config(model_type, **over)
    tensors = build_tensors(cfg, seed, dtype, std)
    if quantize:
        from .quantizer import DEFAULT_Q4_FILTER, quantize_tensor

        tensors = {k: (quantize_tensor(v) if DEFAULT_Q4_FILTER(k) and v.dim() >= 2 and v.shape[-1] % 32 == 0 else v)
                   for k, v in tensors.items()}
    with open(os.path.join(out_dir, "config.json"), "w") as f:
        json.dump(cfg, f, indent=1)
    if sharded:
        write_sharded(out_dir, tensors, max_shard_bytes=256 * 1024)
    else:
        write_safetensors(os.path.join(out_dir, "model.safetensors"), tensors)
    return cfg
