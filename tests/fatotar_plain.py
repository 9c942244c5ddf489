"""Slow, plain statement of the Fatotar decoder: one function per mechanism, loops and dense matrices, nothing shared with the
package. ``W`` maps tensor names to tensors, ``cfg`` is the parsed ``config.json``. Everything runs in the dtype of ``real``
(float64 by default), one sequence at a time, whole prefix at once: no cache, no batch, no chunk."""
import math

import torch

real = torch.float64


def bigram_rows(tokens, mul_prev, mul_cur, buckets):
    """Table row per token; the first token of a sequence has no predecessor and takes the row behind the hashed ones."""
    rows = [buckets]
    for prev, cur in zip(tokens[:-1], tokens[1:]):
        rows.append((prev * mul_prev + cur * mul_cur) % buckets)
    return rows


def embed(W, cfg, tokens):
    e = cfg["embedding"]
    x = W["embed"].to(real)[torch.tensor(tokens)] * e["scale"]
    b = e["bigram"]
    return x + W["bigram"].to(real)[torch.tensor(bigram_rows(tokens, b["mul_prev"], b["mul_cur"], b["buckets"]))]


def layer_norm(x, w, b, eps):
    out = torch.empty_like(x)
    for t in range(x.shape[0]):
        mean = x[t].sum() / x.shape[1]
        var = ((x[t] - mean) ** 2).sum() / x.shape[1]
        out[t] = (x[t] - mean) / torch.sqrt(var + eps) * w.to(real) + b.to(real)
    return out


def rms_norm(x, w, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps) * w.to(real)


def yarn_frequencies(dims, base, scaling):
    """(frequencies of the dims / 2 pairs, factor on cos and sin)"""
    if not scaling:
        return [base ** (-2.0 * i / dims) for i in range(dims // 2)], 1.0

    def turn_dim(turns):  # the (fractional) pair index that makes `turns` full turns over the original context
        return dims * math.log(scaling["original"] / (2 * math.pi * turns)) / (2 * math.log(base))

    lo = max(math.floor(turn_dim(scaling["fast"])), 0)
    hi = min(math.ceil(turn_dim(scaling["slow"])), dims - 1)
    out = []
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / scaling["factor"] * ramp + f * (1.0 - ramp))
    return out, 0.1 * math.log(scaling["factor"]) + 1.0


def rotate(v, pos, freqs, mult):
    """Rotate-half pairs (i, i + n) of the first 2 n entries of vector v; the rest passes."""
    n = len(freqs)
    a = torch.tensor([pos * f for f in freqs], dtype=torch.float64)
    c, s = (torch.cos(a) * mult).to(v.dtype), (torch.sin(a) * mult).to(v.dtype)
    u, w = v[:n], v[n:2 * n]
    return torch.cat([u * c - w * s, w * c + u * s, v[2 * n:]])


def latent_attention(W, m, p, h, eps):
    """Latent attention of one sequence over its own prefix; h [T, width] is the mixer's input, p the tensor prefix."""
    T = h.shape[0]
    H, dn, dr, dv, R = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    g = lambda n: W[p + n].to(real)  # noqa: E731
    freqs, mult = yarn_frequencies(m["rot"]["dims"], m["rot"]["base"], m["rot"].get("scaling"))
    q = (h @ g("q").T).reshape(T, H, dn + dr)
    down = h @ g("dkv").T
    c = rms_norm(down[:, :R], g("dkv.norm"), eps)
    kr = torch.stack([rotate(down[t, R:], t, freqs, mult) for t in range(T)])
    k = (c @ g("uk").T).reshape(T, H, dn)
    v = (c @ g("uv").T).reshape(T, H, dv)
    out = torch.zeros(T, H, dv, dtype=h.dtype)
    for t in range(T):
        first = max(0, t - m["mask"]["size"] + 1)
        for n in range(H):
            qr = rotate(q[t, n, dn:], t, freqs, mult)
            s = (k[first:t + 1, n] @ q[t, n, :dn] + kr[first:t + 1] @ qr) * m["scale"]
            e = torch.exp(s - s.max())
            out[t, n] = (e / e.sum()) @ v[first:t + 1, n]
    gate = torch.sigmoid(h @ g("g").T)
    return (out.reshape(T, H * dv) * gate) @ g("o").T


def feed_forward(W, p, h):
    lin = lambda n, x: x @ W[p + n].to(real).T + W[p + n + ".b"].to(real)  # noqa: E731
    return lin("down", torch.clamp(lin("gate", h), min=0) * lin("up", h))


def layer_order(cfg):
    """Weight-layer index of every layer run."""
    n, lp = len(cfg["layers"]), cfg.get("loop")
    if not lp:
        return list(range(n))
    return list(range(lp["start"])) + list(range(lp["start"], lp["stop"])) * lp["times"] + list(range(lp["stop"], n))


def forward(W, cfg, tokens, want_layers=False):
    """Logits [T, vocab]; with ``want_layers`` also the residual stream after every layer run."""
    eps = cfg["norm"]["eps"]
    x = embed(W, cfg, tokens)
    stream = []
    for i in layer_order(cfg):
        L, p = cfg["layers"][i], f"l{i}."
        a = latent_attention(W, L["mixer"], p + "mix.", layer_norm(x, W[p + "norm1"], W[p + "norm1.b"], eps), eps)
        f = feed_forward(W, p + "mlp.", layer_norm(x, W[p + "norm2"], W[p + "norm2.b"], eps)) if L.get("mlp") else 0
        x = x + (a + f)
        stream.append(x)
    logits = layer_norm(x, W["final.norm"], W["final.norm.b"], eps) @ W["head"].to(real).T
    return (logits, stream) if want_layers else logits
