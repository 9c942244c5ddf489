"""Slow, plain statement of the Gevovik decoder: one function per mechanism, loops and dense matrices, nothing shared with the package.
``W`` maps tensor names to tensors, ``cfg`` is the parsed ``config.json``. Everything runs in the dtype of ``real`` (float64), one
sequence at a time, whole prefix at once: no cache, no state slot, no batch, no chunk."""
import math

import torch

real = torch.float64


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def silu(z):
    return z * torch.sigmoid(z)


def softplus(z):
    return torch.where(z > 40, z, torch.log1p(torch.exp(torch.clamp(z, max=40))))


# --------------------------------------------------------------------------------------------------- embedding, norm, feed-forward
def embed(W, cfg, tokens):
    """Token rows times a constant plus the row of the pair (previous token, token); the last row where there is no previous token."""
    e = cfg["embedding"]
    bg = e.get("bigram")
    rows = []
    for t, tok in enumerate(tokens):
        x = W["embed"][tok].to(real) * e["scale"]
        if bg:
            row = (tokens[t - 1] * bg["mul_prev"] + tok * bg["mul_cur"]) % bg["buckets"] if t else bg["buckets"]
            x = x + W["bigram"][row].to(real)
        rows.append(x)
    return torch.stack(rows)


def add_normed(x, y, gain, eps):
    """The sublayer's output is normed, with one gain for all columns, and added; nothing is normed in front of a sublayer."""
    return x + rms(y, eps) * gain.to(real).reshape(())


def dense(W, p, h):
    a = torch.clamp(h @ W[p + "up"].to(real).T, min=0)
    return (a * a) @ W[p + "down"].to(real).T


# --------------------------------------------------------------------------------------------------- rotations
def frequencies(rot):
    dims, base = rot["dims"], rot["base"]
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    sc = rot.get("scaling")
    if not sc:
        return f, 1.0
    turn = lambda t: dims * math.log(sc["original"] / (2 * math.pi * t)) / (2 * math.log(base))  # noqa: E731
    lo, hi = max(math.floor(turn(sc["fast"])), 0), min(math.ceil(turn(sc["slow"])), dims - 1)
    out = []
    for i, w in enumerate(f):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(w / sc["factor"] * r + w * (1 - r))
    return out, 0.1 * math.log(sc["factor"]) + 1.0


def rotate(x, rot, pairs):
    """x [T, heads, d], row t at position t. ``pairs``: entries 2 i and 2 i + 1 turn together, else i and i + dims / 2."""
    f, mult = frequencies(rot)
    n, out, t = rot["dims"] // 2, x.clone(), torch.arange(x.shape[0], dtype=real).unsqueeze(1)
    for i in range(n):
        a, b = (2 * i, 2 * i + 1) if pairs else (i, i + n)
        c, s = torch.cos(t * f[i]) * mult, torch.sin(t * f[i]) * mult
        out[..., a] = x[..., a] * c - x[..., b] * s
        out[..., b] = x[..., b] * c + x[..., a] * s
    return out


# --------------------------------------------------------------------------------------------------- convolution
def causal_conv(x, w, bias=None):
    """Per channel over time: x [T, C], w [C, taps], the last column is the current token's, zeros in front of the sequence."""
    T, taps = x.shape[0], w.shape[1]
    out = torch.zeros_like(x)
    for j in range(taps):
        back = taps - 1 - j
        out[back:] += w[:, j].to(real) * x[: T - back] if back < T else 0
    return out if bias is None else out + bias.to(real)


# --------------------------------------------------------------------------------------------------- Mamba-2
def ssd(x, B, C, dt, A_log, D):
    """x [T, H, dv], B and C [T, G, N], dt [T, H] (positive) -> y [T, H, dv]: S <- exp(-exp(A_log) dt) S + dt B x^T, y = S^T C + D x."""
    T, H, dv = x.shape
    G, N = B.shape[1:]
    S, y = torch.zeros(H, N, dv, dtype=real), torch.zeros(T, H, dv, dtype=real)
    group = [h // (H // G) for h in range(H)]
    for t in range(T):
        decay, b, c = torch.exp(-torch.exp(A_log) * dt[t]), B[t, group], C[t, group]
        S = decay.view(H, 1, 1) * S + dt[t].view(H, 1, 1) * b.unsqueeze(2) * x[t].unsqueeze(1)
        y[t] = (S * c.unsqueeze(2)).sum(dim=1) + D.view(H, 1) * x[t]
    return y


def mamba2(W, m, p, h, eps):
    T, H, dv, N, G = h.shape[0], m["heads"], m["vdim"], m["state"], m["groups"]
    I = H * dv
    g = lambda n: W[p + n].to(real)  # noqa: E731
    z, xbc, dt = (h @ g("in").T).split([I, I + 2 * G * N, H], dim=-1)
    x, B, C = silu(causal_conv(xbc, g("conv"), g("conv.b"))).split([I, G * N, G * N], dim=-1)
    y = ssd(x.reshape(T, H, dv), B.reshape(T, G, N), C.reshape(T, G, N), softplus(dt + g("dt_bias")), g("A_log"), g("D")).reshape(T, I)
    y = rms((y * silu(z)).reshape(T, m["norm_groups"], -1), eps).reshape(T, I) * g("norm")
    return y @ g("o").T


# --------------------------------------------------------------------------------------------------- attention with mixed scores
def mixed_head_attention(q, k, v, scale, temp, talk, window):
    """q [T, H, d], k [T, G, d], v [T, G, dv] -> [T, H, dv]: every head's score has its own factor, then the heads' scores are mixed (``talk``:
    to, from), in front of a softmax over the last ``window`` keys."""
    T, H, G = q.shape[0], q.shape[1], k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=real)
    own = [n // (H // G) for n in range(H)]
    for t in range(T):
        lo = max(0, t - window + 1) if window else 0
        raw = (k[lo : t + 1, own] * q[t]).sum(dim=-1).T * scale * temp.unsqueeze(1)  # [H, keys]
        s = torch.softmax(talk @ raw, dim=-1)
        out[t] = (s.T.unsqueeze(2) * v[lo : t + 1, own]).sum(dim=0)
    return out


def attention(W, m, p, h, eps):
    T, H, G = h.shape[0], m["heads"], m["kv_heads"]
    g = lambda n: W[p + n].to(real)  # noqa: E731
    head = lambda n, k: rotate(rms((h @ g(n).T).reshape(T, k, m["dim"]), eps) * g(n + ".norm"), m["rot"], False)  # noqa: E731
    v = (h @ g("v").T).reshape(T, G, m["vdim"])
    o = mixed_head_attention(head("q", H), head("k", G), v, m["scale"], g("temp").reshape(-1), g("talk"), m["mask"]["size"])
    o = o * torch.sigmoid(h @ g("g").T).unsqueeze(-1)
    return o.reshape(T, -1) @ g("o").T


# --------------------------------------------------------------------------------------------------- gated delta rule
def delta_rule(q, k, v, a, beta):
    """q, k, a [T, H, d], v [T, H, dv], beta [T, H] -> [T, H, dv]: decay every key channel, correct what the key reads, write, read."""
    T, H, d = q.shape
    S, out = torch.zeros(H, d, v.shape[2], dtype=real), torch.zeros(v.shape, dtype=real)
    for t in range(T):
        S = a[t].unsqueeze(2) * S
        u = beta[t].unsqueeze(1) * (v[t] - (S * k[t].unsqueeze(2)).sum(dim=1))
        S = S + k[t].unsqueeze(2) * u.unsqueeze(1)
        out[t] = (S * q[t].unsqueeze(2)).sum(dim=1)
    return out


def unit(x):
    return x / torch.sqrt((x * x).sum(dim=-1, keepdim=True) + 1e-6)


def gated_delta(W, m, p, h, eps):
    T, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    g = lambda n: W[p + n].to(real)  # noqa: E731
    q, k, v = (silu(causal_conv(h @ g(n).T, g(n + ".conv"))).reshape(T, k_, -1) for n, k_ in (("q", G), ("k", G), ("v", H)))
    own = [n // (H // G) for n in range(H)]
    q, k = unit(q)[:, own] * d ** -0.5, unit(k)[:, own]
    beta = torch.sigmoid(h @ g("b").T)
    step = softplus((h @ g("a1").T) @ g("a2").T + g("dt_bias")).reshape(T, H, d)
    a = torch.exp(-torch.exp(g("A_log")).reshape(1, H, 1) * step)
    o = rms(delta_rule(q, k, v, a, beta), eps) * g("norm")
    return (o.reshape(T, -1) * torch.sigmoid((h @ g("g1").T) @ g("g2").T)) @ g("o").T


def parallel(W, m, p, h, eps):
    return m["left_scale"] * attention(W, m["left"], p + "left.", h, eps) + m["right_scale"] * gated_delta(W, m["right"], p + "right.", h, eps)


# --------------------------------------------------------------------------------------------------- latent attention
def latent_rows(W, m, p, h, eps):
    """What a layer with a down projection caches per token: the normed latent and the rotated key part."""
    g = lambda n: W[p + n].to(real)  # noqa: E731
    c, r = (h @ g("dkv").T).split([m["kv_rank"], m["rot_dim"]], dim=-1)
    return rms(c, eps) * g("dkv.norm"), rotate(r.unsqueeze(1), m["rot"], True).squeeze(1)


def sink_softmax(s, sink):
    """Weights of scores s [H, n] beside a sink per head that has neither key nor value."""
    top = torch.maximum(s.max(dim=-1).values, sink).unsqueeze(1)
    e = torch.exp(s - top)
    return e / (e.sum(dim=-1, keepdim=True) + torch.exp(sink.unsqueeze(1) - top))


def latent_attention(W, m, p, h, c, r):
    T, H, d, dr, dv = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    g = lambda n: W[p + n].to(real)  # noqa: E731
    q = (h @ g("q").T).reshape(T, H, d + dr)
    qr = rotate(q[..., d:], m["rot"], True)
    k, v = (c @ g("uk").T).reshape(T, H, d), (c @ g("uv").T).reshape(T, H, dv)
    out = torch.zeros(T, H, dv, dtype=real)
    for t in range(T):
        s = ((k[: t + 1] * q[t, :, :d]).sum(dim=-1).T + qr[t] @ r[: t + 1].T) * m["scale"]
        out[t] = (sink_softmax(s, g("sink").reshape(-1)).T.unsqueeze(2) * v[: t + 1]).sum(dim=0)
    return out.reshape(T, -1) @ g("o").T


# --------------------------------------------------------------------------------------------------- model
def layer(W, cfg, i, x, caches):
    L, p, eps = cfg["layers"][i], f"l{i}.", cfg["norm"]["eps"]
    m = L["mixer"]
    if L["type"] == "mamba2":
        y = mamba2(W, m, p + "mix.", x, eps)
    elif L["type"] == "parallel":
        y = parallel(W, m, p + "mix.", x, eps)
    else:
        src = m.get("kv_from")
        caches[i] = caches[src] if src is not None else latent_rows(W, m, p + "mix.", x, eps)
        y = latent_attention(W, m, p + "mix.", x, *caches[i])
    x = add_normed(x, y, W[p + "norm1"], eps)
    if L.get("mlp"):
        x = add_normed(x, dense(W, p + "mlp.", x), W[p + "norm2"], eps)
    return x


def forward(W, cfg, tokens, want_layers=False):
    """Logits [T, vocab]; with ``want_layers`` also the residual stream after every layer."""
    x, outs, caches = embed(W, cfg, tokens), [], {}
    for i in range(len(cfg["layers"])):
        x = layer(W, cfg, i, x, caches)
        outs.append(x)
    logits = (rms(x, cfg["norm"]["eps"]) * W["final.norm"].to(real).reshape(())) @ W["head"].to(real).T
    return (logits, outs) if want_layers else logits
