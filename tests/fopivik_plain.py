"""Slow, plain statement of the Fopivik decoder: one function per mechanism, loops and dense matrices, nothing shared with the package.
``W`` maps tensor names to tensors, ``cfg`` is the parsed ``config.json``. Everything runs in the dtype of ``real`` (float64), one
sequence at a time, whole prefix at once: no cache, no state slot, no batch, no chunk."""
import math

import torch

real = torch.float64


def layer_norm(x, w, eps):
    mean = x.mean(dim=-1, keepdim=True)
    var = ((x - mean) ** 2).mean(dim=-1, keepdim=True)
    return (x - mean) / torch.sqrt(var + eps) * w.to(real)


def rms_norm(x, w, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps) * w.to(real)


def banded_frequencies(dims, base, scaling):
    """Rotary frequencies of the dims / 2 pairs: long wavelengths slowed down by a factor, short ones kept, a linear blend in between."""
    out = []
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        if scaling:
            wave = 2 * math.pi / f
            if wave > scaling["original"] / scaling["low"]:
                f = f / scaling["factor"]
            elif not wave < scaling["original"] / scaling["high"]:
                s = (scaling["original"] / wave - scaling["low"]) / (scaling["high"] - scaling["low"])
                f = (1 - s) * f / scaling["factor"] + s * f
        out.append(f)
    return out


def rotate_pairs(v, pos, freqs):
    """Neighbouring entries (2 i, 2 i + 1) of vector v are a pair; entries behind the rotated ones pass."""
    v = v.clone()
    for i, f in enumerate(freqs):
        c, s = math.cos(pos * f), math.sin(pos * f)
        a, b = v[2 * i].item(), v[2 * i + 1].item()
        v[2 * i], v[2 * i + 1] = a * c - b * s, b * c + a * s
    return v


def visible(i, j, mask):
    """Does position i see position j: a sliding window plus the first tokens of the sequence."""
    return j <= i and (i - j < mask["size"] or j < mask["keep_first"])


def attention(W, m, p, h):
    T, H, G, dk, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    g = lambda n: W[p + n].to(real)  # noqa: E731
    freqs = banded_frequencies(m["rot"]["dims"], m["rot"]["base"], m["rot"].get("scaling"))
    q = (h @ g("q").T).reshape(T, H, dk)
    k = (h @ g("k").T).reshape(T, G, dk)
    v = (h @ g("v").T).reshape(T, G, dv)
    for t in range(T):
        for n in range(H):
            q[t, n] = rotate_pairs(q[t, n], t, freqs)
        for n in range(G):
            k[t, n] = rotate_pairs(k[t, n], t, freqs)
    out = torch.zeros(T, H, dv, dtype=real)
    for t in range(T):
        seen = [j for j in range(t + 1) if visible(t, j, m["mask"])]
        for n in range(H):
            kv = n // (H // G)
            s = (k[seen, kv] @ q[t, n]) * m["scale"]
            s = m["softcap"] * torch.tanh(s / m["softcap"])
            top = max(0.0, s.max().item())
            e = torch.exp(s - top)
            out[t, n] = (e / (math.exp(-top) + e.sum())) @ v[seen, kv]  # a sink of score 0 takes part in the sum only
    return out.reshape(T, H * dv) @ g("o").T


def gla(W, m, p, h, eps, state=None):
    """Gated linear attention, token by token. ``state``: [heads, dim, vdim] to start from, updated in place."""
    T, H, dk, dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    g = lambda n: W[p + n].to(real)  # noqa: E731
    q = (h @ g("q").T).reshape(T, H, dk) * dk ** -0.5
    k = (h @ g("k").T).reshape(T, H, dk)
    v = (h @ g("v").T).reshape(T, H, dv)
    z = ((h @ g("a1").T) @ g("a2").T + g("a2.b").reshape(-1)).reshape(T, H, dk)
    alpha = torch.exp(torch.nn.functional.logsigmoid(z) / m["tau"])
    S = torch.zeros(H, dk, dv, dtype=real) if state is None else state
    out = torch.zeros(T, H, dv, dtype=real)
    for t in range(T):
        for n in range(H):
            S[n] = alpha[t, n].unsqueeze(1) * S[n] + torch.outer(k[t, n], v[t, n])
            out[t, n] = S[n].T @ q[t, n]
    o = rms_norm(out, g("norm").reshape(-1), eps).reshape(T, H * dv)
    z = h @ g("g").T
    return (o * (z * torch.sigmoid(z))) @ g("o").T


def route(z, top):
    """Chosen experts and their weights for router logits z [experts]: softmax over all, the largest ones, not renormalised."""
    s = torch.softmax(z, dim=0)
    idx = sorted(range(len(s)), key=lambda e: (-s[e].item(), e))[:top]
    return idx, s[idx]


def moe(W, ff, p, h):
    g = lambda n: W[p + n].to(real)  # noqa: E731
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        idx, w = route(g("router") @ h[t], ff["router"]["top"])
        for e, s in zip(idx, w):
            a = g(f"e{e}.gate") @ h[t]
            out[t] += s * (g(f"e{e}.down") @ (a * torch.sigmoid(a) * (g(f"e{e}.up") @ h[t])))
    return out


def layer(W, cfg, i, x):
    L, p, eps, m = cfg["layers"][i], f"l{i}.", cfg["norm"]["eps"], cfg["residual_mult"]
    h = layer_norm(x, W[p + "norm1"], eps)
    a = attention(W, L["mixer"], p + "mix.", h) if L["type"] == "attention" else gla(W, L["mixer"], p + "mix.", h, eps)
    x = x + m * layer_norm(a, W[p + "norm1b"], eps)
    if L.get("mlp"):
        f = moe(W, L["mlp"], p + "mlp.", layer_norm(x, W[p + "norm2"], eps))
        x = x + m * layer_norm(f, W[p + "norm2b"], eps)
    return x


def pass_input(W, x, x0, t):
    """What the first layer of pass t of the loop reads: the stream and the embedding output mixed, plus the pass's own vector."""
    return torch.cat([x, x0], dim=1) @ W["loop.in"].to(real).T + W["loop.step"][t].to(real)


def forward(W, cfg, tokens, want_layers=False):
    """Logits [T, vocab]; with ``want_layers`` also the residual stream after every layer run."""
    x = x0 = W["embed"].to(real)[torch.tensor(tokens)]
    lp, stream = cfg.get("loop"), []

    def run(i, x):
        x = layer(W, cfg, i, x)
        stream.append(x)
        return x

    n = len(cfg["layers"])
    start, stop, times = (lp["start"], lp["stop"], lp["times"]) if lp else (n, n, 0)
    for i in range(start):
        x = run(i, x)
    for t in range(times):
        x = pass_input(W, x, x0, t)
        for i in range(start, stop):
            x = run(i, x)
    for i in range(stop, n):
        x = run(i, x)
    logits = layer_norm(x, W["final.norm"], cfg["norm"]["eps"]) @ W["head"].to(real).T
    logits = cfg["logit_softcap"] * torch.tanh(logits / cfg["logit_softcap"])
    return (logits, stream) if want_layers else logits
