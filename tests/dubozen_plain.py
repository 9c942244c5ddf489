"""Slow, plain statement of the Dubozen decoder: one function per mechanism, loops and dense matrices, nothing shared with the package.
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


def rotate_halves(v, pos, dims, base):
    """Entries i and i + dims / 2 of vector v are a pair, i < dims / 2; entries from dims on pass."""
    v, old, n = v.clone(), v, dims // 2
    for i in range(n):
        a = pos * base ** (-2.0 * i / dims)
        c, s = math.cos(a), math.sin(a)
        v[i], v[i + n] = old[i] * c - old[i + n] * s, old[i + n] * c + old[i] * s
    return v


def rotate_all(x, rot):
    """x [T, heads, dim]; row t is position t."""
    return torch.stack([torch.stack([rotate_halves(head, t, rot["dims"], rot["base"]) for head in row]) for t, row in enumerate(x)])


def softmax_heads(q, k, v, scale, sink=None):
    """Causal attention of grouped heads: q [T, H, dk], k [T, G, dk], v [T, G, dv] -> [T, H, dv]. ``sink`` [H]: a score per head that counts
    in the denominator only."""
    T, H, G = q.shape[0], q.shape[1], k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=real)
    for t in range(T):
        for n in range(H):
            kv = n // (H // G)
            s = (k[: t + 1, kv] @ q[t, n]) * scale
            top = max(s.max().item(), sink[n].item() if sink is not None else -math.inf)
            e = torch.exp(s - top)
            den = e.sum() + (math.exp(sink[n].item() - top) if sink is not None else 0.0)
            out[t, n] = (e / den) @ v[: t + 1, kv]
    return out


def mixed_values(v, first, lam):
    """What a later value-mixing layer uses and caches: its own values blended with those of the first such layer."""
    return (1 - lam) * v + lam * first


def attention(W, m, p, h, v_first=None):
    """Returns the mixer's output and the values that attention used (the first mixing layer's are every later one's ``v_first``)."""
    T, H, G = h.shape[0], m["heads"], m["kv_heads"]
    g = lambda n: W[p + n].to(real)  # noqa: E731
    q = rotate_all((h @ g("q").T).reshape(T, H, m["dim"]), m["rot"])
    k = rotate_all((h @ g("k").T).reshape(T, G, m["dim"]), m["rot"])
    v = (h @ g("v").T).reshape(T, G, m["vdim"])
    if m.get("v_mix") and v_first is not None:
        v = mixed_values(v, v_first, g("vmix").reshape(()))
    o = softmax_heads(q, k, v, m["scale"], g("sink").reshape(-1)).reshape(T, -1)
    return (o * torch.sigmoid(h @ g("g").T)) @ g("o").T, v


def tied_attention(W, m, p, h, eps):
    """Grouped attention whose values are the projected keys (before norm and rotation), with per-head norms and one gate per head."""
    T, H, G, d = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    g = lambda n: W[p + n].to(real)  # noqa: E731
    q, k = (h @ g("q").T).reshape(T, H, d), (h @ g("k").T).reshape(T, G, d)
    o = softmax_heads(rotate_all(rms_norm(q, g("q.norm"), eps), m["rot"]), rotate_all(rms_norm(k, g("k.norm"), eps), m["rot"]), k, m["scale"])
    o = o * torch.sigmoid(h @ g("g").T).unsqueeze(-1)
    return o.reshape(T, H * d) @ g("o").T


def silu(z):
    return z * torch.sigmoid(z)


def lightning(W, m, p, h, eps, state=None):
    """Linear attention with one constant decay per head, token by token. ``state``: [heads, dim, vdim] to start from, updated in place."""
    T, H, dk, dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    g = lambda n: W[p + n].to(real)  # noqa: E731
    q, k, v = (silu(h @ g(n).T).reshape(T, H, d) for n, d in (("q", dk), ("k", dk), ("v", dv)))
    S = torch.zeros(H, dk, dv, dtype=real) if state is None else state
    out = torch.zeros(T, H, dv, dtype=real)
    for t in range(T):
        for n in range(H):
            S[n] = m["decay"][n] * S[n] + torch.outer(k[t, n], v[t, n])
            out[t, n] = S[n].T @ q[t, n]
    o = rms_norm(out.reshape(T, H * dv), g("norm").reshape(-1), eps)
    return (o * torch.sigmoid(h @ g("g").T)) @ g("o").T


def parallel(W, m, p, h, eps, state=None):
    return m["left_scale"] * tied_attention(W, m["left"], p + "left.", h, eps) + m["right_scale"] * lightning(W, m["right"], p + "right.", h, eps, state)


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def dense(W, p, h):
    g = lambda n: W[p + n].to(real)  # noqa: E731
    return (gelu_tanh(h @ g("gate").T) * (h @ g("up").T)) @ g("down").T


def route(z, correction, r):
    """Chosen experts and their weights for router logits z [experts]."""
    s = torch.sigmoid(z)
    choice = (s + correction).tolist()
    n, groups = len(choice), r.get("groups") or {"count": 1, "keep": 1}
    size = n // groups["count"]
    value = [sum(sorted(choice[j * size : (j + 1) * size])[-2:]) for j in range(groups["count"])]
    kept = sorted(range(groups["count"]), key=lambda j: (-value[j], j))[: groups["keep"]]
    idx = sorted((e for e in range(n) if e // size in kept), key=lambda e: (-choice[e], e))[: r["top"]]
    return idx, s[idx] / (s[idx].sum() + 1e-20) * r["scale"]


def moe(W, ff, p, h):
    g = lambda n: W[p + n].to(real)  # noqa: E731
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        idx, w = route(g("router") @ h[t], g("correction").reshape(-1), ff["router"])
        for e, s in zip(idx, w):
            out[t] += s * (g(f"e{e}.down") @ (silu(g(f"e{e}.gate") @ h[t]) * (g(f"e{e}.up") @ h[t])))
    return out


def read_streams(X, w_in):
    """X [T, streams, width] -> the sublayer's input row, a weighted sum of the streams."""
    return (X * w_in.to(real).reshape(-1, 1)).sum(dim=1)


def write_streams(X, y, mix, w_out):
    """New streams from the old ones (mix[from, to]) plus the sublayer's output, weighted per stream."""
    n = X.shape[1]
    return torch.stack([sum(mix[a, b].to(real) * X[:, a] for a in range(n)) + w_out.reshape(-1)[b].to(real) * y for b in range(n)], dim=1)


def sublayer(W, p, q, X, eps, fn):
    h = layer_norm(read_streams(X, W[f"{p}hc{q}.in"]), W[f"{p}norm{q}"], eps)
    return write_streams(X, fn(h), W[f"{p}hc{q}.mix"], W[f"{p}hc{q}.out"])


def layer(W, cfg, i, X, shared):
    L, p, eps = cfg["layers"][i], f"l{i}.", cfg["norm"]["eps"]

    def mixer(h):
        if L["type"] == "parallel":
            return parallel(W, L["mixer"], p + "mix.", h, eps)
        y, v = attention(W, L["mixer"], p + "mix.", h, shared.get("v"))
        if L["mixer"].get("v_mix"):
            shared.setdefault("v", v)
        return y

    X = sublayer(W, p, 1, X, eps, mixer)
    if L.get("mlp"):
        X = sublayer(W, p, 2, X, eps, (lambda h: dense(W, p + "mlp.", h)) if L["mlp"]["kind"] == "dense" else lambda h: moe(W, L["mlp"], p + "mlp.", h))
    return X


def forward(W, cfg, tokens, want_layers=False):
    """Logits [T, vocab]; with ``want_layers`` also the sum of the streams after every layer."""
    eps = cfg["norm"]["eps"]
    x = layer_norm(W["embed"].to(real)[torch.tensor(tokens)], W["embed.norm"], eps)
    X, sums, shared = torch.stack([x] * cfg["streams"], dim=1), [], {}
    for i in range(len(cfg["layers"])):
        X = layer(W, cfg, i, X, shared)
        sums.append(X.sum(dim=1))
    logits = layer_norm(X.sum(dim=1), W["final.norm"], eps) @ W["embed"].to(real).T
    return (logits, sums) if want_layers else logits
