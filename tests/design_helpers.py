"""Shared by the tests of designs with a plain statement of their own: devices and precisions, an in-memory loader, replay of a plan."""
import pytest
import torch

from deliverance_b200.engine.engine import Engine, EngineConfig
from deliverance_b200.kv.paged import KvCacheSettings

gpu = pytest.mark.gpu
RUNS = [pytest.param(("cpu", torch.float32), id="cpu-f32"), pytest.param(("cuda", torch.float32), id="cuda-f32", marks=gpu),
        pytest.param(("cuda", torch.bfloat16), id="cuda-bf16", marks=gpu)]


def tol(dtype, f32=2e-5, bf16=2.5e-2):
    return f32 if dtype == torch.float32 else bf16


def rel(got, want):
    """RMS of the difference over the RMS of the expected values, worst row."""
    got, want = got.detach().double().cpu(), want.double()
    return ((got - want).pow(2).mean(-1).sqrt() / want.pow(2).mean().sqrt().clamp_min(1e-12)).max().item()


def tokens_of(n, vocab, seed):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


class Dict2Loader:
    """Loader interface over tensors in memory."""

    def __init__(self, tensors):
        self.t = tensors

    def has(self, n):
        return n in self.t

    def load_dense(self, n, dtype=torch.float32, shard=None):
        return self.t[n].to(dtype)


def engine_for(model, tokens=4096, **kw):
    kw.setdefault("max_seqs", 8)
    kv = kw.pop("kv", KvCacheSettings(enabled=False))
    return Engine(model, EngineConfig(num_pages=(tokens + 31) // 32 + 1, kv=kv, **kw))


def replay(engine, plan, requests):
    """Run ``plan`` = steps of (name, count); returns logits of every position per name."""
    at, live, out = {}, {}, {}
    for step in plan:
        entries, spans = [], []
        for name, n in step:
            lo = at.get(name, 0)
            if name not in live:
                live[name] = engine.open_replay()
            entries.append((live[name], requests[name][lo : lo + n], list(range(n))))
            spans.append((name, n))
            at[name] = lo + n
        logits, row = engine.replay_step(entries), 0
        for name, n in spans:
            out.setdefault(name, []).append(logits[row : row + n])
            row += n
            if at[name] == len(requests[name]):
                engine.close_replay(live.pop(name))
    assert not live
    return {k: torch.cat(v) for k, v in out.items()}


class _Stage:
    def __enter__(self):
        return self

    def __exit__(self, *a):
        return False
