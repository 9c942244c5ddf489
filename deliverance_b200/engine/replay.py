"""Trace replay: given token ids instead of sampled ones, logits instead of tokens.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N < steps.jsonl

Every input line is one batch, ``{"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": ["b"]}``: the next
tokens of each request, the places among them whose logits are wanted, and the requests that are finished afterwards (their pages go
back to the pool). For a step in which something is wanted the logits go to ``<out>/<step>.f32`` (little-endian fp32
``[wanted, vocab]``, in the order of the entries and of ``want``); after every step ``done <step>`` is printed. The batches run through
:meth:`Engine.replay_step`, i.e. the model, paged cache, kernels and captured decode steps that generation uses. The page pool holds
``--max-tokens`` tokens (every live request rounded up to whole pages), for at most four live requests.

``bfloat16`` is the serving precision; ``float32`` runs everything in 32-bit for the families whose kernels have that form (exit
code 3 otherwise). The CUDA extension is compiled when it is missing or older than its sources.
"""
from __future__ import annotations

import argparse
import json
import os
import sys

MAX_LIVE = 4
FLOAT32_FAMILIES = ("fatotar", "fopivik", "dubozen", "gevovik")  # CUDA families with a true 32-bit path


def open_engine(model_dir: str, dtype: str, max_tokens: int, device: str = "auto", max_live: int = MAX_LIVE):
    """Engine over the model in ``model_dir`` with a pool of ``max_tokens`` tokens."""
    import torch

    from ..api import AutoModelForCausalLM
    from ..kv.paged import KvCacheSettings
    from .engine import Engine, EngineConfig

    b = AutoModelForCausalLM.new_builder(model_dir).with_device(device).with_working_memory_type({"bfloat16": "bf16", "float32": "f32"}[dtype])
    model, _ = b.build_local_transformer_model()
    kv = KvCacheSettings(enabled=False)  # every given token runs: no prefix of another request stands in for it
    pages = (max_tokens + kv.block_size - 1) // kv.block_size + 1  # + the scratch page
    torch.set_grad_enabled(False)
    return Engine(model, EngineConfig(max_seqs=max_live, num_pages=pages, kv=kv))


class Replay:
    def __init__(self, engine, out_dir: str):
        self.engine, self.out_dir = engine, out_dir
        self.live: dict = {}

    def step(self, d: dict) -> None:
        entries = []
        for e in d.get("entries", []):
            if e["id"] not in self.live:
                self.live[e["id"]] = self.engine.open_replay()
            entries.append((self.live[e["id"]], [int(t) for t in e["tokens"]], [int(w) for w in e.get("want", [])]))
        logits = self.engine.replay_step(entries) if entries else None
        if logits is not None:
            rows = logits.float().cpu().contiguous().numpy().astype("<f4", copy=False)
            rows.tofile(os.path.join(self.out_dir, f"{d['step']}.f32"))
        for i in d.get("end", []):
            self.engine.close_replay(self.live.pop(i))
        if self.engine.device.type == "cuda":
            from .. import ops

            ops.check_status(self.engine.device.index)


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="Replay token ids through a model and write logits.")
    ap.add_argument("--model", required=True, help="folder with config.json and safetensors weights")
    ap.add_argument("--dtype", required=True, choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder for <step>.f32 files")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens that live requests hold at any time")
    ap.add_argument("--device", default="auto")
    a = ap.parse_args(argv)

    import torch

    from ..config import load_config

    cuda = a.device.startswith("cuda") or (a.device == "auto" and torch.cuda.is_available())
    if not cuda and a.device != "cpu":
        print("trace_run: no CUDA device (use --device cpu for the CPU operator set)", file=sys.stderr)
        return 2
    if cuda:
        if a.dtype == "float32" and load_config(a.model).model_type not in FLOAT32_FAMILIES:
            print("trace_run: this model family's CUDA kernels have no 32-bit form", file=sys.stderr)
            return 3
        from ..ops.build import build_extension

        build_extension()
    os.makedirs(a.out, exist_ok=True)
    replay = Replay(open_engine(a.model, a.dtype, a.max_tokens, a.device), a.out)
    for line in sys.stdin:
        if not line.strip():
            continue
        d = json.loads(line)
        replay.step(d)
        print(f"done {d['step']}", flush=True)
    return 0
