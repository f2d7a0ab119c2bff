"""Replaying a trace: given token ids through a model step by step, logits out, nothing sampled.

The steps run on the engine and request bookkeeping that generation uses (``HostBatcher.extend`` ->
``Engine.forward_batch``): a request is admitted when its first tokens come, every step is one batch of
prompt portions and single tokens, and what a finished request held is given back.
"""
from __future__ import annotations

import json
from pathlib import Path

import numpy as np

from .engine import EngineConfig
from .host_batch import HostBatcher
from .models import load_model, read_config

PAGE_SIZE = 64
MAX_LIVE = 4    # state slots: live requests at any time


class TraceReplay:
    def __init__(self, model_dir, dtype: str, max_tokens: int, page_size: int = PAGE_SIZE, max_live: int = MAX_LIVE):
        pages = max(1, -(-max_tokens // page_size))
        tokens = pages * page_size
        self.engine = load_model(model_dir, EngineConfig(page_size, pages, max_live, tokens, tokens), dtype,
                                 read_config(model_dir, dtype))
        self.engine.capture_graphs(range(1, max_live + 1))   # steps of single tokens replay as decode graphs
        # a trace says what it caches: nothing is shared between its requests
        self.batcher = HostBatcher(self.engine, pages, page_size, max_live, enable_prefix_cache=False)
        self.max_len = tokens
        self.live: dict = {}

    def step(self, entries, end) -> np.ndarray:
        """Run one step; the wanted logits, fp32 [wanted, vocab], in the order of the entries."""
        reqs, portions, wanted, at = [], [], [], 0
        for e in entries:
            if not e["tokens"]:
                continue
            if e["id"] not in self.live:
                self.live[e["id"]] = self.batcher.open_request(self.max_len)
            reqs.append(self.live[e["id"]])
            portions.append(e["tokens"])
            wanted += [at + int(k) for k in e.get("want", [])]
            at += len(e["tokens"])
        logits = np.zeros((0, self.engine.model_config.vocab_size), np.float32)
        if reqs:
            self.batcher.extend(reqs, portions).synchronize()
            if wanted:
                logits = self.engine.token_logits(wanted).numpy()
        for name in end:
            if name in self.live:
                self.batcher.release(self.live.pop(name))
        return logits


def replay(lines, out_dir, run: TraceReplay, report) -> None:
    """Steps from an iterable of JSON lines; logits to ``out_dir/<step>.f32``; ``report(step)`` after each."""
    out = Path(out_dir)
    out.mkdir(parents=True, exist_ok=True)
    for line in lines:
        if not line.strip():
            continue
        s = json.loads(line)
        logits = run.step(s.get("entries", []), s.get("end", []))
        if len(logits):
            logits.astype("<f4", copy=False).tofile(out / f"{s['step']}.f32")
        report(s["step"])
