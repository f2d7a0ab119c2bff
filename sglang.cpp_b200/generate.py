"""Batch generation through the scheduler: prompts in, token ids out."""
from __future__ import annotations

from typing import Optional, Sequence

from .host_batch import HostScheduler


def generate(engine, prompts: Sequence, max_new_tokens: int, temperature: float = 0.0, top_k: int = -1,
             top_p: float = 1.0, seed: int = 0, prefix_cache: bool = True,
             scheduler: Optional[HostScheduler] = None) -> list:
    """Run every prompt (a sequence of token ids) for ``max_new_tokens`` tokens; returns the generated
    ids per prompt.  Greedy unless ``temperature`` > 0.  Requests are admitted, chunked, batched and
    retired by ``HostScheduler``, as the reference's scheduler does it."""
    c = engine.config
    sched = scheduler or HostScheduler(engine, c.num_pages, c.page_size, c.max_running_req, c.max_seq_len,
                                       c.max_extend_tokens, prefix_cache)
    for uid, p in enumerate(prompts):
        # HostScheduler counts the token a prefill samples as the first new one
        if len(p) + max_new_tokens > c.max_seq_len:
            raise ValueError(f"prompt {uid}: {len(p)} + {max_new_tokens} tokens exceed max_seq_len {c.max_seq_len}")
        sched.submit(uid, p, max_new_tokens)
    out: list = [[] for _ in prompts]
    while True:
        batch = sched.next_batch()
        if batch is None:
            break
        reqs = batch.reqs
        sampling = {}
        if temperature > 0:
            sampling = dict(temperatures=[temperature] * len(reqs), top_k=[top_k] * len(reqs),
                            top_p=[top_p] * len(reqs), seeds=[seed + r.uid for r in reqs])
        fo = engine.forward_batch(batch.phase, [r.table_idx for r in reqs], [r.cached_len for r in reqs],
                                  [r.extend_len() for r in reqs], write_pos=[r.write_pos() for r in reqs], **sampling)
        fo.synchronize()
        tokens = fo.next_tokens_cpu[:len(reqs)].numpy().copy()
        chunked = [r.is_chunked_prefill for r in reqs]
        sched.finish_batch(batch, tokens)
        for r, tok, part in zip(reqs, tokens, chunked):
            if not part:
                out[r.uid].append(int(tok))
    return [o[:max_new_tokens] for o in out]
