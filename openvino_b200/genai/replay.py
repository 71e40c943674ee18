"""Replay of given tokens: the serving program's steps, cache and kernels, driven by the caller's batches instead of a sampler.

A step names requests and their next tokens; the logits at any of those tokens can be asked for. Blocks and state slots come from
the scheduler's block manager and go back when a request ends. A step that exceeds the executor's token or sequence limits is run
in portions.
"""
from __future__ import annotations

from typing import Dict, List, Sequence as Seq, Tuple

import numpy as np
import torch

from ..runtime.cuda_llm import LlmExecutor
from .pipeline import step_shape
from .scheduler import Scheduler, SchedulerConfig, Sequence


class Replay:
    def __init__(self, executor: LlmExecutor):
        self.ex = executor
        self.scheduler = Scheduler(SchedulerConfig(max_num_batched_tokens=executor.prefill.Tcap, max_num_seqs=executor.max_seqs,
                                                   num_kv_blocks=executor.num_kv_blocks, block_size=executor.block_size))
        self.requests: Dict[object, Sequence] = {}
        self._count = 0
        self._views = {id(sb): {name: sb.view(name, host=0).numpy() for name in sb.offsets} for sb in (executor.prefill, executor.decode)}

    def step(self, entries: Seq[Tuple[object, Seq[int], Seq[int]]]) -> torch.Tensor:
        """entries: (request, next tokens, places among these tokens whose logits are wanted); a request that is not known yet
        starts. Returns fp32 logits [wanted, vocab] on the host, in the order of the entries and of their places."""
        todo: List[Tuple[int, Sequence, int, int]] = []      # (entry, sequence, first new token, end)
        for i, (rid, tokens, want) in enumerate(entries):
            if len(tokens) == 0:
                raise ValueError("request %s brings no token" % (rid,))
            if any(not 0 <= w < len(tokens) for w in want):
                raise ValueError("request %s asks for a place outside its tokens" % (rid,))
            seq = self.requests.get(rid)
            if seq is None:
                seq = Sequence(self._count, np.zeros(0, dtype=np.int32), 0)
                self._count += 1
                self.scheduler.admit(seq)
                self.requests[rid] = seq
            base = len(seq.prompt)
            seq.prompt = np.concatenate([seq.prompt, np.asarray(tokens, dtype=np.int32)])
            todo.append((i, seq, base, base + len(tokens)))
        rows: Dict[Tuple[int, int], torch.Tensor] = {}
        at = {i: base for i, _, base, _ in todo}
        while True:
            batch, left = [], self.ex.prefill.Tcap
            for i, seq, base, end in todo:
                n = min(end - at[i], left)
                if n > 0 and len(batch) < self.ex.max_seqs:
                    batch.append((i, seq, base, n))
                    left -= n
            if not batch:
                break
            self._run(batch, at, entries, rows)
        out = [rows[(i, w)] for i, (_, _, want) in enumerate(entries) for w in want]
        return torch.stack(out) if out else torch.empty((0, self.ex.cfg.vocab_size), dtype=torch.float32)

    def _run(self, batch, at, entries, rows) -> None:
        ex = self.ex
        st = self.scheduler.place([b[1] for b in batch], [b[3] for b in batch])
        sb = ex.decode if st.max_q_len == 1 and len(st.seqs) <= ex.decode.Bcap else ex.prefill
        self.scheduler.fill(st, self._views[id(sb)])
        ex.upload(sb, 0)
        ex.run(sb, step_shape(st))
        self.scheduler.advance(st)
        keys, where, t = [], [], 0
        for i, _, base, n in batch:
            lo = at[i] - base                                  # places of this entry that the portion covers
            for w in entries[i][2]:
                if lo <= w < lo + n:
                    keys.append((i, w))
                    where.append(t + w - lo)
            at[i] += n
            t += n
        if where:
            rows.update(zip(keys, ex.logits_at(sb, where).cpu()))
        torch.cuda.current_stream().synchronize()              # the pinned descriptor may be rewritten

    def end(self, rid) -> None:
        """The request is finished: its blocks and state slot are free again."""
        self.scheduler.retire(self.requests.pop(rid))
