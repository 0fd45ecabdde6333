"""Sequences over a runner's slots: portions, single steps and greedy generation.

A runner decodes its slots 0 .. batch-1 side by side; the scheduler keeps which request is in which slot, gives slots
back and reuses them, and picks the kernels: one token of the only sequence goes through the decode step's graph,
anything longer is a portion of a prompt.
"""
from __future__ import annotations

from typing import Dict, Iterable, List, Optional, Sequence

import numpy as np


class Scheduler:
    def __init__(self, model):
        self.model = model
        self.slots: Dict[object, int] = {}
        self.free: List[int] = list(range(model.max_batch))

    # -- requests -------------------------------------------------------------------
    def slot(self, request) -> int:
        if request not in self.slots:
            if not self.free:
                raise RuntimeError(f"all {self.model.max_batch} slots are taken")
            s = self.free.pop(0)
            self.model.release(s)
            self.slots[request] = s
        return self.slots[request]

    def finish(self, request):
        """Give back what a request holds (unknown requests hold nothing)."""
        s = self.slots.pop(request, None)
        if s is not None:
            self.model.release(s)
            self.free.append(s)
            self.free.sort()

    # -- steps ----------------------------------------------------------------------
    def step(self, request, tokens: Sequence[int], want: Sequence[int] = ()) -> np.ndarray:
        """Run a request's next tokens; logits [len(want), vocab] at the wanted places among them, in that order."""
        s, want = self.slot(request), list(want)
        if any(w < 0 or w >= len(tokens) for w in want):
            raise ValueError("a wanted place lies outside the tokens")
        if len(tokens) == 1 and s == 0 and len(self.slots) == 1:
            self.model.decode([tokens[0]], 1)
            rows = self.model.read_logits(self.model.cfg["vocab"]).reshape(1, -1) if want else np.empty((0, self.model.cfg["vocab"]), np.float32)
            return rows[want] if want else rows
        order = sorted(set(want))
        rows = self.model.extend(tokens, order, s)
        return rows[[order.index(w) for w in want]] if want else rows

    # -- greedy generation -----------------------------------------------------------
    def generate(self, prompts: Iterable[Sequence[int]], max_new_tokens: int, stop: Optional[Iterable[int]] = None, block: int = 32) -> List[List[int]]:
        """Greedy continuation of every prompt (a token of ``stop`` ends a sequence and is kept).  Prompts are taken in
        groups of at most max_batch; a group decodes together, ``block`` steps between two looks at the stop tokens."""
        if self.slots:
            raise RuntimeError("generate needs every slot free")
        prompts, stop, out = [list(p) for p in prompts], set(stop or ()), []
        m = self.model
        for g0 in range(0, len(prompts), m.max_batch):
            group = prompts[g0:g0 + m.max_batch]
            if max_new_tokens < 1:
                out += [[] for _ in group]
                continue
            for i in range(len(group)):
                m.release(i)
            done = [[m.prefill(p, seq=i)] for i, p in enumerate(group)]
            left = max_new_tokens - 1
            while left > 0 and not all(stop.intersection(d) for d in done):
                room = min(m.cfg["max_seq"] - m.seq_len(i) for i in range(len(group)))
                n = min(block, left, room)
                if n < 1:
                    break
                toks = m.decode([d[-1] for d in done], n)
                for i, d in enumerate(done):
                    d.extend(int(t) for t in toks[:, i])
                left -= n
            for i, d in enumerate(done):
                hit = next((j for j, t in enumerate(d) if t in stop), None)
                out.append(d if hit is None else d[:hit + 1])
                m.release(i)
        return out
