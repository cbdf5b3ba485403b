"""Serving loop over a decoder: requests named by id, each bound to a sequence slot from its first tokens to its end.

``step`` runs given tokens of given requests (what a trace replay does); ``generate`` admits prompts in order as slots
come free and decodes greedily.  Works with any ``decoder.GreedyDecoder``.
"""
from __future__ import annotations

from collections import deque
from dataclasses import dataclass

import torch


@dataclass
class Entry:
    id: str
    tokens: list
    want: list


class Engine:
    def __init__(self, model):
        self.model = model
        self._slots: dict[str, int] = {}

    def step(self, entries, end=()) -> torch.Tensor | None:
        """Runs every entry's tokens from the state its earlier steps left; returns the wanted logits, rows in the order
        of the entries and of ``want`` (None if nothing is wanted).  ``end``: requests that give back their slot."""
        rows = []
        for e in entries:
            if e.id not in self._slots:
                self._slots[e.id] = self.model.open_slot()
            slot = self._slots[e.id]
            order = sorted(range(len(e.want)), key=lambda j: e.want[j])
            got = self.model.extend(slot, torch.tensor(e.tokens, dtype=torch.int32), [e.want[j] for j in order])
            back = torch.empty(len(order), dtype=torch.long)
            back[order] = torch.arange(len(order))
            if len(order):
                rows.append(got[back.to(got.device)])
        for i in end:
            self.model.close_slot(self._slots.pop(i))
        return torch.cat(rows) if rows else None

    def generate(self, prompts, n_new: int) -> list[list[int]]:
        """Greedy continuations of the prompts (lists of token ids), n_new tokens each."""
        waiting = deque(enumerate(prompts))
        out: list = [None] * len(prompts)
        while waiting:
            active = []
            while waiting and len(active) < self.model.n_slots:
                i, ids = waiting.popleft()
                slot = self.model.open_slot()
                self.model.extend(slot, torch.tensor(ids, dtype=torch.int32), [])
                active.append((i, slot))
            for i, slot in active:
                self.model.bind(slot)
                first = int(self.model.tok[0])
                more = self.model.generate(n_new - 1).tolist() if n_new > 1 else []
                out[i] = [first] + more
                self.model.close_slot(slot)
        return out
