"""Per-sequence state of a decoder: a pool of slots, each holding what one sequence carries from step to step.

A model declares its buffers once -- ``recurrent`` ones start a sequence as zeros (matrix memories, convolution and
token-shift rings), ``ring`` ones are caches whose validity follows from the position and need no clearing.  Recurrent
buffers of a slot are views into one flat f32 arena, so giving a slot to a new sequence is a single fill.
"""
from __future__ import annotations

from dataclasses import dataclass

import torch


class StatePool:
    def __init__(self, n_slots: int, device):
        self.n_slots, self.device = n_slots, device
        self._recurrent: dict[str, tuple[tuple[int, ...], int]] = {}      # name -> (shape, offset in floats)
        self._arena_floats = 0
        self._rings: dict[str, tuple[tuple[int, ...], torch.dtype]] = {}
        self._free = list(range(n_slots))
        self.length = [0] * n_slots                                       # tokens of the slot's sequence so far
        self._views: list[dict[str, torch.Tensor]] = []
        self._arena = None
        i32 = dict(dtype=torch.int32, device=device)
        # device-resident loop state of every slot: position of the token to be processed, its id, the id before it
        self.pos, self.tok, self.prev = torch.zeros((n_slots, 32), **i32), torch.zeros((n_slots, 32), **i32), torch.zeros((n_slots, 32), **i32)

    def recurrent(self, name: str, *shape: int) -> None:
        n = 1
        for s in shape:
            n *= s
        self._recurrent[name] = (shape, self._arena_floats)
        self._arena_floats += (n + 63) // 64 * 64                         # 256-byte aligned views

    def ring(self, name: str, shape, dtype) -> None:
        self._rings[name] = (tuple(shape), dtype)

    def allocate(self) -> None:
        self._arena = torch.zeros((self.n_slots, max(self._arena_floats, 64)), dtype=torch.float32, device=self.device)
        for s in range(self.n_slots):
            views = {}
            for name, (shape, off) in self._recurrent.items():
                n = 1
                for d in shape:
                    n *= d
                views[name] = self._arena[s, off:off + n].view(shape)
            for name, (shape, dtype) in self._rings.items():
                views[name] = torch.zeros(shape, dtype=dtype, device=self.device)
            self._views.append(views)

    def views(self, slot: int) -> dict:
        return self._views[slot]

    def arena(self, slot: int) -> torch.Tensor:
        return self._arena[slot]

    def open(self) -> int:
        """A free slot, reset for a new sequence."""
        if not self._free:
            raise RuntimeError("no free sequence slot")
        slot = self._free.pop(0)
        self._arena[slot].zero_()
        self.pos[slot].zero_()
        self.prev[slot].zero_()
        self.length[slot] = 0
        return slot

    def close(self, slot: int) -> None:
        if slot in self._free:
            raise RuntimeError(f"slot {slot} is not in use")
        self._free.append(slot)

    @property
    def n_free(self) -> int:
        return len(self._free)


@dataclass
class Workspace:
    """Named scratch buffers that grow to the largest use; a name is one buffer for all layers."""
    device: object

    def __post_init__(self):
        self._bufs = {}

    def get(self, name: str, rows: int, cols: int, dtype=torch.float32) -> torch.Tensor:
        key = (name, dtype)
        need = rows * cols
        b = self._bufs.get(key)
        if b is None or b.numel() < need:
            b = torch.zeros(need, dtype=dtype, device=self.device)
            self._bufs[key] = b
        return b[:need].view(rows, cols)


class LayerRun:
    """What a mixer needs from the model for one execution of a layer on one sequence."""

    def __init__(self, views: dict, prefix: str, pos: torch.Tensor, start: int | None = None):
        """``pos``: the position on the device; ``start``: the same on the host, known for portions only."""
        self._views, self._prefix, self.pos, self.start = views, prefix, pos, start

    def state(self, name: str) -> torch.Tensor:
        return self._views[self._prefix + name]
