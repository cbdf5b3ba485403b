"""Gated feed-forward layers with bf16 weights, shared by decoder designs.

Like a mixer, a feed-forward owns its weights and runs two ways: ``decode`` takes the row prologue that stands in front of
its first product, ``prefill`` the normed rows of a portion.  Both return (output, parts): the layer's output is the sum of
``parts`` consecutive rows per token, added up by whoever reads it next.  Gate and up rows alternate in one matrix, so
that a product's epilogue holds both of a pair.
"""
from __future__ import annotations

import torch

from .seqops import (EPI_CLAMP_GLU, EPI_NONE, EPI_SWIGLU, GROUP_TILE, PRO_HYPER, PRO_NONE, DenseWeight, ExpertStep, Hyper, Matvec, RowGroups, SeqOps, pad8,
                     struct)
from .state import Workspace


def _pairs(gate: torch.Tensor, up: torch.Tensor) -> torch.Tensor:
    """Rows gate 0, up 0, gate 1, up 1, ... with zero rows up to a multiple of 8 pairs (they give zeros: the pitch the next
    product reads)."""
    both = torch.stack([gate, up], dim=1).reshape(2 * gate.shape[0], *gate.shape[1:])
    return torch.cat([both, both.new_zeros(2 * (pad8(gate.shape[0]) - gate.shape[0]), *gate.shape[1:])])


class ClampedGlu:
    """g = min(gate, limit), u = clamp(up, -limit, limit): down(g sigmoid(1.702 g) (u + 1)); biases on all three."""

    def __init__(self, sop: SeqOps, cfg: dict, width: int, load, load_f32, device, act):
        self.sop, self.width, self.act, self.limit = sop, width, act, float(cfg["limit"])
        ff = cfg["ff"]
        self.gate_up = DenseWeight(_pairs(load("gate", ff, width), load("up", ff, width)), device)
        self.gate_up_b = _pairs(load_f32("gate.b", ff), load_f32("up.b", ff)).to(device)
        self.down, self.down_b = DenseWeight(load("down", width, ff), device), load_f32("down.b", width).to(device)

    def decode(self, ws: Workspace, pre: Hyper):
        act, y = ws.get("d.act", 1, self.down.k), ws.get("d.y", 1, self.width)
        self.sop.matvec(PRO_HYPER, struct(Matvec, w=self.gate_up.w, y=act, hyper=pre, n=self.gate_up.n, k=self.gate_up.k, epilogue=EPI_CLAMP_GLU, cap=self.limit,
                                          bias=self.gate_up_b))
        self.sop.matvec(PRO_NONE, struct(Matvec, w=self.down.w, y=y, x=act, n=self.down.n, k=self.down.k, epilogue=EPI_NONE, bias=self.down_b))
        return y, 1

    def prefill(self, ws: Workspace, h, m: int):
        act, y = ws.get("act", m, self.down.k, self.act), ws.get("y", m, self.width)
        self.sop.matmul(h, self.gate_up, act, m, EPI_CLAMP_GLU, cap=self.limit, bias=self.gate_up_b)
        self.sop.matmul(act, self.down, y, m, bias=self.down_b)
        return y, 1

    def decode_bytes(self) -> int:
        return self.gate_up.nbytes + self.down.nbytes


class RoutedExperts:
    """Sigmoid-scored routing to ``top`` of the experts, scores not renormalised and applied to the expert's input (which,
    gate and up being linear, is the same as scaling both of their outputs); expert: down(silu(gate) up)."""

    def __init__(self, sop: SeqOps, cfg: dict, width: int, load, load_f32, device, act):
        self.sop, self.width, self.act = sop, width, act
        self.experts, self.top, ff = cfg["router"]["experts"], cfg["router"]["top"], cfg["expert"]["ff"]
        if not 1 <= self.top <= self.experts:
            raise ValueError(f"routed experts: {self.top} of {self.experts}")
        self.router = DenseWeight(load("router", self.experts, width), device)
        self.gate_up = DenseWeight(torch.cat([_pairs(load(f"e{e}.gate", ff, width), load(f"e{e}.up", ff, width)) for e in range(self.experts)]), device)
        self.down = DenseWeight(torch.cat([load(f"e{e}.down", width, ff) for e in range(self.experts)]), device)

    def decode(self, ws: Workspace, pre: Hyper):
        h, logits = ws.get("d.h", 1, self.router.k), ws.get("d.router", 1, self.experts)
        act, y, ids = ws.get("d.act", self.top, self.down.k), ws.get("d.y", 1, self.width), ws.get("d.ids", 1, self.top, torch.int32)
        pre.h_out = h.data_ptr()
        self.sop.matvec(PRO_HYPER, struct(Matvec, w=self.router.w, y=logits, hyper=pre, n=self.experts, k=self.router.k))
        self.sop.expert_step(struct(ExpertStep, gate_up=self.gate_up.w, down=self.down.w, logits=logits, h=h, ids=ids, act=act, y=y, experts=self.experts,
                                    top=self.top, ff=self.down.k, width=self.width, k_in=self.router.k))
        return y, 1

    def prefill(self, ws: Workspace, h, m: int):
        sop, rows, i32, tile = self.sop, m * self.top, torch.int32, GROUP_TILE[h.dtype]
        logits = ws.get("moe.logits", m, pad8(self.experts))[:, :self.experts]
        ids, scores, perm = ws.get("moe.ids", m, self.top, i32), ws.get("moe.scores", m, self.top), ws.get("moe.perm", m, self.top, i32)
        header, tiles = ws.get("moe.header", 1, 64, i32), ws.get("moe.tiles", rows // tile + min(rows, self.experts), 4, i32)
        xg, act, y = ws.get("moe.x", rows, self.router.k, h.dtype), ws.get("moe.act", rows, self.down.k, self.act), ws.get("y", rows, self.width)
        sop.matmul(h, self.router, logits, m)
        sop.sigmoid_topk(logits, ids, scores, m, self.experts, self.top)
        sop.sort_rows(ids, m, self.top, self.experts, h, header, tiles, perm, xg)
        group = dict(header=header, tiles=tiles, perm=perm, groups=self.experts, tile_rows=tile)
        sop.grouped(struct(RowGroups, row_scale=scores, **group), xg, self.gate_up, act, rows, EPI_SWIGLU)
        sop.grouped(struct(RowGroups, scatter=1, **group), act, self.down, y, rows)
        return y, self.top

    def decode_bytes(self) -> int:
        return self.router.nbytes + (self.gate_up.nbytes + self.down.nbytes) * self.top // self.experts


FEED_FORWARDS = {"dense": ClampedGlu, "moe": RoutedExperts}
