"""Token mixers with bf16 weights, shared by decoder designs.

A mixer owns its weights, declares its per-sequence state in a ``StatePool`` and runs two ways on the current stream:
``decode`` (one token, prologues and epilogues fused into the products, capturable) and ``prefill`` (a portion of
m tokens).  Both get the fused projection of the layer's input and leave the mixer's result either added to the
residual stream (``adds_residual``) or as the two vectors that the next row prologue combines (``combines``).
"""
from __future__ import annotations

from dataclasses import dataclass

import torch

from .seqops import EPI_ADD, PRO_GATED, Delta, DenseWeight, GatedHeads, MLstm, Matvec, SeqOps, WindowAttn, pad8, pad32, struct
from .ops import DT_BF16, DT_F32


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

    def __init__(self, views: dict, prefix: str, pos: torch.Tensor):
        self._views, self._prefix, self.pos = views, prefix, pos

    def state(self, name: str) -> torch.Tensor:
        return self._views[self._prefix + name]


def _off(t: torch.Tensor, cols: int) -> int:
    return t.data_ptr() + cols * t.element_size()


class ParallelWindowMLstm:
    """Sliding-window attention (per-head q / k norm, logarithmic distance term, sigmoid output gate) and an mLSTM matrix
    memory side by side on the same input; the result is half the sum of the two RMS-normed outputs."""
    combines, adds_residual = True, False

    def __init__(self, sop: SeqOps, cfg: dict, eps: float, width: int, load, load_f32, device, act, window_cap: int):
        self.sop, self.eps, self.width, self.act = sop, eps, width, act
        left, right = cfg["left"], cfg["right"]
        self.left, self.right = left, right
        self.window = min(left["mask"]["size"], window_cap)
        names = ["left.q", "left.k", "left.v", "left.g", "right.q", "right.k", "right.v", "right.g", "right.i", "right.f"]
        rows = [left["heads"] * left["dim"], left["kv_heads"] * left["dim"], left["kv_heads"] * left["vdim"], left["heads"] * left["vdim"],
                right["heads"] * right["dim"], right["heads"] * right["dim"], right["heads"] * right["vdim"], right["heads"] * right["vdim"],
                right["heads"], right["heads"]]
        self.proj = DenseWeight([load(n, r, width) for n, r in zip(names, rows)], device)
        self.off = dict(zip(names, self.proj.offsets))
        self.lo = DenseWeight(load("left.o", width, left["heads"] * left["vdim"]), device)
        self.ro = DenseWeight(load("right.o", width, right["heads"] * right["vdim"]), device)
        f = lambda n, *s: load_f32(n, *s).to(device)
        self.q_norm, self.k_norm = f("left.q.norm", left["dim"]), f("left.k.norm", left["dim"])
        self.r1, self.r2 = f("left.r1", left["heads"]), f("left.r2", left["heads"])
        self.r_norm = f("right.norm", right["heads"] * right["vdim"])
        self.i_b, self.f_b = f("right.i.b", right["heads"]), f("right.f.b", right["heads"])
        self.a_norm, self.b_norm = f("left.out", width), f("right.out", width)
        self.scratch = None

    def declare(self, pool, prefix: str, max_portion: int, cache_dtype) -> None:
        left, right = self.left, self.right
        self.capacity, self.cache_dtype = self.window - 1 + max_portion, cache_dtype
        pool.ring(prefix + "k", (left["kv_heads"], self.capacity, pad8(left["dim"])), cache_dtype)
        pool.ring(prefix + "v", (left["kv_heads"], self.capacity, pad8(left["vdim"])), cache_dtype)
        slices = (right["vdim"] + 15) // 16
        pool.recurrent(prefix + "s", right["heads"], right["vdim"], pad32(right["dim"]))
        pool.recurrent(prefix + "n", right["heads"], slices, pad32(right["dim"]))
        pool.recurrent(prefix + "mx", right["heads"], slices)

    def _attn(self, run: LayerRun, proj) -> WindowAttn:
        c, o = self.left, self.off
        return struct(WindowAttn, qkv=proj, ld=self.proj.n, q_off=o["left.q"], k_off=o["left.k"], v_off=o["left.v"], q_norm=self.q_norm, k_norm=self.k_norm,
                      r1=self.r1, r2=self.r2, k_cache=run.state("k"), v_cache=run.state("v"), heads=c["heads"], kv_heads=c["kv_heads"], dim=c["dim"],
                      vdim=c["vdim"], window=self.window, capacity=self.capacity, cache_dtype=DT_F32 if self.cache_dtype == torch.float32 else DT_BF16,
                      scale=c["scale"], eps=self.eps, pos=run.pos)

    def _mlstm(self, run: LayerRun, proj) -> MLstm:
        c, o = self.right, self.off
        return struct(MLstm, proj=proj, ld=self.proj.n, q_off=o["right.q"], k_off=o["right.k"], v_off=o["right.v"], i_off=o["right.i"], f_off=o["right.f"],
                      i_bias=self.i_b, f_bias=self.f_b, s=run.state("s"), n=run.state("n"), mx=run.state("mx"), heads=c["heads"], dim=c["dim"],
                      vdim=c["vdim"], gate_cap=c["gate_cap"])

    def _right_gate(self, o, proj) -> GatedHeads:
        c = self.right
        return struct(GatedHeads, o=o, gate=_off(proj, self.off["right.g"]), norm=self.r_norm, ldo=o.shape[1], ldg=self.proj.n, heads=c["heads"],
                      head_dim=c["vdim"], norm_all=1, eps=self.eps)

    def decode(self, run: LayerRun, ws: Workspace, proj, x):
        left, right, sop = self.left, self.right, self.sop
        att = ws.get("d.att", 1, left["heads"] * left["vdim"])
        mem = ws.get("d.mem", 1, right["heads"] * right["vdim"])
        a, b = ws.get("d.a", 1, self.width), ws.get("d.b", 1, self.width)
        attn = self._attn(run, proj)
        if self.scratch is None:
            self.scratch = sop.window_scratch(attn, ws.device)
        sop.window_decode(attn, att, self.scratch)
        sop.mlstm(self._mlstm(run, proj), 1, mem)
        gate = struct(GatedHeads, o=att, gate=_off(proj, self.off["left.g"]), ldo=att.shape[1], ldg=self.proj.n, heads=left["heads"], head_dim=left["vdim"],
                      eps=self.eps)
        sop.matvec(PRO_GATED, struct(Matvec, w=self.lo.w, y=a, gated=gate, n=self.lo.n, k=self.lo.k),
                   struct(Matvec, w=self.ro.w, y=b, gated=self._right_gate(mem, proj), n=self.ro.n, k=self.ro.k))
        return a, b

    def prefill(self, run: LayerRun, ws: Workspace, proj, x, m: int):
        left, right, sop = self.left, self.right, self.sop
        attn = self._attn(run, proj)
        q = ws.get("q", m, left["heads"] * pad8(left["dim"]), self.cache_dtype)
        att = ws.get("att", m, self.lo.k, self.act)
        mem = ws.get("mem", m, right["heads"] * right["vdim"])
        gated = ws.get("gated", m, self.ro.k, self.act)
        a, b = ws.get("a", m, self.width), ws.get("b", m, self.width)
        sop.window_append(attn, m, q)
        sop.window_prefill(attn, m, q, _off(proj, self.off["left.g"]), self.proj.n, att)
        sop.mlstm(self._mlstm(run, proj), m, mem)
        sop.gated_heads(self._right_gate(mem, proj), m, gated)
        sop.matmul(att, self.lo, a, m)
        sop.matmul(gated, self.ro, b, m)
        return a, b

    def delta(self, run, proj):
        return None                                    # no convolution state

    def decode_bytes(self) -> int:
        """Bytes one decode step reads and writes besides activations: weights and state."""
        left, right = self.left, self.right
        kv = self.window * left["kv_heads"] * (pad8(left["dim"]) + pad8(left["vdim"])) * (4 if self.act == torch.float32 else 2)
        return self.proj.nbytes + self.lo.nbytes + self.ro.nbytes + kv + 8 * right["heads"] * right["vdim"] * pad32(right["dim"])


class ChannelDelta:
    """Gated delta rule with one decay per head and key channel, short convolutions on q, k and v, low-rank decay and
    output-gate projections."""
    combines, adds_residual = False, True

    def __init__(self, sop: SeqOps, cfg: dict, eps: float, width: int, load, load_f32, device, act, window_cap: int):
        self.sop, self.eps, self.width, self.act, self.c = sop, eps, width, act, cfg
        H, G, d, dv, taps = cfg["heads"], cfg["kv_heads"], cfg["dim"], cfg["vdim"], cfg["conv"]
        a1, g1 = load("a1", None, width), load("g1", None, width)          # the ranks are the tensors' own
        names = ["q", "k", "v", "b", "a1", "g1"]
        self.proj = DenseWeight([load("q", G * d, width), load("k", G * d, width), load("v", H * dv, width), load("b", H, width), a1, g1], device)
        self.off = dict(zip(names, self.proj.offsets))
        self.a2, self.g2 = DenseWeight(load("a2", H * d, a1.shape[0]), device), DenseWeight(load("g2", H * dv, g1.shape[0]), device)
        self.o = DenseWeight(load("o", width, H * dv), device)
        f = lambda n, *s: load_f32(n, *s).to(device)
        self.q_conv, self.k_conv, self.v_conv = f("q.conv", G * d, taps), f("k.conv", G * d, taps), f("v.conv", H * dv, taps)
        self.a_log, self.dt_bias, self.norm = f("A_log", H), f("dt_bias", H * d), f("norm", dv)

    def declare(self, pool, prefix: str, max_portion: int, cache_dtype) -> None:
        c = self.c
        pool.recurrent(prefix + "conv", 2 * c["kv_heads"] * c["dim"] + c["heads"] * c["vdim"], c["conv"])
        pool.recurrent(prefix + "s", c["heads"], c["vdim"], pad32(c["dim"]))

    def delta(self, run: LayerRun, proj) -> Delta:
        c, o = self.c, self.off
        return struct(Delta, proj=proj, ld=self.proj.n, q_off=o["q"], k_off=o["k"], v_off=o["v"], b_off=o["b"], a1_off=o["a1"], g1_off=o["g1"],
                      q_conv=self.q_conv, k_conv=self.k_conv, v_conv=self.v_conv, a_log=self.a_log, dt_bias=self.dt_bias, a2=self.a2.w, g2=self.g2.w,
                      conv_state=run.state("conv"), s=run.state("s"), heads=c["heads"], kv_heads=c["kv_heads"], dim=c["dim"], vdim=c["vdim"],
                      taps=c["conv"], a_rank_ld=self.a2.k, g_rank_ld=self.g2.k, pos=run.pos)

    def _gate(self, o, gate) -> GatedHeads:
        c = self.c
        return struct(GatedHeads, o=o, gate=gate, norm=self.norm, ldo=o.shape[1], ldg=gate.shape[1], heads=c["heads"], head_dim=c["vdim"], norm_all=0,
                      eps=self.eps)

    def decode(self, run: LayerRun, ws: Workspace, proj, x):
        n = self.c["heads"] * self.c["vdim"]
        o, gate = ws.get("d.mem", 1, n), ws.get("d.gate", 1, n)
        self.sop.delta_step(self.delta(run, proj), o, gate)
        self.sop.matvec(PRO_GATED, struct(Matvec, w=self.o.w, y=x, residual=x, gated=self._gate(o, gate), n=self.o.n, k=self.o.k, epilogue=EPI_ADD))

    def prefill(self, run: LayerRun, ws: Workspace, proj, x, m: int):
        c, sop = self.c, self.sop
        H, G, d, dv = c["heads"], c["kv_heads"], c["dim"], c["vdim"]
        a = self.delta(run, proj)
        qkv, beta = ws.get("qkv", m, 2 * G * d + H * dv), ws.get("beta", m, H)
        a1, g1 = ws.get("a1", m, self.a2.k, self.act), ws.get("g1", m, self.g2.k, self.act)
        g, gate, mem = ws.get("decay", m, H * d), ws.get("gate", m, H * dv), ws.get("mem", m, H * dv)
        gated = ws.get("gated", m, self.o.k, self.act)
        sop.delta_prep(a, m, qkv, beta, a1, g1)
        sop.matmul(a1, self.a2, g, m)
        sop.matmul(g1, self.g2, gate, m)
        sop.delta_decay(a, m, g)
        sop.delta_scan(a, m, qkv, beta, g, mem)
        sop.gated_heads(self._gate(mem, gate), m, gated)
        sop.matmul(gated, self.o, x, m, epilogue=EPI_ADD, residual=x)

    def decode_bytes(self) -> int:
        c = self.c
        return self.proj.nbytes + self.a2.nbytes + self.g2.nbytes + self.o.nbytes + 8 * c["heads"] * c["vdim"] * pad32(c["dim"])


MIXERS = {"parallel": ParallelWindowMLstm, "channel_delta": ChannelDelta}
