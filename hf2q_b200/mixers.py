"""Token mixers with bf16 weights, shared by decoder designs.

A mixer owns its weights, declares its per-sequence state in a ``StatePool`` and runs two ways on the current stream:
``decode`` (one token, prologues and epilogues fused into the products, capturable) and ``prefill`` (a portion of
m tokens).  Both get the fused projection of the layer's input and leave the mixer's result added to the residual
stream (``adds_residual``), as the two vectors that the next row prologue combines (``combines``), or else return it.
"""
from __future__ import annotations

import torch

from .ops import DT_BF16, DT_F32
from .seqops import (EPI_ADD, GATE_SILU_FIRST, PRO_GATED, PRO_NONE, Delta, DenseWeight, GatedHeads, LatentAttn, MLstm, Matvec, SeqOps, Ssd, WindowAttn, pad8,
                     pad32, struct)
from .state import LayerRun, Workspace


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


class Mamba2:
    """State-space layer with a scalar decay per head and token; short convolution on x, B and C; the output is gated
    before it is normed in equal parts."""
    combines, adds_residual = False, False

    def __init__(self, sop: SeqOps, cfg: dict, eps: float, width: int, load, load_f32, device, act, window_cap: int):
        self.sop, self.eps, self.width, self.act, self.c = sop, eps, width, act, cfg
        H, G, N, taps = cfg["heads"], cfg["groups"], cfg["state"], cfg["conv"]
        self.inner = H * cfg["vdim"]
        self.channels = self.inner + 2 * G * N
        if H % G or self.inner % cfg["norm_groups"]:
            raise ValueError(f"mamba2: {H} heads in {G} groups, {self.inner} outputs in {cfg['norm_groups']} normed parts")
        self.proj = DenseWeight(load("in", self.inner + self.channels + H, width), device)
        self.o = DenseWeight(load("o", width, self.inner), device)
        f = lambda n, *s: load_f32(n, *s).to(device)
        self.conv, self.conv_b = f("conv", self.channels, taps), f("conv.b", self.channels)
        self.dt_bias, self.a_log, self.d, self.norm = f("dt_bias", H), f("A_log", H), f("D", H), f("norm", self.inner)

    def declare(self, pool, prefix: str, max_portion: int, cache_dtype) -> None:
        c = self.c
        pool.recurrent(prefix + "conv", self.channels, c["conv"])
        pool.recurrent(prefix + "s", c["heads"], c["vdim"], pad32(c["state"]))

    def _ssd(self, run: LayerRun, proj) -> Ssd:
        c = self.c
        return struct(Ssd, proj=proj, ld=proj.stride(0), off=self.inner, conv=self.conv, conv_bias=self.conv_b, dt_bias=self.dt_bias, a_log=self.a_log, d=self.d,
                      conv_state=run.state("conv"), s=run.state("s"), heads=c["heads"], groups=c["groups"], state=c["state"], vdim=c["vdim"], taps=c["conv"],
                      pos=run.pos)

    def _gate(self, y, proj) -> GatedHeads:
        n = self.c["norm_groups"]
        return struct(GatedHeads, o=y, gate=proj, norm=self.norm, ldo=y.stride(0), ldg=proj.stride(0), heads=n, head_dim=self.inner // n, norm_all=1,
                      eps=self.eps, kind=GATE_SILU_FIRST)

    def decode(self, run: LayerRun, ws: Workspace, proj, x=None):
        y, out = ws.get("d.mem", 1, self.inner), ws.get("d.y", 1, self.width)
        self.sop.ssd_step(self._ssd(run, proj), y)
        self.sop.matvec(PRO_GATED, struct(Matvec, w=self.o.w, y=out, gated=self._gate(y, proj), n=self.o.n, k=self.o.k))
        return out

    def prefill(self, run: LayerRun, ws: Workspace, proj, x, m: int):
        sop, a, H = self.sop, self._ssd(run, proj), self.c["heads"]
        xbc, dt, la = ws.get("xbc", m, self.channels), ws.get("dt", m, H), ws.get("la", m, H)
        y, gated, out = ws.get("mem", m, self.inner), ws.get("gated", m, self.o.k, self.act), ws.get("y", m, self.width)
        sop.ssd_prep(a, m, xbc, dt, la)
        sop.ssd_scan(a, m, xbc, dt, la, y)
        sop.gated_heads(self._gate(y, proj), m, gated)
        sop.matmul(gated, self.o, out, m)
        return out

    def decode_bytes(self) -> int:
        c = self.c
        return self.proj.nbytes + self.o.nbytes + 8 * c["heads"] * c["vdim"] * pad32(c["state"])


class LatentAttention:
    """Sliding-window attention whose keys and values are expanded from one cached latent vector per token; a rotated part
    of every key is shared by the heads.  Decoding moves the query into the latent space instead, portions expand the
    window's latents."""
    combines, adds_residual = False, False

    def __init__(self, sop: SeqOps, cfg: dict, eps: float, width: int, load, load_f32, device, act, window_cap: int):
        self.sop, self.eps, self.width, self.act, self.c = sop, eps, width, act, cfg
        H, d, r, dv, rank, rot = cfg["heads"], cfg["dim"], cfg["rot_dim"], cfg["vdim"], cfg["kv_rank"], cfg["rot"]
        if rot["dims"] % 2 or rot["dims"] > r:
            raise ValueError(f"latent attention: {rot['dims']} turned dimensions of {r}")
        self.window = min(cfg["mask"]["size"], window_cap)
        self.proj = DenseWeight([load("q", H * (d + r), width), load("dkv", rank + r, width)], device)
        uk, uv = load("uk", H * d, rank), load("uv", H * dv, rank)
        self.dp, self.vp, self.rp, self.row = pad8(d), pad8(dv), pad8(rank), pad8(rank) + pad8(r)
        # portions: every head's keys, then every head's values, at multiples of 8 columns
        self.ukv = DenseWeight(list(uk.split(d)) + list(uv.split(dv)), device)
        # decoding: uk transposed per head
        self.uk_t = DenseWeight(uk.view(H, d, rank).transpose(1, 2).reshape(H * rank, d), device)
        self.uv = DenseWeight(uv, device)
        self.o = DenseWeight(load("o", width, H * dv), device)
        self.norm = load_f32("dkv.norm", rank).to(device)
        i = torch.arange(rot["dims"] // 2, dtype=torch.float64)
        self.freq = (float(rot["base"]) ** (-2.0 * i / rot["dims"])).float().to(device)
        if self.freq.numel() == 0:
            self.freq = torch.zeros(1, device=device)
        self.scratch = None

    def declare(self, pool, prefix: str, max_portion: int, cache_dtype) -> None:
        self.capacity, self.cache_dtype = self.window - 1 + max_portion, cache_dtype
        pool.ring(prefix + "latent", (self.capacity, self.row), cache_dtype)

    def _attn(self, run: LayerRun, proj) -> LatentAttn:
        c = self.c
        return struct(LatentAttn, proj=proj, ld=proj.stride(0), q_off=self.proj.offsets[0], c_off=self.proj.offsets[1], norm=self.norm, freq=self.freq,
                      uk_t=self.uk_t.w, uv=self.uv.w, cache=run.state("latent"), heads=c["heads"], dim=c["dim"], rot_dim=c["rot_dim"],
                      rot_pairs=c["rot"]["dims"] // 2, vdim=c["vdim"], kv_rank=c["kv_rank"], window=self.window, capacity=self.capacity,
                      cache_dtype=DT_F32 if self.cache_dtype == torch.float32 else DT_BF16, scale=c["scale"], eps=self.eps, pos=run.pos)

    def decode(self, run: LayerRun, ws: Workspace, proj, x=None):
        c, sop = self.c, self.sop
        att, out = ws.get("d.att", 1, self.o.k), ws.get("d.y", 1, self.width)
        a = self._attn(run, proj)
        if self.scratch is None:
            self.scratch = sop.latent_scratch(a, ws.device)
        sop.latent_decode(a, att, self.scratch)
        sop.matvec(PRO_NONE, struct(Matvec, w=self.o.w, y=out, x=att, n=self.o.n, k=self.o.k))
        return out

    def prefill(self, run: LayerRun, ws: Workspace, proj, x, m: int):
        c, sop, H, dt = self.c, self.sop, self.c["heads"], self.cache_dtype
        a, cache = self._attn(run, proj), run.state("latent")
        q = ws.get("q", m, H * (self.dp + pad8(c["rot_dim"])), dt)
        sop.latent_append(a, m, q)
        # keys and values of the window's tokens, oldest first; the ring's end cuts them in two at most
        first = max(0, run.start - (self.window - 1))
        n, at = run.start + m - first, first % self.capacity
        kv = ws.get("kv", n, self.ukv.n, dt)
        for lo, hi, slot in ((0, min(n, self.capacity - at), at), (min(n, self.capacity - at), n, 0)):
            if hi > lo:
                sop.matmul(cache[slot:slot + hi - lo], self.ukv, kv[lo:hi], hi - lo)
        att, out = ws.get("att", m, self.o.k, self.act), ws.get("y", m, self.width)
        w = struct(WindowAttn, qkv=proj, k_cache=kv, v_cache=_off(kv, H * self.dp), heads=H, kv_heads=H, dim=c["dim"], vdim=c["vdim"], window=self.window,
                   capacity=self.capacity, cache_dtype=a.cache_dtype, scale=c["scale"], eps=self.eps, pos=run.pos, linear=1, row_stride=self.ukv.n,
                   k_head_stride=self.dp, v_head_stride=self.vp, k_shared=_off(cache, self.rp), shared_dim=c["rot_dim"], shared_stride=self.row,
                   shared_capacity=self.capacity)
        sop.window_prefill(w, m, q, None, 0, att)
        sop.matmul(att, self.o, out, m)
        return out

    def decode_bytes(self) -> int:
        kv = self.window * self.row * (4 if self.act == torch.float32 else 2)
        return self.proj.nbytes + self.uk_t.nbytes + self.uv.nbytes + self.o.nbytes + kv


MIXERS = {"parallel": ParallelWindowMLstm, "channel_delta": ChannelDelta, "mamba2": Mamba2, "latent_attention": LatentAttention}
