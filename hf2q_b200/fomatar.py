"""The Fomatar decoder design: pre-norm layers whose mixers are windowed attention beside an mLSTM memory, or a gated
delta rule with channel decays; a token shift in front of every mixer, a hashed bigram embedding, a looped span of
layers that runs several times with its own state per pass, and soft-capped logits.

The mixers live in ``mixers.py``, their state in ``state.StatePool``, the kernels behind ``seqops``; this file reads the
configuration and the weights and orders the calls.  ``dtype`` bfloat16 serves with bf16 weights and tensor-core operands
(scores, norms, residual stream and recurrences in 32-bit); float32 keeps every activation and product in 32-bit.
"""
from __future__ import annotations

import json
from dataclasses import dataclass
from pathlib import Path

import torch

from . import _lib, ops
from .decoder import SlotDecoder
from .mixers import MIXERS
from .safetensors import SafetensorsFile
from .seqops import (EPI_ADD, EPI_GELU, EPI_NONE, EPI_SOFTCAP, PRO_NONE, PRO_NORM, DenseWeight, Embed, Matvec, PreNorm, SeqOps, pad8, struct)


def _bad(msg: str):
    return ops.Hf2qError(_lib.ERR_INVALID_ARGUMENT, msg)


@dataclass(frozen=True)
class Run:
    """One execution of a layer: its index, and for the first layer of a pass of the looped span the number of the pass."""
    layer: int
    begins_pass: int | None


@dataclass(frozen=True)
class FomatarConfig:
    raw: dict

    @classmethod
    def load(cls, path) -> "FomatarConfig":
        return cls(json.loads(Path(path).read_text()))

    def __post_init__(self):
        for i, e in enumerate(self.layers):
            if e["type"] not in ("parallel", "channel_delta"):
                raise _bad(f"layer {i}: unknown mixer '{e['type']}'")
            if e.get("mlp") and e["mlp"].get("kind", "dense") != "dense":
                raise _bad(f"layer {i}: unknown feed-forward '{e['mlp']['kind']}'")
        lp = self.loop
        if lp and not (0 <= lp["start"] < lp["stop"] <= len(self.layers) and lp["times"] >= 1):
            raise _bad("loop: the span lies outside the layers")

    @property
    def layers(self) -> list:
        return self.raw["layers"]

    @property
    def width(self) -> int:
        return self.raw["width"]

    @property
    def vocab(self) -> int:
        return self.raw["vocab"]

    @property
    def eps(self) -> float:
        return self.raw["norm"]["eps"]

    @property
    def loop(self):
        return self.raw.get("loop")

    @property
    def softcap(self):
        return self.raw.get("logit_softcap")

    @property
    def bigram(self):
        return (self.raw.get("embedding") or {}).get("bigram")

    def runs(self) -> list[Run]:
        n, lp = len(self.layers), self.loop
        if not lp:
            return [Run(i, None) for i in range(n)]
        out = [Run(i, None) for i in range(lp["start"])]
        for t in range(lp["times"]):
            out += [Run(i, t if i == lp["start"] else None) for i in range(lp["start"], lp["stop"])]
        return out + [Run(i, None) for i in range(lp["stop"], n)]


class _Layer:
    def __init__(self, sop, cfg: FomatarConfig, i: int, get, device, act, window_cap):
        entry, p, w = cfg.layers[i], f"l{i}.", cfg.width

        def load(prefix):
            def f(name, rows, cols):
                t = get(prefix + name)
                if t.dim() != 2 or t.shape[1] != cols or (rows is not None and t.shape[0] != rows):
                    raise _bad(f"{prefix + name}: shape {tuple(t.shape)}, expected [{'*' if rows is None else rows}, {cols}]")
                return t
            return f

        def load_f32(prefix):
            def f(name, *shape):
                t = get(prefix + name)
                if tuple(t.shape) != shape:
                    raise _bad(f"{prefix + name}: shape {tuple(t.shape)}, expected {list(shape)}")
                return t.float().contiguous()
            return f

        vec = load_f32(p)
        self.norm1, self.shift = vec("norm1", w).to(device), vec("shift", w).to(device)
        self.mixer = MIXERS[entry["type"]](sop, entry["mixer"], cfg.eps, w, load(p + "mix."), load_f32(p + "mix."), device, act, window_cap)
        self.norm2 = self.up = self.down = None
        if entry.get("mlp"):
            ff = entry["mlp"]["ff"]
            self.norm2 = vec("norm2", w).to(device)
            # up's output rows are padded to the pitch down reads: the extra rows are zero, and so is gelu of them
            up = load(p)("mlp.up", ff, w)
            self.up = DenseWeight(torch.cat([up, up.new_zeros(pad8(ff) - ff, w)]), device)
            self.down = DenseWeight(load(p)("mlp.down", w, ff), device)


class FomatarDecoder(SlotDecoder):
    """n_slots sequences may be open; steps run one sequence at a time."""

    def __init__(self, ctx: ops.GpuContext, cfg: FomatarConfig, get, dtype=torch.bfloat16, max_seq: int = 32768, n_slots: int = 1,
                 prefill_chunk: int = 2048):
        """``get(name)`` returns a weight as a CPU tensor.  ``max_seq``: most tokens of one sequence."""
        if dtype not in (torch.bfloat16, torch.float32):
            raise _bad(f"dtype {dtype} (want bfloat16 or float32)")
        super().__init__(ctx, cfg, dtype, max_seq, n_slots, prefill_chunk)
        self.sop = SeqOps(ctx)
        w, dev = cfg.width, self.dev
        bf = lambda name: get(name).to(torch.bfloat16).contiguous().to(dev)
        self.embed_w = bf("embed")
        if tuple(self.embed_w.shape) != (cfg.vocab, w):
            raise _bad(f"embed: shape {tuple(self.embed_w.shape)}, expected {[cfg.vocab, w]}")
        self.bigram_w = None
        if cfg.bigram:
            self.bigram_w = bf("bigram")
            if tuple(self.bigram_w.shape) != (cfg.bigram["buckets"] + 1, w):
                raise _bad(f"bigram: shape {tuple(self.bigram_w.shape)}, expected {[cfg.bigram['buckets'] + 1, w]}")
        self.layers = [_Layer(self.sop, cfg, i, get, dev, dtype, max_seq) for i in range(len(cfg.layers))]
        self.runs = cfg.runs()
        self.steps = None
        if cfg.loop:
            self.steps = get("loop.step").float().contiguous().to(dev)
            if tuple(self.steps.shape) != (cfg.loop["times"], w):
                raise _bad(f"loop.step: shape {tuple(self.steps.shape)}, expected {[cfg.loop['times'], w]}")
        self.final_norm = get("final.norm").float().contiguous().to(dev)
        self.head = DenseWeight(get("head"), dev)
        if (self.head.n, self.head.k_raw) != (cfg.vocab, w):
            raise _bad(f"head: shape {[self.head.n, self.head.k_raw]}, expected {[cfg.vocab, w]}")

        for r, run in enumerate(self.runs):
            self.pool.recurrent(f"r{r}.shift", 2, w)
            self.layers[run.layer].mixer.declare(self.pool, f"r{r}.", self.chunk, dtype)
        self.pool.allocate()

    @classmethod
    def from_directory(cls, ctx, path, **kw) -> "FomatarDecoder":
        path = Path(path)
        st = SafetensorsFile(path / "model.safetensors")
        try:
            return cls(ctx, FomatarConfig.load(path / "config.json"), st.load_tensor, **kw)
        finally:
            st.close()

    # ---- pieces shared by the two ways to run -----------------------------------------------------
    def _embed(self, ids, m, x):
        bg = self.cfg.bigram
        e = struct(Embed, embed=self.embed_w, bigram=self.bigram_w, vocab=self.cfg.vocab, width=self.cfg.width, ld=self.cfg.width,
                   buckets=bg["buckets"] if bg else None, mul_prev=bg["mul_prev"] if bg else None, mul_cur=bg["mul_cur"] if bg else None, pos=self.pos,
                   prev=self.prev)
        self.sop.embed(e, ids, m, x)

    def _pre(self, x, pending, norm, x_out=None, run=None, layer=None, x0=None) -> PreNorm:
        """The row prologue: a pending pair of mixer outputs, the additions at the start of a pass, norm, token shift."""
        kw = dict(x=x, norm=norm, eps=self.cfg.eps, width=self.cfg.width)
        if pending is not None:
            a, b, mixer = pending
            kw.update(a=a, b=b, a_norm=mixer.a_norm, b_norm=mixer.b_norm)
        if run is not None:
            t = self.runs[run].begins_pass
            if t is not None:
                kw.update(step=self.steps[t], add0=x0 if t > 0 else None)
            kw.update(shift=layer.shift, shift_state=self._run(run).state("shift"), pos=self.pos)
        if pending is not None or kw.get("step") is not None:
            kw.update(x_out=x_out)
        return struct(PreNorm, **kw)

    # ---- one decode step --------------------------------------------------------------------------
    def decode_step(self) -> None:
        c, sop, ws = self.cfg, self.sop, self.ws
        w = c.width
        x0 = ws.get("d.x0", 1, w)
        bufs, cur = [ws.get("d.x1", 1, w), ws.get("d.x2", 1, w)], 0
        self._embed(self.tok, 1, x0)
        x, pending = x0, None

        def product(pre, weight, y, epilogue=EPI_NONE, cap=0.0):
            nonlocal x, cur
            sop.matvec(PRO_NORM, struct(Matvec, w=weight.w, y=y, pre=pre, n=weight.n, k=weight.k, epilogue=epilogue, cap=cap))
            if pre.x_out:
                x, cur = bufs[cur], cur ^ 1

        for r, run in enumerate(self.runs):
            layer = self.layers[run.layer]
            if layer.mixer.adds_residual and x is x0 and run.begins_pass is None:
                # the residual is updated in place from here on; the embedding output must survive for later passes
                bufs[cur].copy_(x0)
                x, cur = bufs[cur], cur ^ 1
            proj = ws.get("d.proj", 1, layer.mixer.proj.n)
            product(self._pre(x, pending, layer.norm1, bufs[cur], r, layer, x0), layer.mixer.proj, proj)
            pending = None
            res = layer.mixer.decode(self._run(r), ws, proj, x)
            if layer.mixer.combines:
                pending = (*res, layer.mixer)
            if layer.up is not None:
                act = ws.get("d.act", 1, layer.up.n)
                if pending is None and x is x0:
                    bufs[cur].copy_(x0)
                    x, cur = bufs[cur], cur ^ 1
                product(self._pre(x, pending, layer.norm2, bufs[cur]), layer.up, act, EPI_GELU)
                pending = None
                sop.matvec(PRO_NONE, struct(Matvec, w=layer.down.w, y=x, residual=x, x=act, n=layer.down.n, k=layer.down.k, epilogue=EPI_ADD))
        product(self._pre(x, pending, self.final_norm, bufs[cur]), self.head, self.logits, EPI_SOFTCAP if c.softcap else EPI_NONE, c.softcap or 0.0)
        sop.argmax(self.logits, self.tok, self.pos)

    # ---- a portion of a prompt ----------------------------------------------------------------------
    def _portion(self, ids, m: int):
        """Runs m tokens from position *pos; returns the residual rows [m, width]."""
        c, sop, ws = self.cfg, self.sop, self.ws
        w = c.width
        x0 = ws.get("x0", m, w)
        bufs, cur = [ws.get("x1", m, w), ws.get("x2", m, w)], 0
        xn, h_last = ws.get("xn", m, pad8(w), self.act), ws.get("h_last", 1, w)
        self._embed(ids, m, x0)
        bufs[cur].copy_(x0)
        x, cur, pending = bufs[cur], 1, None

        def pre(p, last=None):
            nonlocal x, cur, pending
            sop.pre_norm(p, m, xn, last)
            if p.x_out:
                x, cur = bufs[cur], cur ^ 1
            pending = None

        for r, run in enumerate(self.runs):
            layer, mixer = self.layers[run.layer], self.layers[run.layer].mixer
            lr = self._run(r)
            pre(self._pre(x, pending, layer.norm1, bufs[cur], r, layer, x0), h_last)
            proj = ws.get("proj", m, mixer.proj.n)
            sop.matmul(xn, mixer.proj, proj, m)
            res = mixer.prefill(lr, ws, proj, x, m)
            if m > 1:
                sop.state_tail(self.pos, m, h_last, lr.state("shift"), w, mixer.delta(lr, proj))
            if mixer.combines:
                pending = (*res, mixer)
            if layer.up is not None:
                pre(self._pre(x, pending, layer.norm2, bufs[cur]))
                act = ws.get("act", m, layer.up.n, self.act)
                sop.matmul(xn, layer.up, act, m, epilogue=EPI_GELU)
                sop.matmul(act, layer.down, x, m, epilogue=EPI_ADD, residual=x)
            if self.on_layer is not None:
                if pending is not None:
                    pre(self._pre(x, pending, self.final_norm, bufs[cur]))
                self.on_layer(r, x)
        if pending is not None:
            pre(self._pre(x, pending, self.final_norm, bufs[cur]))
        return x

    def _head_rows(self, x, rows) -> torch.Tensor:
        """Final norm and output head of the given residual rows."""
        c, n = self.cfg, len(rows)
        xs = x if n == x.shape[0] else x.index_select(0, torch.tensor(rows, device=self.dev))
        xn = self.ws.get("head.xn", n, pad8(c.width), self.act)
        self.sop.pre_norm(self._pre(xs, None, self.final_norm), n, xn)
        out = torch.empty((n, c.vocab), dtype=torch.float32, device=self.dev)
        self.sop.matmul(xn, self.head, out, n, epilogue=EPI_SOFTCAP if c.softcap else EPI_NONE, cap=c.softcap or 0.0)
        return out

    # ---- sizes --------------------------------------------------------------------------------------
    def decode_bytes_per_token(self) -> int:
        """Bytes of weights and state one decode step moves (full window)."""
        total = self.head.nbytes
        for run in self.runs:
            layer = self.layers[run.layer]
            total += layer.mixer.decode_bytes() + (layer.up.nbytes + layer.down.nbytes if layer.up is not None else 0)
        return total
