"""The Runopel decoder design: a residual in several streams (hyper-connections), mixers that are a Mamba-2 state-space
layer or latent attention over a sliding window, and feed-forwards that are a clamped gated layer or routed experts; the
output head is the embedding table.

The mixers live in ``mixers.py``, the feed-forwards in ``feedforward.py``, their state in ``state.StatePool``, the kernels
behind ``seqops``; this file reads the configuration and the weights and orders the calls.  Every sublayer starts with one
row prologue: the pending output of the sublayer before it enters the streams, the streams are read into one row, the row is
normed.  ``dtype`` bfloat16 serves with bf16 weights and tensor-core operands (scores, norms, router, streams and
recurrences in 32-bit); float32 keeps every activation and product in 32-bit.
"""
from __future__ import annotations

import json
from dataclasses import dataclass
from pathlib import Path

import torch

from . import _lib, ops
from .decoder import SlotDecoder
from .feedforward import FEED_FORWARDS
from .mixers import MIXERS
from .safetensors import SafetensorsFile
from .seqops import EPI_SCALE, PRO_HYPER, DenseWeight, Embed, Hyper, Matvec, SeqOps, pad8, struct


def _bad(msg: str):
    return ops.Hf2qError(_lib.ERR_INVALID_ARGUMENT, msg)


@dataclass(frozen=True)
class RunopelConfig:
    raw: dict

    @classmethod
    def load(cls, path) -> "RunopelConfig":
        return cls(json.loads(Path(path).read_text()))

    def __post_init__(self):
        for i, e in enumerate(self.layers):
            if e["type"] not in ("mamba2", "latent_attention"):
                raise _bad(f"layer {i}: unknown mixer '{e['type']}'")
            if e.get("mlp") and e["mlp"].get("kind") not in FEED_FORWARDS:
                raise _bad(f"layer {i}: unknown feed-forward '{e['mlp'].get('kind')}'")
        if self.streams < 1:
            raise _bad("streams: at least one")

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
    def streams(self) -> int:
        return self.raw["streams"]

    @property
    def residual_mult(self) -> float:
        return self.raw["residual_mult"]

    @property
    def logit_scale(self) -> float:
        return self.raw["logit_scale"]


class _Streams:
    """How a sublayer reads the streams and how its output enters them."""

    def __init__(self, load_f32, name: str, n: int, mult: float, device):
        self.c_in, self.mix = load_f32(name + ".in", n).to(device), load_f32(name + ".mix", n, n).to(device)
        self.out = (mult * load_f32(name + ".out", n)).to(device)


class _Layer:
    def __init__(self, sop, cfg: RunopelConfig, i: int, get, device, act, window_cap):
        entry, p, w = cfg.layers[i], f"l{i}.", cfg.width

        def shaped(name, shape):
            t = get(name)
            if tuple(t.shape) != shape:
                raise _bad(f"{name}: shape {tuple(t.shape)}, expected {list(shape)}")
            return t

        load = lambda prefix: lambda name, rows, cols: shaped(prefix + name, (rows, cols))
        load_f32 = lambda prefix: lambda name, *shape: shaped(prefix + name, shape).float().contiguous()
        vec = load_f32(p)
        try:
            self.norm1, self.hc1 = vec("norm1", w).to(device), _Streams(vec, "hc1", cfg.streams, cfg.residual_mult, device)
            self.mixer = MIXERS[entry["type"]](sop, entry["mixer"], cfg.eps, w, load(p + "mix."), load_f32(p + "mix."), device, act, window_cap)
            self.ff = None
            if entry.get("mlp"):
                self.norm2, self.hc2 = vec("norm2", w).to(device), _Streams(vec, "hc2", cfg.streams, cfg.residual_mult, device)
                self.ff = FEED_FORWARDS[entry["mlp"]["kind"]](sop, entry["mlp"], w, load(p + "mlp."), load_f32(p + "mlp."), device, act)
        except ValueError as e:
            raise _bad(f"layer {i}: {e}") from e


@dataclass
class _Rows:
    """The streams of some tokens: x [m, x_streams * width] and the sublayer output that has yet to enter them."""
    x: torch.Tensor
    x_streams: int
    pending: tuple | None = None        # (y [m * parts, width], parts, _Streams of its sublayer)


class RunopelDecoder(SlotDecoder):
    """n_slots sequences may be open; steps run one sequence at a time."""

    def __init__(self, ctx: ops.GpuContext, cfg: RunopelConfig, get, dtype=torch.bfloat16, max_seq: int = 32768, n_slots: int = 1, prefill_chunk: int = 2048):
        """``get(name)`` returns a weight as a CPU tensor.  ``max_seq``: most tokens of one sequence."""
        super().__init__(ctx, cfg, dtype, max_seq, n_slots, prefill_chunk)
        self.sop = SeqOps(ctx)
        self.head = DenseWeight(get("embed"), self.dev)
        if (self.head.n, self.head.k_raw) != (cfg.vocab, cfg.width):
            raise _bad(f"embed: shape {[self.head.n, self.head.k_raw]}, expected {[cfg.vocab, cfg.width]}")
        self.layers = [_Layer(self.sop, cfg, i, get, self.dev, dtype, max_seq) for i in range(len(cfg.layers))]
        self.final_norm = get("final.norm").float().contiguous().to(self.dev)
        if tuple(self.final_norm.shape) != (cfg.width,):
            raise _bad(f"final.norm: shape {tuple(self.final_norm.shape)}, expected {[cfg.width]}")
        for r, layer in enumerate(self.layers):
            layer.mixer.declare(self.pool, f"r{r}.", self.chunk, dtype)
        self.pool.allocate()

    @classmethod
    def from_directory(cls, ctx, path, **kw) -> "RunopelDecoder":
        path = Path(path)
        st = SafetensorsFile(path / "model.safetensors")
        try:
            return cls(ctx, RunopelConfig.load(path / "config.json"), st.load_tensor, **kw)
        finally:
            st.close()

    # ---- pieces shared by the two ways to run -----------------------------------------------------
    def _embed(self, ids, m, x) -> _Rows:
        """Until the first sublayer's output arrives all streams equal the embedding rows."""
        c = self.cfg
        self.sop.embed(struct(Embed, embed=self.head.w, vocab=c.vocab, width=c.width, ld=self.head.k, pos=self.pos, prev=self.prev), ids, m, x)
        return _Rows(x, 1)

    def _prologue(self, rows: _Rows, c_in, norm, x_out=None) -> Hyper:
        """c_in None: the sum of the streams."""
        c, kw = self.cfg, {}
        if rows.pending is not None:
            y, parts, hc = rows.pending
            kw = dict(y=y, y_parts=parts, mix=hc.mix, out=hc.out, x_out=x_out)
        return struct(Hyper, x=rows.x, x_streams=rows.x_streams, streams=c.streams, width=c.width, c_in=c_in, norm=norm, eps=c.eps, **kw)

    # ---- one decode step --------------------------------------------------------------------------
    def decode_step(self) -> None:
        c, sop, ws = self.cfg, self.sop, self.ws
        rows = self._embed(self.tok, 1, ws.get("d.x0", 1, c.width))
        # every CTA of a product reads the old streams while some store the new ones
        bufs = [ws.get("d.s0", 1, c.streams * c.width), ws.get("d.s1", 1, c.streams * c.width)]

        def sublayer(hc, norm, run):
            nonlocal rows
            x_out = bufs[0]
            pre = self._prologue(rows, hc.c_in, norm, x_out)
            entered = rows.pending is not None
            y, parts = run(pre)
            rows = _Rows(x_out, c.streams, (y, parts, hc)) if entered else _Rows(rows.x, rows.x_streams, (y, parts, hc))
            bufs.reverse()

        def mixer(pre):
            proj = ws.get("d.proj", 1, pad8(layer.mixer.proj.n))
            sop.matvec(PRO_HYPER, struct(Matvec, w=layer.mixer.proj.w, y=proj, hyper=pre, n=layer.mixer.proj.n, k=layer.mixer.proj.k))
            return layer.mixer.decode(self._run(r), ws, proj), 1

        for r, layer in enumerate(self.layers):
            sublayer(layer.hc1, layer.norm1, mixer)
            if layer.ff is not None:
                sublayer(layer.hc2, layer.norm2, lambda pre: layer.ff.decode(ws, pre))
        sop.matvec(PRO_HYPER, struct(Matvec, w=self.head.w, y=self.logits, hyper=self._prologue(rows, None, self.final_norm), n=self.head.n, k=self.head.k,
                                     epilogue=EPI_SCALE, cap=c.logit_scale))
        sop.argmax(self.logits, self.tok, self.pos)

    # ---- a portion of a prompt ----------------------------------------------------------------------
    def _portion(self, ids, m: int) -> _Rows:
        """Runs m tokens from position *pos."""
        c, sop, ws = self.cfg, self.sop, self.ws
        rows = self._embed(ids, m, ws.get("x0", m, c.width))
        x, h = ws.get("x", m, c.streams * c.width), ws.get("xn", m, pad8(c.width), self.act)

        def sublayer(hc, norm, run):
            nonlocal rows
            sop.hyper_norm(self._prologue(rows, hc.c_in, norm, x), m, h)
            if rows.pending is not None:
                rows = _Rows(x, c.streams)
            rows.pending = (*run(), hc)

        def mixer():
            proj = ws.get("proj", m, pad8(layer.mixer.proj.n))
            sop.matmul(h, layer.mixer.proj, proj, m)
            return layer.mixer.prefill(self._run(r), ws, proj, None, m), 1

        for r, layer in enumerate(self.layers):
            sublayer(layer.hc1, layer.norm1, mixer)
            if layer.ff is not None:
                sublayer(layer.hc2, layer.norm2, lambda: layer.ff.prefill(ws, h, m))
            if self.on_layer is not None:
                total = torch.empty((m, c.width), device=self.dev)
                sop.hyper_norm(self._prologue(rows, None, None), m, total)
                self.on_layer(r, total)
        return rows

    def _head_rows(self, portion: _Rows, rows) -> torch.Tensor:
        """Final norm and output head of the given tokens."""
        c, n, m = self.cfg, len(rows), portion.x.shape[0]
        if n != m or rows != list(range(m)):
            at = torch.tensor(rows, device=self.dev)
            pending = portion.pending
            if pending is not None:
                y, parts, hc = pending
                pending = (y.reshape(m, -1).index_select(0, at), parts, hc)
            portion = _Rows(portion.x.index_select(0, at), portion.x_streams, pending)
        h = self.ws.get("head.xn", n, pad8(c.width), self.act)
        self.sop.hyper_norm(self._prologue(portion, None, self.final_norm), n, h)
        out = torch.empty((n, c.vocab), dtype=torch.float32, device=self.dev)
        self.sop.matmul(h, self.head, out, n, EPI_SCALE, cap=c.logit_scale)
        return out

    # ---- sizes --------------------------------------------------------------------------------------
    def decode_bytes_per_token(self) -> int:
        """Bytes of weights and state one decode step moves (full window)."""
        return self.head.nbytes + sum(l.mixer.decode_bytes() + (l.ff.decode_bytes() if l.ff is not None else 0) for l in self.layers)
