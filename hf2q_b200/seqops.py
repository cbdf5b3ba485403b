"""ctypes view of the bf16-weight product, recurrent-mixer and windowed-attention entries of the C ABI: the parameter
structs of include/hf2q_cuda.h and one thin function per entry (torch's current stream, no allocation)."""
from __future__ import annotations

import ctypes as C

import torch

from . import ops
from .ops import DT_BF16, DT_F32, _TORCH_DT

EPI_NONE, EPI_GELU, EPI_ADD, EPI_SOFTCAP, EPI_SCALE, EPI_SWIGLU, EPI_CLAMP_GLU = range(7)
PRO_NONE, PRO_NORM, PRO_GATED, PRO_HYPER = range(4)
GATE_SIGMOID_LAST, GATE_SILU_FIRST = range(2)
GROUP_TILE = {torch.float32: 64, torch.bfloat16: 128}        # rows per tile of the grouped products
_vp, _u32, _u64, _f32 = C.c_void_p, C.c_uint32, C.c_uint64, C.c_float


def pad8(n: int) -> int:
    return (n + 7) // 8 * 8


def pad32(n: int) -> int:
    return (n + 31) // 32 * 32


def _fields(ptrs: str, u32s: str = "", f32s: str = ""):
    return [(n, _vp) for n in ptrs.split()] + [(n, _u32) for n in u32s.split()] + [(n, _f32) for n in f32s.split()]


class PreNorm(C.Structure):
    _fields_ = _fields("x a b a_norm b_norm add0 step x_out norm shift shift_state pos") + [("eps", _f32), ("width", _u32)]


class GatedHeads(C.Structure):
    _fields_ = _fields("o gate norm", "ldo ldg heads head_dim norm_all", "eps") + [("kind", _u32)]


class Hyper(C.Structure):
    _fields_ = _fields("x x_out y mix out c_in norm h_out", "x_streams streams y_parts width", "eps")


class Matvec(C.Structure):
    _fields_ = _fields("w y residual x") + [("pre", PreNorm), ("gated", GatedHeads)] + _fields("", "n k epilogue", "cap") + [("hyper", Hyper), ("bias", _vp)]


class RowGroups(C.Structure):
    _fields_ = _fields("header tiles perm row_scale", "groups tile_rows scatter reserved")


class ExpertStep(C.Structure):
    _fields_ = _fields("gate_up down logits h ids act y", "experts top ff width k_in")


class Embed(C.Structure):
    _fields_ = _fields("embed bigram", "vocab width ld buckets") + [("mul_prev", _u64), ("mul_cur", _u64)] + _fields("pos prev")


class WindowAttn(C.Structure):
    _fields_ = _fields("qkv", "ld q_off k_off v_off") + _fields("q_norm k_norm r1 r2 k_cache v_cache",
                                                                "heads kv_heads dim vdim window capacity cache_dtype", "scale eps") + _fields(
        "pos", "linear row_stride k_head_stride v_head_stride") + _fields("k_shared", "shared_dim shared_stride shared_capacity reserved")


class LatentAttn(C.Structure):
    _fields_ = _fields("proj", "ld q_off c_off") + _fields("norm freq uk_t uv cache", "heads dim rot_dim rot_pairs vdim kv_rank window capacity cache_dtype",
                                                           "scale eps") + _fields("pos")


class Ssd(C.Structure):
    _fields_ = _fields("proj", "ld off") + _fields("conv conv_bias dt_bias a_log d conv_state s", "heads groups state vdim taps") + _fields("pos")


class MLstm(C.Structure):
    _fields_ = _fields("proj", "ld q_off k_off v_off i_off f_off") + _fields("i_bias f_bias s n mx", "heads dim vdim", "gate_cap")


class Delta(C.Structure):
    _fields_ = _fields("proj", "ld q_off k_off v_off b_off a1_off g1_off") + _fields(
        "q_conv k_conv v_conv a_log dt_bias a2 g2 conv_state s", "heads kv_heads dim vdim taps a_rank_ld g_rank_ld") + _fields("pos")


def ptr(t):
    return None if t is None else t.data_ptr()


def struct(cls, **kw):
    return cls(**{k: (v.data_ptr() if isinstance(v, torch.Tensor) else v) for k, v in kw.items() if v is not None})


class DenseWeight:
    """bf16 [n][k] on the device, k padded with zero columns to a multiple of 8.  Built from one or several row blocks
    that share k; every block but a lone one starts at a multiple of 8 rows (``offsets``)."""

    def __init__(self, blocks, device):
        if isinstance(blocks, torch.Tensor):
            blocks = [blocks]
        self.k_raw = blocks[0].shape[1]
        self.k = pad8(self.k_raw)
        self.offsets, rows = [], 0
        for b in blocks:
            self.offsets.append(rows)
            rows += pad8(b.shape[0]) if len(blocks) > 1 else b.shape[0]
        self.n = rows
        w = torch.zeros((self.n, self.k), dtype=torch.bfloat16)
        for o, b in zip(self.offsets, blocks):
            w[o:o + b.shape[0], :self.k_raw] = b
        self.w = w.to(device)

    @property
    def nbytes(self) -> int:
        return self.w.numel() * 2


class SeqOps:
    """The entries bound to one context."""

    def __init__(self, ctx: ops.GpuContext):
        self.ctx, self.lib = ctx, ctx._lib

    def _call(self, name, *args):
        self.ctx._check(getattr(self.lib, "hf2q_cuda_" + name)(self.ctx._h, self.ctx._stream(), *args))

    def embed(self, e: Embed, ids, m, x):
        self._call("embed", C.byref(e), ptr(ids), m, ptr(x))

    def matmul(self, x, w: DenseWeight, y, m, epilogue=EPI_NONE, residual=None, cap=0.0, bias=None):
        self._call("dense_matmul", ptr(x), _TORCH_DT[x.dtype], x.stride(0), ptr(w.w), ptr(y), _TORCH_DT[y.dtype], y.stride(0), m, w.n, w.k, epilogue,
                   ptr(residual), cap, ptr(bias))

    def grouped(self, g: RowGroups, x, w: DenseWeight, y, rows, epilogue=EPI_NONE, cap=0.0):
        """``w`` holds the matrices of all groups one below the other."""
        self._call("dense_grouped", C.byref(g), ptr(x), _TORCH_DT[x.dtype], x.stride(0), ptr(w.w), ptr(y), _TORCH_DT[y.dtype], y.stride(0), rows,
                   w.n // g.groups, w.k, epilogue, cap)

    def sigmoid_topk(self, logits, ids, weights, m, experts, top):
        self._call("moe_sigmoid_topk", ptr(logits), logits.stride(0), ptr(ids), ptr(weights), m, experts, top)

    def sort_rows(self, ids, m, top, experts, x, header, tiles, perm, xg):
        self._call("sort_rows", ptr(ids), m, top, experts, GROUP_TILE[x.dtype], ptr(x), _TORCH_DT[x.dtype], x.stride(0), ptr(header), ptr(tiles), ptr(perm), ptr(xg))

    def expert_step(self, e: ExpertStep):
        self._call("expert_glu_step", C.byref(e))
        self._call("expert_down_step", C.byref(e))

    def hyper_norm(self, p: Hyper, m, out):
        self._call("hyper_norm", C.byref(p), m, ptr(out), _TORCH_DT[out.dtype], out.stride(0))

    def matvec(self, prologue, *segs: Matvec):
        self._call("dense_matvec", prologue, (Matvec * len(segs))(*segs), len(segs))

    def pre_norm(self, p: PreNorm, m, out, h_last=None):
        self._call("pre_norm", C.byref(p), m, ptr(out), _TORCH_DT[out.dtype], out.stride(0), ptr(h_last))

    def gated_heads(self, g: GatedHeads, m, out):
        self._call("gated_heads", C.byref(g), m, ptr(out), _TORCH_DT[out.dtype], out.stride(0))

    def window_scratch(self, a: WindowAttn, device) -> torch.Tensor:
        need = C.c_uint64()
        self.ctx._check(self.lib.hf2q_cuda_window_attn_scratch_bytes(self.ctx._h, C.byref(a), C.byref(need)))
        return torch.zeros(need.value, dtype=torch.uint8, device=device)

    def window_decode(self, a: WindowAttn, out, scratch):
        self._call("window_attn_decode", C.byref(a), ptr(out), ptr(scratch), scratch.numel())

    def window_append(self, a: WindowAttn, m, q_out):
        self._call("window_attn_append", C.byref(a), m, ptr(q_out))

    def window_prefill(self, a: WindowAttn, m, q, gate_ptr, ldg, out):
        self._call("window_attn_prefill", C.byref(a), m, ptr(q), gate_ptr, ldg, ptr(out), _TORCH_DT[out.dtype], out.stride(0))

    def latent_scratch(self, a: LatentAttn, device) -> torch.Tensor:
        need = C.c_uint64()
        self.ctx._check(self.lib.hf2q_cuda_latent_scratch_bytes(self.ctx._h, C.byref(a), C.byref(need)))
        return torch.zeros(need.value, dtype=torch.uint8, device=device)

    def latent_decode(self, a: LatentAttn, out, scratch):
        self._call("latent_decode", C.byref(a), ptr(out), ptr(scratch), scratch.numel())

    def latent_append(self, a: LatentAttn, m, q_out):
        self._call("latent_append", C.byref(a), m, ptr(q_out))

    def ssd_step(self, a: Ssd, y):
        self._call("ssd_step", C.byref(a), ptr(y))

    def ssd_prep(self, a: Ssd, m, xbc, dt, la):
        self._call("ssd_prep", C.byref(a), m, ptr(xbc), ptr(dt), ptr(la))

    def ssd_scan(self, a: Ssd, m, xbc, dt, la, y):
        self._call("ssd_scan", C.byref(a), m, ptr(xbc), ptr(dt), ptr(la), ptr(y))

    def mlstm(self, a: MLstm, m, out):
        self._call("mlstm", C.byref(a), m, ptr(out))

    def delta_step(self, a: Delta, out, gate):
        self._call("delta_step", C.byref(a), ptr(out), ptr(gate))

    def delta_prep(self, a: Delta, m, qkv, beta, a1, g1):
        self._call("delta_prep", C.byref(a), m, ptr(qkv), ptr(beta), ptr(a1), ptr(g1), _TORCH_DT[a1.dtype])

    def delta_decay(self, a: Delta, m, g):
        self._call("delta_decay", C.byref(a), m, ptr(g))

    def delta_scan(self, a: Delta, m, qkv, beta, g, out):
        self._call("delta_scan", C.byref(a), m, ptr(qkv), ptr(beta), ptr(g), ptr(out))

    def state_tail(self, pos, m, h_last, shift_state, width, delta: Delta | None = None):
        self._call("state_tail", ptr(pos), m, ptr(h_last), ptr(shift_state), width, C.byref(delta) if delta is not None else None)

    def argmax(self, logits_row, tok, pos=None):
        self._call("argmax", ptr(logits_row), logits_row.numel(), ptr(tok), ptr(pos))
