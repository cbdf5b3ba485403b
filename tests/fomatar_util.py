"""Small Fomatar configurations and random weights for the tests."""
import numpy as np
import torch

from oracle import fomatar_forward as F


def parallel(width, lh, lg, ld, lv, window, scale, rh, rd, rv, cap, ff=None):
    return {"type": "parallel", "mlp": {"kind": "dense", "ff": ff} if ff else None,
            "mixer": {"left": {"heads": lh, "kv_heads": lg, "dim": ld, "vdim": lv, "mask": {"size": window}, "scale": scale},
                      "right": {"heads": rh, "dim": rd, "vdim": rv, "gate_cap": cap}}}


def delta(h, g, d, dv, conv, ff=None):
    return {"type": "channel_delta", "mlp": {"kind": "dense", "ff": ff} if ff else None,
            "mixer": {"heads": h, "kv_heads": g, "dim": d, "vdim": dv, "conv": conv}}


# grouped heads, sizes that are no multiple of 16, a looped span with a layer before and behind it
CFG_A = {"architecture": "Fomatar", "width": 72, "vocab": 301, "norm": {"eps": 1e-6}, "logit_softcap": 7.0,
         "embedding": {"bigram": {"buckets": 97, "mul_prev": 31, "mul_cur": 5}},
         "layers": [delta(6, 3, 24, 40, 4, ff=52), parallel(72, 6, 2, 40, 24, 33, 0.21, 3, 20, 36, 5.0, ff=100), delta(2, 2, 32, 16, 2),
                    parallel(72, 4, 4, 16, 32, 7, 0.5, 2, 48, 17, 9.0)],
         "loop": {"start": 1, "stop": 3, "times": 3}}
# odd sizes, nothing optional: no bigram table, no loop, no cap; one tap
CFG_B = {"architecture": "Fomatar", "width": 52, "vocab": 75, "norm": {"eps": 1e-5}, "layers": [
    parallel(52, 3, 1, 17, 9, 5, 0.3, 1, 11, 21, 3.0), delta(3, 1, 13, 7, 1), parallel(52, 2, 2, 8, 8, 1, 1.0, 2, 8, 8, 4.0, ff=30)]}
# head sizes of a real layer; ten query heads on a key head
CFG_C = {"architecture": "Fomatar", "width": 256, "vocab": 500, "norm": {"eps": 1e-5}, "logit_softcap": 20.0,
         "embedding": {"bigram": {"buckets": 211, "mul_prev": 1000003, "mul_cur": 7919}},
         "layers": [parallel(256, 10, 1, 128, 128, 150, 0.09, 2, 128, 128, 12.0, ff=384), delta(4, 2, 128, 128, 4),
                    parallel(256, 2, 1, 160, 144, 64, 0.08, 1, 256, 72, 15.0), delta(2, 1, 256, 40, 3)],
         "loop": {"start": 0, "stop": 4, "times": 2}}
CONFIGS = {"a": CFG_A, "b": CFG_B, "c": CFG_C}


def shapes(cfg, rank=12):
    w, out = cfg["width"], {"embed": (cfg["vocab"], cfg["width"])}
    if cfg.get("embedding"):
        out["bigram"] = (cfg["embedding"]["bigram"]["buckets"] + 1, w)
    if cfg.get("loop"):
        out["loop.step"] = (cfg["loop"]["times"], w)
    for i, e in enumerate(cfg["layers"]):
        p, m = f"l{i}.mix.", e["mixer"]
        out[f"l{i}.norm1"] = out[f"l{i}.shift"] = (w,)
        if e["type"] == "parallel":
            L, R = m["left"], m["right"]
            out |= {p + "left.q": (L["heads"] * L["dim"], w), p + "left.k": (L["kv_heads"] * L["dim"], w), p + "left.v": (L["kv_heads"] * L["vdim"], w),
                    p + "left.q.norm": (L["dim"],), p + "left.k.norm": (L["dim"],), p + "left.r1": (L["heads"],), p + "left.r2": (L["heads"],),
                    p + "left.g": (L["heads"] * L["vdim"], w), p + "left.o": (w, L["heads"] * L["vdim"]), p + "left.out": (w,), p + "right.out": (w,),
                    p + "right.q": (R["heads"] * R["dim"], w), p + "right.k": (R["heads"] * R["dim"], w), p + "right.v": (R["heads"] * R["vdim"], w),
                    p + "right.g": (R["heads"] * R["vdim"], w), p + "right.o": (w, R["heads"] * R["vdim"]), p + "right.norm": (R["heads"] * R["vdim"],),
                    p + "right.i": (R["heads"], w), p + "right.f": (R["heads"], w), p + "right.i.b": (R["heads"],), p + "right.f.b": (R["heads"],)}
        else:
            H, G, d, dv, K = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"]
            out |= {p + "q": (G * d, w), p + "k": (G * d, w), p + "v": (H * dv, w), p + "q.conv": (G * d, K), p + "k.conv": (G * d, K),
                    p + "v.conv": (H * dv, K), p + "b": (H, w), p + "A_log": (H,), p + "dt_bias": (H * d,), p + "a1": (rank, w), p + "a2": (H * d, rank),
                    p + "g1": (rank + 6, w), p + "g2": (H * dv, rank + 6), p + "norm": (dv,), p + "o": (w, H * dv)}
        if e["mlp"]:
            out |= {f"l{i}.norm2": (w,), f"l{i}.mlp.up": (e["mlp"]["ff"], w), f"l{i}.mlp.down": (w, e["mlp"]["ff"])}
    return out | {"final.norm": (w,), "head": (cfg["vocab"], w)}


def weights(cfg, seed=0):
    """{name: bf16 tensor}; sizes such that gates, decays and distance terms all matter."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, s in shapes(cfg).items():
        r = torch.randn(s, generator=g)
        leaf = name.rsplit(".", 1)[-1]
        if leaf in ("norm1", "norm2", "norm", "out"):
            t = 1.0 + 0.2 * r
        elif leaf == "shift":
            t = torch.rand(s, generator=g)
        elif leaf == "r1":
            t = 0.5 + torch.rand(s, generator=g)
        elif leaf == "r2":
            t = 0.05 + 0.5 * torch.rand(s, generator=g)
        elif leaf == "b" and len(s) == 1:
            t = r + (2.0 if ".f.b" in name else -1.0)
        elif leaf == "A_log":
            t = r - 1.0
        elif leaf == "dt_bias":
            t = r - 2.0
        elif leaf == "conv":
            t = 0.6 * r
        elif leaf in ("embed", "bigram", "step"):
            t = r
        else:
            t = r * 1.5 / s[-1] ** 0.5
        out[name] = t.to(torch.bfloat16)
    return out


def as_f64(w):
    return {k: v.double().numpy() for k, v in w.items()}


def tokens(cfg, n, seed=1):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], n).tolist()


def oracle_logits(cfg, w, ids):
    return F.forward(cfg, as_f64(w), ids)


def errors(got, want):
    """Root mean square difference over the vocabulary at every position, in units of the logits' own spread."""
    got = got.detach().cpu().double().numpy() if isinstance(got, torch.Tensor) else got
    return np.sqrt(((got - want) ** 2).mean(-1)) / want.std()


def error(got, want):
    return float(errors(got, want).max())


def close(got, want, dtype):
    """f32: every position to rounding.  bf16: product operands carry 8 bits, and an mLSTM quotient whose denominator is
    near its floor magnifies that at single positions, so those have room while nineteen of twenty have little."""
    e = errors(got, want)
    if dtype == torch.float32:
        return e.max() < 1e-4
    return np.quantile(e, 0.95) < 6e-2 and e.max() < 0.3
