"""Small Runopel configurations and random weights for the tests."""
import copy

import numpy as np
import torch

from oracle import runopel_forward as F


def mamba(heads, vdim, state, groups, norm_groups, conv, mlp=None):
    return {"type": "mamba2", "mlp": mlp, "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "norm_groups": norm_groups, "conv": conv}}


def latent(heads, dim, rot, vdim, rank, window, scale, base, mlp=None):
    return {"type": "latent_attention", "mlp": mlp,
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank, "mask": {"size": window}, "rot": {"base": base, "dims": rot},
                      "scale": scale}}


def dense(ff, limit):
    return {"kind": "dense", "ff": ff, "limit": limit}


def moe(experts, top, ff):
    return {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}


# three streams; grouped heads, sizes that are no multiple of 16, a layer without feed-forward, several experts per token
CFG_A = {"architecture": "Runopel", "width": 72, "vocab": 301, "streams": 3, "residual_mult": 0.6, "logit_scale": 1.7, "norm": {"eps": 1e-6},
         "layers": [latent(5, 24, 12, 20, 44, 33, 0.2, 1e4, dense(52, 1.5)), mamba(6, 24, 20, 3, 2, 4, moe(5, 2, 28)), mamba(2, 16, 40, 1, 4, 2),
                    latent(3, 16, 8, 40, 24, 7, 0.3, 50.0, moe(3, 3, 20))]}
# odd sizes, a single stream, one tap, a window of one token, one expert per token
CFG_B = {"architecture": "Runopel", "width": 52, "vocab": 75, "streams": 1, "residual_mult": 1.0, "logit_scale": 1.0, "norm": {"eps": 1e-5},
         "layers": [mamba(3, 7, 13, 1, 3, 1, moe(4, 1, 10)), latent(1, 9, 2, 11, 17, 5, 0.4, 100.0, dense(30, 0.7)), latent(2, 8, 6, 8, 8, 1, 1.0, 10.0),
                    mamba(2, 9, 5, 2, 1, 6, dense(9, 3.0))]}
# head sizes of a real layer; more heads than a decode group holds, streams beyond four
CFG_C = {"architecture": "Runopel", "width": 256, "vocab": 500, "streams": 5, "residual_mult": 0.4, "logit_scale": 0.5, "norm": {"eps": 1e-5},
         "layers": [mamba(4, 64, 128, 1, 1, 4, moe(12, 4, 96)), latent(18, 128, 64, 128, 320, 150, 0.07, 1e4, moe(9, 2, 136)), mamba(3, 72, 160, 3, 3, 3, dense(384, 2.5)),
                    latent(20, 48, 16, 72, 512, 64, 0.12, 5e5)]}
CONFIGS = {"a": CFG_A, "b": CFG_B, "c": CFG_C}


def all_experts(cfg):
    """Every token goes through all experts: no choice that rounding could turn."""
    cfg = copy.deepcopy(cfg)
    for e in cfg["layers"]:
        if e["mlp"] and e["mlp"]["kind"] == "moe":
            e["mlp"]["router"]["top"] = e["mlp"]["router"]["experts"]
    return cfg


def shapes(cfg):
    w, s, out = cfg["width"], cfg["streams"], {"embed": (cfg["vocab"], cfg["width"])}
    for i, e in enumerate(cfg["layers"]):
        p, m, H = f"l{i}.mix.", e["mixer"], e["mixer"]["heads"]
        if e["type"] == "mamba2":
            inner, bc = H * m["vdim"], 2 * m["groups"] * m["state"]
            out |= {p + "in": (2 * inner + bc + H, w), p + "conv": (inner + bc, m["conv"]), p + "conv.b": (inner + bc,), p + "dt_bias": (H,), p + "A_log": (H,),
                    p + "D": (H,), p + "norm": (inner,), p + "o": (w, inner)}
        else:
            out |= {p + "q": (H * (m["dim"] + m["rot_dim"]), w), p + "dkv": (m["kv_rank"] + m["rot_dim"], w), p + "dkv.norm": (m["kv_rank"],),
                    p + "uk": (H * m["dim"], m["kv_rank"]), p + "uv": (H * m["vdim"], m["kv_rank"]), p + "o": (w, H * m["vdim"])}
        p, f = f"l{i}.mlp.", e["mlp"]
        if f and f["kind"] == "dense":
            out |= {p + "gate": (f["ff"], w), p + "gate.b": (f["ff"],), p + "up": (f["ff"], w), p + "up.b": (f["ff"],), p + "down": (w, f["ff"]), p + "down.b": (w,)}
        elif f:
            out[p + "router"] = (f["router"]["experts"], w)
            for x in range(f["router"]["experts"]):
                out |= {f"{p}e{x}.gate": (f["expert"]["ff"], w), f"{p}e{x}.up": (f["expert"]["ff"], w), f"{p}e{x}.down": (w, f["expert"]["ff"])}
        for q in (1, 2) if f else (1,):
            out |= {f"l{i}.norm{q}": (w,), f"l{i}.hc{q}.in": (s,), f"l{i}.hc{q}.out": (s,), f"l{i}.hc{q}.mix": (s, s)}
    return out | {"final.norm": (w,)}


def weights(cfg, seed=0):
    """{name: bf16 tensor}; sizes such that decays, gates, clamps and the streams' differences all matter."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, s in shapes(cfg).items():
        r = torch.randn(s, generator=g)
        leaf = name.rsplit(".", 1)[-1]
        if leaf in ("norm", "norm1", "norm2"):
            t = 1.0 + 0.2 * r
        elif leaf == "in" and len(s) == 1:
            t = (1.0 + 0.5 * r) / s[0] ** 0.5
        elif leaf == "out":
            t = 1.0 + 0.4 * r
        elif leaf == "mix":
            t = 0.8 * torch.eye(s[0]) + 0.2 * r
        elif leaf == "A_log":
            t = r - 1.0
        elif leaf == "dt_bias":
            t = r - 1.0
        elif leaf == "conv":
            t = 0.8 * r / s[1] ** 0.5
        elif leaf in ("b", "D"):
            t = 0.5 * r
        elif leaf == "embed":
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
    """Root mean square difference over the last axis at every position, in units of the wanted values' own spread."""
    got = got.detach().cpu().double().numpy() if isinstance(got, torch.Tensor) else got
    return np.sqrt(((got - want) ** 2).mean(-1)) / want.std()


def error(got, want):
    return float(errors(got, want).max())


def close(got, want, dtype):
    """f32: every position to rounding.  bf16: product operands carry 8 bits."""
    e = errors(got, want)
    if dtype == torch.float32:
        return e.max() < 1e-4
    return np.quantile(e, 0.95) < 6e-2 and e.max() < 0.2
