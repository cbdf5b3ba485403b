"""Streams, gated products, routed experts, state-space and latent-attention kernels, each against plain f64 arithmetic."""
import numpy as np
import pytest
import torch

from hf2q_b200 import seqops as S
from hf2q_b200.feedforward import ClampedGlu, RoutedExperts
from hf2q_b200.mixers import LatentAttention, Mamba2
from hf2q_b200.ops import Hf2qError
from hf2q_b200.state import LayerRun, StatePool, Workspace
from oracle import runopel_forward as F
from tests import runopel_util as U

pytestmark = pytest.mark.gpu
DEV = "cuda"


@pytest.fixture(scope="module")
def sop(gpu_ctx):
    return S.SeqOps(gpu_ctx)


def f32(a):
    return torch.tensor(np.asarray(a), dtype=torch.float32, device=DEV)


def rel(got, want):
    got = got.detach().cpu().double().numpy().reshape(want.shape)
    return float(np.linalg.norm(got - want) / max(np.linalg.norm(want), 1e-30))


# ---- streams ------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("streams,parts,width", [(1, 1, 52), (2, 1, 53), (3, 2, 344), (4, 1, 4096), (5, 3, 72), (8, 1, 30), (16, 2, 260)])
@pytest.mark.parametrize("m", [1, 3])
def test_streams_and_norm_alone_and_in_the_matvec(sop, streams, parts, width, m):
    rng = np.random.default_rng(streams * 10 + m)
    eps, ldo = 1e-3, S.pad8(width)
    y, norm = rng.standard_normal((m, parts, width)), rng.standard_normal(width)
    mix, out, c_in = rng.standard_normal((streams, streams)), rng.standard_normal(streams), rng.standard_normal(streams)
    dy, dn, dm, do, di = f32(y), f32(norm), f32(mix), f32(out), f32(c_in)
    for x_streams in {1, streams}:
        x = rng.standard_normal((m, x_streams, width))
        X = np.repeat(x, streams, 1) if x_streams == 1 else x
        for pending, summed in ((True, False), (True, True), (False, False)):
            Xn = F.write_streams(X.transpose(1, 0, 2), y.sum(1), mix, out, 1.0) if pending else X.transpose(1, 0, 2)
            u = F.read_streams(Xn, np.ones(streams) if summed else c_in)
            want = F.rms(u, eps) * norm
            dx, xo, h = f32(x), torch.zeros(m, streams, width, device=DEV), torch.full((m, ldo), 5.0, device=DEV)
            p = S.struct(S.Hyper, x=dx, x_streams=x_streams, streams=streams, width=width, norm=dn, eps=eps, c_in=None if summed else di,
                         **(dict(y=dy, y_parts=parts, mix=dm, out=do, x_out=xo) if pending else {}))
            sop.hyper_norm(p, m, h)
            assert rel(h[:, :width], want) < 1e-5 and not h[:, width:].any()
            if pending:
                assert rel(xo, Xn.transpose(1, 0, 2)) < 1e-6
            hb = torch.zeros((m, ldo), dtype=torch.bfloat16, device=DEV)
            sop.hyper_norm(p, m, hb)
            assert rel(hb[:, :width], want) < 4e-3
            if m == 1:
                n = 37
                w = S.DenseWeight(torch.randn(n, width).to(torch.bfloat16), DEV)
                xo2, hh, yy = torch.zeros_like(xo), torch.zeros(1, ldo, device=DEV), torch.zeros(1, n, device=DEV)
                p.h_out, p.x_out = hh.data_ptr(), xo2.data_ptr() if pending else None
                sop.matvec(S.PRO_HYPER, S.struct(S.Matvec, w=w.w, y=yy, hyper=p, n=n, k=w.k))
                assert rel(yy, want @ w.w[:, :width].cpu().double().numpy().T) < 2e-5 and rel(hh[:, :width], want) < 1e-5
                if pending:
                    assert rel(xo2, Xn.transpose(1, 0, 2)) < 1e-6
            if pending and x_streams == streams:                            # in place, without a norm
                p.x_out, p.norm, p.h_out = dx.data_ptr(), None, None
                sop.hyper_norm(p, m, h)
                assert rel(dx, Xn.transpose(1, 0, 2)) < 1e-6 and rel(h[:, :width], u) < 1e-5


def test_streams_refuse_bad_arguments(sop):
    x = torch.zeros(1, 17 * 8, device=DEV)
    with pytest.raises(Hf2qError):
        sop.hyper_norm(S.struct(S.Hyper, x=x, x_streams=17, streams=17, width=8), 1, torch.zeros(1, 8, device=DEV))
    with pytest.raises(Hf2qError):
        sop.hyper_norm(S.struct(S.Hyper, x=x, x_streams=2, streams=3, width=8), 1, torch.zeros(1, 8, device=DEV))


# ---- products -----------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("m,n,k", [(1, 10, 8), (2, 300, 72), (8, 130, 1000), (9, 24, 8), (64, 616, 312), (257, 1030, 200), (600, 4096, 512), (1500, 2304, 264)])
@pytest.mark.parametrize("xd", [torch.float32, torch.bfloat16])
def test_paired_epilogues_bias_and_scale(sop, m, n, k, xd):
    g = torch.Generator().manual_seed(m * 7 + n)
    x, b = torch.randn(m, k, generator=g).to(xd), torch.randn(n, generator=g)
    w = S.DenseWeight((torch.randn(n, k, generator=g) / k ** 0.5).to(torch.bfloat16), DEV)
    z = x.double().numpy() @ w.w.cpu().double().numpy().T
    zb, xg, bg = z + b.double().numpy(), x.to(DEV), b.to(DEV)
    gate, up = np.minimum(zb[:, ::2], 0.8), np.clip(zb[:, 1::2], -0.8, 0.8)
    cases = [(S.EPI_NONE, bg, 0.0, zb), (S.EPI_SCALE, None, -1.3, -1.3 * z), (S.EPI_SWIGLU, None, 0.0, F.silu(z[:, ::2]) * z[:, 1::2]),
             (S.EPI_CLAMP_GLU, bg, 0.8, gate * F.sigmoid(1.702 * gate) * (up + 1))]
    for epi, bias, cap, want in cases:
        cols = want.shape[1]
        y = torch.full((m, cols), 7.0, device=DEV)
        sop.matmul(xg, w, y, m, epi, cap=cap, bias=bias)
        assert rel(y, want) < 2e-5
        yb = torch.full((m, S.pad8(cols) + 8), 7.0, dtype=torch.bfloat16, device=DEV)
        sop.matmul(xg, w, yb[:, :cols], m, epi, cap=cap, bias=bias)
        assert rel(yb[:, :cols], want) < 4e-3 and bool((yb[:, cols:] == 7).all())
        if m == 1 and xd == torch.float32:
            y.zero_()
            sop.matvec(S.PRO_NONE, S.struct(S.Matvec, w=w.w, y=y, x=xg, n=n, k=k, epilogue=epi, cap=cap, bias=bias))
            assert rel(y, want) < 2e-5
    sop.ctx.check_status()
    with pytest.raises(Hf2qError):
        sop.matmul(xg, w, torch.zeros(m, n, device=DEV), m, S.EPI_CLAMP_GLU)           # no limit


@pytest.mark.parametrize("groups,size", [(1, 21), (2, 72), (4, 8), (16, 5), (20, 3), (3, 256), (1, 4096)])
def test_gate_then_group_norm(sop, groups, size):
    rng = np.random.default_rng(groups)
    m, n, eps = 3, groups * size, 1e-4
    y, z, w = rng.standard_normal((m, n)), rng.standard_normal((m, n + 4)), rng.standard_normal(n)
    want = F.gated_group_norm(y, z[:, :n], w, groups, eps)
    yg, zg, wg = f32(y), f32(z), f32(w)
    g = S.struct(S.GatedHeads, o=yg, gate=zg, norm=wg, ldo=n, ldg=n + 4, heads=groups, head_dim=size, norm_all=1, eps=eps, kind=S.GATE_SILU_FIRST)
    out = torch.full((m, n + 5), 2.0, device=DEV)
    sop.gated_heads(g, m, out)
    assert rel(out[:, :n], want) < 1e-6 and not out[:, n:].any()
    p = S.DenseWeight(torch.randn(50, n).to(torch.bfloat16), DEV)
    o = torch.zeros(1, 50, device=DEV)
    sop.matvec(S.PRO_GATED, S.struct(S.Matvec, w=p.w, y=o, gated=g, n=p.n, k=p.k))
    assert rel(o, want[:1] @ p.w[:, :n].cpu().double().numpy().T) < 1e-5


# ---- feed-forwards ------------------------------------------------------------------------------------------------
def ff_getters(w):
    return lambda n, *s: w[n], lambda n, *s: w[n].float()


@pytest.mark.parametrize("dt", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("width,ff,limit", [(52, 30, 0.5), (256, 384, 3.0), (72, 52, 1.0)])
def test_clamped_feed_forward(sop, dt, width, ff, limit):
    cfg = {"kind": "dense", "ff": ff, "limit": limit}
    g = torch.Generator().manual_seed(ff)
    w = {"gate": (ff, width), "up": (ff, width), "down": (width, ff), "gate.b": (ff,), "up.b": (ff,), "down.b": (width,)}
    w = {n: (torch.randn(s, generator=g) / (s[-1] ** 0.5 if len(s) > 1 else 1)).to(torch.bfloat16) for n, s in w.items()}
    w64 = [w[n].double().numpy() for n in ("gate", "gate.b", "up", "up.b", "down", "down.b")]
    f, ws = ClampedGlu(sop, cfg, width, *ff_getters(w), DEV, dt), Workspace(DEV)
    for m in (2, 40, 130):
        h = torch.zeros(m, S.pad8(width), dtype=dt, device=DEV)
        h[:, :width] = torch.randn(m, width, generator=g).to(DEV)
        y, parts = f.prefill(ws, h, m)
        assert parts == 1 and rel(y, F.clamped_glu(h[:, :width].cpu().double().numpy(), *w64, limit)) < (1e-5 if dt == torch.float32 else 6e-3)
    x = torch.randn(1, width, generator=g).to(DEV)
    y, _ = f.decode(ws, S.struct(S.Hyper, x=x, x_streams=1, streams=1, width=width))
    assert rel(y, F.clamped_glu(x.cpu().double().numpy(), *w64, limit)) < 1e-5


@pytest.mark.parametrize("dt", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("width,ff,experts,top", [(52, 10, 4, 1), (72, 28, 5, 2), (256, 96, 40, 8), (64, 136, 3, 3), (1100, 1200, 2, 1), (48, 16, 300, 33)])
def test_routed_experts(sop, dt, width, ff, experts, top):
    cfg = {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}
    g = torch.Generator().manual_seed(width)
    w = {"router": (experts, width)}
    for e in range(experts):
        w |= {f"e{e}.gate": (ff, width), f"e{e}.up": (ff, width), f"e{e}.down": (width, ff)}
    w = {n: (2.0 * torch.randn(s, generator=g) / s[-1] ** 0.5).to(torch.bfloat16) for n, s in w.items()}
    f, ws = RoutedExperts(sop, cfg, width, *ff_getters(w), DEV, dt), Workspace(DEV)
    router, ex = w["router"].double().numpy(), [tuple(w[f"e{e}.{n}"].double().numpy() for n in ("gate", "up", "down")) for e in range(experts)]
    for m in (2, 3, 60, 400):
        h = torch.zeros(m, S.pad8(width), dtype=dt, device=DEV)
        h[:, :width] = torch.randn(m, width, generator=g).to(DEV)
        if m == 60:
            h[:, :width] = h[0, :width].clone()                             # all tokens to the same experts
        y, parts = f.prefill(ws, h, m)
        assert parts == top
        # (scores that nearly tie may choose the other expert: single tokens have room)
        e = U.errors(y.view(m, top, width).sum(1), F.expert_mixture(h[:, :width].cpu().double().numpy(), router, ex, top))
        assert np.quantile(e, 0.97) < (1e-5 if dt == torch.float32 else 1e-2)
    for k in range(3):
        x = torch.randn(1, width, generator=g).to(DEV)
        y, parts = f.decode(ws, S.struct(S.Hyper, x=x, x_streams=1, streams=1, width=width))
        assert parts == 1 and rel(y, F.expert_mixture(x.cpu().double().numpy(), router, ex, top)) < 1e-5
    sop.ctx.check_status()


def test_choice_of_experts(sop):
    z = np.array([[0.0, 3.0, -2.0, 3.0, 1.0], [30.0, 40.0, -1.0, 50.0, 0.0], [-1.0, -1.0, -1.0, -1.0, -1.0]])
    logits = torch.full((3, 8), 99.0, device=DEV)
    logits[:, :5] = f32(z)
    ids, w = torch.zeros(3, 3, dtype=torch.int32, device=DEV), torch.zeros(3, 3, device=DEV)
    sop.sigmoid_topk(logits[:, :5], ids, w, 3, 5, 3)
    assert ids.tolist() == [[1, 3, 4], [0, 1, 3], [0, 1, 2]]               # equal scores (also saturated ones): the lower index first
    assert rel(w, F.sigmoid(np.take_along_axis(z, ids.cpu().numpy(), 1))) < 1e-6


# ---- state space --------------------------------------------------------------------------------------------------
def mixer_of(sop, cls, c, dt, width=24, portion=1 << 12, edit=None):
    cfg = {"width": width, "vocab": 8, "streams": 1, "layers": [{"type": "mamba2" if cls is Mamba2 else "latent_attention", "mlp": None, "mixer": c}]}
    w = {n[len("l0.mix."):]: t for n, t in U.weights(cfg).items() if n.startswith("l0.mix.")}
    if edit:
        edit(w)
    m = cls(sop, c, 1e-5, width, lambda n, *s: w[n], lambda n, *s: w[n].float(), DEV, dt, 1 << 20)
    pool = StatePool(1, DEV)
    m.declare(pool, "r0.", portion, dt)
    pool.allocate()
    return m, w, pool


def run_mixer(sop, m, pool, h, cuts, dt):
    """The mixer over rows h [T, width] (f32, on the device) in portions; a portion of one token is a decode step."""
    ws, out, at = Workspace(DEV), [], 0
    slot = pool.open()
    pos = pool.pos[slot, :1]
    for c in cuts:
        pos.fill_(at)
        run = LayerRun(pool.views(slot), "r0.", pos, at)
        rows = torch.zeros(c, m.proj.k, dtype=dt, device=DEV)
        rows[:, :h.shape[1]] = h[at:at + c]
        proj = torch.zeros(c, S.pad8(m.proj.n), device=DEV)
        sop.matmul(rows, m.proj, proj, c)
        out.append((m.decode(run, ws, proj) if c == 1 else m.prefill(run, ws, proj, None, c)).clone())
        at += c
    pool.close(slot)
    sop.ctx.check_status()
    return torch.cat(out)


def spread(n, pattern):
    out = []
    while sum(out) < n:
        out.append(min(pattern[len(out) % len(pattern)], n - sum(out)))
    return out


MAMBAS = {"plain": (4, 16, 32, 1, 1, 4), "groups": (6, 24, 20, 3, 2, 3), "odd": (3, 7, 13, 1, 3, 1), "wide": (2, 64, 128, 2, 1, 4), "long": (1, 130, 200, 1, 2, 2),
          "taps": (2, 9, 5, 2, 1, 6)}


@pytest.mark.parametrize("name", list(MAMBAS))
@pytest.mark.parametrize("dt", [torch.float32, torch.bfloat16])
def test_mamba2_whole_in_portions_and_token_by_token(sop, name, dt):
    c = U.mamba(*MAMBAS[name])["mixer"]
    m, w, pool = mixer_of(sop, Mamba2, c, dt)
    T = 150
    h = torch.randn(T, 24, generator=torch.Generator().manual_seed(3)).to(dt).float().to(DEV)
    want = F.mixer_mamba2(c, U.as_f64(w), "", h.cpu().double().numpy(), 1e-5)
    tol = 2e-5 if dt == torch.float32 else 1.5e-2
    for cuts in ([T], [1] * T, spread(T, [2]), spread(T, [3, 64, 2, 1, 7, 65]), [T - 4] + [1] * 4, [63, 64, 23], [64, 86], [65, 2, 83]):
        assert rel(run_mixer(sop, m, pool, h, cuts, dt), want) < tol, cuts[:5]


def test_mamba2_state_reaches_far_and_forgets_as_told(sop):
    """The first token's write alone, read a long way on, with slow decays; and heads whose decay is fast."""
    H, P, N, T = 3, 20, 24, 700
    rng = np.random.default_rng(0)
    a_log = np.array([-6.0, -3.0, 1.0])
    x, B, C = np.zeros((T, H, P)), np.zeros((T, 1, N)), rng.standard_normal((T, 1, N))
    x[0], B[0] = rng.standard_normal((H, P)), rng.standard_normal((1, N))
    step = 0.5 + rng.random((T, H))
    want = F.state_space(x, B, C, step, a_log, np.zeros(H))
    xbc, dd = f32(np.concatenate([x.reshape(T, -1), B.reshape(T, -1), C.reshape(T, -1)], 1)), f32(step)
    la, zero = f32(-np.exp(a_log) * step), torch.zeros(H * P + 2 * N, device=DEV)
    al, s, pos = f32(a_log), torch.zeros(H, P, 32, device=DEV), torch.zeros(1, dtype=torch.int32, device=DEV)
    for cuts in ([T], [1, T - 1], spread(T, [97]), spread(T, [2, 64, 5])):
        y = torch.zeros(T, H * P, device=DEV)
        s.zero_()
        a = S.struct(S.Ssd, proj=xbc, ld=xbc.shape[1], conv=zero, conv_bias=zero, dt_bias=zero, a_log=al, d=zero, conv_state=zero, s=s,
                     heads=H, groups=1, state=N, vdim=P, taps=1, pos=pos)
        at = 0
        for c in cuts:
            sop.ssd_scan(a, c, xbc[at:at + c], dd[at:at + c], la[at:at + c], y[at:at + c])
            at += c
        got = y.cpu().double().numpy().reshape(T, H, P)
        for h in range(H):
            for lo, hi in ((0, 5), (90, 100), (600, 700)):
                ref = want[lo:hi, h]
                assert np.linalg.norm(got[lo:hi, h] - ref) <= 1e-4 * np.linalg.norm(ref) + 1e-7 * np.linalg.norm(want[:3, h]), (cuts[:3], h, lo)


# ---- latent attention ---------------------------------------------------------------------------------------------
LATENTS = {"small": (5, 24, 12, 20, 44, 33, 0.2, 1e4), "odd": (1, 9, 2, 11, 17, 5, 0.4, 100.0), "one": (2, 8, 6, 8, 8, 1, 1.0, 10.0), "many": (18, 16, 8, 16, 40, 70, 0.2, 50.0),
           "real": (4, 128, 64, 128, 512, 100, 0.07, 1e4), "group": (17, 128, 64, 64, 256, 64, 0.07, 5e5), "big": (2, 200, 32, 160, 700, 40, 0.05, 1e4)}


@pytest.mark.parametrize("name", list(LATENTS))
@pytest.mark.parametrize("dt", [torch.float32, torch.bfloat16])
def test_latent_attention_whole_in_portions_and_token_by_token(sop, name, dt):
    c = U.latent(*LATENTS[name])["mixer"]
    m, w, pool = mixer_of(sop, LatentAttention, c, dt, portion=256)
    T = 150
    h = torch.randn(T, 24, generator=torch.Generator().manual_seed(3)).to(dt).float().to(DEV)
    want = F.mixer_latent_attention(c, U.as_f64(w), "", h.cpu().double().numpy(), 1e-5)
    tol = 3e-5 if dt == torch.float32 else 2.5e-2
    for cuts in ([T], [1] * T, spread(T, [2]), spread(T, [3, 64, 2, 1, 7, 65]), [T - 4] + [1] * 4):
        got = run_mixer(sop, m, pool, h, cuts, dt)
        assert rel(got, want) < tol, cuts[:5]
        assert U.errors(got, want).max() < 3 * tol


@pytest.mark.parametrize("dt", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("window", [2, 31, 32, 33, 64, 65, 130])
def test_edge_of_the_window(sop, dt, window):
    """A key that outweighs all others is seen for exactly `window` tokens, in portions and in decode steps, and the ring
    (short portions make it wrap) hands it over."""
    c = U.latent(2, 16, 4, 16, 24, window, 1.0, 100.0)["mixer"]

    def edit(w):                                                            # every query asks for element 1 of the latent
        w["dkv"][:24] = torch.eye(24)
        w["dkv"][24:] *= 0.1
        w["q"] *= 0.1
        for h in range(2):
            w["q"][20 * h] = 0.0
            w["q"][20 * h, 0] = 2.0
            w["uk"][16 * h] = 0.0
            w["uk"][16 * h, 1] = 1.0
    T = 300
    m, w, pool = mixer_of(sop, LatentAttention, c, dt, portion=16, edit=edit)
    h = 0.5 * torch.randn(T, 24, generator=torch.Generator().manual_seed(5))
    h[:, 0], h[:, 1] = 1.0, 0.0
    h[[0, 3, 120], 1] = 8.0
    h = h.to(dt).float()
    want = F.mixer_latent_attention(c, U.as_f64(w), "", h.double().numpy(), 1e-5)
    for other in (window - 1, window + 1):                                  # the planted key shows where it enters or leaves
        e = F.mixer_latent_attention({**c, "mask": {"size": other}}, U.as_f64(w), "", h.double().numpy(), 1e-5)
        at = 120 + min(other, window)
        assert U.errors(e, want)[at] > 0.3
    for cuts in (spread(T, [16]), [1] * T, spread(T, [2, 16, 1, 5]), spread(T, [15, 3, 1, 1])):
        e = U.errors(run_mixer(sop, m, pool, h.to(DEV), cuts, dt), want)
        assert e.max() < (1e-4 if dt == torch.float32 else 0.06), (cuts[:4], int(e.argmax()))


def test_positions_far_out(sop):
    """Rotations at large positions: the same rows far from the start give the same output as near it (only distances
    count), to the rounding of 32-bit angles."""
    c = U.latent(3, 16, 8, 16, 24, 20, 0.3, 1e4)["mixer"]
    m, w, pool = mixer_of(sop, LatentAttention, c, torch.float32, portion=256)
    h = torch.randn(24, 24, generator=torch.Generator().manual_seed(1)).to(DEV)
    want = F.mixer_latent_attention(c, U.as_f64(w), "", h.cpu().double().numpy(), 1e-5)
    slot, ws, start = pool.open(), Workspace(DEV), 20000
    pos = pool.pos[slot, :1]
    proj = torch.zeros(24, S.pad8(m.proj.n), device=DEV)
    sop.matmul(h, m.proj, proj, 24)
    out = []
    for at, cnt in ((0, 20), (20, 2), (22, 1), (23, 1)):
        pos.fill_(start + at)
        run = LayerRun(pool.views(slot), "r0.", pos, start + at)
        p = proj[at:at + cnt].clone()
        out.append((m.decode(run, ws, p) if cnt == 1 else m.prefill(run, ws, p, None, cnt)).clone())
    assert U.errors(torch.cat(out)[19:], want[19:]).max() < 5e-3            # rows whose whole window lies in the run


def test_latent_attention_refuses_bad_arguments(sop):
    m, _, pool = mixer_of(sop, LatentAttention, U.latent(1, 8, 2, 8, 8, 4, 1.0, 10.0)["mixer"], torch.float32, portion=8)
    run = LayerRun(pool.views(0), "r0.", pool.pos[0, :1], 0)
    proj = torch.zeros(9, S.pad8(m.proj.n), device=DEV)
    with pytest.raises(Hf2qError):
        m.prefill(run, Workspace(DEV), proj, None, 9)                       # more tokens than the ring holds
