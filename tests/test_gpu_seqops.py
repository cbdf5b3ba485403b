"""The bf16-weight products, row prologues, windowed attention and recurrent mixers, each against plain f64 arithmetic."""
import numpy as np
import pytest
import torch

from hf2q_b200 import seqops as S
from hf2q_b200.ops import DT_BF16, DT_F32, Hf2qError
from oracle import fomatar_forward as F

pytestmark = pytest.mark.gpu
DEV = "cuda"


@pytest.fixture(scope="module")
def sop(gpu_ctx):
    return S.SeqOps(gpu_ctx)


def f32(a):
    return torch.tensor(np.asarray(a), dtype=torch.float32, device=DEV)


def dev_pos(p):
    return torch.tensor([p], dtype=torch.int32, device=DEV)


def rel(got, want):
    got = got.detach().cpu().double().numpy().reshape(want.shape)
    return float(np.linalg.norm(got - want) / max(np.linalg.norm(want), 1e-30))


# ---- products ---------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("m,n,k", [(1, 5, 8), (2, 300, 72), (3, 64, 4096), (8, 129, 1000), (9, 24, 8), (64, 616, 312), (130, 301, 72), (257, 1030, 200),
                                   (600, 4096, 512), (1500, 2304, 264)])
@pytest.mark.parametrize("xd", [torch.float32, torch.bfloat16])
def test_product_and_epilogues(sop, m, n, k, xd):
    g = torch.Generator().manual_seed(m * 7 + n)
    x = torch.randn(m, k, generator=g).to(xd)
    w = S.DenseWeight((torch.randn(n, k, generator=g) / k ** 0.5).to(torch.bfloat16), DEV)
    want = x.double().numpy() @ w.w.cpu().double().numpy().T
    res = torch.randn(m, n, generator=g)
    xg = x.to(DEV)
    tol = 2e-6 if k <= 512 else 2e-5
    y = torch.full((m, n), 7.0, device=DEV)
    sop.matmul(xg, w, y, m)
    assert rel(y, want) < tol
    y.copy_(res.to(DEV))
    sop.matmul(xg, w, y, m, S.EPI_ADD, residual=y)                      # in place
    assert rel(y, want + res.double().numpy()) < tol
    sop.matmul(xg, w, y, m, S.EPI_SOFTCAP, cap=1.5)
    assert rel(y, 1.5 * np.tanh(want / 1.5)) < tol
    yb = torch.empty((m, n), dtype=torch.bfloat16, device=DEV)
    sop.matmul(xg, w, yb, m, S.EPI_GELU)
    assert rel(yb, F.gelu_tanh(want)) < 3e-3
    sop.ctx.check_status()


def test_product_reads_and_writes_with_a_row_pitch(sop):
    g = torch.Generator().manual_seed(3)
    for m in (4, 40):
        big = torch.randn(m, 96, generator=g).to(torch.bfloat16).to(DEV)
        w = S.DenseWeight(torch.randn(20, 64, generator=g).to(torch.bfloat16), DEV)
        out = torch.zeros(m, 32, device=DEV)
        sop.matmul(big[:, 16:80], w, out[:, :20], m)
        assert rel(out[:, :20], big[:, 16:80].cpu().double().numpy() @ w.w.cpu().double().numpy().T) < 1e-5
        assert float(out[:, 20:].abs().sum()) == 0.0


def test_product_refuses_bad_arguments(sop):
    w = S.DenseWeight(torch.zeros(4, 16, dtype=torch.bfloat16), DEV)
    y = torch.zeros(2, 4, device=DEV)
    with pytest.raises(Hf2qError):
        sop.matmul(torch.zeros(2, 8, device=DEV), w, y, 2)              # rows shorter than k
    with pytest.raises(Hf2qError):
        sop.matmul(torch.zeros(2, 16, device=DEV), w, y, 2, S.EPI_ADD)  # no residual


# ---- row prologues ------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("width", [1, 52, 344, 4096])
@pytest.mark.parametrize("m", [1, 2, 7])
def test_pre_norm_and_token_shift(sop, width, m):
    rng = np.random.default_rng(width + m)
    eps, ldo = 1e-3, S.pad8(width)
    x, a, b, add0 = (rng.standard_normal((m, width)) for _ in range(4))
    an, bn, step, norm, mu, before = (rng.standard_normal(width) for _ in range(6))
    for pos in (0, 5, 6):
        rows = x + 0.5 * (F.rms(a, eps) * an + F.rms(b, eps) * bn) + add0 + step
        h = F.rms(rows, eps) * norm
        prev = np.vstack([before[None] if pos else np.zeros((1, width)), h[:-1]])
        want = h + (prev - h) * mu
        st = np.full((2, width), 9.0)
        st[(pos + 1) & 1] = prev[0]
        state, x_out, out = f32(st), torch.zeros(m, width, device=DEV), torch.full((m, ldo), 3.0, device=DEV)
        last = torch.zeros(1, width, device=DEV)
        keep = [f32(v) for v in (x, a, b, an, bn, add0, step, norm, mu)] + [dev_pos(pos)]
        p = S.struct(S.PreNorm, x=keep[0], a=keep[1], b=keep[2], a_norm=keep[3], b_norm=keep[4], add0=keep[5], step=keep[6], x_out=x_out, norm=keep[7],
                     shift=keep[8], shift_state=state, pos=keep[9], eps=eps, width=width)
        sop.pre_norm(p, m, out, last)
        if m > 1:
            sop.state_tail(keep[9], m, last, state, width)
        assert rel(x_out, rows) < 1e-6 and rel(out[:, :width], want) < 2e-6 and float(out[:, width:].abs().sum()) == 0.0
        assert rel(state[(pos + m - 1) & 1], h[-1]) < 1e-6
        if m == 1:
            # the same prologue inside the mat-vec, against the state as it was
            w = S.DenseWeight(torch.randn(37, width).to(torch.bfloat16), DEV)
            state2, y, xo2 = f32(st), torch.zeros(1, 37, device=DEV), torch.zeros(1, width, device=DEV)
            p.shift_state, p.x_out = state2.data_ptr(), xo2.data_ptr()
            sop.matvec(S.PRO_NORM, S.struct(S.Matvec, w=w.w, y=y, pre=p, n=w.n, k=w.k))
            assert rel(y, want @ w.w[:, :width].cpu().double().numpy().T) < 1e-5
            assert torch.allclose(state2, state, rtol=1e-5, atol=1e-6) and torch.allclose(xo2, x_out, rtol=1e-5, atol=1e-6)


@pytest.mark.parametrize("m", [600, 2501])
def test_pre_norm_of_long_portions(sop, m):
    """Several rows per CTA: the row in front of a CTA's first one is recomputed."""
    rng = np.random.default_rng(m)
    w = 68
    x, norm, mu, step = rng.standard_normal((m, w)), rng.standard_normal(w), rng.random(w), rng.standard_normal(w)
    h = F.rms(x + step, 1e-5) * norm
    xg, ng, mg, sg, state, last, pos = f32(x), f32(norm), f32(mu), f32(step), torch.zeros(2, w, device=DEV), torch.zeros(1, w, device=DEV), dev_pos(0)
    out, x_out = torch.zeros(m, 72, device=DEV), torch.zeros(m, w, device=DEV)
    p = S.struct(S.PreNorm, x=xg, step=sg, x_out=x_out, norm=ng, shift=mg, shift_state=state, pos=pos, eps=1e-5, width=w)
    sop.pre_norm(p, m, out, last)
    assert rel(out[:, :w], F.token_shift(h, mu)) < 2e-6 and rel(last, h[-1:]) < 1e-6 and rel(x_out, x + step) < 1e-6


@pytest.mark.parametrize("norm_all", [0, 1])
def test_gated_heads_alone_and_in_the_matvec(sop, norm_all):
    rng = np.random.default_rng(2)
    m, H, d, eps = 5, 3, 19, 1e-4
    o, gate = rng.standard_normal((m, H * d)), rng.standard_normal((m, H * d + 4))
    w = rng.standard_normal(H * d if norm_all else d)
    want = (F.rms(o.reshape(m, H, d), eps) * (w.reshape(H, d) if norm_all else w)).reshape(m, -1) * F.sigmoid(gate[:, 2:2 + H * d])
    og, gg, wg = f32(o), f32(gate), f32(w)
    g = S.struct(S.GatedHeads, o=og, gate=gg.data_ptr() + 8, norm=wg, ldo=H * d, ldg=H * d + 4, heads=H, head_dim=d, norm_all=norm_all, eps=eps)
    out = torch.full((m, 64), 2.0, device=DEV)
    sop.gated_heads(g, m, out)
    assert rel(out[:, :H * d], want) < 1e-6 and float(out[:, H * d:].abs().sum()) == 0.0
    pr = S.DenseWeight(torch.randn(50, H * d).to(torch.bfloat16), DEV)
    pr2 = S.DenseWeight(torch.randn(11, H * d).to(torch.bfloat16), DEV)
    y, y2, res = torch.zeros(1, 50, device=DEV), torch.zeros(1, 11, device=DEV), torch.randn(1, 50, device=DEV)
    plain = S.struct(S.GatedHeads, o=og, gate=gg.data_ptr() + 8, ldo=H * d, ldg=H * d + 4, heads=H, head_dim=d)
    sop.matvec(S.PRO_GATED, S.struct(S.Matvec, w=pr.w, y=y, residual=res, gated=g, n=pr.n, k=pr.k, epilogue=S.EPI_ADD),
               S.struct(S.Matvec, w=pr2.w, y=y2, gated=plain, n=pr2.n, k=pr2.k))
    assert rel(y, want[:1] @ pr.w[:, :H * d].cpu().double().numpy().T + res.cpu().double().numpy()) < 1e-5
    assert rel(y2, (o[0] * F.sigmoid(gate[0, 2:2 + H * d]))[None] @ pr2.w[:, :H * d].cpu().double().numpy().T) < 1e-5


def test_embedding_rows(sop):
    g = torch.Generator().manual_seed(0)
    emb, big = torch.randn(50, 33, generator=g).to(torch.bfloat16), torch.randn(14, 33, generator=g).to(torch.bfloat16)
    cfg = {"embedding": {"bigram": {"buckets": 13, "mul_prev": 2 ** 33 + 1, "mul_cur": 12345678901}}}
    ids = [3, 49, 0, 7, 7, 21]
    want = F.embedding(cfg, {"embed": emb.double().numpy(), "bigram": big.double().numpy()}, np.array(ids))
    eg, bg, prev = emb.to(DEV), big.to(DEV), dev_pos(40)
    for cuts in ([6], [1, 1, 4], [2, 3, 1]):
        out, at = torch.zeros(6, 33, device=DEV), 0
        for c in cuts:
            pos = dev_pos(at)
            e = S.struct(S.Embed, embed=eg, bigram=bg, vocab=50, width=33, ld=33, buckets=13, mul_prev=2 ** 33 + 1, mul_cur=12345678901, pos=pos, prev=prev)
            part = torch.tensor(ids[at:at + c], dtype=torch.int32, device=DEV)
            sop.embed(e, part, c, out[at:])
            at += c
        assert rel(out, want) < 1e-7, cuts
    sop.ctx.check_status()
    e = S.struct(S.Embed, embed=eg, vocab=50, width=33, ld=33, pos=prev, prev=prev)
    sop.embed(e, torch.tensor([50], dtype=torch.int32, device=DEV), 1, out)       # out of range: zero row and a status
    with pytest.raises(Hf2qError):
        sop.ctx.check_status()
    assert float(out[0].abs().sum()) == 0.0


# ---- windowed attention ----------------------------------------------------------------------------------------------
def run_window(sop, q, k, v, window, scale, r1, r2, dtype, cuts, capacity=None, qn=None, kn=None, eps=1e-5, gate=None):
    """Runs the tokens in the given portions (one token: the decode kernel); returns [T, H * dv]."""
    T, H, d = q.shape
    G, dv = v.shape[1], v.shape[2]
    row = np.concatenate([q.reshape(T, -1), k.reshape(T, -1), v.reshape(T, -1)] + ([gate] if gate is not None else []), 1)
    qkv = f32(row)
    cap = capacity or window - 1 + max(cuts)
    kc = torch.full((G, cap, S.pad8(d)), 0.0, dtype=dtype, device=DEV)
    vc = torch.full((G, cap, S.pad8(dv)), 0.0, dtype=dtype, device=DEV)
    consts = [f32(c) if c is not None else None for c in (qn, kn, r1, r2)]
    out, at, scratch = torch.zeros(T, H * dv, device=DEV), 0, None
    ld = row.shape[1]
    for c in cuts:
        pos = dev_pos(at)
        a = S.struct(S.WindowAttn, qkv=qkv.data_ptr() + at * ld * 4, ld=ld, q_off=0, k_off=H * d, v_off=H * d + G * d, q_norm=consts[0], k_norm=consts[1],
                     r1=consts[2], r2=consts[3], k_cache=kc, v_cache=vc, heads=H, kv_heads=G, dim=d, vdim=dv, window=window, capacity=cap,
                     cache_dtype=DT_F32 if dtype == torch.float32 else DT_BF16, scale=scale, eps=eps, pos=pos)
        if c == 1:
            scratch = sop.window_scratch(a, DEV) if scratch is None else scratch
            sop.window_decode(a, out[at:at + 1], scratch)
            if gate is not None:
                out[at] *= torch.sigmoid(qkv[at, -H * dv:])
        else:
            qb = torch.zeros(c, H * S.pad8(d), dtype=dtype, device=DEV)
            sop.window_append(a, c, qb)
            gp = qkv.data_ptr() + (at * ld + ld - H * dv) * 4 if gate is not None else None
            sop.window_prefill(a, c, qb, gp, ld, out[at:at + c])
        at += c
    return out


WSHAPES = [(6, 2, 40, 24, 33), (3, 1, 17, 9, 5), (2, 2, 64, 64, 64), (10, 1, 128, 128, 150), (2, 1, 160, 144, 65), (1, 1, 256, 256, 1), (4, 1, 48, 96, 400)]


@pytest.mark.parametrize("H,G,d,dv,window", WSHAPES)
@pytest.mark.parametrize("dtype,tol", [(torch.float32, 3e-6), (torch.bfloat16, 1e-2)])
def test_window_attention_in_portions(sop, H, G, d, dv, window, dtype, tol):
    rng = np.random.default_rng(H * d + window)
    T = 215
    q, k, v = rng.standard_normal((T, H, d)), rng.standard_normal((T, G, d)), rng.standard_normal((T, G, dv))
    qn, kn, r1, r2 = 1 + 0.3 * rng.standard_normal(d), 1 + 0.3 * rng.standard_normal(d), rng.random(H) + 0.2, rng.random(H) * 0.3
    gate, scale, eps = rng.standard_normal((T, H * dv)), d ** -0.5, 1e-3
    want = F.window_attention(F.rms(q, eps) * qn, F.rms(k, eps) * kn, v, window, scale, r1, r2).reshape(T, -1) * F.sigmoid(gate)
    for cuts in ([T], [1] * 12 + [2, 3, 64, 2, 65, 3, 64], [150] + [1] * 65):
        got = run_window(sop, q, k, v, window, scale, r1, r2, dtype, cuts, qn=qn, kn=kn, eps=eps, gate=gate)
        assert rel(got, want) < tol, cuts


@pytest.mark.parametrize("window", [1, 2, 63, 64, 65, 130])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_a_key_just_inside_and_just_outside_the_window(sop, window, dtype):
    """One key outscores all others; its value must show at the last query that sees it and vanish one later."""
    T, d, at = 300, 32, 101
    q, k, v = np.zeros((T, 1, d)), np.zeros((T, 1, d)), np.zeros((T, 1, 8))
    q[:, 0, 0] = 4.0
    k[at, 0, 0] = 8.0
    v[at] = 1.0
    want = np.zeros(T)
    want[at:at + window] = 1.0
    last = at + window - 1
    for cuts in ([T], [90] + [1] * 210, [at, 2, 3] + [64] * 2 + [T - at - 133], [last, 2, T - last - 2], [last + 1, T - last - 1]):
        got = run_window(sop, q, k, v, window, 1.0, None, None, dtype, [c for c in cuts if c], capacity=window - 1 + max(cuts))
        assert np.abs(got[:, 0].cpu().numpy() - want).max() < 1e-3, cuts


def test_the_distance_term_against_a_far_key(sop):
    """Two keys of equal score: the weights' ratio is (1 + r2 distance) to the power of -r1."""
    T, d = 200, 16
    q, k, v = np.zeros((T, 1, d)), np.zeros((T, 1, d)), np.zeros((T, 1, 8))
    q[:, 0, 0], k[:, 0, 0] = 1.0, -60.0
    k[10, 0, 0] = k[190, 0, 0] = 0.0
    v[10] = 1.0
    for dtype in (torch.float32, torch.bfloat16):
        for cuts in ([T], [T - 4] + [1] * 4):
            got = run_window(sop, q, k, v, 190, 1.0, np.array([0.7]), np.array([0.25]), dtype, cuts)
            a, b = (1 + 0.25 * 189) ** -0.7, (1 + 0.25 * 9) ** -0.7
            assert float(got[199, 0]) == pytest.approx(a / (a + b), rel=2e-3 if dtype == torch.bfloat16 else 1e-5)
            assert float(got[5, 0]) == 0.0


def test_window_attention_refuses_what_does_not_fit(sop):
    x = torch.zeros(8, 64, device=DEV)
    c = torch.zeros(4096, device=DEV)
    pos = dev_pos(0)
    kw = dict(qkv=x, ld=64, k_cache=c, v_cache=c, heads=1, kv_heads=1, dim=8, vdim=8, window=4, capacity=6, cache_dtype=DT_F32, scale=1.0, pos=pos)
    with pytest.raises(Hf2qError):
        sop.window_append(S.struct(S.WindowAttn, **kw), 4, c.view(8, -1))          # 3 + 4 tokens in a ring of 6
    with pytest.raises(Hf2qError):
        sop.window_append(S.struct(S.WindowAttn, **{**kw, "dim": 300}), 2, c.view(8, -1))


# ---- recurrences --------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("H,d,dv", [(3, 20, 36), (1, 11, 21), (2, 128, 128), (1, 256, 17), (2, 64, 16)])
@pytest.mark.parametrize("bias", [0.0, -6.0])
def test_mlstm_in_portions(sop, H, d, dv, bias):
    """bias -6: weak input gates against the maximum that starts at zero, so that the normaliser's floor decides."""
    rng = np.random.default_rng(d + dv)
    T, cap = 150, 8.0
    q, k, v = rng.standard_normal((T, H, d)), rng.standard_normal((T, H, d)), rng.standard_normal((T, H, dv))
    ir, fr, ib, fb = rng.standard_normal((T, H)) * 3, rng.standard_normal((T, H)) * 3, rng.standard_normal(H) + bias, rng.standard_normal(H) + 2
    want = F.mlstm(q * d ** -0.5, k, v, cap * np.tanh((ir + ib) / cap), -F.softplus(-cap * np.tanh((fr + fb) / cap)))
    row = np.concatenate([x.reshape(T, -1) for x in (q, k, v, ir, fr)], 1)
    proj, ld, dp, sl = f32(row), row.shape[1], S.pad32(d), (dv + 15) // 16
    o = np.cumsum([0, H * d, H * d, H * dv, H])
    ibg, fbg = f32(ib), f32(fb)
    for cuts in ([T], [1] * 20 + [2, 3, 16, 17, 92], [33, 117]):
        s, n, mx = torch.zeros(H, dv, dp, device=DEV), torch.zeros(H, sl, dp, device=DEV), torch.zeros(H, sl, device=DEV)
        out, at = torch.zeros(T, H * dv, device=DEV), 0
        for c in cuts:
            a = S.struct(S.MLstm, proj=proj.data_ptr() + at * ld * 4, ld=ld, q_off=int(o[0]), k_off=int(o[1]), v_off=int(o[2]), i_off=int(o[3]),
                         f_off=int(o[4]), i_bias=ibg, f_bias=fbg, s=s, n=n, mx=mx, heads=H, dim=d, vdim=dv, gate_cap=cap)
            sop.mlstm(a, c, out[at:])
            at += c
        assert rel(out, want) < 5e-5, cuts              # the quotient magnifies rounding where n . q is near its floor
        assert float(s[:, :, d:].abs().sum()) == 0.0


@pytest.mark.parametrize("H,G,d,dv,taps,rank", [(6, 3, 24, 40, 4, 12), (3, 1, 13, 7, 1, 5), (4, 2, 128, 128, 4, 64), (2, 1, 256, 40, 3, 8), (2, 2, 64, 32, 7, 16)])
def test_gated_delta_in_portions(sop, H, G, d, dv, taps, rank):
    rng = np.random.default_rng(d * dv + taps)
    T, rp = 130, S.pad8(rank)
    q, k, v, b = rng.standard_normal((T, G * d)), rng.standard_normal((T, G * d)), rng.standard_normal((T, H * dv)), rng.standard_normal((T, H)) * 2
    lr = [np.pad(rng.standard_normal((T, rank)), ((0, 0), (0, rp - rank))) for _ in range(2)]
    qc, kc, vc = (rng.standard_normal((c, taps)) for c in (G * d, G * d, H * dv))
    a_log, dt = rng.standard_normal(H) * 2 - 1, rng.standard_normal(H * d) - 1               # decays from near 0 to near 1
    a2 = S.DenseWeight(torch.tensor(rng.standard_normal((H * d, rank))).to(torch.bfloat16), DEV)
    g2 = S.DenseWeight(torch.tensor(rng.standard_normal((H * dv, rank))).to(torch.bfloat16), DEV)
    unit = lambda x: x / np.sqrt((x * x).sum(-1, keepdims=True) + 1e-6)
    qh = np.repeat(unit(F.short_conv(q, qc).reshape(T, G, d)) * d ** -0.5, H // G, axis=1)
    kh = np.repeat(unit(F.short_conv(k, kc).reshape(T, G, d)), H // G, axis=1)
    raw = (lr[0] @ a2.w.cpu().double().numpy().T + dt).reshape(T, H, d)
    decay = np.exp(-np.exp(a_log)[:, None] * F.softplus(raw))
    want = F.gated_delta(qh, kh, F.short_conv(v, vc).reshape(T, H, dv), F.sigmoid(b), decay)
    row = np.concatenate([q, k, v, b, *lr], 1)
    proj, ld, o = f32(row), row.shape[1], np.cumsum([0, G * d, G * d, H * dv, H, rp])
    consts = [f32(c) for c in (qc, kc, vc, a_log, dt)]
    for cuts in ([T], [1] * 9 + [2, 3, 16, 17, 2, 81], [40] + [1] * 40 + [50]):
        conv, s = torch.zeros(2 * G * d + H * dv, taps, device=DEV), torch.zeros(H, dv, S.pad32(d), device=DEV)
        out, at = torch.zeros(T, H * dv, device=DEV), 0
        for c in cuts:
            pos = dev_pos(at)
            a = S.struct(S.Delta, proj=proj.data_ptr() + at * ld * 4, ld=ld, q_off=int(o[0]), k_off=int(o[1]), v_off=int(o[2]), b_off=int(o[3]),
                         a1_off=int(o[4]), g1_off=int(o[5]), q_conv=consts[0], k_conv=consts[1], v_conv=consts[2], a_log=consts[3], dt_bias=consts[4],
                         a2=a2.w, g2=g2.w, conv_state=conv, s=s, heads=H, kv_heads=G, dim=d, vdim=dv, taps=taps, a_rank_ld=rp, g_rank_ld=rp, pos=pos)
            if c == 1:
                gate = torch.zeros(1, H * dv, device=DEV)
                sop.delta_step(a, out[at:], gate)
                assert rel(gate, lr[1][at:at + 1] @ g2.w.cpu().double().numpy().T) < 1e-5
            else:
                qkv, beta, g = torch.zeros(c, 2 * G * d + H * dv, device=DEV), torch.zeros(c, H, device=DEV), torch.zeros(c, H * d, device=DEV)
                a1, g1 = torch.zeros(c, rp, device=DEV), torch.zeros(c, rp, device=DEV)
                sop.delta_prep(a, c, qkv, beta, a1, g1)
                sop.matmul(a1, a2, g, c)
                sop.delta_decay(a, c, g)
                sop.delta_scan(a, c, qkv, beta, g, out[at:])
                sop.state_tail(pos, c, None, None, 0, a)
            at += c
        assert rel(out, want) < 2e-5, cuts
