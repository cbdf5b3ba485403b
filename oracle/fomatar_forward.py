"""Plain forward pass of the Fomatar decoder design in numpy / f64: one function per mechanism, one token
after the other wherever the design has a recurrence.  Test infrastructure; shares no code with the product.

A model is a ``config`` dict (the keys of its config.json) and ``w``: {tensor name: float array}.
"""
import numpy as np


def rms(x, eps):
    """x over its root mean square along the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def sigmoid(x):
    return 1.0 / (1.0 + np.exp(-x))


def softplus(x):
    return np.logaddexp(0.0, x)


def silu(x):
    return x * sigmoid(x)


def gelu_tanh(x):
    return 0.5 * x * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (x + 0.044715 * x ** 3)))


def embedding(cfg, w, tokens):
    """Token rows plus the row of (previous token, token) in the hashed bigram table."""
    x = w["embed"][tokens]
    bg = (cfg.get("embedding") or {}).get("bigram")
    if bg:
        rows = [bg["buckets"]]
        for a, b in zip(tokens[:-1], tokens[1:]):
            rows.append((int(a) * bg["mul_prev"] + int(b) * bg["mul_cur"]) % bg["buckets"])
        x = x + w["bigram"][np.array(rows)]
    return x


def token_shift(h, mu):
    before = np.vstack([np.zeros_like(h[:1]), h[:-1]])
    return h + (before - h) * mu


def short_conv(x, taps):
    """Causal depth-wise convolution, x [T, C], taps [C, K] (last column: the current token), then SiLU."""
    K = taps.shape[1]
    ext = np.vstack([np.zeros((K - 1, x.shape[1])), x])
    y = np.zeros_like(x)
    for j in range(K):
        y += ext[j:j + len(x)] * taps[:, j]
    return silu(y)


def window_attention(q, k, v, window, scale, r1, r2):
    """q [T, H, d], k [T, G, d], v [T, G, dv]; key j is visible to i when 0 <= i - j < window; the score loses
    r1 ln(1 + r2 (i - j)) of its head."""
    T, H, _ = q.shape
    rep = H // k.shape[1]
    out = np.zeros((T, H, v.shape[2]))
    for i in range(T):
        j0 = max(0, i - window + 1)
        dist = i - np.arange(j0, i + 1)
        for h in range(H):
            s = k[j0:i + 1, h // rep] @ q[i, h] * scale - r1[h] * np.log1p(r2[h] * dist)
            p = np.exp(s - s.max())
            out[i, h] = (p / p.sum()) @ v[j0:i + 1, h // rep]
    return out


def mlstm(q, k, v, ig, fg):
    """Matrix memory with exponential gates: q, k [T, H, d], v [T, H, dv], log gates ig, fg [T, H]."""
    T, H, d = q.shape
    out = np.zeros((T, H, v.shape[2]))
    for h in range(H):
        S, n, m = np.zeros((d, v.shape[2])), np.zeros(d), 0.0
        for t in range(T):
            m_new = max(fg[t, h] + m, ig[t, h])
            keep, write = np.exp(fg[t, h] + m - m_new), np.exp(ig[t, h] - m_new)
            S = keep * S + write * np.outer(k[t, h], v[t, h])
            n = keep * n + write * k[t, h]
            m = m_new
            out[t, h] = (q[t, h] @ S) / (max(abs(n @ q[t, h]), np.exp(-m)) + 1e-6)
    return out


def gated_delta(q, k, v, beta, g):
    """Delta rule with one decay per key channel: q, k, g [T, H, d], v [T, H, dv], beta [T, H]."""
    T, H, d = q.shape
    out = np.zeros((T, H, v.shape[2]))
    for h in range(H):
        S = np.zeros((d, v.shape[2]))
        for t in range(T):
            S = g[t, h][:, None] * S
            u = beta[t, h] * (v[t, h] - k[t, h] @ S)
            S = S + np.outer(k[t, h], u)
            out[t, h] = q[t, h] @ S
    return out


def mixer_parallel(c, w, p, h, eps):
    T = len(h)
    lin = lambda name: h @ w[p + name].T
    L, R = c["left"], c["right"]
    q = rms(lin("left.q").reshape(T, L["heads"], L["dim"]), eps) * w[p + "left.q.norm"]
    k = rms(lin("left.k").reshape(T, L["kv_heads"], L["dim"]), eps) * w[p + "left.k.norm"]
    v = lin("left.v").reshape(T, L["kv_heads"], L["vdim"])
    o = window_attention(q, k, v, L["mask"]["size"], L["scale"], w[p + "left.r1"], w[p + "left.r2"])
    left = (o.reshape(T, -1) * sigmoid(lin("left.g"))) @ w[p + "left.o"].T

    q = lin("right.q").reshape(T, R["heads"], R["dim"]) * R["dim"] ** -0.5
    k = lin("right.k").reshape(T, R["heads"], R["dim"])
    v = lin("right.v").reshape(T, R["heads"], R["vdim"])
    cap = R["gate_cap"]
    ig = cap * np.tanh((lin("right.i") + w[p + "right.i.b"]) / cap)
    fg = -softplus(-cap * np.tanh((lin("right.f") + w[p + "right.f.b"]) / cap))
    o = rms(mlstm(q, k, v, ig, fg), eps).reshape(T, -1) * w[p + "right.norm"]
    right = (o * sigmoid(lin("right.g"))) @ w[p + "right.o"].T
    return 0.5 * (rms(left, eps) * w[p + "left.out"] + rms(right, eps) * w[p + "right.out"])


def mixer_channel_delta(c, w, p, h, eps):
    T, H, G, d, dv = len(h), c["heads"], c["kv_heads"], c["dim"], c["vdim"]
    conv = lambda name: short_conv(h @ w[p + name].T, w[p + name + ".conv"])
    unit = lambda x: x / np.sqrt(np.sum(x * x, axis=-1, keepdims=True) + 1e-6)
    q = np.repeat(unit(conv("q").reshape(T, G, d)) * d ** -0.5, H // G, axis=1)
    k = np.repeat(unit(conv("k").reshape(T, G, d)), H // G, axis=1)
    v = conv("v").reshape(T, H, dv)
    beta = sigmoid(h @ w[p + "b"].T)
    a = (h @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "dt_bias"]
    g = np.exp(-np.exp(w[p + "A_log"])[:, None] * softplus(a.reshape(T, H, d)))
    o = rms(gated_delta(q, k, v, beta, g), eps) * w[p + "norm"]
    gate = sigmoid((h @ w[p + "g1"].T) @ w[p + "g2"].T)
    return (o.reshape(T, -1) * gate) @ w[p + "o"].T


MIXERS = {"parallel": mixer_parallel, "channel_delta": mixer_channel_delta}


def layer(entry, w, i, x, eps):
    p = f"l{i}."
    h = token_shift(rms(x, eps) * w[p + "norm1"], w[p + "shift"])
    x = x + MIXERS[entry["type"]](entry["mixer"], w, p + "mix.", h, eps)
    if entry.get("mlp"):
        h = rms(x, eps) * w[p + "norm2"]
        x = x + gelu_tanh(h @ w[p + "mlp.up"].T) @ w[p + "mlp.down"].T
    return x


def layer_runs(cfg):
    """[(layer, pass or None if outside the loop, first layer of its pass)] in execution order."""
    n = len(cfg["layers"])
    loop = cfg.get("loop")
    if not loop:
        return [(i, None, False) for i in range(n)]
    runs = [(i, None, False) for i in range(loop["start"])]
    for t in range(loop["times"]):
        runs += [(i, t, i == loop["start"]) for i in range(loop["start"], loop["stop"])]
    return runs + [(i, None, False) for i in range(loop["stop"], n)]


def forward(cfg, w, tokens, layers_out=None):
    """Logits [T, vocab]; layers_out (a list) collects the residual stream after every layer run."""
    eps = cfg["norm"]["eps"]
    x0 = x = embedding(cfg, w, np.asarray(tokens))
    for i, t, first in layer_runs(cfg):
        if first:
            if t > 0:
                x = x + x0
            x = x + w["loop.step"][t]
        x = layer(cfg["layers"][i], w, i, x, eps)
        if layers_out is not None:
            layers_out.append(x.copy())
    logits = (rms(x, eps) * w["final.norm"]) @ w["head"].T
    cap = cfg.get("logit_softcap")
    return cap * np.tanh(logits / cap) if cap else logits
