"""Plain forward pass of the Runopel decoder design in numpy / f64: one function per mechanism, one token after the
other wherever the design has a recurrence.  Test infrastructure; shares no code with the product.

A model is a ``config`` dict (the keys of its config.json) and ``w``: {tensor name: float array}.
"""
import numpy as np


def rms(x, eps):
    """x over its root mean square along the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def sigmoid(x):
    return 1.0 / (1.0 + np.exp(-x))


def silu(x):
    return x * sigmoid(x)


def softplus(x):
    return np.logaddexp(0.0, x)


# ---- hyper-connections: X [streams, T, width]
def read_streams(X, c_in):
    return np.einsum("s,stw->tw", c_in, X)


def write_streams(X, y, mix, c_out, mult):
    """Every stream from all old ones (mix is indexed [from, to]) plus its share of the sublayer's output."""
    return np.einsum("ab,atw->btw", mix, X) + mult * c_out[:, None, None] * y


# ---- mamba2
def short_conv(x, taps, bias):
    """Causal depth-wise convolution, x [T, C], taps [C, K] (last column: the current token), bias [C], then SiLU."""
    K = taps.shape[1]
    y = np.zeros_like(x)
    for t in range(len(x)):
        for j in range(K):
            if t - j >= 0:
                y[t] += x[t - j] * taps[:, K - 1 - j]
    return silu(y + bias)


def state_space(x, B, C, dt, a_log, D):
    """x [T, H, P], B, C [T, G, N], dt [T, H] > 0: a scalar decay per head and token, rank-one writes."""
    T, H, P = x.shape
    G, N = B.shape[1:]
    y = np.zeros_like(x)
    for h in range(H):
        g = h // (H // G)
        S = np.zeros((N, P))
        for t in range(T):
            S = np.exp(-np.exp(a_log[h]) * dt[t, h]) * S + dt[t, h] * np.outer(B[t, g], x[t, h])
            y[t, h] = C[t, g] @ S + D[h] * x[t, h]
    return y


def gated_group_norm(y, z, weight, groups, eps):
    """The gate first, then every one of the equal parts over its own root mean square."""
    v = y * silu(z)
    return rms(v.reshape(len(v), groups, -1), eps).reshape(v.shape) * weight


def mixer_mamba2(c, w, p, h, eps):
    T, H, P, N, G = len(h), c["heads"], c["vdim"], c["state"], c["groups"]
    inner = H * P
    z, xbc, dt = np.split(h @ w[p + "in"].T, [inner, 2 * inner + 2 * G * N], axis=1)
    xbc = short_conv(xbc, w[p + "conv"], w[p + "conv.b"])
    x, B, C = np.split(xbc, [inner, inner + G * N], axis=1)
    y = state_space(x.reshape(T, H, P), B.reshape(T, G, N), C.reshape(T, G, N), softplus(dt + w[p + "dt_bias"]), w[p + "A_log"], w[p + "D"])
    return gated_group_norm(y.reshape(T, inner), z, w[p + "norm"], c["norm_groups"], eps) @ w[p + "o"].T


# ---- latent attention
def rotate(x, base, first=0):
    """x [T, ..., d]: pair (2i, 2i + 1) of the token at position first + t turned by position * base^(-2i / d)."""
    d = x.shape[-1]
    out = np.array(x)
    for t in range(len(x)):
        for i in range(d // 2):
            a = (first + t) * base ** (-2.0 * i / d)
            u, v = x[t, ..., 2 * i], x[t, ..., 2 * i + 1]
            out[t, ..., 2 * i], out[t, ..., 2 * i + 1] = u * np.cos(a) - v * np.sin(a), v * np.cos(a) + u * np.sin(a)
    return out


def window_softmax(q, k, v, window, scale):
    """q, k [T, H, d], v [T, H, dv]; key j is visible to i when 0 <= i - j < window."""
    T, H, _ = q.shape
    out = np.zeros((T, H, v.shape[2]))
    for i in range(T):
        j0 = max(0, i - window + 1)
        for h in range(H):
            s = k[j0:i + 1, h] @ q[i, h] * scale
            e = np.exp(s - s.max())
            out[i, h] = (e / e.sum()) @ v[j0:i + 1, h]
    return out


def mixer_latent_attention(c, w, p, h, eps):
    T, H, d, r, dv, base = len(h), c["heads"], c["dim"], c["rot_dim"], c["vdim"], c["rot"]["base"]
    q = (h @ w[p + "q"].T).reshape(T, H, d + r)
    low = h @ w[p + "dkv"].T
    lat = rms(low[:, :c["kv_rank"]], eps) * w[p + "dkv.norm"]
    k_rot = rotate(low[:, None, c["kv_rank"]:], base)
    q = np.concatenate([q[..., :d], rotate(q[..., d:], base)], axis=2)
    k = np.concatenate([(lat @ w[p + "uk"].T).reshape(T, H, d), np.repeat(k_rot, H, axis=1)], axis=2)
    v = (lat @ w[p + "uv"].T).reshape(T, H, dv)
    return window_softmax(q, k, v, c["mask"]["size"], c["scale"]).reshape(T, H * dv) @ w[p + "o"].T


MIXERS = {"mamba2": mixer_mamba2, "latent_attention": mixer_latent_attention}


# ---- feed-forward
def clamped_glu(h, wg, bg, wu, bu, wd, bd, limit):
    g = np.minimum(h @ wg.T + bg, limit)
    u = np.clip(h @ wu.T + bu, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ wd.T + bd


def route(h, router, top):
    """Scores of all experts and, per token, the chosen ones (largest score first)."""
    s = sigmoid(h @ router.T)
    return s, np.argsort(-s, axis=1, kind="stable")[:, :top]


def expert_mixture(h, router, experts, top):
    """experts: [(gate, up, down)]; a chosen expert's score scales its input."""
    s, ids = route(h, router, top)
    y = np.zeros((len(h), experts[0][2].shape[0]))
    for t in range(len(h)):
        for e in ids[t]:
            gate, up, down = experts[e]
            x = s[t, e] * h[t]
            y[t] += down @ (silu(gate @ x) * (up @ x))
    return y


def feed_forward(mlp, w, p, h):
    if mlp["kind"] == "dense":
        return clamped_glu(h, *[w[p + n] for n in ("gate", "gate.b", "up", "up.b", "down", "down.b")], mlp["limit"])
    r = mlp["router"]
    return expert_mixture(h, w[p + "router"], [[w[f"{p}e{e}.{n}"] for n in ("gate", "up", "down")] for e in range(r["experts"])], r["top"])


# ---- the model
def forward(cfg, w, tokens, layers_out=None):
    """Logits [T, vocab]; layers_out (a list) collects the sum of the streams after every layer."""
    eps, mult = cfg["norm"]["eps"], cfg["residual_mult"]
    x = w["embed"][np.asarray(tokens)]
    X = np.stack([x] * cfg["streams"])
    for i, e in enumerate(cfg["layers"]):
        p = f"l{i}."
        subs = [lambda h: MIXERS[e["type"]](e["mixer"], w, p + "mix.", h, eps)]
        if e.get("mlp"):
            subs.append(lambda h: feed_forward(e["mlp"], w, p + "mlp.", h))
        for q, sub in enumerate(subs, 1):
            hc = f"{p}hc{q}."
            y = sub(rms(read_streams(X, w[hc + "in"]), eps) * w[f"{p}norm{q}"])
            X = write_streams(X, y, w[hc + "mix"], w[hc + "out"], mult)
        if layers_out is not None:
            layers_out.append(X.sum(0))
    return (rms(X.sum(0), eps) * w["final.norm"]) @ w["embed"].T * cfg["logit_scale"]
