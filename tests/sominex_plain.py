"""A plain NumPy implementation of the Sominex decoder, one function per mechanism.

Slow, sequential and in float64: it is what the CUDA path is compared with. It takes the parsed
config.json and a dict of arrays (tensor name -> array) and shares no code with the library.
A sequence is always evaluated whole, from its first token; there is no cache here.
"""

from __future__ import annotations

import numpy as np

F = np.float64


# ------------------------------------------------------------------ element-wise pieces
def sigmoid(z):
    return 0.5 * (1.0 + np.tanh(0.5 * z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.logaddexp(0.0, z)


def logsigmoid(z):
    return -np.logaddexp(0.0, -z)


def unit_rms(x, eps):
    return x / np.sqrt((x * x).mean(axis=-1, keepdims=True) + eps)


# ------------------------------------------------------------------ mechanisms
def token_shift(h, s):
    """row t becomes (1 - s) h_t + s h_(t-1), with a zero row before the first"""
    before = np.concatenate([np.zeros((1, h.shape[1]), F), h[:-1]])
    return h + (before - h) * s


def rope_frequencies(rot):
    """(frequencies [dims/2], factor on cos and sin)"""
    dims, base = rot["dims"], rot["base"]
    i = np.arange(dims // 2, dtype=F)
    f = base ** (-2.0 * i / dims)
    sc = rot.get("scaling")
    if not sc:
        return f, 1.0

    def dim_of(turns):
        return dims * np.log(sc["original"] / (2 * np.pi * turns)) / (2 * np.log(base))

    lo, hi = max(np.floor(dim_of(sc["fast"])), 0), min(np.ceil(dim_of(sc["slow"])), dims - 1)
    ramp = np.clip((i - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return f / sc["factor"] * ramp + f * (1 - ramp), 0.1 * np.log(sc["factor"]) + 1.0


def rotate(x, rot):
    """x [T, heads, dim], row t at position t; first `dims` dimensions, i paired with i + dims/2"""
    if not rot:
        return x
    f, m = rope_frequencies(rot)
    a = np.arange(x.shape[0], dtype=F)[:, None, None] * f
    c, s, n = np.cos(a) * m, np.sin(a) * m, rot["dims"] // 2
    u, v = x[..., :n], x[..., n:2 * n]
    return np.concatenate([u * c - v * s, v * c + u * s, x[..., 2 * n:]], axis=-1)


def pooled_blocks(x, pool):
    """means of the complete blocks of `pool` rows: [T // pool, ...]"""
    n = x.shape[0] // pool
    return x[:n * pool].reshape((n, pool) + x.shape[1:]).mean(axis=1)


def visible(T, window, pool=0):
    """[T, T + T // pool] bool: the tokens, then the pooled blocks, that query i sees"""
    i, j = np.arange(T)[:, None], np.arange(T)[None, :]
    tok = (j <= i) & (i - j < window)
    if not pool:
        return tok
    b = np.arange(T // pool)[None, :]
    return np.concatenate([tok, (b + 1) * pool - 1 <= i - window], axis=1)


def attention(q, k, v, scale, window, pool=0):
    """q [T, H, dim], k [T, G, dim], v [T, G, vdim] -> [T, H, vdim]"""
    T, H, _ = q.shape
    per = H // k.shape[1]
    see = visible(T, window, pool)
    if pool:
        k, v = np.concatenate([k, pooled_blocks(k, pool)]), np.concatenate([v, pooled_blocks(v, pool)])
    out = np.zeros((T, H, v.shape[2]), F)
    for h in range(H):
        s = np.where(see, q[:, h] @ k[:, h // per].T * scale, -np.inf)
        p = np.exp(s - s.max(axis=1, keepdims=True))
        out[:, h] = (p / p.sum(axis=1, keepdims=True)) @ v[:, h // per]
    return out


def conv_silu(x, w, b):
    """causal convolution over time per channel with a bias, then silu: x [T, C], w [C, taps]"""
    T, taps = x.shape[0], w.shape[1]
    pad = np.concatenate([np.zeros((taps - 1, x.shape[1]), F), x])
    y = np.zeros_like(x) + b
    for j in range(taps):
        y += w[:, j] * pad[j:j + T]
    return silu(y)


def ssm(x, B, C, dt, A_log, D):
    """x [T, H, vdim], B, C [T, G, N], dt [T, H] step sizes -> y [T, H, vdim]"""
    T, H, vd = x.shape
    per = H // B.shape[1]
    S = np.zeros((H, B.shape[2], vd), F)
    y = np.zeros_like(x)
    for t in range(T):
        for h in range(H):
            S[h] = np.exp(-np.exp(A_log[h]) * dt[t, h]) * S[h] + dt[t, h] * np.outer(B[t, h // per], x[t, h])
            y[t, h] = S[h].T @ C[t, h // per] + D[h] * x[t, h]
    return y


def mlstm(q, k, v, i, f):
    """q, k [T, H, dim], v [T, H, vdim], i, f [T, H] log gates -> o [T, H, vdim]"""
    T, H, dim = q.shape
    S, n, m = np.zeros((H, dim, v.shape[2]), F), np.zeros((H, dim), F), np.zeros(H, F)
    o = np.zeros((T, H, v.shape[2]), F)
    for t in range(T):
        for h in range(H):
            new = max(f[t, h] + m[h], i[t, h])
            a, b = np.exp(f[t, h] + m[h] - new), np.exp(i[t, h] - new)
            S[h] = a * S[h] + b * np.outer(k[t, h], v[t, h])
            n[h] = a * n[h] + b * k[t, h]
            m[h] = new
            o[t, h] = S[h].T @ q[t, h] / (max(abs(n[h] @ q[t, h]), np.exp(-new)) + 1e-6)
    return o


def route(z, top, scale):
    """[T, E] logits -> (chosen experts [T, top], weights [T, top])"""
    s = np.exp(z - z.max(axis=1, keepdims=True))
    s /= s.sum(axis=1, keepdims=True)
    e = np.argsort(-s, axis=1, kind="stable")[:, :top]
    return e, np.take_along_axis(s, e, axis=1) * scale


def clamped_glu(g, u, limit):
    g, u = np.minimum(g, limit), np.clip(u, -limit, limit)
    return g * sigmoid(1.702 * g) * (u + 1)


# ------------------------------------------------------------------ blocks
def attention_mixer(h, W, p, c, eps):
    T = h.shape[0]
    q = rotate((h @ W[p + "q"].T).reshape(T, c["heads"], c["dim"]), c.get("rot"))
    k = rotate((h @ W[p + "k"].T).reshape(T, c["kv_heads"], c["dim"]), c.get("rot"))
    v = unit_rms((h @ W[p + "v"].T).reshape(T, c["kv_heads"], c["vdim"]), eps)
    return attention(q, k, v, c["scale"], c["mask"]["size"], c["mask"].get("pool", 0)).reshape(T, -1) @ W[p + "o"].T


def mamba2_mixer(h, W, p, c, eps):
    T, H, N, G, vd = h.shape[0], c["heads"], c["state"], c["groups"], c["vdim"]
    inner = H * vd
    z, xbc, dt = np.split(h @ W[p + "in"].T, [inner, 2 * inner + 2 * G * N], axis=1)
    x, B, C = np.split(conv_silu(xbc, W[p + "conv"], W[p + "conv.b"]), [inner, inner + G * N], axis=1)
    y = ssm(x.reshape(T, H, vd), B.reshape(T, G, N), C.reshape(T, G, N), softplus(dt + W[p + "dt_bias"]), W[p + "A_log"], W[p + "D"])
    y = (y.reshape(T, inner) * silu(z)).reshape(T, c["norm_groups"], -1)
    return (unit_rms(y, eps).reshape(T, inner) * W[p + "norm"]) @ W[p + "o"].T


def mlstm_mixer(h, W, p, c, eps):
    T, H, dim, vd, cap = h.shape[0], c["heads"], c["dim"], c["vdim"], c["gate_cap"]
    q = (h @ W[p + "q"].T).reshape(T, H, dim) * dim ** -0.5
    k = (h @ W[p + "k"].T).reshape(T, H, dim)
    v = (h @ W[p + "v"].T).reshape(T, H, vd)
    i = cap * np.tanh((h @ W[p + "i"].T + W[p + "i.b"]) / cap)
    f = logsigmoid(cap * np.tanh((h @ W[p + "f"].T + W[p + "f.b"]) / cap))
    o = unit_rms(mlstm(q, k, v, i, f), eps).reshape(T, -1) * W[p + "norm"]
    return (o * sigmoid(h @ W[p + "g"].T)) @ W[p + "o"].T


MIXERS = {"attention": attention_mixer, "mamba2": mamba2_mixer, "mlstm": mlstm_mixer}


def expert(h, W, p):
    return (silu(h @ W[p + "gate"].T) * (h @ W[p + "up"].T)) @ W[p + "down"].T


def feed_forward(h, W, p, c):
    if c["kind"] == "dense":
        return clamped_glu(h @ W[p + "gate"].T, h @ W[p + "up"].T, c["limit"]) @ W[p + "down"].T
    y = expert(h, W, p + "shared.") if c.get("shared") else np.zeros_like(h)
    chosen, weight = route(h @ W[p + "router"].T, c["router"]["top"], c["router"]["scale"])
    for t in range(h.shape[0]):
        for e, w in zip(chosen[t], weight[t]):
            y[t] += w * expert(h[t], W, p + "e%d." % e)
    return y


def layer(x, W, i, cfg):
    p, spec, eps = "l%d." % i, cfg["layers"][i], cfg["norm"]["eps"]
    h = unit_rms(x, eps) * W[p + "norm1"]
    y = MIXERS[spec["type"]](token_shift(h, W[p + "shift"]), W, p + "mix.", spec["mixer"], eps)
    if spec.get("mlp"):
        y = y + feed_forward(h, W, p + "mlp.", spec["mlp"])
    return x + y


def forward(tokens, W, cfg, trace=None):
    """logits [T, vocab]; the residual stream after every layer is appended to `trace`"""
    W = {k: np.asarray(v, F) for k, v in W.items()}
    x = W["embed"][np.asarray(tokens)] * cfg["embedding"]["scale"]
    for i in range(len(cfg["layers"])):
        x = layer(x, W, i, cfg)
        if trace is not None:
            trace.append(x)
    return (unit_rms(x, cfg["norm"]["eps"]) * W["final.norm"]) @ W["head"].T
