"""A plain NumPy implementation of the Nabelix decoder, one function per mechanism.

Slow, sequential and in float64: it is what the CUDA path is compared with. It takes the parsed
config.json and a dict of arrays (tensor name -> array) and shares no code with the library.
A sequence is always evaluated whole, from its first token; there is no cache here.
"""

from __future__ import annotations

import json
import struct

import numpy as np

F = np.float64


# ------------------------------------------------------------------ element-wise pieces
def sigmoid(z):
    return 0.5 * (1.0 + np.tanh(0.5 * z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.logaddexp(0.0, z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (z + 0.044715 * z ** 3)))


def layer_norm(x, w, eps):
    c = x - x.mean(axis=-1, keepdims=True)
    return c / np.sqrt((c * c).mean(axis=-1, keepdims=True) + eps) * w


def rms_norm(x, w, eps):
    return x / np.sqrt((x * x).mean(axis=-1, keepdims=True) + eps) * w


def softcap(x, cap):
    return cap * np.tanh(x / cap) if cap else x


# ------------------------------------------------------------------ mechanisms
def causal_conv(x, w):
    """depth-wise causal convolution over time: x [T, C], w [C, taps], the last tap meets the current row"""
    T, taps = x.shape[0], w.shape[1]
    pad = np.concatenate([np.zeros((taps - 1, x.shape[1]), F), x])
    y = np.zeros_like(x)
    for j in range(taps):
        y += w[:, j] * pad[j:j + T]
    return y


def visible(T, window, keep_first):
    """[T, T] bool: query i sees key j"""
    i, j = np.arange(T)[:, None], np.arange(T)[None, :]
    return (j <= i) & ((i - j < window) | (j < keep_first))


def distance_bias(T, r1, r2):
    """[T, T]: what is taken off a head's scores (only j <= i is meaningful)"""
    d = np.maximum(np.arange(T)[:, None] - np.arange(T)[None, :], 0)
    return r1 * np.log1p(r2 * d)


def attention(q, k, v, scale, window, keep_first, r1, r2):
    """q [T, H, dim], k [T, G, dim], v [T, G, vdim] -> [T, H, vdim]"""
    T, H, _ = q.shape
    per = H // k.shape[1]
    see = visible(T, window, keep_first)
    out = np.zeros((T, H, v.shape[2]), F)
    for h in range(H):
        s = q[:, h] @ k[:, h // per].T * scale - distance_bias(T, r1[h], r2[h])
        s = np.where(see, s, -np.inf)
        p = np.exp(s - s.max(axis=1, keepdims=True))
        out[:, h] = (p / p.sum(axis=1, keepdims=True)) @ v[:, h // per]
    return out


def unit(x):
    return x / np.sqrt((x * x).sum(axis=-1, keepdims=True) + 1e-6)


def delta_rule(q, k, v, g, beta):
    """q, k [T, KH, dim], v [T, H, vdim], g [T, H, dim] decays, beta [T, H] -> (o [T, H, vdim], state)"""
    T, H, vd = v.shape
    per = H // q.shape[1]
    S = np.zeros((H, q.shape[2], vd), F)
    o = np.zeros((T, H, vd), F)
    for t in range(T):
        for h in range(H):
            kk, qq = k[t, h // per], q[t, h // per]
            S[h] *= g[t, h][:, None]
            u = beta[t, h] * (v[t, h] - S[h].T @ kk)
            S[h] += np.outer(kk, u)
            o[t, h] = S[h].T @ qq
    return o, S


# ------------------------------------------------------------------ blocks
def left_mixer(h, W, p, c):
    T = h.shape[0]
    q = (h @ W[p + "q"].T).reshape(T, c["heads"], c["dim"])
    k = (h @ W[p + "k"].T).reshape(T, c["kv_heads"], c["dim"])
    v = (h @ W[p + "v"].T).reshape(T, c["kv_heads"], c["vdim"])
    o = attention(q, k, v, c["scale"], c["mask"]["size"], c["mask"]["keep_first"], W[p + "r1"], W[p + "r2"]).reshape(T, -1)
    return (o * sigmoid(h @ W[p + "g"].T)) @ W[p + "o"].T


def right_mixer(h, W, p, c, eps):
    T, H, KH, dim, vd = h.shape[0], c["heads"], c["kv_heads"], c["dim"], c["vdim"]

    def proj(n, heads, size):
        return silu(causal_conv(h @ W[p + n].T, W[p + n + ".conv"])).reshape(T, heads, size)

    q = unit(proj("q", KH, dim)) * dim ** -0.5
    k = unit(proj("k", KH, dim))
    v = proj("v", H, vd)
    beta = sigmoid(h @ W[p + "b"].T)
    z = ((h @ W[p + "a1"].T) @ W[p + "a2"].T + W[p + "dt_bias"]).reshape(T, H, dim)
    g = np.exp(-np.exp(W[p + "A_log"])[:, None] * softplus(z))
    o, _ = delta_rule(q, k, v, g, beta)
    gate = sigmoid((h @ W[p + "g1"].T) @ W[p + "g2"].T)
    return (rms_norm(o, W[p + "norm"], eps).reshape(T, -1) * gate) @ W[p + "o"].T


def feed_forward(n, W, p):
    return (gelu_tanh(n @ W[p + "gate"].T) * (n @ W[p + "up"].T)) @ W[p + "down"].T


def layer(x, W, i, cfg):
    p, spec, eps = "l%d." % i, cfg["layers"][i], cfg["norm"]["eps"]
    h = layer_norm(x, W[p + "norm1"], eps)
    h = h + causal_conv(h, W[p + "canon1"])
    mx = spec["mixer"]
    x = x + mx["left_scale"] * left_mixer(h, W, p + "mix.left.", mx["left"]) \
          + mx["right_scale"] * right_mixer(h, W, p + "mix.right.", mx["right"], eps)
    if spec.get("mlp"):
        x = x + feed_forward(layer_norm(x, W[p + "norm2"], eps), W, p + "mlp.")
    return x


def run_order(cfg):
    """[(layer, adds the embedding output first)] with the loop written out"""
    n, lp = len(cfg["layers"]), cfg.get("loop")
    if not lp:
        return [(i, False) for i in range(n)]
    order = [(i, False) for i in range(lp["start"])]
    for t in range(lp["times"]):
        order += [(i, t > 0 and i == lp["start"]) for i in range(lp["start"], lp["stop"])]
    return order + [(i, False) for i in range(lp["stop"], n)]


def forward(tokens, W, cfg, trace=None):
    """logits [T, vocab]; the residual stream after every layer run is appended to `trace`"""
    W = {k: np.asarray(v, F) for k, v in W.items()}
    e = W["embed"][np.asarray(tokens)]
    x = e
    for i, again in run_order(cfg):
        x = layer(x + e if again else x, W, i, cfg)
        if trace is not None:
            trace.append(x)
    return softcap(layer_norm(x, W["final.norm"], cfg["norm"]["eps"]) @ W["embed"].T, cfg.get("logit_softcap"))


# ------------------------------------------------------------------ model folders
def to_bf16(x):
    """float32 values rounded to bfloat16 (nearest even), as float32"""
    b = np.asarray(x, np.float32).view(np.uint32)
    return ((b + 0x7FFF + ((b >> 16) & 1)) & 0xFFFF0000).astype(np.uint32).view(np.float32)


def write_model(folder, cfg, W):
    """config.json + model.safetensors (bfloat16) in `folder`"""
    import os

    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    head, blobs, at = {}, [], 0
    for name, a in W.items():
        raw = (np.ascontiguousarray(to_bf16(a)).view(np.uint32) >> 16).astype("<u2").tobytes()
        head[name] = {"dtype": "BF16", "shape": list(np.shape(a)), "data_offsets": [at, at + len(raw)]}
        blobs.append(raw)
        at += len(raw)
    h = json.dumps(head).encode()
    with open(os.path.join(folder, "model.safetensors"), "wb") as f:
        f.write(struct.pack("<Q", len(h)) + h + b"".join(blobs))
    return folder


def read_model(folder):
    """(config, weights) of a folder"""
    import os

    with open(os.path.join(folder, "config.json")) as f:
        cfg = json.load(f)
    with open(os.path.join(folder, "model.safetensors"), "rb") as f:
        n = struct.unpack("<Q", f.read(8))[0]
        head = json.loads(f.read(n))
        data = f.read()
    W = {}
    for name, t in head.items():
        if name == "__metadata__":
            continue
        raw = data[t["data_offsets"][0]:t["data_offsets"][1]]
        if t["dtype"] == "BF16":
            a = (np.frombuffer(raw, "<u2").astype(np.uint32) << 16).view(np.float32)
        else:
            a = np.frombuffer(raw, {"F32": "<f4", "I32": "<i4"}[t["dtype"]])
        W[name] = a.reshape(t["shape"])
    return cfg, W
