"""Small configurations and random weights for the Sominex tests."""

import copy

import numpy as np

from nabelix_plain import to_bf16

YARN = dict(factor=5.0, original=300, fast=20.0, slow=1.5)


def dense(ff=48, limit=1.7):
    return dict(kind="dense", ff=ff, limit=limit)


def moe(experts=6, top=2, ff=24, shared=40, scale=1.5):
    c = dict(kind="moe", expert=dict(ff=ff), router=dict(experts=experts, top=top, scale=scale))
    if shared:
        c["shared"] = dict(ff=shared)
    return c


def attn(mlp=None, size=20, pool=6, base=10000.0, rot=24, scaling=YARN, **kw):
    mx = dict(heads=4, kv_heads=2, dim=32, vdim=48, scale=0.21, mask=dict(size=size))
    if pool:
        mx["mask"]["pool"] = pool
    mx.update(kw)
    if rot:
        mx["rot"] = dict(base=base, dims=rot)
        if scaling:
            mx["rot"]["scaling"] = dict(scaling)
    return dict(type="attention", mixer=mx, mlp=mlp)


def mamba(mlp=None, **kw):
    mx = dict(heads=4, vdim=24, state=40, groups=2, conv=4, norm_groups=3)
    mx.update(kw)
    return dict(type="mamba2", mixer=mx, mlp=mlp)


def mlstm(mlp=None, **kw):
    mx = dict(heads=3, dim=40, vdim=24, gate_cap=7.0)
    mx.update(kw)
    return dict(type="mlstm", mixer=mx, mlp=mlp)


def config(layers, width=96, vocab=160, eps=1e-5, scale=2.0):
    return dict(architecture="Sominex", width=width, vocab=vocab, layers=copy.deepcopy(layers), norm=dict(eps=eps), embedding=dict(scale=scale))


# sizes that are not multiples of anything, sizes above a tile, every kind of layer with every feed-forward
CONFIGS = {
    "plain": config([attn(dense()), mamba(moe()), mlstm(dense(72, 0.9)), mlstm(moe(5, 3, 16, 0))]),
    "order": config([mlstm(moe()), attn(moe(9, 4, 20, 24), size=33, pool=5), mamba(dense()), attn(None, size=9, pool=4, scaling=None)], width=100, vocab=77),
    "odd": config([mamba(dense(37), heads=5, vdim=19, state=21, groups=1, conv=2, norm_groups=5),
                   mlstm(moe(3, 3, 13, 7, 0.7), heads=5, dim=21, vdim=33),
                   attn(moe(4, 1, 9, 11, 3.0), heads=3, kv_heads=1, dim=21, vdim=19, rot=10, size=17, pool=3),
                   mamba(None, heads=3, vdim=8, state=7, groups=3, conv=1, norm_groups=1)], width=52, vocab=131, scale=1.0),
    "wide": config([attn(dense(200), heads=2, kv_heads=1, dim=160, vdim=208, scale=0.07, size=70, pool=16, rot=160),
                    mamba(moe(40, 5, 48, 72), heads=3, vdim=136, state=144, groups=1, norm_groups=2, conv=5),
                    mlstm(dense(130), heads=2, dim=136, vdim=200)], width=136, vocab=300),
    "big_heads": config([attn(dense(64), heads=2, kv_heads=2, dim=264, vdim=272, scale=0.05, size=33, pool=2, rot=128),
                         mlstm(None, heads=1, dim=272, vdim=300), mamba(None, heads=2, vdim=40, state=300, groups=2, norm_groups=2)], width=64, vocab=96),
    "no_pool": config([attn(dense(), pool=0, size=12, rot=0), attn(moe(), size=1, pool=1, rot=32), mlstm(dense(), heads=1, gate_cap=2.0),
                       attn(None, heads=8, kv_heads=8, size=64, pool=64)]),
    # the shape of real layers' heads
    "real_heads": config([attn(dense(256), heads=4, kv_heads=2, dim=128, vdim=128, scale=0.09, size=150, pool=16, rot=128),
                          mamba(moe(16, 4, 64, 128), heads=8, vdim=64, state=128, groups=2, norm_groups=2),
                          mlstm(dense(256), heads=2, dim=128, vdim=256, gate_cap=15.0)], width=256, vocab=512),
}


def weights(cfg, seed, gain=1.0):
    g = np.random.default_rng(seed)
    D = cfg["width"]

    def lin(n, k, s=1.0):
        return g.standard_normal((n, k)) * (gain * s / np.sqrt(k))

    def glu(W, p, ff):
        W[p + "gate"], W[p + "up"], W[p + "down"] = lin(ff, D), lin(ff, D), lin(D, ff)

    W = {"embed": g.standard_normal((cfg["vocab"], D))}
    for i, sp in enumerate(cfg["layers"]):
        p, m, c = "l%d." % i, "l%d.mix." % i, sp["mixer"]
        W[p + "norm1"] = 1.0 + 0.2 * g.standard_normal(D)
        W[p + "shift"] = g.uniform(-0.2, 0.9, D)
        if sp["type"] == "attention":
            W[m + "q"] = lin(c["heads"] * c["dim"], D, 1.2)
            W[m + "k"] = lin(c["kv_heads"] * c["dim"], D, 1.2)
            W[m + "v"] = lin(c["kv_heads"] * c["vdim"], D, 0.7)
            W[m + "o"] = lin(D, c["heads"] * c["vdim"])
        elif sp["type"] == "mamba2":
            inner, ch = c["heads"] * c["vdim"], c["heads"] * c["vdim"] + 2 * c["groups"] * c["state"]
            W[m + "in"] = lin(inner + ch + c["heads"], D, 1.3)
            W[m + "conv"] = g.standard_normal((ch, c["conv"])) * 0.6
            W[m + "conv.b"] = g.standard_normal(ch) * 0.2
            W[m + "dt_bias"] = g.uniform(-3.0, 1.0, c["heads"])
            W[m + "A_log"] = g.uniform(-4.0, 2.5, c["heads"])
            W[m + "D"] = g.standard_normal(c["heads"])
            W[m + "norm"] = 1.0 + 0.2 * g.standard_normal(inner)
            W[m + "o"] = lin(D, inner)
        else:
            inner = c["heads"] * c["vdim"]
            for n, rows in (("q", c["heads"] * c["dim"]), ("k", c["heads"] * c["dim"]), ("v", inner), ("g", inner)):
                W[m + n] = lin(rows, D)
            W[m + "norm"] = 1.0 + 0.2 * g.standard_normal(inner)
            W[m + "i"], W[m + "f"] = lin(c["heads"], D, 2.0), lin(c["heads"], D, 2.0)
            W[m + "i.b"], W[m + "f.b"] = g.uniform(-3.0, 2.0, c["heads"]), g.uniform(0.0, 6.0, c["heads"])
            W[m + "o"] = lin(D, inner)
        ff = sp["mlp"]
        if ff and ff["kind"] == "dense":
            glu(W, p + "mlp.", ff["ff"])
        elif ff:
            W[p + "mlp.router"] = lin(ff["router"]["experts"], D, 5.0)  # (few close calls)
            for e in range(ff["router"]["experts"]):
                glu(W, p + "mlp.e%d." % e, ff["expert"]["ff"])
            if ff.get("shared"):
                glu(W, p + "mlp.shared.", ff["shared"]["ff"])
    W["final.norm"] = 1.0 + 0.2 * g.standard_normal(D)
    W["head"] = lin(cfg["vocab"], D)
    return {k: to_bf16(v) for k, v in W.items()}


def tokens(cfg, n, seed):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], n).astype(np.int32)


# ------------------------------------------------------------------ a model in which one key decides
# Token KEY's key and token QUERY's query point the same way (strongly enough for the mean of a block to stand out);
# everybody else's are nearly zero. At a QUERY position the attention either finds the KEY, itself or in a pooled block, or
# is spread evenly, so whether one certain position is visible decides the output.
KEY, QUERY = 1, 2


def beacon(window, pool, seed=5, **kw):
    cfg = config([attn(None, size=window, pool=pool, heads=2, kv_heads=1, dim=32, vdim=32, scale=0.4, rot=0)], **kw)
    W = weights(cfg, seed)
    e, m = np.array(W["embed"]), "l0.mix."
    e[:, :2] = 0.0
    e[KEY, 0] = e[QUERY, 1] = 12.0
    W["embed"] = e
    W["l0.shift"] = np.zeros_like(W["l0.shift"])
    W["l0.norm1"] = np.ones_like(W["l0.norm1"])
    q, k = 0.02 * np.array(W[m + "q"]), 0.02 * np.array(W[m + "k"])
    q[::32, 1] = k[::32, 0] = 3.0
    W[m + "q"], W[m + "k"] = q, k
    v = np.array(W[m + "v"])
    v[:, 0] = 4.0 * np.random.default_rng(seed).standard_normal(v.shape[0])
    W[m + "v"] = v
    W[m + "o"] = 4.0 * np.array(W[m + "o"])
    return cfg, {k_: to_bf16(x) for k_, x in W.items()}


def without_mixers(W, cfg):
    """the same weights with every mixer's output projection zero: what a layer adds is its feed-forward's"""
    W = dict(W)
    for i in range(len(cfg["layers"])):
        W["l%d.mix.o" % i] = np.zeros_like(W["l%d.mix.o" % i])
    return W
