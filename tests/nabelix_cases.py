"""Small configurations and random weights for the Nabelix tests."""

import copy

import numpy as np

import nabelix_plain as P


def layer(left=None, right=None, ff=48, left_scale=0.8, right_scale=1.3):
    lf = dict(heads=4, kv_heads=2, dim=32, vdim=48, scale=0.21, mask=dict(size=24, keep_first=3))
    rt = dict(heads=4, kv_heads=2, dim=32, vdim=24, conv=3)
    lf.update(left or {})
    rt.update(right or {})
    return dict(type="parallel", mixer=dict(left=lf, right=rt, left_scale=left_scale, right_scale=right_scale),
                mlp=dict(kind="dense", ff=ff) if ff else None)


def config(layers, width=96, vocab=160, taps=3, eps=1e-5, softcap=9.0, loop=None):
    c = dict(architecture="Nabelix", width=width, vocab=vocab, layers=copy.deepcopy(layers), norm=dict(eps=eps), canon=dict(taps=taps))
    if softcap:
        c["logit_softcap"] = softcap
    if loop:
        c["loop"] = dict(start=loop[0], stop=loop[1], times=loop[2])
    return c


def mask(size, keep):
    return dict(size=size, keep_first=keep)


# sizes that are not multiples of anything, sizes above a tile, switches in both positions
CONFIGS = {
    "plain": config([layer(), layer(), layer()], loop=(1, 3, 2)),
    "odd": config([layer(dict(heads=5, kv_heads=5, dim=20, vdim=36, scale=0.3, mask=mask(17, 1)),
                         dict(heads=3, kv_heads=1, dim=21, vdim=19, conv=5), ff=37),
                   layer(dict(heads=3, kv_heads=1, dim=24, vdim=8, mask=mask(9, 4)),
                         dict(heads=2, kv_heads=2, dim=8, vdim=33, conv=2), ff=23)], width=52, vocab=131, taps=2, loop=(0, 1, 3)),
    "wide": config([layer(dict(heads=2, kv_heads=1, dim=160, vdim=208, scale=0.07, mask=mask(70, 66)),
                          dict(heads=3, kv_heads=3, dim=130, vdim=72, conv=4), ff=200)], width=136, vocab=300, taps=4),
    "big_heads": config([layer(dict(heads=2, kv_heads=2, dim=264, vdim=272, scale=0.05, mask=mask(33, 2)),
                               dict(heads=1, kv_heads=1, dim=256, vdim=300, conv=4), ff=64)], width=64, vocab=96, taps=5, softcap=0),
    "no_kept": config([layer(dict(mask=mask(12, 0)), ff=0), layer(dict(mask=mask(1, 2)), dict(heads=6, kv_heads=2), ff=64)], taps=6,
                      softcap=0, loop=(1, 2, 2)),
    "one_tap": config([layer(dict(heads=8, kv_heads=1, dim=64, vdim=64, mask=mask(40, 50)), dict(conv=1, dim=64, vdim=64)),
                       layer(dict(heads=1, kv_heads=1), dict(heads=1, kv_heads=1))], taps=1, width=100, vocab=77, loop=(0, 2, 2)),
    # the shape of a real layer's heads
    "real_heads": config([layer(dict(heads=4, kv_heads=2, dim=128, vdim=128, scale=0.09, mask=mask(150, 5)),
                                dict(heads=2, kv_heads=1, dim=128, vdim=128, conv=4), ff=256)], width=256, vocab=512, taps=4),
}


def weights(cfg, seed, rank=20, gain=1.0):
    g = np.random.default_rng(seed)
    D = cfg["width"]

    def lin(n, k, s=1.0):
        return g.standard_normal((n, k)) * (gain * s / np.sqrt(k))

    W = {"embed": g.standard_normal((cfg["vocab"], D)) * 1.5}
    for i, sp in enumerate(cfg["layers"]):
        p, lf, rt = "l%d." % i, sp["mixer"]["left"], sp["mixer"]["right"]
        W[p + "norm1"] = 1.0 + 0.2 * g.standard_normal(D)
        W[p + "canon1"] = g.standard_normal((D, cfg["canon"]["taps"])) * 0.4
        m = p + "mix.left."
        W[m + "q"] = lin(lf["heads"] * lf["dim"], D, 1.2)
        W[m + "k"] = lin(lf["kv_heads"] * lf["dim"], D, 1.2)
        W[m + "v"] = lin(lf["kv_heads"] * lf["vdim"], D)
        W[m + "r1"] = g.uniform(0.2, 1.5, lf["heads"])
        W[m + "r2"] = g.uniform(0.05, 0.8, lf["heads"])
        W[m + "g"] = lin(lf["heads"] * lf["vdim"], D)
        W[m + "o"] = lin(D, lf["heads"] * lf["vdim"])
        m = p + "mix.right."
        kc, vc = rt["kv_heads"] * rt["dim"], rt["heads"] * rt["vdim"]
        for n, c in (("q", kc), ("k", kc), ("v", vc)):
            W[m + n] = lin(c, D, 1.5)
            W[m + n + ".conv"] = g.standard_normal((c, rt["conv"])) * 0.6
        W[m + "b"] = lin(rt["heads"], D)
        W[m + "A_log"] = g.uniform(-3.0, 0.5, rt["heads"])
        W[m + "norm"] = 1.0 + 0.2 * g.standard_normal(rt["vdim"])
        W[m + "a1"] = lin(rank, D)
        W[m + "a2"] = lin(rt["heads"] * rt["dim"], rank)
        W[m + "dt_bias"] = g.uniform(-3.0, 0.5, rt["heads"] * rt["dim"])
        W[m + "g1"] = lin(rank + 3, D)
        W[m + "g2"] = lin(vc, rank + 3)
        W[m + "o"] = lin(D, vc)
        if sp["mlp"]:
            W[p + "norm2"] = 1.0 + 0.2 * g.standard_normal(D)
            W[p + "mlp.gate"] = lin(sp["mlp"]["ff"], D)
            W[p + "mlp.up"] = lin(sp["mlp"]["ff"], D)
            W[p + "mlp.down"] = lin(D, sp["mlp"]["ff"])
    W["final.norm"] = 1.0 + 0.2 * g.standard_normal(D)
    return {k: P.to_bf16(v) for k, v in W.items()}


def tokens(cfg, n, seed):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], n).astype(np.int32)


# ------------------------------------------------------------------ a model in which one key decides
# Token KEY's key and token QUERY's query point the same way (strongly); everybody else's are nearly zero, and the
# distance bias is small. At a QUERY position the attention either finds a KEY among the visible positions or is
# spread evenly, so whether one certain position is visible decides the output.
KEY, QUERY = 1, 2


def beacon(window, keep, seed=5, **kw):
    cfg = config([layer(dict(mask=mask(window, keep), heads=2, kv_heads=1, dim=32, vdim=32, scale=1.0), ff=0, right_scale=0.05)],
                 taps=2, softcap=0, **kw)
    W = weights(cfg, seed)
    D = cfg["width"]
    e, p = np.array(W["embed"]), "l0."
    e[:, :2] = 0.0
    e[KEY, 0] = e[QUERY, 1] = 12.0
    W["embed"] = e
    W[p + "canon1"] = np.zeros_like(W[p + "canon1"])
    W[p + "norm1"] = np.ones(D)
    q, k = 0.02 * np.array(W[p + "mix.left.q"]), 0.02 * np.array(W[p + "mix.left.k"])
    q[::32, 1] = 3.0
    k[::32, 0] = 3.0
    W[p + "mix.left.q"], W[p + "mix.left.k"] = q, k
    W[p + "mix.left.r1"] = np.full(2, 0.05)
    v = np.array(W[p + "mix.left.v"])
    v[:, 0] = 4.0 * np.random.default_rng(seed).standard_normal(v.shape[0])
    W[p + "mix.left.v"] = v
    return cfg, {k_: P.to_bf16(x) for k_, x in W.items()}
