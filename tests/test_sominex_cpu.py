"""Sominex without a GPU: the plain implementation's mechanisms against independent statements of them, the chunked form
of the recurrences that the kernels use against the token-by-token rules, and what opening a model folder refuses."""

import json

import numpy as np
import pytest

import nabelix_plain as F
import sominex_cases as C
import sominex_plain as P


def test_visible_tokens_and_blocks():
    see = P.visible(30, 7, 4)
    tok = [j for j in range(30) if see[20, j]]
    blk = [b for b in range(7) if see[20, 30 + b]]
    assert tok == list(range(14, 21)) and blk == [0, 1, 2]  # block 3 is 12 .. 15: 15 is still in the window
    assert [b for b in range(7) if see[22, 30 + b]] == [0, 1, 2, 3]
    assert not see[6, 30:].any() and [b for b in range(7) if see[10, 30 + b]] == [0]
    assert P.visible(9, 3).shape == (9, 9)


def test_attention_shares_one_softmax_between_tokens_and_block_means():
    g = np.random.default_rng(0)
    q, k, v = g.standard_normal((12, 4, 5)), g.standard_normal((12, 2, 5)), g.standard_normal((12, 2, 3))
    o = P.attention(q, k, v, 0.3, 3, 2)
    i, h = 9, 3
    keys = [k[0:2, 1].mean(0), k[2:4, 1].mean(0), k[4:6, 1].mean(0)] + [k[j, 1] for j in (7, 8, 9)]  # token 6: neither
    vals = [v[0:2, 1].mean(0), v[2:4, 1].mean(0), v[4:6, 1].mean(0)] + [v[j, 1] for j in (7, 8, 9)]
    w = np.exp([0.3 * (q[i, h] @ kk) for kk in keys])
    assert np.allclose(o[i, h], sum(a * b for a, b in zip(w / w.sum(), vals)))


def test_rotation_depends_on_the_distance_only():
    g = np.random.default_rng(1)
    u, w = g.standard_normal(8), g.standard_normal(8)
    rot = dict(base=100.0, dims=6)
    x, y = P.rotate(np.tile(u, (9, 1, 1)), rot), P.rotate(np.tile(w, (9, 1, 1)), rot)
    assert np.isclose(x[7, 0] @ y[4, 0], x[5, 0] @ y[2, 0]) and np.allclose(x[3, 0, 6:], u[6:]) and np.allclose(x[0, 0], u)
    c, s = np.cos(3 * 100.0 ** (-2 / 6)), np.sin(3 * 100.0 ** (-2 / 6))  # pair 1 (dimensions 1 and 4) at position 3
    assert np.isclose(x[3, 0, 1], u[1] * c - u[4] * s) and np.isclose(x[3, 0, 4], u[4] * c + u[1] * s)


def test_yarn_keeps_fast_pairs_and_stretches_slow_ones():
    rot = dict(base=10000.0, dims=64, scaling=dict(factor=4.0, original=1000, fast=32.0, slow=1.0))
    f, m = P.rope_frequencies(rot)
    plain, one = P.rope_frequencies(dict(base=10000.0, dims=64))
    turns = 1000 * plain / (2 * np.pi)  # over the original context
    assert np.allclose(f[turns > 60], plain[turns > 60]) and np.allclose(f[turns < 0.5], plain[turns < 0.5] / 4)
    assert (np.diff(f / plain) <= 1e-12).all() and np.isclose(m, 0.1 * np.log(4) + 1) and one == 1.0


def test_token_shift_and_convolution():
    g = np.random.default_rng(2)
    h, s = g.standard_normal((5, 3)), g.uniform(0, 1, 3)
    y = P.token_shift(h, s)
    assert np.allclose(y[3], h[3] + (h[2] - h[3]) * s) and np.allclose(y[0], (1 - s) * h[0])
    w, b = g.standard_normal((3, 2)), g.standard_normal(3)
    z = P.conv_silu(h, w, b)
    a = w[:, 0] * h[1] + w[:, 1] * h[2] + b
    assert np.allclose(z[2], a / (1 + np.exp(-a)))


def test_mlstm_is_attention_with_accumulated_gates():
    """the running maximum cancels: o_t = sum_s d_ts (q_t.k_s) v_s / max(|sum_s d_ts q_t.k_s|, 1), d_ts = exp(i_s + f_(s+1) + .. + f_t)"""
    g = np.random.default_rng(3)
    T, dim = 9, 4
    q, k, v = g.standard_normal((T, 1, dim)), g.standard_normal((T, 1, dim)), g.standard_normal((T, 1, 3))
    i, f = g.uniform(-2, 2, (T, 1)), P.logsigmoid(g.uniform(-2, 4, (T, 1)))
    o = P.mlstm(q, k, v, i, f)
    for t in range(T):
        d = np.array([np.exp(i[s, 0] + f[s + 1:t + 1, 0].sum()) * (q[t, 0] @ k[s, 0]) for s in range(t + 1)])
        assert np.allclose(o[t, 0], d @ v[:t + 1, 0] / max(abs(d.sum()), 1.0), rtol=1e-4)


def test_scan_of_the_running_maximum():
    """(F1, M1)(F2, M2) = (F1 + F2, max(M1 + F2, M2)) is associative and gives m_t = max(f + m, i) from any start"""
    g = np.random.default_rng(4)
    f, i = -g.uniform(0, 4, 12), g.uniform(-9, 3, 12)

    def join(a, b):
        return a[0] + b[0], max(a[1] + b[0], b[1])

    m, m0, left = 0.7, 0.7, (0.0, -np.inf)
    for t in range(12):
        m = max(f[t] + m, i[t])
        left = join(left, (f[t], i[t]))
        right = (f[t], i[t])
        for s in range(t - 1, -1, -1):
            right = join((f[s], i[s]), right)
        assert np.allclose(left, right) and np.isclose(m, max(m0 + left[0], left[1]))


@pytest.mark.parametrize("n", [1, 7, 128])
def test_chunked_form_of_the_recurrence(n):
    """o = exp(c_t) q_t S0 + sum exp(c_t - c_s) b_s (q_t.k_s) v_s and S1 = exp(c_n) S0 + sum ..., with c in pairs of floats: strong
    decays before weak ones included"""
    g = np.random.default_rng(n)
    N, vd = 6, 5
    k, q, v, b = g.standard_normal((n, N)), g.standard_normal((n, N)), g.standard_normal((n, vd)), g.uniform(0, 2, n)
    la = -np.exp(g.uniform(-7, 6, n))  # decays down to exp(-400)
    S = S0 = g.standard_normal((N, vd))
    want = []
    for t in range(n):
        S = np.exp(la[t]) * S + b[t] * np.outer(k[t], v[t])
        want.append(S.T @ q[t])
    c = np.cumsum(la)
    hi = c.astype(np.float32)
    lo = (c - hi).astype(np.float32)
    d = (hi[:, None] - hi[None, :]).astype(np.float32) + (lo[:, None] - lo[None, :]).astype(np.float32)
    w = np.where(np.tril(np.ones((n, n), bool)), np.exp(np.minimum(d, 0).astype(np.float64)), 0.0)
    o = np.exp(c)[:, None] * (q @ S0) + (w * b * (q @ k.T)) @ v
    assert np.allclose(o, want, rtol=2e-5, atol=2e-6)
    S1 = np.exp(c[-1]) * S0 + k.T @ ((w[-1] * b)[:, None] * v)
    assert np.allclose(S1, S, rtol=2e-5, atol=2e-6)


def test_router_takes_the_largest_scores():
    z = np.array([[0.0, 2.0, 1.0, 2.0, -1.0]])
    e, w = P.route(z, 3, 2.0)
    s = np.exp(z[0]) / np.exp(z[0]).sum()
    assert list(e[0]) == [1, 3, 2] and np.allclose(w[0], 2.0 * s[[1, 3, 2]]) and w.sum() < 2.0


def test_clamped_gate():
    g, u = np.array([0.5, 9.0, -9.0]), np.array([-5.0, 0.3, 5.0])
    y = P.clamped_glu(g, u, 2.0)
    assert np.allclose(y, [0.5 / (1 + np.exp(-0.851)) * -1.0, 2.0 / (1 + np.exp(-3.404)) * 1.3, -9.0 / (1 + np.exp(15.318)) * 3.0])


def test_model_folder_round_trip(tmp_path):
    cfg = C.CONFIGS["odd"]
    W = C.weights(cfg, 1)
    c2, W2 = F.read_model(F.write_model(str(tmp_path), cfg, W))
    assert c2 == cfg and set(W2) == set(W) and all(np.array_equal(W[k], W2[k]) for k in W)


# ------------------------------------------------------------------ opening a folder
@pytest.mark.parametrize("path,value,word", [
    (("layers", 0, "type"), "other", "other"), (("layers", 0, "mixer", "dim"), None, "dim"), (("layers", 0, "mixer", "heads"), 3, "kv_heads"),
    (("layers", 0, "mixer", "mask", "size"), 0, "size"), (("layers", 0, "mixer", "rot", "dims"), 7, "rot"),
    (("layers", 0, "mixer", "rot", "dims"), 40, "rot"), (("layers", 0, "mixer", "rot", "scaling", "factor"), 0, "scaling"),
    (("layers", 1, "mixer", "groups"), 3, "groups"), (("layers", 1, "mixer", "norm_groups"), 7, "norm_groups"), (("layers", 1, "mixer", "conv"), 2.5, "conv"),
    (("layers", 1, "mlp", "router", "top"), 7, "top"), (("layers", 1, "mlp", "expert"), None, "expert"), (("layers", 1, "mlp", "kind"), "sparse", "sparse"),
    (("layers", 0, "mlp", "limit"), None, "limit"), (("layers", 2, "mixer", "gate_cap"), 0, "gate_cap"), (("embedding",), None, "embedding"),
    (("norm",), None, "norm"), (("width",), "wide", "width"), (("layers",), [], "layers")])
def test_bad_configs_are_refused(capi, tmp_path, path, value, word):
    cfg = json.loads(json.dumps(C.CONFIGS["plain"]))
    at = cfg
    for k in path[:-1]:
        at = at[k]
    at[path[-1]] = value
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    with pytest.raises(capi.TgError) as e:
        capi.Model.open(str(tmp_path)).close()
    assert e.value.code in (capi.TG_EINVAL, capi.TG_ESHAPE) and word in str(e.value)


def test_no_cpu_fallback(capi, tmp_path):
    if capi.device_count() > 0:
        return
    F.write_model(str(tmp_path), C.CONFIGS["plain"], C.weights(C.CONFIGS["plain"], 0))
    with pytest.raises(capi.TgError) as e:
        capi.Model.open(str(tmp_path)).close()
    assert e.value.code == capi.TG_ENODEVICE


def test_random_models_of_the_benchmark_have_every_tensor(synth, tmp_path):
    cfg = synth.sominex_config("270m")
    cfg["layers"], cfg["vocab"], cfg["width"] = cfg["layers"][:3], 64, 64
    for sp in cfg["layers"]:
        if sp["type"] == "mamba2":
            sp["mixer"]["heads"] = 2
    c2, W = F.read_model(synth.write_random_layered(str(tmp_path), cfg))
    want = C.weights(c2, 0)
    assert {k: v.shape for k, v in W.items()} == {k: v.shape for k, v in want.items()}
    assert np.isfinite(P.forward([1, 2, 3], W, c2)).all()
