"""Nabelix without a GPU: the plain implementation's mechanisms against independent statements of them, the block form
of the delta rule that the kernels use against the token-by-token rule, and what opening a model folder refuses."""

import json
import os
import subprocess
import sys

import numpy as np
import pytest

import nabelix_cases as N
import nabelix_plain as P

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


def test_window_with_kept_first_tokens():
    see = P.visible(12, 4, 2)
    assert [j for j in range(12) if see[9, j]] == [0, 1, 6, 7, 8, 9]
    assert [j for j in range(12) if see[4, j]] == [0, 1, 2, 3, 4]  # 1 = last position inside the window, 0 kept
    assert [j for j in range(12) if P.visible(12, 1, 0)[7, j]] == [7]


def test_attention_is_a_softmax_over_the_visible_keys():
    g = np.random.default_rng(0)
    q, k, v = g.standard_normal((7, 4, 5)), g.standard_normal((7, 2, 5)), g.standard_normal((7, 2, 3))
    r1, r2 = g.uniform(0.1, 1, 4), g.uniform(0.1, 1, 4)
    o = P.attention(q, k, v, 0.3, 3, 1, r1, r2)
    i, h = 6, 3
    js = [0, 4, 5, 6]
    s = np.array([0.3 * (q[i, h] @ k[j, 1]) - r1[h] * np.log(1 + r2[h] * (i - j)) for j in js])
    w = np.exp(s) / np.exp(s).sum()
    assert np.allclose(o[i, h], sum(a * v[j, 1] for a, j in zip(w, js)))


def test_causal_conv_is_a_dot_with_the_last_taps():
    g = np.random.default_rng(1)
    x, w = g.standard_normal((9, 4)), g.standard_normal((4, 3))
    y = P.causal_conv(x, w)
    assert np.allclose(y[5], w[:, 0] * x[3] + w[:, 1] * x[4] + w[:, 2] * x[5])
    assert np.allclose(y[0], w[:, 2] * x[0])


def test_delta_rule_overwrites_what_a_key_held():
    """no decay, beta = 1, orthonormal keys: the state maps each key to its last value"""
    k = np.eye(4)[[0, 1, 0, 2]][:, None]
    v = np.random.default_rng(2).standard_normal((4, 1, 3))
    o, S = P.delta_rule(k, k, v, np.ones((4, 1, 4)), np.ones((4, 1)))
    assert np.allclose(S[0][0], v[2, 0]) and np.allclose(S[0][1], v[1, 0]) and np.allclose(S[0][3], 0)
    assert np.allclose(o, v)  # the read-out sees the write of its own token


@pytest.mark.parametrize("n", [1, 5, 16])
def test_block_form_of_the_delta_rule(n):
    """u = T (V - Kt S0), S' = D S0 + sum (D / D_s) k_s u_s^T ... equals the token-by-token rule, strong decays included"""
    g = np.random.default_rng(n)
    dk, dv, n0 = 6, 5, 4
    k = P.unit(g.standard_normal((n0 + n, 1, dk)))
    q, v = g.standard_normal((n0 + n, 1, dk)), g.standard_normal((n0 + n, 1, dv))
    dec = np.exp(-np.exp(g.uniform(-4, 3.5, (n0 + n, 1, dk))))  # down to exp(-33)
    beta = g.uniform(0, 1, (n0 + n, 1))
    o, S = P.delta_rule(q, k, v, dec, beta)
    _, S0 = P.delta_rule(q[:n0], k[:n0], v[:n0], dec[:n0], beta[:n0])
    K, Q, V, G, b, S0 = k[n0:, 0], q[n0:, 0], v[n0:, 0], dec[n0:, 0], beta[n0:, 0], S0[0]

    def ratio(t, s):  # D_t / D_s as a product, s <= t
        return np.prod(G[s + 1:t + 1], axis=0)

    D = np.cumprod(G, axis=0)
    A = np.array([[K[t] @ (ratio(t, s) * K[s]) if s < t else 0.0 for s in range(n)] for t in range(n)])
    M = np.array([[Q[t] @ (ratio(t, s) * K[s]) if s <= t else 0.0 for s in range(n)] for t in range(n)])
    T = np.linalg.inv(np.eye(n) + b[:, None] * A) @ np.diag(b)
    u = T @ (V - (D * K) @ S0)
    assert np.allclose((D * Q) @ S0 + M @ u, o[n0:, 0])
    S1 = D[-1][:, None] * S0 + sum(np.outer(ratio(n - 1, s) * K[s], u[s]) for s in range(n))
    assert np.allclose(S1, S[0])


def test_loop_order():
    cfg = N.config([N.layer()] * 4, loop=(1, 3, 3))
    assert P.run_order(cfg) == [(0, False), (1, False), (2, False), (1, True), (2, False), (1, True), (2, False), (3, False)]
    assert P.run_order(N.config([N.layer()] * 2)) == [(0, False), (1, False)]


def test_model_folder_round_trip(tmp_path):
    cfg = N.CONFIGS["odd"]
    W = N.weights(cfg, 1)
    c2, W2 = P.read_model(P.write_model(str(tmp_path), cfg, W))
    assert c2 == cfg and set(W2) == set(W) and all(np.array_equal(W[k], W2[k]) for k in W)


# ------------------------------------------------------------------ opening a folder
def _open(capi, folder):
    with pytest.raises(capi.TgError) as e:
        capi.Model.open(str(folder)).close()
    return e.value


def test_bad_folders_are_refused(capi, tmp_path):
    assert _open(capi, tmp_path).code == capi.TG_EIO
    (tmp_path / "config.json").write_text("{\"architecture\": \"Nabelix\", ")
    assert _open(capi, tmp_path).code == capi.TG_EIO
    (tmp_path / "config.json").write_text("{}")
    assert _open(capi, tmp_path).code == capi.TG_EINVAL
    (tmp_path / "config.json").write_text("{\"architecture\": \"Nothing\"}")
    e = _open(capi, tmp_path)
    assert e.code == capi.TG_EINVAL and "Nothing" in str(e)
    cfg = json.loads(json.dumps(N.CONFIGS["plain"]))
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    assert _open(capi, tmp_path).code == capi.TG_EIO  # no weights


@pytest.mark.parametrize("path,value,word", [
    (("layers", 0, "type"), "other", "other"), (("layers", 0, "mixer", "left", "dim"), None, "dim"),
    (("layers", 0, "mixer", "left", "heads"), 3, "kv_heads"), (("layers", 0, "mixer", "right", "conv"), 2.5, "conv"),
    (("layers", 1, "mlp", "kind"), "sparse", "feed-forward"), (("loop", "stop"), 9, "loop"), (("norm",), None, "norm"),
    (("layers", 0, "mixer", "left", "mask", "size"), 0, "size"), (("width",), "wide", "width")])
def test_bad_configs_are_refused(capi, tmp_path, path, value, word):
    cfg = json.loads(json.dumps(N.CONFIGS["plain"]))
    at = cfg
    for k in path[:-1]:
        at = at[k]
    at[path[-1]] = value
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    e = _open(capi, tmp_path)
    assert e.code in (capi.TG_EINVAL, capi.TG_ESHAPE) and word in str(e)


def test_no_cpu_fallback(capi, tmp_path):
    if capi.device_count() > 0:
        return
    P.write_model(str(tmp_path), N.CONFIGS["plain"], N.weights(N.CONFIGS["plain"], 0))
    assert _open(capi, tmp_path).code == capi.TG_ENODEVICE
    r = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", "bfloat16",
                        "--out", str(tmp_path), "--max-tokens", "10"], input="", capture_output=True, text=True)
    assert r.returncode not in (0, 3) and "CUDA device" in r.stderr
