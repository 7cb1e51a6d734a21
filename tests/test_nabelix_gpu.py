"""Nabelix on the GPU against the plain implementation (nabelix_plain.py), through the library's own step, cache and
generation loop. float32 states must agree to rounding; bfloat16 states to the rounding of their activations.

The state's passes are kept small (TG_PASS_ROWS) where the point is the cache's ring, so that it wraps many times.
"""

import json
import os
import subprocess
import sys

import numpy as np
import pytest

import nabelix_cases as N
import nabelix_plain as P
from conftest import rel_l2

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
TOL = {"float32": 2e-5, "bfloat16": 3e-2}
DTYPES = ["float32", "bfloat16"]


@pytest.fixture(scope="module")
def folder(tmp_path_factory):
    made = {}

    def get(key, cfg=None, W=None):
        if key not in made:
            cfg = cfg or N.CONFIGS[key]
            W = N.weights(cfg, 3) if W is None else W
            made[key] = (P.write_model(str(tmp_path_factory.mktemp(key)), cfg, W), cfg, W)
        return made[key]

    return get


class Ref:
    """plain logits (and layer traces) of token lists, computed once"""
    cache = {}

    @classmethod
    def get(cls, key, cfg, W, toks):
        k = (key, tuple(int(t) for t in toks))
        if k not in cls.cache:
            tr = []
            cls.cache[k] = (P.forward(toks, W, cfg, tr), np.array(tr))
        return cls.cache[k]


def row_err(a, b):
    return np.linalg.norm(a - b, axis=-1) / np.maximum(np.linalg.norm(b, axis=-1), 1e-9)


def close(got, want, dtype, factor=1.0):
    e = row_err(np.asarray(got, np.float64), want)
    assert np.isfinite(got).all() and e.max() <= factor * TOL[dtype], (dtype, float(e.max()), np.unravel_index(e.argmax(), e.shape))


def replay(st, seq, toks, cuts, every=True):
    """the logits of all tokens, brought in portions of the given sizes (the rest in one)"""
    out, at, i = [], 0, 0
    while at < len(toks):
        n = min(cuts[i] if i < len(cuts) else len(toks), len(toks) - at)
        out.append(st.step([(seq, toks[at:at + n], list(range(n)))]))
        at += n
        i += 1
    return np.concatenate(out)


# ------------------------------------------------------------------ whole prompts, layer by layer
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("key", sorted(N.CONFIGS))
def test_prompt_matches_plain_layer_by_layer(capi, folder, key, dtype):
    path, cfg, W = folder(key)
    toks = N.tokens(cfg, 150, 1)
    want, tr = Ref.get(key, cfg, W, toks)
    m = capi.Model.open(path, dtype)
    st = m.state(1, 256)
    st.trace_enable()
    got = st.step([(0, toks, list(range(len(toks))))])
    t = st.trace()
    assert t.shape == tr.shape
    for i in range(len(tr)):
        close(t[i], tr[i], dtype)
    close(got, want, dtype)
    # and token by token: the decode kernels
    st.free_sequence(0)
    n = 40
    close(replay(st, 0, toks[:n], [1] * n), want[:n], dtype)
    st.close()
    m.close()


# ------------------------------------------------------------------ one mechanism at a time
def _only(part):
    """configurations whose layer output is one mechanism's"""
    left, right, ff = (1.0, 0.0, 0) if part in ("attention", "gate", "bias", "conv") else ((0.0, 1.0, 0) if part == "delta" else (0.0, 0.0, 80))
    cfg = N.config([N.layer(ff=ff, left_scale=left, right_scale=right)], taps=5 if part == "conv" else 2, softcap=0)
    W = N.weights(cfg, 17)
    if part != "conv":
        W["l0.canon1"] = np.zeros_like(W["l0.canon1"])
    if part in ("attention", "bias"):
        W["l0.mix.left.g"] = np.zeros_like(W["l0.mix.left.g"])  # every gate 1/2
    if part == "attention":
        W["l0.mix.left.r1"] = np.zeros_like(W["l0.mix.left.r1"])
    if part == "bias":
        W["l0.mix.left.q"] = np.zeros_like(W["l0.mix.left.q"])  # the distance alone weighs the keys
        W["l0.mix.left.r1"] = P.to_bf16(np.full_like(W["l0.mix.left.r1"], 2.0))
    return cfg, W


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("part", ["attention", "bias", "gate", "conv", "delta", "feed_forward"])
def test_mechanism_alone(capi, folder, part, dtype):
    cfg, W = _only(part)
    path, _, _ = folder("only_" + part, cfg, W)
    toks = N.tokens(cfg, 90, 2)
    tr = []
    P.forward(toks, W, cfg, tr)
    x0 = W["embed"][toks]
    m = capi.Model.open(path, dtype)
    st = m.state(1, 128)
    st.trace_enable()
    for cuts in ([90], [70] + [1] * 20):
        got, at = [], 0
        for n in cuts:
            st.step([(0, toks[at:at + n], [])])
            got.append(st.trace()[0])
            at += n
        # what the layer added to the stream is the mechanism's own output
        d, w = np.concatenate(got) - x0, tr[0] - x0
        assert rel_l2(d, w) <= TOL[dtype], rel_l2(d, w)
        st.free_sequence(0)
    st.close()
    m.close()


# ------------------------------------------------------------------ portions, decoding, the ring
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("cuts", [[2] * 400, [3, 1, 5, 2, 7, 1, 1, 13, 2, 64, 65, 63, 16, 17, 15, 128], [1, 127, 2, 129], [700]])
@pytest.mark.parametrize("key", ["plain", "odd", "real_heads"])
def test_portions(capi, folder, monkeypatch, key, cuts, dtype):
    monkeypatch.setenv("TG_PASS_ROWS", "128")
    path, cfg, W = folder(key)
    toks = N.tokens(cfg, 330, 4)
    want, _ = Ref.get(key, cfg, W, toks)
    m = capi.Model.open(path, dtype)
    st = m.state(1, 400)
    close(replay(st, 0, toks, cuts), want, dtype)
    assert st.position(0) == len(toks)
    st.close()
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding(capi, folder, monkeypatch, dtype):
    """the ring (window 24 + 128 rows -> 192 slots) wraps more than once in decoding alone"""
    monkeypatch.setenv("TG_PASS_ROWS", "128")
    path, cfg, W = folder("plain")
    toks = N.tokens(cfg, 520, 6)
    want, _ = Ref.get("plain", cfg, W, toks)
    m = capi.Model.open(path, dtype)
    st = m.state(1, 1000)
    close(replay(st, 0, toks, [30] + [1] * 490), want, dtype)
    st.close()
    m.close()


# ------------------------------------------------------------------ batches
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("B", [3, 7])
def test_unequal_requests_in_one_batch(capi, folder, monkeypatch, B, dtype):
    """prompts of different lengths, portions beside single tokens, slots freed and used again; every request equals
    the plain result (and so itself alone)"""
    monkeypatch.setenv("TG_PASS_ROWS", "128")
    path, cfg, W = folder("plain")
    g = np.random.default_rng(B)
    m = capi.Model.open(path, dtype)
    st = m.state(B, 400)
    todo = [N.tokens(cfg, int(n), 50 + i) for i, n in enumerate([70, 5, 130, 1, 33, 260, 2, 90, 17, 64, 40][:B + 4])]
    slot, at, got = {}, {}, {}
    nxt = 0
    while nxt < len(todo) or slot:
        for b in range(B):
            if b not in slot and nxt < len(todo):
                slot[b], at[nxt], got[nxt] = nxt, 0, []
                nxt += 1
        entries = []
        for b, r in slot.items():
            if g.random() < 0.25 and len(slot) > 1:
                continue  # this request waits
            n = min(int(g.choice([1, 1, 2, 9, 40, 150])), len(todo[r]) - at[r])
            entries.append((b, todo[r][at[r]:at[r] + n], list(range(n)), r))
        if not entries:
            continue
        order = g.permutation(len(entries))
        entries = [entries[i] for i in order]
        out, k = st.step([e[:3] for e in entries]), 0
        for b, t, w, r in entries:
            got[r].append(out[k:k + len(w)])
            k += len(w)
            at[r] += len(t)
            if at[r] == len(todo[r]):
                st.free_sequence(b)
                del slot[b]
    for r, toks in enumerate(todo):
        close(np.concatenate(got[r]), Ref.get("plain", cfg, W, toks)[0], dtype)
    st.close()
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_lockstep_decode_in_batches(capi, folder, dtype):
    """tg_prefill + tg_decode: few rows (matrix-vector pipeline) and more (tensor cores), several prompts at once"""
    path, cfg, W = folder("plain")
    m = capi.Model.open(path, dtype)
    for B in (1, 2, 3, 4, 5, 9):
        toks = np.stack([N.tokens(cfg, 48, 200 + b) for b in range(B)])
        st = m.state(B, 64)
        want = np.stack([Ref.get("plain", cfg, W, t)[0] for t in toks])
        close(st.prefill(toks[:, :40]), want[:, 39], dtype)
        for i in range(40, 48):
            close(st.decode(toks[:, i]), want[:, i], dtype)
        assert all(st.position(b) == 48 for b in range(B))
        st.reset()
        close(st.prefill(toks[:, :1]), want[:, 0], dtype)
        st.close()
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_large_batch_of_equal_requests(capi, folder, dtype):
    """150 sequences, several pieces of keys per CTA: every row has the same bits, and they are the plain result"""
    path, cfg, W = folder("real_heads")
    toks, B = N.tokens(cfg, 190, 31), 150
    want = Ref.get("real_heads", cfg, W, toks)[0]
    m = capi.Model.open(path, dtype)
    st = m.state(B, 200)
    for b0 in range(0, B, 50):
        st.step([(b, toks[:150], []) for b in range(b0, b0 + 50)])
    for i in range(150, 190):
        got = st.decode(np.full(B, toks[i]))
        assert np.array_equal(got, np.broadcast_to(got[0], got.shape)), (i, np.nonzero((got != got[0]).any(1))[0])
        close(got[0], want[i], dtype)
    st.close()
    m.close()


# ------------------------------------------------------------------ edges
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("window,keep", [(24, 3), (64, 1), (65, 64), (130, 70), (7, 0)])
def test_keys_just_inside_and_outside(capi, folder, monkeypatch, window, keep, dtype):
    monkeypatch.setenv("TG_PASS_ROWS", "128")
    cfg, W = N.beacon(window, keep)
    path, _, _ = folder("beacon_%d_%d" % (window, keep), cfg, W)
    m = capi.Model.open(path, dtype)
    st = m.state(1, 600)
    T = 300
    base = np.random.default_rng(8).integers(3, cfg["vocab"], T).astype(np.int32)
    shows = 0
    for q in (window + keep + 3, 191, 192, 193, 255, 299):
        cases = [q - window + 1, q - window, q - window - 1, keep - 1, keep, 0]  # inside, outside; last kept, first not kept
        for k in sorted({c for c in cases if 0 <= c < q}):
            toks = base.copy()
            toks[k], toks[q] = N.KEY, N.QUERY
            want = P.forward(toks[:q + 1], W, cfg)[q]
            # the case tells: an oracle whose edges are off by one at this key gives something else
            seen = bool(P.visible(q + 1, window, keep)[q, k])
            flip = json.loads(json.dumps(cfg))
            mk = flip["layers"][0]["mixer"]["left"]["mask"]
            if q - k == window or q - k == window - 1:
                mk["size"] += 1 if not seen else -1
            else:
                mk["keep_first"] = k + 1 if not seen else k
            other = P.forward(toks[:q + 1], W, flip)[q] if mk["size"] > 0 else want
            if bool(P.visible(q + 1, mk["size"], mk["keep_first"])[q, k]) != seen:
                shows += 1
                assert row_err(other, want) > 0.15
            # in a prompt; then with the query decoded alone
            for cuts in ([q + 1], [q, 1], [q - 1, 2]):
                st.free_sequence(0)
                got = replay(st, 0, toks[:q + 1], cuts)[q]
                assert row_err(got, want) <= 2 * TOL[dtype], (q, k, cuts, row_err(got, want))
    assert shows >= 6
    st.close()
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_first_tokens(capi, folder, dtype):
    """prompts of 1 .. 9 tokens, in one step and cut after every place"""
    path, cfg, W = folder("odd")
    m = capi.Model.open(path, dtype)
    st = m.state(1, 16)
    toks = N.tokens(cfg, 9, 11)
    want, _ = Ref.get("odd", cfg, W, toks)
    for n in range(1, 10):
        for c in range(0, n):
            st.free_sequence(0)
            close(replay(st, 0, toks[:n], [c, n - c] if c else [n]), want[:n], dtype)
    st.close()
    m.close()


def test_freed_slots_leave_nothing_behind(capi, folder):
    """the same request in a fresh state and in one whose slots have held others: the same bits"""
    path, cfg, W = folder("plain")
    m = capi.Model.open(path, "bfloat16")
    a, b = m.state(2, 300), m.state(2, 300)
    toks, other = N.tokens(cfg, 100, 21), N.tokens(cfg, 260, 22)
    b.step([(0, other, []), (1, other[:50], [])])
    b.step([(0, other[:30], [])])
    b.free_sequence(0)
    b.free_sequence(1)
    for st in (a, b):
        st.last = [replay(st, 1, toks, [60, 3, 1, 1, 20])]
        st.free_sequence(1)
    assert np.array_equal(a.last[0], b.last[0])
    a.close()
    b.close()
    m.close()


# ------------------------------------------------------------------ generation
def test_greedy_generation_matches_plain(capi, folder):
    path, cfg, W = folder("plain")
    m = capi.Model.open(path, "float32")
    for B in (1, 5):
        prompts = np.stack([N.tokens(cfg, 20, 300 + b) for b in range(B)])
        st = m.state(B, 64)
        st.prefill(prompts, want_logits=False)
        first = st.sample_argmax()
        more = st.generate(first, 24)
        toks = np.concatenate([first[None], more]).T
        for b in range(B):
            seq = list(prompts[b])
            for t in toks[b]:
                lg = P.forward(seq, W, cfg)[-1]
                top = np.sort(lg)[-2:]
                assert int(t) == int(lg.argmax()) or top[1] - top[0] < 1e-4
                seq.append(int(t))
        # step by step (the tokens stay on the device), and continuing a context, give the same
        st.reset()
        st.prefill(prompts, want_logits=False)
        step = [st.sample_argmax()]
        for _ in range(24):
            st.decode(None, want_logits=False)
            step.append(st.sample_argmax())
        assert np.array_equal(np.array(step).T, toks)
        if B == 1:
            st.reset()
            st.prefill(prompts[:, :9], want_logits=False)
            st.append(prompts[0, 9:], want_logits=False)
            assert st.sample_argmax()[0] == toks[0, 0]
            assert np.array_equal(st.generate([toks[0, 0]], 24)[:, 0], toks[0, 1:])
        st.close()
    m.close()


def test_sampled_generation_and_vocabulary_edge(capi, folder):
    """min-p sampling with a vocabulary that is no multiple of 4: ids stay inside it, runs repeat, and the device loop
    equals sampling step by step"""
    path, cfg, W = folder("odd")
    assert cfg["vocab"] % 4
    m = capi.Model.open(path, "bfloat16")
    st = m.state(2, 200)
    prompts = np.stack([N.tokens(cfg, 10, 400 + b) for b in range(2)])
    u = np.random.default_rng(3).random((60, 2)).astype(np.float32)
    runs = []
    for _ in range(2):
        st.reset()
        st.prefill(prompts, want_logits=False)
        first = st.sample_minp(0.05, 0.9, u[0])
        runs.append(np.concatenate([first[None], st.generate(first, 59, 0.05, 0.9, u[1:])]))
    assert np.array_equal(runs[0], runs[1]) and runs[0].min() >= 0 and runs[0].max() < cfg["vocab"]
    st.reset()
    st.prefill(prompts, want_logits=False)
    step = [st.sample_minp(0.05, 0.9, u[0])]
    for i in range(1, 60):
        st.decode(step[-1], want_logits=False)
        step.append(st.sample_minp(0.05, 0.9, u[i]))
    assert np.array_equal(np.array(step), runs[0])
    # after a sampler has overwritten the row, greedy decoding still finds a real token
    st.decode(step[-1], want_logits=False)
    assert (st.sample_argmax() < cfg["vocab"]).all() and (st.sample_argmax() >= 0).all()
    st.close()
    m.close()


def test_command_lines(capi, folder, tmp_path):
    """gemma_tokens on a model folder; trace_run against the plain logits"""
    path, cfg, W = folder("plain")
    capi.load()
    lib = os.path.join(ROOT, "tiny-gemma_b200")
    exe = str(tmp_path / "gemma_tokens")
    subprocess.check_call(["g++", "-std=c++20", "-O1", "-o", exe, os.path.join(lib, "host", "gemma_tokens.cpp"), "-L", lib,
                           "-ltinygemma_b200", "-Wl,-rpath," + lib])
    toks = N.tokens(cfg, 30, 77)
    (tmp_path / "ids.txt").write_text(" ".join(map(str, toks)))
    m = capi.Model.open(path, "float32")
    st = m.state(1, 64)
    st.prefill(toks[None], want_logits=False)
    first = st.sample_argmax()
    want = [int(first[0])] + [int(t) for t in st.generate(first, 12)[:, 0]]
    st.close()
    m.close()
    for extra in ([], ["2.0", "1.0", "0", "--device-loop"]):
        r = subprocess.run([exe, path, "float32", str(tmp_path / "ids.txt"), "12"] + extra, capture_output=True, text=True, timeout=300)
        assert r.returncode == 0, r.stderr
        assert [int(t) for t in r.stdout.split()] == want
    out = tmp_path / "out"
    out.mkdir()
    other = N.tokens(cfg, 12, 78)
    steps = [dict(step=0, entries=[dict(id="a", tokens=[int(t) for t in toks[:25]], want=[0, 24])], end=[]),
             dict(step=1, entries=[dict(id="a", tokens=[int(toks[25])], want=[])], end=[]),
             dict(step=2, entries=[dict(id="a", tokens=[int(toks[26])], want=[0])], end=["a"]),
             dict(step=3, entries=[dict(id="b", tokens=[int(t) for t in other], want=[11])], end=["b"])]
    r = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", path, "--dtype", "float32", "--out", str(out),
                        "--max-tokens", "40"], input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr
    assert r.stdout.split("\n")[:4] == ["done 0", "done 1", "done 2", "done 3"]
    ref, ref_b = Ref.get("plain", cfg, W, toks)[0], Ref.get("plain", cfg, W, other)[0]
    V = cfg["vocab"]
    close(np.fromfile(out / "0.f32", "<f4").reshape(-1, V), ref[[0, 24]], "float32")
    close(np.fromfile(out / "2.f32", "<f4").reshape(-1, V), ref[[26]], "float32")
    close(np.fromfile(out / "3.f32", "<f4").reshape(-1, V), ref_b[[11]], "float32")
    assert not (out / "1.f32").exists()


# ------------------------------------------------------------------ what is refused
def test_errors(capi, folder, tmp_path):
    path, cfg, W = folder("plain")
    bad = dict(W)
    del bad["l1.mix.right.a2"]
    with pytest.raises(capi.TgError) as e:
        capi.Model.open(P.write_model(str(tmp_path / "missing"), cfg, bad))
    assert e.value.code == capi.TG_EIO and "l1.mix.right.a2" in str(e.value)
    bad = dict(W)
    bad["l0.mlp.up"] = bad["l0.mlp.up"][:-1]
    with pytest.raises(capi.TgError) as e:
        capi.Model.open(P.write_model(str(tmp_path / "shape"), cfg, bad))
    assert e.value.code == capi.TG_ESHAPE and "l0.mlp.up" in str(e.value)
    m = capi.Model.open(path)
    st = m.state(2, 20)

    def code(f):
        with pytest.raises(capi.TgError) as e:
            f()
        return e.value.code

    assert code(lambda: st.step([(0, [cfg["vocab"]], [])])) == capi.TG_EINVAL
    assert code(lambda: st.step([(2, [1], [])])) == capi.TG_EINVAL
    assert code(lambda: st.step([(0, [1], []), (0, [2], [])])) == capi.TG_EINVAL
    assert code(lambda: st.step([(0, [1, 2], [2])])) == capi.TG_EINVAL
    assert code(lambda: st.step([(0, [1] * 21, [])])) == capi.TG_ESTATE
    st.step([(0, [1] * 20, [])])
    assert code(lambda: st.step([(0, [1], [])])) == capi.TG_ESTATE
    assert code(lambda: st.decode([1, 1])) == capi.TG_ESTATE
    assert code(lambda: st.prefill([[1], [1]])) == capi.TG_ESTATE
    st.step([(1, [1, 2, 3], [])])  # the other sequence still works
    # entry points of another family
    assert code(lambda: st.decode_hidden([1, 1])) == capi.TG_EINVAL
    assert code(lambda: m.build_tables()) == capi.TG_EINVAL
    st.close()
    m.close()
