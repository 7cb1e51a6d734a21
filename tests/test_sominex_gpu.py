"""Sominex on the GPU against the plain implementation (sominex_plain.py), through the library's own step, cache and
generation loop. float32 states must agree to rounding. bfloat16 states agree to the rounding of their activations: nearly
all rows closely, and a few (a router's close call, a read-out that nearly cancels) still roughly.

The state's passes are kept small (TG_PASS_ROWS) where the point is the cache's ring, so that it wraps many times.
"""

import json
import os
import subprocess
import sys

import numpy as np
import pytest

import nabelix_plain as F
import sominex_cases as C
import sominex_plain as P
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
            cfg = cfg or C.CONFIGS[key]
            W = C.weights(cfg, 3) if W is None else W
            made[key] = (F.write_model(str(tmp_path_factory.mktemp(key)), cfg, W), cfg, W)
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


def close(got, want, dtype):
    e = np.atleast_1d(row_err(np.asarray(got, np.float64), want))
    assert np.isfinite(got).all()
    if dtype == "float32":
        assert e.max() <= TOL[dtype], (float(e.max()), np.unravel_index(e.argmax(), e.shape))
    else:
        over, far = int((e > TOL[dtype]).sum()), int((e > 0.2).sum())
        assert over <= max(1, 0.04 * e.size) and far <= max(1, 0.015 * e.size), (over, far, e.size, float(e.max()), int(e.argmax()))


def replay(st, seq, toks, cuts):
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
@pytest.mark.parametrize("key", sorted(C.CONFIGS))
def test_prompt_matches_plain_layer_by_layer(capi, folder, key, dtype):
    path, cfg, W = folder(key)
    toks = C.tokens(cfg, 150, 1)
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
    st.trace_enable(False)
    n = 60
    close(replay(st, 0, toks[:n], [1] * n), want[:n], dtype)
    st.close()
    m.close()


# ------------------------------------------------------------------ one mechanism at a time
MECHANISMS = {
    "window": C.config([C.attn(None, pool=0, rot=0)]),
    "pooled": C.config([C.attn(None, rot=0, size=11, pool=7)]),
    "rotation": C.config([C.attn(None, pool=0, size=90, scaling=None, base=300.0)]),
    "yarn": C.config([C.attn(None, pool=0, size=90)]),
    "pooled_rotation": C.config([C.attn(None, size=7, pool=3, rot=32)]),
    "state_space": C.config([C.mamba(None)]),
    "state_space_strong": C.config([C.mamba(None, heads=6, groups=3)]),
    "matrix_memory": C.config([C.mlstm(None)]),
    "matrix_memory_extreme": C.config([C.mlstm(None, heads=4, gate_cap=15.0)]),
    "clamped_ff": C.config([C.mlstm(C.dense(90, 0.6))]),
    "mixture": C.config([C.mlstm(C.moe(7, 3, 24, 0, 2.5))]),
    "mixture_shared": C.config([C.mamba(C.moe(5, 2, 16, 56, 0.5))]),
    "mixture_all": C.config([C.mamba(C.moe(4, 4, 32, 0))]),
    "mixture_one": C.config([C.mamba(C.moe(12, 1, 40, 0, 6.0))]),
}


def mechanism(part):
    cfg = MECHANISMS[part]
    W = C.weights(cfg, 17)
    if "mixture" in part or part == "clamped_ff":
        W = C.without_mixers(W, cfg)
        W = {k: np.asarray(v) * (6.0 if k.endswith("router") else 1.0) for k, v in W.items()}  # (no close calls to speak of)
    if part == "state_space_strong":  # heads that forget at once beside heads that hardly forget, large steps beside small ones
        W["l0.mix.A_log"] = F.to_bf16(np.array([5.0, -6.0, 3.0, -2.0, 4.0, 0.0]))
        W["l0.mix.dt_bias"] = F.to_bf16(np.array([3.0, -4.0, 5.0, 2.0, -1.0, 0.0]))
        W["l0.mix.in"] = F.to_bf16(np.concatenate([W["l0.mix.in"][:-6], 3.0 * W["l0.mix.in"][-6:]]))
    if part == "matrix_memory_extreme":  # input gates from e^-15 to e^15, forget gates from nothing to everything
        W["l0.mix.i.b"] = F.to_bf16(np.array([-12.0, 12.0, 0.0, 4.0]))
        W["l0.mix.f.b"] = F.to_bf16(np.array([-9.0, 9.0, 0.0, 14.0]))
        for n in "if":
            W["l0.mix." + n] = F.to_bf16(4.0 * np.asarray(W["l0.mix." + n]))
    return cfg, {k: F.to_bf16(v) for k, v in W.items()}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("part", sorted(MECHANISMS))
def test_mechanism_alone(capi, folder, part, dtype):
    cfg, W = mechanism(part)
    path, _, _ = folder("only_" + part, cfg, W)
    toks = C.tokens(cfg, 300, 2)
    tr = []
    P.forward(toks, W, cfg, tr)
    x0 = np.asarray(W["embed"], np.float64)[toks] * cfg["embedding"]["scale"]
    m = capi.Model.open(path, dtype)
    st = m.state(1, 320)
    st.trace_enable()
    for cuts in ([300], [270] + [1] * 30, [5, 123, 2, 129, 1, 40]):
        got, at = [], 0
        for n in cuts:
            st.step([(0, toks[at:at + n], [])])
            got.append(st.trace()[0])
            at += n
        # what the layer added to the stream is the mechanism's own output
        d, w = np.concatenate(got) - x0, tr[0] - x0
        assert rel_l2(d, w) <= TOL[dtype] * (2 if "extreme" in part and dtype == "float32" else 1), rel_l2(d, w)
        st.free_sequence(0)
    st.close()
    m.close()


def test_chunks_and_token_by_token_agree(capi, folder, monkeypatch):
    """the two ways a portion goes through a recurrence"""
    path, cfg, W = folder("real_heads")
    toks = C.tokens(cfg, 330, 4)
    m = capi.Model.open(path, "bfloat16")
    got = []
    for tc in ("1", "0"):
        monkeypatch.setenv("TG_LIN_TC", tc)
        st = m.state(1, 400)
        got.append(replay(st, 0, toks, [200, 130]))
        st.close()
    m.close()
    e = row_err(got[0], got[1])
    assert np.median(e) < 5e-3 and np.quantile(e, 0.95) < 2e-2


# ------------------------------------------------------------------ portions, decoding, the ring
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("cuts", [[2] * 400, [3, 1, 5, 2, 7, 1, 1, 13, 2, 64, 65, 63, 16, 17, 15, 128], [1, 127, 2, 129], [9, 8, 10, 256], [700]])
@pytest.mark.parametrize("key", ["plain", "order", "odd", "real_heads"])
def test_portions(capi, folder, monkeypatch, key, cuts, dtype):
    monkeypatch.setenv("TG_PASS_ROWS", "128")
    path, cfg, W = folder(key)
    toks = C.tokens(cfg, 330, 4)
    want, _ = Ref.get(key, cfg, W, toks)
    m = capi.Model.open(path, dtype)
    st = m.state(1, 400)
    close(replay(st, 0, toks, cuts), want, dtype)
    assert st.position(0) == len(toks)
    st.close()
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_one_long_pass(capi, folder, dtype):
    """several chunks, several tiles of rows per expert, in one pass"""
    path, cfg, W = folder("plain")
    toks = C.tokens(cfg, 700, 14)
    want, _ = Ref.get("plain", cfg, W, toks)
    m = capi.Model.open(path, dtype)
    st = m.state(1, 800)
    close(replay(st, 0, toks, [690]), want, dtype)
    st.close()
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding(capi, folder, monkeypatch, dtype):
    """the ring (window 20 + 128 rows -> 192 slots) wraps more than once in decoding alone; the pooled blocks do not"""
    monkeypatch.setenv("TG_PASS_ROWS", "128")
    path, cfg, W = folder("plain")
    toks = C.tokens(cfg, 520, 6)
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
    todo = [C.tokens(cfg, int(n), 50 + i) for i, n in enumerate([70, 5, 130, 1, 33, 260, 2, 90, 17, 64, 40][:B + 4])]
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
@pytest.mark.parametrize("key", ["plain", "odd"])
def test_lockstep_decode_in_batches(capi, folder, key, dtype):
    """tg_prefill + tg_decode: few rows (matrix-vector pipeline) and more (tensor cores), several prompts at once"""
    path, cfg, W = folder(key)
    m = capi.Model.open(path, dtype)
    for B in (1, 2, 3, 4, 5, 9):
        toks = np.stack([C.tokens(cfg, 48, 200 + b) for b in range(B)])
        st = m.state(B, 64)
        want = np.stack([Ref.get(key, cfg, W, t)[0] for t in toks])
        got = [st.prefill(toks[:, :40])] + [st.decode(toks[:, i]) for i in range(40, 48)]
        close(np.stack(got, axis=1), want[:, 39:], dtype)
        assert all(st.position(b) == 48 for b in range(B))
        st.reset()
        close(st.prefill(toks[:, :1]), want[:, 0], dtype)
        st.close()
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_large_batch_of_equal_requests(capi, folder, dtype):
    """150 sequences, several pieces of keys per CTA: every row has the same bits, and they are the plain result"""
    path, cfg, W = folder("real_heads")
    toks, B = C.tokens(cfg, 190, 31), 150
    want = Ref.get("real_heads", cfg, W, toks)[0]
    m = capi.Model.open(path, dtype)
    st = m.state(B, 200)
    for at in range(0, 150, 25):  # (in one pass each, so that every sequence's rows meet the same kernels)
        st.step([(b, toks[at:at + 25], []) for b in range(B)])
    rows = []
    for i in range(150, 190):
        got = st.decode(np.full(B, toks[i]))
        assert np.array_equal(got, np.broadcast_to(got[0], got.shape)), (i, np.nonzero((got != got[0]).any(1))[0])
        rows.append(got[0])
    close(np.array(rows), want[150:], dtype)
    st.close()
    m.close()


# ------------------------------------------------------------------ edges
def sees(q, k, window, pool):
    return bool(P.visible(q + 1, window)[q, k]) or (pool > 0 and (k // pool + 1) * pool - 1 <= q - window)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("window,pool", [(24, 6), (64, 8), (65, 16), (130, 5), (7, 0), (3, 20)])
def test_keys_just_inside_and_outside(capi, folder, monkeypatch, window, pool, dtype):
    monkeypatch.setenv("TG_PASS_ROWS", "128")
    cfg, W = C.beacon(window, pool)
    path, _, _ = folder("beacon_%d_%d" % (window, pool), cfg, W)
    m = capi.Model.open(path, dtype)
    st = m.state(1, 600)
    T = 300
    base = np.random.default_rng(8).integers(3, cfg["vocab"], T).astype(np.int32)
    seen = unseen = 0
    for q in (window + 2 * max(pool, 1) + 1, 191, 192, 193, 255, 299):
        nb = max(0, (q - window + 1) // pool) if pool else 0  # blocks that the query sees
        cases = [q - window + 1, q - window, q - window - 1, q - 1, 0, nb * pool - 1, nb * pool, (nb - 1) * pool, nb * pool // 2]
        for k in sorted({c for c in cases if 0 <= c < q}):
            toks = base.copy()
            toks[k], toks[q] = C.KEY, C.QUERY
            want = P.forward(toks[:q + 1], W, cfg)[q]
            without = base.copy()
            without[q] = C.QUERY
            # the case tells: a key that is seen shows, one that is not leaves no trace in the logits
            e = row_err(P.forward(without[:q + 1], W, cfg)[q], want)
            if sees(q, k, window, pool):
                seen += 1
                assert e > 0.15, (q, k)
            else:
                unseen += 1
                assert e < 1e-12
            # in a prompt; then with the query decoded alone
            for cuts in ([q + 1], [q, 1], [q - 1, 2]):
                st.free_sequence(0)
                got = replay(st, 0, toks[:q + 1], cuts)[q]
                assert row_err(got, want) <= 2 * TOL[dtype], (q, k, cuts, row_err(got, want))
    assert seen >= 6 and unseen >= (6 if pool != 1 else 0)
    st.close()
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("key", ["order", "odd"])
def test_first_tokens(capi, folder, key, dtype):
    """prompts of 1 .. 9 tokens, in one step and cut after every place"""
    path, cfg, W = folder(key)
    m = capi.Model.open(path, dtype)
    st = m.state(1, 16)
    toks = C.tokens(cfg, 9, 11)
    want, _ = Ref.get(key, cfg, W, toks)
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
    toks, other = C.tokens(cfg, 100, 21), C.tokens(cfg, 260, 22)
    b.step([(0, other, []), (1, other[:50], [])])
    b.step([(0, other[:30], [])])
    b.free_sequence(0)
    b.free_sequence(1)
    for st in (a, b):
        st.last = replay(st, 1, toks, [60, 3, 1, 1, 20])
        st.free_sequence(1)
    assert np.array_equal(a.last, b.last)
    a.close()
    b.close()
    m.close()


# ------------------------------------------------------------------ generation
def test_greedy_generation_matches_plain(capi, folder):
    path, cfg, W = folder("plain")
    m = capi.Model.open(path, "float32")
    for B in (1, 5):
        prompts = np.stack([C.tokens(cfg, 20, 300 + b) for b in range(B)])
        st = m.state(B, 64)
        st.prefill(prompts, want_logits=False)
        first = st.sample_argmax()
        more = st.generate(first, 24)
        toks = np.concatenate([first[None], more]).T
        for b in range(B):
            seq = list(prompts[b]) + [int(t) for t in toks[b]]
            lg = P.forward(seq[:-1], W, cfg)[len(prompts[b]) - 1:]
            for t, row in zip(toks[b], lg):
                top = np.sort(row)[-2:]
                assert int(t) == int(row.argmax()) or top[1] - top[0] < 1e-4
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
    """min-p sampling with a vocabulary that is no multiple of 4: ids stay inside it, and runs repeat"""
    path, cfg, W = folder("odd")
    assert cfg["vocab"] % 4
    m = capi.Model.open(path, "bfloat16")
    st = m.state(2, 200)
    prompts = np.stack([C.tokens(cfg, 10, 400 + b) for b in range(2)])
    u = np.random.default_rng(3).random((60, 2)).astype(np.float32)
    runs = []
    for _ in range(2):
        st.reset()
        st.prefill(prompts, want_logits=False)
        first = st.sample_minp(0.05, 0.9, u[0])
        runs.append(np.concatenate([first[None], st.generate(first, 59, 0.05, 0.9, u[1:])]))
    assert np.array_equal(runs[0], runs[1]) and runs[0].min() >= 0 and runs[0].max() < cfg["vocab"]
    st.close()
    m.close()


def test_command_lines(capi, folder, tmp_path):
    """gemma_tokens on a model folder; trace_run against the plain logits"""
    path, cfg, W = folder("order")
    capi.load()
    lib = os.path.join(ROOT, "tiny-gemma_b200")
    exe = str(tmp_path / "gemma_tokens")
    subprocess.check_call(["g++", "-std=c++20", "-O1", "-o", exe, os.path.join(lib, "host", "gemma_tokens.cpp"), "-L", lib,
                           "-ltinygemma_b200", "-Wl,-rpath," + lib])
    toks = C.tokens(cfg, 30, 77)
    (tmp_path / "ids.txt").write_text(" ".join(map(str, toks)))
    m = capi.Model.open(path, "float32")
    st = m.state(1, 64)
    st.prefill(toks[None], want_logits=False)
    first = st.sample_argmax()
    want = [int(first[0])] + [int(t) for t in st.generate(first, 12)[:, 0]]
    st.close()
    m.close()
    r = subprocess.run([exe, path, "float32", str(tmp_path / "ids.txt"), "12"], capture_output=True, text=True, timeout=300)
    assert r.returncode == 0 and [int(t) for t in r.stdout.split()] == want, r.stderr
    out = tmp_path / "out"
    out.mkdir()
    other = C.tokens(cfg, 12, 78)
    steps = [dict(step=0, entries=[dict(id="a", tokens=[int(t) for t in toks[:25]], want=[0, 24])], end=[]),
             dict(step=1, entries=[dict(id="a", tokens=[int(toks[25])], want=[])], end=[]),
             dict(step=2, entries=[dict(id="a", tokens=[int(toks[26])], want=[0])], end=["a"]),
             dict(step=3, entries=[dict(id="b", tokens=[int(t) for t in other], want=[11])], end=["b"])]
    r = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", path, "--dtype", "float32", "--out", str(out),
                        "--max-tokens", "40"], input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr
    assert r.stdout.split("\n")[:4] == ["done 0", "done 1", "done 2", "done 3"]
    ref, ref_b = Ref.get("order", cfg, W, toks)[0], Ref.get("order", cfg, W, other)[0]
    V = cfg["vocab"]
    close(np.fromfile(out / "0.f32", "<f4").reshape(-1, V), ref[[0, 24]], "float32")
    close(np.fromfile(out / "2.f32", "<f4").reshape(-1, V), ref[[26]], "float32")
    close(np.fromfile(out / "3.f32", "<f4").reshape(-1, V), ref_b[[11]], "float32")


# ------------------------------------------------------------------ what is refused
def test_errors(capi, folder, tmp_path):
    path, cfg, W = folder("plain")
    for name, cut, code in (("l2.mix.f.b", None, capi.TG_EIO), ("l3.mlp.e4.down", 1, capi.TG_ESHAPE), ("l1.mix.in", 1, capi.TG_ESHAPE), ("head", None, capi.TG_EIO)):
        bad = dict(W)
        if cut:
            bad[name] = bad[name][:-cut]
        else:
            del bad[name]
        with pytest.raises(capi.TgError) as e:
            capi.Model.open(F.write_model(str(tmp_path / name), cfg, bad))
        assert e.value.code == code and name in str(e.value)
    m = capi.Model.open(path)
    st = m.state(2, 20)

    def code(f):
        with pytest.raises(capi.TgError) as e:
            f()
        return e.value.code

    assert code(lambda: st.step([(0, [cfg["vocab"]], [])])) == capi.TG_EINVAL
    assert code(lambda: st.step([(0, [1] * 21, [])])) == capi.TG_ESTATE
    st.step([(0, [1] * 20, [])])
    assert code(lambda: st.step([(0, [1], [])])) == capi.TG_ESTATE
    st.step([(1, [1, 2, 3], [])])  # the other sequence still works
    st.close()
    m.close()
