"""Seeded random-init Gemma-3 weights in the ``gemma_i8.bin`` layout, plus prompts.

There is no checkpoint to download where this runs, so benchmarks and parity
tests use random weights of the real architecture. The file produced here is
byte-for-byte what the reference converter would write for the same float
tensors:

* layout and order  — reference ``py/gemma.py:27-77``
  (``write_from_transformer_weights_quantized``), read back by
  ``csrc/include/transformer.hpp:99-165`` (``read_weights``);
* quantiser         — reference ``py/weight_handlers.py:10-20``: one fp32 scale
  per column of the stored 2-D array, ``scale = max|W| / 127`` over axis 0,
  ``q = rint(W / scale)`` as int8.

No header, no padding, native little-endian.
"""

from __future__ import annotations

import os
from dataclasses import dataclass

import numpy as np


@dataclass(frozen=True)
class Config:
    """Field order follows reference ``csrc/include/config.hpp:7-20``."""

    hidden_size: int
    intermediate_size: int
    n_layers: int
    n_vocab: int
    n_pos: int
    n_pos_local: int
    head_dim: int
    n_head: int
    n_kv: int
    rope_theta: float
    rope_theta_local: float
    window_pattern: int

    @property
    def q_dim(self) -> int:
        return self.n_head * self.head_dim

    @property
    def kv_dim(self) -> int:
        return self.n_kv * self.head_dim

    def is_local(self, layer: int) -> bool:
        # reference transformer.hpp:43
        return (layer % self.window_pattern) != (self.window_pattern - 1)


# reference config.hpp:46-48
CONFIGS = {
    "270m": Config(640, 2048, 18, 262144, 32768, 512, 256, 4, 1, 1_000_000.0, 10_000.0, 6),
    "1B": Config(1152, 6912, 26, 262144, 32768, 512, 256, 4, 1, 1_000_000.0, 10_000.0, 6),
}


def quantize_weight(w: np.ndarray) -> tuple[np.ndarray, np.ndarray]:
    """Per-column int8 quantiser (reference ``py/weight_handlers.py:10-20``)."""
    assert w.ndim == 2
    scales = (np.max(np.abs(w), axis=0, keepdims=True) / 127.0).astype(np.float32)
    q = np.rint(w / scales).astype(np.int8)
    return q, scales


def layout(size: str) -> list[tuple[str, str, tuple[int, ...], int]]:
    """[(name, dtype, shape, byte offset)] of every tensor in file order."""
    c = CONFIGS[size]
    out = []
    off = 0

    def add(name, dtype, shape):
        nonlocal off
        out.append((name, dtype, shape, off))
        off += int(np.prod(shape)) * (1 if dtype == "i1" else 4)

    def addq(name, rows, cols):
        add(name + ".q", "i1", (rows, cols))
        add(name + ".s", "f4", (cols,))

    addq("wte", c.n_vocab, c.hidden_size)
    add("final_norm", "f4", (c.hidden_size,))
    for l in range(c.n_layers):
        p = f"l{l}."
        addq(p + "q", c.hidden_size, c.q_dim)
        addq(p + "k", c.hidden_size, c.kv_dim)
        addq(p + "v", c.hidden_size, c.kv_dim)
        addq(p + "o", c.q_dim, c.hidden_size)
        add(p + "q_norm", "f4", (c.head_dim,))
        add(p + "k_norm", "f4", (c.head_dim,))
        add(p + "attn_pre", "f4", (c.hidden_size,))
        add(p + "attn_post", "f4", (c.hidden_size,))
        addq(p + "up", c.hidden_size, c.intermediate_size)
        addq(p + "gate", c.hidden_size, c.intermediate_size)
        addq(p + "down", c.intermediate_size, c.hidden_size)
        add(p + "mlp_pre", "f4", (c.hidden_size,))
        add(p + "mlp_post", "f4", (c.hidden_size,))
    addq("lm_head", c.hidden_size, c.n_vocab)
    out.append(("<end>", "i1", (0,), off))
    return out


def file_size(size: str) -> int:
    return layout(size)[-1][3]


def random_tensors(size: str, seed: int = 0, std: float = 0.02):
    """The seeded N(0, std) fp32 tensors of a model in file order, as (name, array): wte [V, D], final_norm,
    then per layer q, k, v, o, q_norm, k_norm, attn_pre, attn_post, up, gate, down, mlp_pre, mlp_post
    (names prefixed l<layer>.). The lm_head is tied: wte.T."""
    c = CONFIGS[size]
    rng = np.random.default_rng(seed)

    def normal(*shape):
        return (rng.standard_normal(shape, dtype=np.float32) * np.float32(std)).astype(np.float32)

    yield "wte", normal(c.n_vocab, c.hidden_size)
    yield "final_norm", normal(c.hidden_size)
    for l in range(c.n_layers):
        p = "l%d." % l
        yield p + "q", normal(c.hidden_size, c.q_dim)
        yield p + "k", normal(c.hidden_size, c.kv_dim)
        yield p + "v", normal(c.hidden_size, c.kv_dim)
        yield p + "o", normal(c.q_dim, c.hidden_size)
        yield p + "q_norm", normal(c.head_dim)
        yield p + "k_norm", normal(c.head_dim)
        yield p + "attn_pre", normal(c.hidden_size)
        yield p + "attn_post", normal(c.hidden_size)
        yield p + "up", normal(c.hidden_size, c.intermediate_size)
        yield p + "gate", normal(c.hidden_size, c.intermediate_size)
        yield p + "down", normal(c.intermediate_size, c.hidden_size)
        yield p + "mlp_pre", normal(c.hidden_size)
        yield p + "mlp_post", normal(c.hidden_size)


def write_random_model(path: str, size: str, seed: int = 0, std: float = 0.02) -> str:
    """Write the tensors of random_tensors (norm weights included, lm_head tied to
    wte before quantisation) to ``path`` in the gemma_i8.bin layout (reference
    ``py/gemma.py:27-77``); returns ``path``. Skips the work if a file of the
    right size is already there (callers encode size/seed in the name)."""
    want = file_size(size)
    if os.path.exists(path) and os.path.getsize(path) == want:
        return path
    tmp = path + ".tmp%d" % os.getpid()
    with open(tmp, "wb") as f:
        wte = None
        for name, w in random_tensors(size, seed, std):
            if w.ndim == 2:
                q, s = quantize_weight(w)
                f.write(np.ascontiguousarray(q).data)
                f.write(np.ascontiguousarray(s).data)
                if name == "wte":
                    wte = w
            else:
                f.write(w.data)
        # tied embeddings: lm_head = wte.T as floats, quantised per vocab column
        s_v = (np.max(np.abs(wte), axis=1) / 127.0).astype(np.float32)  # [V]
        q = np.rint(wte / s_v[:, None]).astype(np.int8)  # [V, D]
        f.write(np.ascontiguousarray(q.T).data)
        f.write(s_v.data)
    assert os.path.getsize(tmp) == want, (os.path.getsize(tmp), want)
    os.replace(tmp, path)
    return path


def random_prompt(n: int, seed: int, vocab: int = 262144) -> np.ndarray:
    """``n`` token ids uniform in [0, vocab) — stands in for the reference's
    ultrachat prompts (mean length 178, reference ``README.md:50``)."""
    return np.random.default_rng(seed).integers(0, vocab, size=n, dtype=np.int32)


def mt19937_uniforms(n: int, seed: int) -> np.ndarray:
    """``n`` draws of ``std::uniform_real_distribution<float>(0,1)`` over
    ``std::mt19937(seed)`` (reference ``transformer.hpp:170-172``): libstdc++'s
    ``generate_canonical<float,24>`` takes one 32-bit word per draw, scales it
    by 2^-32 in float and maps a result of 1.0 to the float just below 1."""
    rs = np.random.RandomState()
    key = np.zeros(624, dtype=np.uint32)
    # std::mt19937 seeding: x[0]=seed, x[i] = 1812433253*(x[i-1]^(x[i-1]>>30)) + i
    x = np.uint64(seed & 0xFFFFFFFF)
    key[0] = x
    for i in range(1, 624):
        x = (np.uint64(1812433253) * (x ^ (x >> np.uint64(30))) + np.uint64(i)) & np.uint64(0xFFFFFFFF)
        key[i] = x
    rs.set_state(("MT19937", key, 624))
    words = rs.randint(0, 2**32, size=n, dtype=np.uint64).astype(np.uint32)
    out = words.astype(np.float32) * np.float32(2.0**-32)
    out[out >= np.float32(1.0)] = np.nextafter(np.float32(1.0), np.float32(0.0))
    return out.astype(np.float32)


# ------------------------------------------------------------------ model folders
#                 width    ff layers  vocab
LAYERED_SIZES = {"270m": (640, 2048, 18, 262144),
                 "1B": (1152, 6912, 26, 262144),
                 "3B": (2560, 9216, 24, 65536)}


# ---- Nabelix
def nabelix_config(name: str) -> dict:
    """config.json of layers that resemble a real model's: the widths, feed-forward sizes, depths and vocabularies of
    the Gemma-3 sizes above (a few more weights per layer than theirs), and a wider one"""
    width, ff, n, vocab = LAYERED_SIZES[name]
    h, g, r = {"270m": (4, 1, 4), "1B": (8, 2, 4), "3B": (20, 4, 20)}[name]  # left heads, its key/value heads, right heads
    layer = {"type": "parallel", "mlp": {"kind": "dense", "ff": ff},
             "mixer": {"left_scale": 1.0, "right_scale": 1.0,
                       "left": {"heads": h, "kv_heads": g, "dim": 128, "vdim": 128, "scale": 128 ** -0.5,
                                "mask": {"size": 512, "keep_first": 4}},
                       "right": {"heads": r, "kv_heads": r, "dim": 128, "vdim": 128, "conv": 4}}}
    return {"architecture": "Nabelix", "width": width, "vocab": vocab, "norm": {"eps": 1e-6}, "canon": {"taps": 4},
            "logit_softcap": 30.0, "layers": [layer] * n}


NABELIX_RANK = 128  # inner size of the two low-rank projections


def nabelix_shapes(cfg: dict):
    """(tensor name, shape) of every tensor of a Nabelix model"""
    D, taps = cfg["width"], cfg["canon"]["taps"]
    yield "embed", (cfg["vocab"], D)
    for i, sp in enumerate(cfg["layers"]):
        p, lf, rt = "l%d." % i, sp["mixer"]["left"], sp["mixer"]["right"]
        yield p + "norm1", (D,)
        yield p + "canon1", (D, taps)
        m = p + "mix.left."
        for n, rows in (("q", lf["heads"] * lf["dim"]), ("k", lf["kv_heads"] * lf["dim"]), ("v", lf["kv_heads"] * lf["vdim"]),
                        ("g", lf["heads"] * lf["vdim"])):
            yield m + n, (rows, D)
        yield m + "r1", (lf["heads"],)
        yield m + "r2", (lf["heads"],)
        yield m + "o", (D, lf["heads"] * lf["vdim"])
        m = p + "mix.right."
        kc, vc = rt["kv_heads"] * rt["dim"], rt["heads"] * rt["vdim"]
        for n, rows in (("q", kc), ("k", kc), ("v", vc)):
            yield m + n, (rows, D)
            yield m + n + ".conv", (rows, rt["conv"])
        yield m + "b", (rt["heads"], D)
        yield m + "A_log", (rt["heads"],)
        yield m + "dt_bias", (rt["heads"] * rt["dim"],)
        yield m + "norm", (rt["vdim"],)
        yield m + "a1", (NABELIX_RANK, D)
        yield m + "a2", (rt["heads"] * rt["dim"], NABELIX_RANK)
        yield m + "g1", (NABELIX_RANK, D)
        yield m + "g2", (vc, NABELIX_RANK)
        yield m + "o", (D, vc)
        if sp["mlp"]:
            yield p + "norm2", (D,)
            yield p + "mlp.gate", (sp["mlp"]["ff"], D)
            yield p + "mlp.up", (sp["mlp"]["ff"], D)
            yield p + "mlp.down", (D, sp["mlp"]["ff"])
    yield "final.norm", (D,)


# ---- Sominex
def sominex_config(name: str) -> dict:
    """the same widths, feed-forward sizes, depths and vocabularies; layers in turns of attention, Mamba-2, mLSTM and
    Mamba-2, the Mamba-2 ones with a mixture of experts of which a token uses as many weights as the dense layers have"""
    width, ff, n, vocab = LAYERED_SIZES[name]
    h, g, groups, lh = {"270m": (4, 1, 2, 4), "1B": (8, 2, 2, 4), "3B": (20, 4, 4, 10)}[name]
    dense = {"kind": "dense", "ff": ff, "limit": 7.0}
    moe = {"kind": "moe", "expert": {"ff": ff // 8}, "router": {"experts": 32, "top": 4, "scale": 1.0}, "shared": {"ff": ff // 2}}
    rot = {"base": 10000.0, "dims": 128, "scaling": {"factor": 4.0, "fast": 32.0, "slow": 1.0, "original": 4096}}
    attention = {"type": "attention", "mlp": dense,
                 "mixer": {"heads": h, "kv_heads": g, "dim": 128, "vdim": 128, "scale": 128 ** -0.5, "rot": rot,
                           "mask": {"size": 512, "pool": 16}}}
    mamba = {"type": "mamba2", "mlp": moe,
             "mixer": {"heads": 2 * width // 64, "vdim": 64, "state": 128, "groups": groups, "conv": 4, "norm_groups": groups}}
    mlstm = {"type": "mlstm", "mlp": dense, "mixer": {"heads": lh, "dim": 128, "vdim": 256, "gate_cap": 15.0}}
    turn = [attention, mamba, mlstm, mamba]
    return {"architecture": "Sominex", "width": width, "vocab": vocab, "norm": {"eps": 1e-6}, "embedding": {"scale": 1.0},
            "layers": [turn[i % 4] for i in range(n)]}


def sominex_shapes(cfg: dict):
    """(tensor name, shape) of every tensor of a Sominex model"""
    D = cfg["width"]
    yield "embed", (cfg["vocab"], D)
    for i, sp in enumerate(cfg["layers"]):
        p, m, c, ff = "l%d." % i, "l%d.mix." % i, sp["mixer"], sp["mlp"]
        yield p + "norm1", (D,)
        yield p + "shift", (D,)
        if sp["type"] == "attention":
            out = c["heads"] * c["vdim"]
            for n, rows in (("q", c["heads"] * c["dim"]), ("k", c["kv_heads"] * c["dim"]), ("v", c["kv_heads"] * c["vdim"])):
                yield m + n, (rows, D)
        elif sp["type"] == "mamba2":
            out = c["heads"] * c["vdim"]
            ch = out + 2 * c["groups"] * c["state"]
            yield m + "in", (out + ch + c["heads"], D)
            yield m + "conv", (ch, c["conv"])
            yield m + "conv.b", (ch,)
            for n in ("dt_bias", "A_log", "D"):
                yield m + n, (c["heads"],)
            yield m + "norm", (out,)
        else:
            out = c["heads"] * c["vdim"]
            for n, rows in (("q", c["heads"] * c["dim"]), ("k", c["heads"] * c["dim"]), ("v", out), ("g", out), ("i", c["heads"]), ("f", c["heads"])):
                yield m + n, (rows, D)
            yield m + "i.b", (c["heads"],)
            yield m + "f.b", (c["heads"],)
            yield m + "norm", (out,)
        yield m + "o", (D, out)
        parts = []
        if ff and ff["kind"] == "dense":
            parts = [("", ff["ff"])]
        elif ff:
            yield p + "mlp.router", (ff["router"]["experts"], D)
            parts = [("e%d." % e, ff["expert"]["ff"]) for e in range(ff["router"]["experts"])] + [("shared.", ff["shared"]["ff"])]
        for q, n in parts:
            yield p + "mlp." + q + "gate", (n, D)
            yield p + "mlp." + q + "up", (n, D)
            yield p + "mlp." + q + "down", (D, n)
    yield "final.norm", (D,)
    yield "head", (cfg["vocab"], D)


LAYERED = {"Nabelix": (nabelix_config, nabelix_shapes), "Sominex": (sominex_config, sominex_shapes)}


def write_random_layered(folder: str, cfg: dict, seed: int = 0) -> str:
    """config.json and model.safetensors with seeded random bfloat16 weights. Matrices are N(0, 1/columns), cut from one
    block of random numbers at random offsets (drawing billions of them would take minutes)."""
    import json

    done = os.path.join(folder, "model.safetensors")
    text = json.dumps(cfg)
    try:
        with open(os.path.join(folder, "config.json")) as f:
            if f.read() == text and os.path.exists(done):
                return folder
    except OSError:
        pass
    os.makedirs(folder, exist_ok=True)
    if os.path.exists(done):
        os.unlink(done)
    g = np.random.default_rng(seed)
    block = g.standard_normal(1 << 24, dtype=np.float32)
    shapes = list(LAYERED[cfg["architecture"]][1](cfg))
    head, at = {}, 0
    for name, shape in shapes:
        n = 2 * int(np.prod(shape))
        head[name] = {"dtype": "BF16", "shape": list(shape), "data_offsets": [at, at + n]}
        at += n
    h = json.dumps(head).encode()
    h += b" " * (-len(h) % 8)

    def bf16(x):
        b = np.ascontiguousarray(x, np.float32).view(np.uint32)
        return ((b + np.uint32(0x7FFF) + ((b >> np.uint32(16)) & np.uint32(1))) >> np.uint32(16)).astype("<u2")

    scaled = {}
    part = done + ".part"
    with open(part, "wb") as f:
        f.write(len(h).to_bytes(8, "little") + h)
        for name, shape in shapes:
            n = int(np.prod(shape))
            if len(shape) == 1:
                leaf = name.split(".mix.")[-1]
                leaf = leaf if leaf in ("i.b", "f.b", "conv.b") else leaf.rsplit(".", 1)[-1]
                x = {"A_log": g.uniform(-3, 0, n), "dt_bias": g.uniform(-4, 0, n), "r1": g.uniform(0.1, 1, n), "r2": g.uniform(0.1, 1, n),
                     "shift": g.uniform(0, 1, n), "i.b": g.uniform(-3, 0, n), "f.b": g.uniform(2, 6, n), "conv.b": 0.1 * g.standard_normal(n)}.get(
                    leaf, 1.0 + 0.1 * g.standard_normal(n))
                f.write(bf16(x).tobytes())
                continue
            k = shape[1]
            if k not in scaled:
                scaled[k] = bf16(block * np.float32(k ** -0.5))
            src = scaled[k]
            o = int(g.integers(0, src.size))
            while n:
                c = min(n, src.size - o)
                f.write(src[o:o + c].tobytes())
                n -= c
                o = 0
    os.replace(part, done)
    with open(os.path.join(folder, "config.json"), "w") as f:
        f.write(text)
    return folder
