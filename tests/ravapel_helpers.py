"""Small Ravapel configurations and model folders with random weights for the tests.

Sizes lie away from powers of two and from each other (key width != value width, heads != kv heads, rotary widths below the
key width and equal to it, heads of 5 to 300 channels, 1 to 6 taps, widths that are no multiple of 8), chunks that do not line
up with the pages of 64, repeated stretches that start at layer 0 or later, run once or several times and hold one layer or
several, layers without a feed-forward, pair tables of few and of many rows.  Weights are drawn here, not by the package's
initialiser, so that the recurrences' memories reach from a few tokens to hundreds, the gates take both branches, and the
norms' weights, biases and scales take values that matter.
"""
import json
import os
import tempfile

import numpy as np
import torch

import ravapel_plain as P

P.PRECISION = torch.float64      # the reference of the tests is the plain implementation in double precision


def hgrn2(dim=12, heads=3, vdim=20):
    return {"dim": dim, "heads": heads, "vdim": vdim}


def attn(dim=20, heads=6, kv_heads=2, vdim=12, rot=(8, 300.0), chunk=37, scale=None):
    m = {"dim": dim, "heads": heads, "kv_heads": kv_heads, "vdim": vdim, "scale": scale or 2.0 * dim ** -0.5}
    if rot:
        m["rot"] = {"dims": rot[0], "base": rot[1]}
    if chunk:
        m["mask"] = {"size": chunk}
    return m


def mlstm(dim=10, heads=2, vdim=14, cap=6.0):
    return {"dim": dim, "heads": heads, "vdim": vdim, "gate_cap": cap}


def parallel(left=None, right=None, left_scale=0.7, right_scale=1.3):
    return {"left": left or attn(), "left_scale": left_scale, "right": right or mlstm(), "right_scale": right_scale}


def layer(kind, mixer, ff=40):
    return {"type": kind, "mixer": mixer, "mlp": {"ff": ff, "kind": "dense"} if ff else None}


def config(layers, loop=None, vocab=211, width=72, eps=1e-5, taps=3, bigram=(97, 31, 11), max_positions=1536):
    cfg = {"architecture": "Ravapel", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width, "canon": {"taps": taps},
           "embedding": {"bigram": {"buckets": bigram[0], "mul_prev": bigram[1], "mul_cur": bigram[2]}}, "max_positions": max_positions}
    if loop:
        cfg["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return cfg


CONFIGS = {
    # both mixers and a layer without a feed-forward; the stretch 1..2 runs twice
    "mixed": lambda: config([layer("hgrn2", hgrn2()), layer("parallel", parallel()), layer("hgrn2", hgrn2(7, 4, 9), None),
                             layer("parallel", parallel(attn(16, 4, 4, 16, (16, 77.0), 50), mlstm(16, 3, 8, 15.0)), 56)], loop=(1, 3, 2)),
    # attention whose scores are sharp: single keys decide a row
    "sharp": lambda: config([layer("hgrn2", hgrn2()), layer("parallel", parallel(attn(scale=2.0), None, 1.5, 0.4)), layer("parallel", parallel(
        attn(chunk=50, scale=2.0), None, 1.5, 0.4), None)], loop=(1, 2, 2)),
    # widths that are multiples of 16, as served models have; the stretch starts at layer 0 and runs three times
    "even": lambda: config([layer("parallel", parallel(attn(48, 4, 2, 32, (32, 10000.0), 130, 0.2), mlstm(32, 4, 64, 15.0), 1.0, 1.0), 176),
                            layer("hgrn2", hgrn2(32, 4, 64), 176), layer("hgrn2", hgrn2(64, 2, 32), 96)], loop=(0, 2, 3), vocab=256, width=128,
                           eps=1e-6, taps=4, bigram=(301, 7, 5)),
    # nothing a multiple of 8; one layer repeated four times; scales of either sign
    "odd": lambda: config([layer("hgrn2", hgrn2(5, 3, 7), 33), layer("parallel", parallel(attn(9, 3, 1, 7, (6, 19.0), 11, 0.9), mlstm(7, 3, 5, 2.5),
                                                                                        -0.6, 1.0), 27), layer("hgrn2", hgrn2(11, 1, 13), None)],
                          loop=(1, 2, 4), vocab=101, width=100, taps=2, bigram=(5, 3, 2), max_positions=700),
    # what a configuration may leave out or make equal: no repeated stretch, no rotation, no chunks, values as wide as keys,
    # every query head with its own keys, one tap, one pair bucket, scales 1
    "plain": lambda: config([layer("parallel", parallel(attn(16, 2, 2, 16, None, None, 0.5), mlstm(16, 2, 16, 1.0), 1.0, 1.0), 32),
                             layer("hgrn2", hgrn2(16, 2, 16), 32)], vocab=97, width=64, taps=1, bigram=(1, 1, 1)),
    # a stretch that runs once, many query heads on one key head, wide heads, many taps
    "wide": lambda: config([layer("parallel", parallel(attn(16, 20, 1, 80, (8, 1000.0), 70, 0.6), mlstm(100, 1, 130)), 24),
                            layer("hgrn2", hgrn2(140, 2, 24), 40), layer("hgrn2", hgrn2(300, 1, 12), None),
                            layer("parallel", parallel(attn(40, 2, 2, 24), mlstm(290, 1, 9)), None)], loop=(0, 3, 1), vocab=97, width=64, taps=6),
    # sizes of a small served model
    "served": lambda: config([layer("hgrn2", hgrn2(128, 4, 128), 1024), layer("parallel", parallel(attn(64, 8, 2, 64, (32, 10000.0), 128, 0.125),
                                                                                               mlstm(64, 4, 128, 15.0), 0.9, 1.1), 1024)],
                             loop=(0, 2, 2), vocab=1000, width=512, eps=1e-6, bigram=(4099, 1009, 17)),
    "hgrn2_only": lambda: config([layer("hgrn2", hgrn2(), None)]),
    "parallel_only": lambda: config([layer("parallel", parallel(), None)]),
    "glu_only": lambda: config([layer("hgrn2", hgrn2(4, 1, 4), 64)]),
    "loop_only": lambda: config([layer("hgrn2", hgrn2(9, 2, 6), None)], loop=(0, 1, 3)),
}

_folders = {}


def make_tensors(cfg: dict, seed: int, sharp: float = 1.0):
    """Random tensors by name (float32 values that bfloat16 holds exactly).  Queries and keys of the recurrences are alike, so
    that a head's result, which is brought to unit size, is rarely the small remainder of a cancellation.  `sharp` scales the attention's queries' norm
    weight: single keys then decide a row."""
    g = torch.Generator().manual_seed(seed)

    def r(t):
        return t.bfloat16().float()

    def mat(o, i, s=1.0):
        return r(torch.randn(o, i, generator=g) * (s / i ** 0.5))

    def vec(n, mean=1.0, s=0.1):
        return r(mean + s * torch.randn(n, generator=g))

    def uni(n, a, b):
        return r(a + (b - a) * torch.rand(n, generator=g))

    w, t = cfg["width"], {}
    t["embed"] = r(torch.randn(cfg["vocab"], w, generator=g))
    t["bigram"] = r(0.7 * torch.randn(cfg["embedding"]["bigram"]["buckets"] + 1, w, generator=g))
    t["pos"] = r(0.5 * torch.randn(cfg["max_positions"], w, generator=g))
    if cfg.get("loop"):
        t["loop.in"] = mat(w, 2 * w)
    for i, l in enumerate(cfg["layers"]):
        p, m = f"l{i}.", l["mixer"]
        for s in ("norm1", "norm1b") + (("norm2", "norm2b") if l.get("mlp") else ()):
            # (what a sublayer adds is half the residual's size: a deep stack of unit-size sublayers would amplify bfloat16's
            # rounding beyond what a tolerance can tell from a fault)
            t[p + s] = vec(w, -0.5 if s.endswith("b") else 0.0, 0.2)
        t[p + "canon1"] = r(0.5 * torch.randn(w, cfg["canon"]["taps"], generator=g))
        if l["type"] == "hgrn2":
            H, D, V = m["heads"], m["dim"], m["vdim"]
            t[p + "mix.q"], t[p + "mix.f"], t[p + "mix.v"] = mat(H * D, w), mat(H * D, w), mat(H * V, w)
            t[p + "mix.f"] = r(0.6 * t[p + "mix.f"] - 0.8 * t[p + "mix.q"])      # (what a query asks for is what its token writes)
            t[p + "mix.f.b"] = uni(H * D, -1.0, 5.0)
            t[p + "mix.lower"] = uni(H * D, 0.0, 0.95)
            t[p + "mix.norm"] = vec(V)
            t[p + "mix.o"] = mat(w, H * V)
        else:
            a, q = m["left"], p + "mix.left."
            H, D = a["heads"], a["dim"]
            G, V = a.get("kv_heads") or H, a.get("vdim") or D
            t[q + "q"], t[q + "k"], t[q + "v"], t[q + "o"] = mat(H * D, w), mat(G * D, w), mat(G * V, w), mat(w, H * V, 0.5)
            t[q + "q.norm"], t[q + "k.norm"] = vec(D, sharp, 0.2), vec(D, 1.0, 0.2)
            t[q + "pb"] = uni(H, -4.0, -1.0)
            a, q = m["right"], p + "mix.right."
            H, D, V = a["heads"], a["dim"], a["vdim"]
            for s, n in (("q", H * D), ("k", H * D), ("v", H * V), ("g", H * V), ("i", H), ("f", H)):
                t[q + s] = mat(n, w)
            t[q + "k"] = r(0.6 * t[q + "k"] + 0.8 * t[q + "q"])
            t[q + "i.b"] = uni(H, -4.0, 2.0)
            t[q + "f.b"] = uni(H, 0.0, 6.0)
            t[q + "norm"] = vec(H * V)
            t[q + "o"] = mat(w, H * V)
        if l.get("mlp"):
            ff = l["mlp"]["ff"]
            for s, o, n in (("gate", ff, w), ("up", ff, w), ("down", w, ff)):
                t[p + "mlp." + s], t[p + "mlp." + s + ".b"] = mat(o, n), vec(o, 0.0, 0.5)
    t["final.norm"] = vec(w, 0.0, 0.2)
    t["head"] = mat(cfg["vocab"], w)
    return t


def write_folder(cfg, tensors, prefix="x0ne_rvp_"):
    from x0ne_engine_b200.weights import write_file
    d = tempfile.mkdtemp(prefix=prefix)
    write_file(os.path.join(d, "model.safetensors"), {k: v.bfloat16() for k, v in tensors.items()})
    with open(os.path.join(d, "config.json"), "w") as f:
        json.dump(cfg, f)
    return d


def folder(name: str, seed: int = 0, sharp: float = 1.0):
    """(folder, config, tensors) of a tiny model written once per (name, seed, sharp)."""
    key = (name, seed, sharp)
    if key not in _folders:
        cfg = CONFIGS[name]()
        tensors = make_tensors(cfg, seed, sharp)
        _folders[key] = (write_folder(cfg, tensors, f"x0ne_rvp_{name}_"), cfg, tensors)
    return _folders[key]


def plain_logits(cfg, tensors, ids, layers_out=None):
    return P.forward(cfg, tensors, list(ids), layers_out=layers_out).numpy()


def plain_greedy(cfg, tensors, prompt, n_new):
    carry, out, ids = {}, [], list(prompt)
    for _ in range(n_new):
        ids = [int(P.forward(cfg, tensors, ids, carry=carry)[-1].argmax())]
        out += ids
    return out


def random_ids(cfg, n, seed=0):
    return [int(t) for t in np.random.default_rng(seed).integers(0, cfg["vocab"], n)]
