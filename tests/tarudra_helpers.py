"""Small Tarudra configurations and model folders with random weights for the tests.

Sizes lie away from powers of two and from each other (key width != value width, heads != kv heads, rotated widths below the
key width and equal to it, latents of 5 to 200 values, delta heads of 5 to 300 channels, 1 to 6 taps, widths that are no
multiple of 8), windows that do not line up with the pages of 64, layers that read an earlier layer's keys under a wider and a
narrower window, layers without a feed-forward.  Weights are drawn here, not by the package's initialiser, so that the delta
states' memories reach from a few tokens to hundreds, and norm weights, layer scales and biases take values that matter.
"""
import json
import os
import tempfile

import numpy as np
import torch

import tarudra_plain as P

P.PRECISION = torch.float64      # the reference of the tests is the plain implementation in double precision

YARN = {"factor": 4.0, "original": 60, "fast": 4.0, "slow": 0.5}


def attn(dim=20, heads=6, kv_heads=2, vdim=12, rot=(8, 300.0, YARN), window=37, scale=None, kv_from=None):
    m = {"dim": dim, "heads": heads, "kv_heads": kv_heads, "vdim": vdim, "scale": scale or dim ** -0.5}
    if rot:
        m["rot"] = {"dims": rot[0], "base": rot[1]}
        if len(rot) > 2:
            m["rot"]["scaling"] = dict(rot[2])
    if window:
        m["mask"] = {"size": window}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return m


def latent(dim=10, heads=5, vdim=14, kv_rank=22, q_rank=13, rot_dim=6, base=90.0, window=45, scale=None):
    m = {"dim": dim, "heads": heads, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank, "rot_dim": rot_dim, "scale": scale or (dim + rot_dim) ** -0.5,
         "rot": {"base": base, "dims": rot_dim}}
    if window:
        m["mask"] = {"size": window}
    return m


def delta(dim=12, heads=6, kv_heads=3, vdim=20, conv=3):
    return {"dim": dim, "heads": heads, "kv_heads": kv_heads, "vdim": vdim, "conv": conv}


def layer(kind, mixer, ff=40):
    return {"type": kind, "mixer": mixer, "mlp": {"ff": ff, "kind": "dense"} if ff else None}


def config(layers, vocab=211, width=72, eps=1e-5, cap=17.0):
    cfg = {"architecture": "Tarudra", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width}
    if cap:
        cfg["logit_softcap"] = cap
    return cfg


A, L, D = "attention", "latent_attention", "delta"

CONFIGS = {
    # every mixer, readers with a wider and a narrower window than the layer whose keys they read (and other head counts), a
    # layer without a feed-forward
    "mixed": lambda: config([layer(L, latent()), layer(A, attn()), layer(D, delta()), layer(A, attn(heads=4, window=90, scale=0.3, kv_from=1)),
                             layer(D, delta(7, 4, 4, 9, 4), None), layer(A, attn(heads=2, window=11, kv_from=1), 24)]),
    # scores sharp enough that single keys decide a row
    "sharp": lambda: config([layer(L, latent(scale=1.3)), layer(A, attn(window=50, scale=0.9)), layer(A, attn(window=70, scale=0.9, kv_from=1), None)], cap=40.0),
    # widths that are multiples of 16, as served models have
    "even": lambda: config([layer(D, delta(32, 4, 2, 64, 4), 176), layer(L, latent(48, 4, 32, 96, 64, 32, 10000.0, 130), 176),
                            layer(A, attn(64, 8, 2, 64, (64, 10000.0, {"factor": 8.0, "original": 128, "fast": 32.0, "slow": 1.0}), 100), 96),
                            layer(D, delta(64, 2, 2, 32, 4), 176)], vocab=256, width=128, eps=1e-6, cap=30.0),
    # nothing a multiple of 8; rotation without scaling
    "odd": lambda: config([layer(D, delta(5, 3, 1, 7, 2), 33), layer(L, latent(7, 3, 5, 11, 5, 2, 19.0, 11), 27), layer(A, attn(9, 3, 1, 7, (6, 19.0), 13, 0.5), None),
                           layer(D, delta(11, 1, 1, 13, 6), None)], vocab=101, width=100, cap=9.0),
    # what a configuration may leave out or make equal: no caps, no windows, no scaled or no rotation at all, values as wide as keys,
    # every head with keys of its own, one tap, ranks equal to one another
    "plain": lambda: config([layer(A, attn(16, 2, 2, 16, None, None, 0.25), 32), layer(L, latent(16, 2, 16, 16, 16, 16, 100.0, None), 32),
                             layer(D, delta(16, 2, 2, 16, 1), 32), layer(A, attn(16, 2, 2, 16, (16, 10000.0), None), 32)], vocab=97, width=64, cap=None),
    # many query heads on one key head, wide heads, wide latents, many taps
    "wide": lambda: config([layer(A, attn(24, 20, 1, 80, (24, 1000.0, YARN), 70, 0.2), 24), layer(L, latent(40, 3, 90, 200, 150, 24, 1000.0, 66), 40),
                            layer(D, delta(140, 2, 1, 24, 6), 40), layer(D, delta(300, 1, 1, 12, 2), None), layer(D, delta(200, 2, 2, 300, 3), None)], vocab=97, width=64),
    # sizes of a small served model
    "served": lambda: config([layer(D, delta(128, 4, 2, 128, 4), 1024), layer(A, attn(64, 8, 2, 64, (64, 10000.0, {"factor": 4.0, "original": 512, "fast": 32.0, "slow": 1.0}),
                                                                                   128, 0.125), 1024),
                              layer(L, latent(64, 4, 64, 128, 192, 32, 10000.0, 200), 1024), layer(A, attn(64, 8, 2, 64, (64, 10000.0, {
                                  "factor": 4.0, "original": 512, "fast": 32.0, "slow": 1.0}), 64, 0.125, 1), 1024)], vocab=1000, width=512, eps=1e-6, cap=50.0),
    "latent_only": lambda: config([layer(L, latent(), None)]),
    "attn_only": lambda: config([layer(A, attn(), None)]),
    "delta_only": lambda: config([layer(D, delta(), None)]),
    "mlp_only": lambda: config([layer(D, delta(4, 1, 1, 4, 1), 64)], cap=3.0),
    "reader_only": lambda: config([layer(A, attn(window=5), None), layer(A, attn(window=60, kv_from=0), None)]),
}

_folders = {}


def make_tensors(cfg: dict, seed: int):
    """Random tensors by name (float32 values that bfloat16 holds exactly).  Queries and keys of the delta rule are alike, so that
    a head's result, which is brought to unit size, is rarely the small remainder of a cancellation."""
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
    t["embed"] = r(0.3 + torch.randn(cfg["vocab"], w, generator=g))          # (rows with a mean: a norm that kept it would show)
    for i, l in enumerate(cfg["layers"]):
        p, m = f"l{i}.", l["mixer"]
        for s in ("1",) + (("2",) if l.get("mlp") else ()):
            t[p + "norm" + s], t[p + "norm" + s + "b"], t[p + "ls" + s] = vec(w, 1.0, 0.2), vec(w, 0.8, 0.2), vec(w, 0.6, 0.2)
        q = p + "mix."
        if l["type"] == "attention":
            H, D_, G, V = m["heads"], m["dim"], m["kv_heads"], m["vdim"]
            rows = {"q": H * D_, "k": G * D_, "v": G * V}
            for s in ("q",) if m.get("kv_from") is not None else ("q", "k", "v"):
                t[q + s], t[q + s + ".b"] = mat(rows[s], w), vec(rows[s], 0.0, 0.5)
            t[q + "o"], t[q + "o.b"] = mat(w, H * V), vec(w, 0.0, 0.3)
        elif l["type"] == "latent_attention":
            H, D_, rr, V, R, Q = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], m["q_rank"]
            t[q + "dq"], t[q + "dq.norm"], t[q + "uq"] = mat(Q, w), vec(Q, 1.0, 0.2), mat(H * (D_ + rr), Q)
            t[q + "dkv"], t[q + "dkv.norm"] = mat(R + rr, w), vec(R, 1.0, 0.2)
            t[q + "uk"], t[q + "uv"], t[q + "g"], t[q + "o"] = mat(H * D_, R), mat(H * V, R), mat(H * V, w), mat(w, H * V)
        else:
            H, G, D_, V, K = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"]
            for s, n in (("q", G * D_), ("k", G * D_), ("v", H * V)):
                t[q + s], t[q + s + ".conv"] = mat(n, w), r(0.6 * torch.randn(n, K, generator=g))
            t[q + "k"] = r(0.6 * t[q + "k"] + 0.8 * t[q + "q"])
            t[q + "k.conv"] = r(0.6 * t[q + "k.conv"] + 0.8 * t[q + "q.conv"])
            t[q + "a"], t[q + "b"], t[q + "g"], t[q + "o"] = mat(H, w), mat(H, w), mat(H * V, w), mat(w, H * V)
            t[q + "A_log"], t[q + "dt_bias"], t[q + "norm"] = uni(H, -2.0, 1.0), uni(H, -6.0, 0.0), vec(V)
        if l.get("mlp"):
            t[p + "mlp.up"], t[p + "mlp.down"] = mat(l["mlp"]["ff"], w), mat(w, l["mlp"]["ff"])
    t["final.norm"] = vec(w, 1.0, 0.2)
    t["head"] = mat(cfg["vocab"], w, 3.0)
    return t


def write_folder(cfg, tensors, prefix="x0ne_trd_"):
    from x0ne_engine_b200.weights import write_file
    d = tempfile.mkdtemp(prefix=prefix)
    write_file(os.path.join(d, "model.safetensors"), {k: v.bfloat16() for k, v in tensors.items()})
    with open(os.path.join(d, "config.json"), "w") as f:
        json.dump(cfg, f)
    return d


def folder(name: str, seed: int = 0):
    """(folder, config, tensors) of a tiny model written once per (name, seed)."""
    key = (name, seed)
    if key not in _folders:
        cfg = CONFIGS[name]()
        tensors = make_tensors(cfg, seed)
        _folders[key] = (write_folder(cfg, tensors, f"x0ne_trd_{name}_"), cfg, tensors)
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
