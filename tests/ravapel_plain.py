"""Ravapel restated in plain PyTorch on the CPU, one function per mechanism.

Nothing here is shared with the package: the functions take a config.json as a dict and the checkpoint tensors by
name (any dtype; they are widened to the working precision), run a sequence with explicit loops over tokens (the
recurrences, the convolution) or full T x T score matrices (the attention), and return the logits of every position.

Notation: T tokens, width W.  Attention: H query heads, G key/value heads, key width D, value width Dv.  Recurrences: H
heads, D state rows, Dv state columns.  K convolution taps.
"""
from __future__ import annotations

import math
from typing import List, Mapping, Optional

import torch

PRECISION = torch.float32      # the tests set float64: the same equations, as a sharper reference


def wide(t: torch.Tensor) -> torch.Tensor:
    return t.detach().to("cpu", PRECISION)


# ------------------------------------------------------------------------------------------ norms, activations
def unit_rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def zero_centred_norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    """The stored weight is what is added to one."""
    return unit_rms(x, eps) * (1.0 + w)


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def log_sigmoid(z: torch.Tensor) -> torch.Tensor:
    return torch.where(z > 0, -torch.log1p(torch.exp(-z.abs())), z - torch.log1p(torch.exp(-z.abs())))


# ------------------------------------------------------------------------------------------ embedding
def bigram_row(prev: Optional[int], cur: int, buckets: int, mul_prev: int, mul_cur: int) -> int:
    return buckets if prev is None else (prev * mul_prev + cur * mul_cur) % buckets


def embed(t: Mapping[str, torch.Tensor], cfg: Mapping, ids: List[int], pos0: int = 0, prev: Optional[int] = None) -> torch.Tensor:
    """`prev`: the token before ids[0] (None: ids[0] is the sequence's first)."""
    b = cfg["embedding"]["bigram"]
    rows = []
    for i, tok in enumerate(ids):
        rows.append(wide(t["embed"][tok]) + wide(t["bigram"][bigram_row(prev, tok, b["buckets"], b["mul_prev"], b["mul_cur"])])
                    + wide(t["pos"][pos0 + i]))
        prev = tok
    return torch.stack(rows)


# ------------------------------------------------------------------------------------------ convolution
def input_conv(h: torch.Tensor, w: torch.Tensor, before: Optional[torch.Tensor] = None):
    """h [T, W], w [W, K]; the last column of w meets the row itself, the one before it the row above, and so on;
    `before` [K - 1, W]: the inputs ahead of row 0.  Returns (h + conv(h), the last K - 1 inputs)."""
    T, W = h.shape
    K = w.shape[1]
    if before is None:
        before = torch.zeros(K - 1, W, dtype=h.dtype)
    ext = torch.cat([before.to(h.dtype), h], dim=0)
    y = torch.empty_like(h)
    for t in range(T):
        y[t] = h[t] + (ext[t:t + K].T * w).sum(dim=-1)
    return y, ext[ext.shape[0] - (K - 1):].clone()


# ------------------------------------------------------------------------------------------ rotation, attention
def rotate_half(x: torch.Tensor, positions: torch.Tensor, dims: int, base: float) -> torch.Tensor:
    """x [T, heads, D]: value i and value i + dims / 2 of every head turn by position * base^(-2i / dims)."""
    if not dims:
        return x
    n = dims // 2
    freq = torch.tensor([float(base) ** (-2.0 * i / dims) for i in range(n)], dtype=PRECISION)
    ang = positions.to(PRECISION)[:, None] * freq[None, :]
    c, s = torch.cos(ang)[:, None, :], torch.sin(ang)[:, None, :]
    u, v = x[..., :n], x[..., n:dims]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], dim=-1)


def sigmoid_attention(q, k, v, scale: float, bias: torch.Tensor, positions: torch.Tensor, chunk: int = 0):
    """q [T, H, D], k [T, G, D], v [T, G, Dv] of ONE sequence, rows at `positions`.  The weight of key j for query i is
    sigmoid(q_i . k_j scale + bias_h) where j <= i and both lie in the same chunk, else 0; nothing is normalised."""
    T, H, _ = q.shape
    rep = H // k.shape[1]
    pi, pj = positions[:, None], positions[None, :]
    seen = pj <= pi
    if chunk:
        seen = seen & (torch.div(pi, chunk, rounding_mode="floor") == torch.div(pj, chunk, rounding_mode="floor"))
    out = torch.zeros(T, H, v.shape[-1], dtype=q.dtype)
    for h in range(H):
        g = h // rep
        w = torch.sigmoid((q[:, h] @ k[:, g].T) * scale + bias[h]) * seen
        out[:, h] = w @ v[:, g]
    return out


def attention_mixer(h, t, p: str, m: Mapping, eps: float, positions):
    T = h.shape[0]
    H, D = m["heads"], m["dim"]
    G, Dv = m.get("kv_heads") or H, m.get("vdim") or D
    rot = m.get("rot") or {"dims": 0, "base": 1.0}
    q = unit_rms((h @ wide(t[p + ".q"]).T).reshape(T, H, D), eps) * wide(t[p + ".q.norm"])
    k = unit_rms((h @ wide(t[p + ".k"]).T).reshape(T, G, D), eps) * wide(t[p + ".k.norm"])
    v = (h @ wide(t[p + ".v"]).T).reshape(T, G, Dv)
    q, k = (rotate_half(x, positions, rot["dims"], rot["base"]) for x in (q, k))
    o = sigmoid_attention(q, k, v, m["scale"], wide(t[p + ".pb"]), positions, (m.get("mask") or {}).get("size", 0))
    return o.reshape(T, H * Dv) @ wide(t[p + ".o"]).T


# ------------------------------------------------------------------------------------------ recurrences
def gated_outer_scan(q, k, v, f, S):
    """q, k, f [T, H, D], v [T, H, Dv]; S [H, D, Dv] is changed in place.  S = f S + k v^T (f on the rows), o = S^T q."""
    out = torch.zeros_like(v)
    for t in range(q.shape[0]):
        S.mul_(f[t][:, :, None]).add_(k[t][:, :, None] * v[t][:, None, :])
        out[t] = (S * q[t][:, :, None]).sum(dim=1)
    return out


def hgrn2_mixer(h, t, p: str, m: Mapping, eps: float, state: Optional[dict] = None):
    T = h.shape[0]
    H, D = m["heads"], m["dim"]
    Dv = m.get("vdim") or D
    low = wide(t[p + ".lower"])
    q = silu(h @ wide(t[p + ".q"]).T).reshape(T, H, D)
    v = (h @ wide(t[p + ".v"]).T).reshape(T, H, Dv)
    z = h @ wide(t[p + ".f"]).T + wide(t[p + ".f.b"])
    f = (low + (1.0 - low) * torch.sigmoid(z)).reshape(T, H, D)
    k = ((1.0 - low) * torch.sigmoid(-z)).reshape(T, H, D)             # 1 - f
    S = torch.zeros(H, D, Dv, dtype=h.dtype) if state is None or "S" not in state else state["S"]
    o = gated_outer_scan(q, k, v, f, S)
    if state is not None:
        state["S"] = S
    o = unit_rms(o, eps) * wide(t[p + ".norm"])
    return o.reshape(T, H * Dv) @ wide(t[p + ".o"]).T


def capped(z, cap: float):
    return cap * torch.tanh(z / cap)


def mlstm_scan(q, k, v, i, f, S, n, m):
    """q, k [T, H, D], v [T, H, Dv], i, f [T, H] (logarithms); S [H, D, Dv], n [H, D], m [H] are changed in place."""
    out = torch.zeros_like(v)
    for t in range(q.shape[0]):
        m_new = torch.maximum(f[t] + m, i[t])
        keep, write = torch.exp(f[t] + m - m_new), torch.exp(i[t] - m_new)
        m.copy_(m_new)
        S.mul_(keep[:, None, None]).add_(write[:, None, None] * k[t][:, :, None] * v[t][:, None, :])
        n.mul_(keep[:, None]).add_(write[:, None] * k[t])
        den = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-m)) + 1e-6
        out[t] = (S * q[t][:, :, None]).sum(dim=1) / den[:, None]
    return out


def mlstm_mixer(h, t, p: str, m: Mapping, eps: float, state: Optional[dict] = None):
    T = h.shape[0]
    H, D = m["heads"], m["dim"]
    Dv, cap = m.get("vdim") or D, float(m["gate_cap"])
    q = (h @ wide(t[p + ".q"]).T).reshape(T, H, D) / math.sqrt(D)
    k = (h @ wide(t[p + ".k"]).T).reshape(T, H, D)
    v = (h @ wide(t[p + ".v"]).T).reshape(T, H, Dv)
    i = capped(h @ wide(t[p + ".i"]).T + wide(t[p + ".i.b"]), cap)
    f = log_sigmoid(capped(h @ wide(t[p + ".f"]).T + wide(t[p + ".f.b"]), cap))
    st = {} if state is None else state
    if "S" not in st:
        st["S"], st["n"], st["m"] = (torch.zeros(*s, dtype=h.dtype) for s in ((H, D, Dv), (H, D), (H,)))
    o = unit_rms(mlstm_scan(q, k, v, i, f, st["S"], st["n"], st["m"]), eps).reshape(T, H * Dv)
    o = o * wide(t[p + ".norm"]) * torch.sigmoid(h @ wide(t[p + ".g"]).T)
    return o @ wide(t[p + ".o"]).T


# ------------------------------------------------------------------------------------------ feed-forward
def biased_glu(h, t, p: str):
    gate = h @ wide(t[p + ".gate"]).T + wide(t[p + ".gate.b"])
    up = h @ wide(t[p + ".up"]).T + wide(t[p + ".up.b"])
    return (silu(gate) * up) @ wide(t[p + ".down"]).T + wide(t[p + ".down.b"])


# ------------------------------------------------------------------------------------------ the model
def run_order(cfg: Mapping) -> List[tuple]:
    """(layer, whether a pass of the repeated stretch opens with this run) for every layer run."""
    n, lp = len(cfg["layers"]), cfg.get("loop")
    if not lp:
        return [(i, False) for i in range(n)]
    stretch = [(i, i == lp["start"]) for i in range(lp["start"], lp["stop"])]
    return [(i, False) for i in range(lp["start"])] + stretch * lp["times"] + [(i, False) for i in range(lp["stop"], n)]


def forward(cfg: Mapping, t: Mapping[str, torch.Tensor], tokens, layers_out: Optional[list] = None, carry: Optional[dict] = None):
    """Logits [T, vocab] of the next `tokens` of a sequence; `layers_out` receives the residual stream after every layer
    run.  `carry` (a dict, empty at a sequence's start) takes the sequence over several calls: position, previous token,
    and per layer run the convolution's inputs, the states, and the attention's inputs of all earlier rows."""
    eps = cfg["norm"]["eps"]
    ids = [int(x) for x in tokens]
    T = len(ids)
    c = {} if carry is None else carry
    pos0 = c.get("pos", 0)
    x = embed(t, cfg, ids, pos0, c.get("prev"))
    c["pos"], c["prev"] = pos0 + T, ids[-1]
    x0 = x
    runs = c.setdefault("runs", {})
    for run, (i, opens) in enumerate(run_order(cfg)):
        L, p = cfg["layers"][i], f"l{i}"
        m, st = L["mixer"], runs.setdefault(run, {})
        if opens:
            x = torch.cat([x, x0], dim=-1) @ wide(t["loop.in"]).T
        h = zero_centred_norm(x, wide(t[p + ".norm1"]), eps)
        h, st["conv"] = input_conv(h, wide(t[p + ".canon1"]), st.get("conv"))
        if L["type"] == "hgrn2":
            y = hgrn2_mixer(h, t, p + ".mix", m, eps, st.setdefault("rec", {}))
        else:
            h_all = st["h"] = torch.cat([st["h"], h], dim=0) if "h" in st else h
            left = attention_mixer(h_all, t, p + ".mix.left", m["left"], eps, torch.arange(pos0 + T))[pos0:]
            right = mlstm_mixer(h, t, p + ".mix.right", m["right"], eps, st.setdefault("rec", {}))
            y = m["left_scale"] * left + m["right_scale"] * right
        x = x + zero_centred_norm(y, wide(t[p + ".norm1b"]), eps)
        if L.get("mlp") is not None:
            y = biased_glu(zero_centred_norm(x, wide(t[p + ".norm2"]), eps), t, p + ".mlp")
            x = x + zero_centred_norm(y, wide(t[p + ".norm2b"]), eps)
        if layers_out is not None:
            layers_out.append(x.clone())
    return zero_centred_norm(x, wide(t["final.norm"]), eps) @ wide(t["head"]).T
