"""Tarudra restated in plain PyTorch on the CPU, one function per mechanism.

Nothing here is shared with the package: the functions take a config.json as a dict and the checkpoint tensors by
name (any dtype; they are widened to the working precision), run a sequence with explicit loops over tokens (the
delta rule, the convolutions) or full T x T score matrices (the attentions), and return the logits of every position.

Notation: T tokens, width W.  Attention: H query heads, G key/value heads, key width D, value width Dv.  Latent
attention: latent width R, rotated width r.  Delta rule: H value heads, G query/key heads, D state rows, Dv columns, K taps.
"""
from __future__ import annotations

import math
from typing import List, Mapping, Optional

import torch

PRECISION = torch.float32      # the tests set float64: the same equations, as a sharper reference
UNIT_EPS = 1e-6                # under the root of the delta rule's unit vectors


def wide(t: torch.Tensor) -> torch.Tensor:
    return t.detach().to("cpu", PRECISION)


# ------------------------------------------------------------------------------------------ norms, activations
def layer_norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    d = x - x.mean(dim=-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(dim=-1, keepdim=True) + eps) * w


def unit_rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def unit_vector(x: torch.Tensor, eps: float = UNIT_EPS) -> torch.Tensor:
    return x / torch.sqrt((x * x).sum(dim=-1, keepdim=True) + eps)


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def softplus(z: torch.Tensor) -> torch.Tensor:
    return torch.clamp(z, min=0.0) + torch.log1p(torch.exp(-z.abs()))


def relu_squared(z: torch.Tensor) -> torch.Tensor:
    return torch.clamp(z, min=0.0) ** 2


def soft_cap(z: torch.Tensor, cap: Optional[float]) -> torch.Tensor:
    return z if not cap else cap * torch.tanh(z / cap)


# ------------------------------------------------------------------------------------------ rotation
def yarn(dims: int, base: float, scaling: Optional[Mapping]):
    """(frequency of every pair, factor on cosine and sine), as Python floats."""
    freq = [float(base) ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not scaling:
        return freq, 1.0

    def pair_of(turns):
        return dims * math.log(scaling["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo = max(math.floor(pair_of(scaling["fast"])), 0)
    hi = min(math.ceil(pair_of(scaling["slow"])), dims - 1)
    out = []
    for i, f in enumerate(freq):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / scaling["factor"] * ramp + f * (1.0 - ramp))
    return out, 0.1 * math.log(scaling["factor"]) + 1.0


def rotate(x: torch.Tensor, positions: torch.Tensor, rot: Optional[Mapping], layout: str) -> torch.Tensor:
    """x [T, heads, D]; the first `dims` values of every head turn: "interleaved" pairs 2i with 2i + 1, "half" i with
    i + dims / 2."""
    if not rot or not rot["dims"]:
        return x
    dims = rot["dims"]
    freq, mag = yarn(dims, rot["base"], rot.get("scaling"))
    ang = positions.to(PRECISION)[:, None] * torch.tensor(freq, dtype=PRECISION)[None, :]
    c, s = mag * torch.cos(ang)[:, None, :], mag * torch.sin(ang)[:, None, :]
    out = x.clone()
    a, b = (slice(0, dims, 2), slice(1, dims, 2)) if layout == "interleaved" else (slice(0, dims // 2), slice(dims // 2, dims))
    u, v = x[..., a], x[..., b]
    out[..., a], out[..., b] = u * c - v * s, v * c + u * s
    return out


# ------------------------------------------------------------------------------------------ attention
def windowed_attention(q, k, v, scale: float, positions: torch.Tensor, window: Optional[int], extra_term: bool):
    """q [T, H, D], k [T, G, D], v [T, G, Dv] of ONE sequence, rows at `positions`.  Query i sees key j where
    0 <= i - j < window; `extra_term` adds one to every softmax denominator."""
    T, H, _ = q.shape
    rep = H // k.shape[1]
    back = positions[:, None] - positions[None, :]
    seen = back >= 0
    if window:
        seen = seen & (back < window)
    out = torch.zeros(T, H, v.shape[-1], dtype=q.dtype)
    for h in range(H):
        s = (q[:, h] @ k[:, h // rep].T) * scale
        s = s.masked_fill(~seen, float("-inf"))
        top = s.max(dim=-1, keepdim=True).values
        if extra_term:
            top = torch.clamp(top, min=0.0)
        e = torch.exp(s - top)
        den = e.sum(dim=-1, keepdim=True) + (torch.exp(-top) if extra_term else 0.0)
        out[:, h] = (e / den) @ v[:, h // rep]
    return out


def attention_keys(h, t, p: str, m: Mapping, positions):
    T, G = h.shape[0], m["kv_heads"]
    k = (h @ wide(t[p + ".k"]).T + wide(t[p + ".k.b"])).reshape(T, G, m["dim"])
    v = (h @ wide(t[p + ".v"]).T + wide(t[p + ".v.b"])).reshape(T, G, m["vdim"])
    return rotate(k, positions, m.get("rot"), "interleaved"), v


def attention_mixer(h, t, p: str, m: Mapping, positions, kv):
    T, H = h.shape[0], m["heads"]
    q = (h @ wide(t[p + ".q"]).T + wide(t[p + ".q.b"])).reshape(T, H, m["dim"])
    q = rotate(q, positions, m.get("rot"), "interleaved")
    o = windowed_attention(q, kv[0], kv[1], m["scale"], positions, (m.get("mask") or {}).get("size"), True)
    return o.reshape(T, H * m["vdim"]) @ wide(t[p + ".o"]).T + wide(t[p + ".o.b"])


def latent_mixer(h, t, p: str, m: Mapping, eps: float, positions):
    T, H, D, r, Dv, R = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    cq = unit_rms(h @ wide(t[p + ".dq"]).T, eps) * wide(t[p + ".dq.norm"])
    q = (cq @ wide(t[p + ".uq"]).T).reshape(T, H, D + r)
    down = h @ wide(t[p + ".dkv"]).T
    c = unit_rms(down[:, :R], eps) * wide(t[p + ".dkv.norm"])
    q_rot = rotate(q[..., D:], positions, m["rot"], "half")
    k_rot = rotate(down[:, None, R:], positions, m["rot"], "half")
    k = torch.cat([(c @ wide(t[p + ".uk"]).T).reshape(T, H, D), k_rot.expand(T, H, r)], dim=-1)
    v = (c @ wide(t[p + ".uv"]).T).reshape(T, H, Dv)
    o = windowed_attention(torch.cat([q[..., :D], q_rot], dim=-1), k, v, m["scale"], positions, (m.get("mask") or {}).get("size"), False)
    o = o.reshape(T, H * Dv) * torch.sigmoid(h @ wide(t[p + ".g"]).T)
    return o @ wide(t[p + ".o"]).T


# ------------------------------------------------------------------------------------------ delta rule
def causal_conv(x: torch.Tensor, w: torch.Tensor, before: Optional[torch.Tensor] = None):
    """x [T, C], w [C, K]; the last column of w meets the row itself; `before` [K - 1, C]: the rows ahead of row 0.
    Returns (convolved rows, the last K - 1 rows)."""
    T, C = x.shape
    K = w.shape[1]
    if before is None:
        before = torch.zeros(K - 1, C, dtype=x.dtype)
    ext = torch.cat([before.to(x.dtype), x], dim=0)
    y = torch.stack([(ext[i:i + K].T * w).sum(dim=-1) for i in range(T)])
    return y, ext[ext.shape[0] - (K - 1):].clone()


def delta_scan(q, k, v, beta, g, S):
    """q, k [T, H, D], v [T, H, Dv], beta, g [T, H]; S [H, D, Dv] is changed in place."""
    out = torch.zeros_like(v)
    for t in range(q.shape[0]):
        S.mul_(g[t][:, None, None])
        u = beta[t][:, None] * (v[t] - (S * k[t][:, :, None]).sum(dim=1))
        S.add_(k[t][:, :, None] * u[:, None, :])
        out[t] = (S * q[t][:, :, None]).sum(dim=1)
    return out


def delta_gates(h, t, p: str):
    beta = torch.sigmoid(h @ wide(t[p + ".b"]).T)
    g = torch.exp(-torch.exp(wide(t[p + ".A_log"])) * softplus(h @ wide(t[p + ".a"]).T + wide(t[p + ".dt_bias"])))
    return beta, g


def delta_mixer(h, t, p: str, m: Mapping, eps: float, state: Optional[dict] = None):
    T, H, D, Dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    G = m.get("kv_heads") or H
    st = {} if state is None else state
    r = {}
    for s in ("q", "k", "v"):
        y, st["conv." + s] = causal_conv(h @ wide(t[f"{p}.{s}"]).T, wide(t[f"{p}.{s}.conv"]), st.get("conv." + s))
        r[s] = silu(y)
    spread = torch.arange(H) // (H // G)
    q = unit_vector(r["q"].reshape(T, G, D))[:, spread] * D ** -0.5
    k = unit_vector(r["k"].reshape(T, G, D))[:, spread]
    beta, g = delta_gates(h, t, p)
    if "S" not in st:
        st["S"] = torch.zeros(H, D, Dv, dtype=h.dtype)
    o = delta_scan(q, k, r["v"].reshape(T, H, Dv), beta, g, st["S"])
    o = unit_rms(o, eps) * wide(t[p + ".norm"]) * silu(h @ wide(t[p + ".g"]).T).reshape(T, H, Dv)
    return o.reshape(T, H * Dv) @ wide(t[p + ".o"]).T


# ------------------------------------------------------------------------------------------ the model
def forward(cfg: Mapping, t: Mapping[str, torch.Tensor], tokens, layers_out: Optional[list] = None, carry: Optional[dict] = None):
    """Logits [T, vocab] of the next `tokens` of a sequence; `layers_out` receives the residual stream after every layer.
    `carry` (a dict, empty at a sequence's start) takes the sequence over several calls: position, and per layer the delta
    rule's state and convolution inputs, or the attention's inputs of all earlier rows."""
    eps = cfg["norm"]["eps"]
    ids: List[int] = [int(x) for x in tokens]
    T = len(ids)
    c = {} if carry is None else carry
    pos0 = c.get("pos", 0)
    c["pos"] = pos0 + T
    positions = torch.arange(pos0 + T)
    x = wide(t["embed"])[ids]
    kept = c.setdefault("layers", {})
    kv = {}
    for i, L in enumerate(cfg["layers"]):
        p, m, st = f"l{i}", L["mixer"], kept.setdefault(i, {})
        h = layer_norm(x, wide(t[p + ".norm1"]), eps)
        if L["type"] == "delta":
            y = delta_mixer(h, t, p + ".mix", m, eps, st)
        else:
            h_all = st["h"] = torch.cat([st["h"], h], dim=0) if "h" in st else h
            if L["type"] == "attention":
                src = m.get("kv_from")
                if src is None:
                    kv[i] = attention_keys(h_all, t, p + ".mix", m, positions)
                y = attention_mixer(h_all, t, p + ".mix", m, positions, kv[i if src is None else src])[pos0:]
            else:
                y = latent_mixer(h_all, t, p + ".mix", m, eps, positions)[pos0:]
        x = x + layer_norm(y, wide(t[p + ".norm1b"]), eps) * wide(t[p + ".ls1"])
        if L.get("mlp") is not None:
            h = layer_norm(x, wide(t[p + ".norm2"]), eps)
            y = relu_squared(h @ wide(t[p + ".mlp.up"]).T) @ wide(t[p + ".mlp.down"]).T
            x = x + layer_norm(y, wide(t[p + ".norm2b"]), eps) * wide(t[p + ".ls2"])
        if layers_out is not None:
            layers_out.append(x.clone())
    return soft_cap(layer_norm(x, wide(t["final.norm"]), eps) @ wide(t["head"]).T, cfg.get("logit_softcap"))
