"""Ravapel on the GPU against the plain implementation (tests/ravapel_plain.py), in float32 and bfloat16: every mechanism
alone, whole prompts, token-by-token decoding, portions down to two tokens, unequal batches with slots, pages and states used
again, the chunk's edge in prompts and in decoding, far keys and a far token in each recurrent state, the first tokens, long
decoding, odd sizes and values a configuration may leave out or make equal, and greedy generation through the entry point."""
import numpy as np
import pytest
import torch

import ravapel_helpers as H
import ravapel_plain as P
from helpers import BF16_KL_TOL, BF16_LOGIT_TOL, BF16_SELF_TOL, assert_close_f32, first_difference, kl_rows

pytestmark = pytest.mark.gpu

DTYPES = ["float32", "bfloat16"]
TORCH = {"float32": torch.float32, "bfloat16": torch.bfloat16}
DEV = "cuda:0"
_engines = {}


def engine(name, dtype, seed=0, sharp=1.0, max_tokens=1024, **kw):
    from x0ne_engine_b200 import Engine
    key = (name, dtype, seed, sharp, max_tokens, tuple(sorted(kw.items())))
    if key not in _engines:
        folder, cfg, tensors = H.folder(name, seed, sharp)
        _engines[key] = (Engine.from_folder(folder, dtype=dtype, max_tokens=max_tokens, max_seq_len=max_tokens, **kw), cfg, tensors)
    return _engines[key]


def rows_within(err, tol, what):
    """Every row within the tolerance, but that of many rows one in fifty (or one) may reach twice that: a head whose result is
    the remainder of a cancellation is brought back to unit size, which amplifies the rounding of what went in."""
    over = int((err > tol).sum())
    assert err.max() <= 2 * tol and over <= max(1, len(err) // 50), f"{what}: worst {err.max():.3e}, {over} of {len(err)} rows over {tol}"


def check(dtype, got, want, what):
    if dtype == "float32":
        assert_close_f32(got, want, what)
        return
    got, want = np.asarray(got, dtype=np.float64), np.asarray(want, dtype=np.float64)
    assert got.shape == want.shape and np.isfinite(got).all(), what
    rows_within(np.abs(got - want).max(-1) / (np.abs(want).max(-1) + 1e-30), BF16_LOGIT_TOL, what + ": logit error")
    rows_within(kl_rows(want, got), BF16_KL_TOL, what + ": KL")


def same_cut(dtype, got, base, what):
    """Another cut of the same work: the same bits in float32, the same to rounding in bfloat16."""
    if dtype == "float32":
        assert first_difference(got, base) is None, f"{what}: first difference at {first_difference(got, base)}"
    else:
        rows_within(np.abs(got - base).max(-1) / np.abs(base).max(-1), 2 * BF16_SELF_TOL, what)


def in_pieces(eng, ids, cuts):
    """Logits of every position, the sequence brought in pieces of the given lengths (the rest in one)."""
    slot, out, at = eng.new_sequence(), [], 0
    cuts = list(cuts) + ([len(ids) - sum(cuts)] if sum(cuts) < len(ids) else [])
    for n in cuts:
        out.append(eng.step([slot], [ids[at:at + n]], [list(range(n))]).cpu().numpy())
        at += n
    eng.free_sequence(slot)
    return np.concatenate(out)


def whole(eng, ids):
    return in_pieces(eng, ids, [])


# ------------------------------------------------------------------------------------------ the recurrences
SCAN_SIZES = [(2, 12, 20), (3, 5, 7), (1, 64, 16), (2, 33, 17), (2, 100, 20), (1, 128, 128), (3, 130, 9), (1, 200, 40), (1, 256, 33), (2, 300, 10)]


def tables(lengths, slots):
    first = torch.tensor(np.concatenate([[0], np.cumsum(lengths)]), dtype=torch.int32, device=DEV)
    return first, torch.tensor(slots, dtype=torch.int32, device=DEV)


class ChannelGated:
    """Raw inputs of a recurrence with a gate per channel, run through the kernels and through the plain scan."""
    head_gates = False

    def __init__(self, heads, dim, vd, rows, seed):
        from x0ne_engine_b200.csrc import ops
        g = torch.Generator().manual_seed(seed)
        self.ops, self.heads, self.dim, self.vd = ops, heads, dim, vd
        hd, hv = heads * dim, heads * vd
        self.cols = [3, 3 + hd, 3 + 2 * hd + 1]                                      # (not aligned on purpose where 3 is added)
        if dim % 4 == 0:
            self.cols = [0, hd, 2 * hd]
        self.width = -(-(self.cols[2] + hv) // 4) * 4
        self.src = torch.randn(rows, self.width, generator=g).to(DEV)
        self.f_bias, self.lower = (2.0 * torch.randn(hd, generator=g)).to(DEV), (0.95 * torch.rand(hd, generator=g)).to(DEV)
        self.g = ops.GatedState(heads, dim, vd, False)

    def run(self, state, rows, first, slots, pos0, step=False):
        ops, hd, hv = self.ops, self.heads * self.dim, self.heads * self.vd
        src = self.src[rows].contiguous()
        n = src.shape[0]
        o = torch.full((n, hv), float("nan"), device=DEV)
        q, f, v = self.cols
        raw = ops.gated_raw(src, q, f, v, self.f_bias, lower=self.lower)
        if step:
            ops.gated_step(self.g, raw, o, None, state, first, slots, len(slots))
        else:
            gates = torch.empty((n, 3 * hd), device=DEV)
            ops.channel_gates(raw, gates, n, hd)
            ops.gated_scan(self.g, gates[:, :hd], gates[:, hd:2 * hd], gates[:, 2 * hd:], src[:, v:v + hv], None, o, None, state, first, slots, len(slots))
        return (o,)

    def plain(self, rows, st):
        x = self.src[rows].double().cpu()
        T, hd = x.shape[0], self.heads * self.dim
        q, f, v = self.cols
        z, low = x[:, f:f + hd] + self.f_bias.double().cpu(), self.lower.double().cpu()
        gate = (low + (1 - low) * torch.sigmoid(z)).view(T, self.heads, self.dim)
        S = st.setdefault("S", torch.zeros(self.heads, self.dim, self.vd, dtype=torch.float64))
        o = P.gated_outer_scan(P.silu(x[:, q:q + hd]).view(T, self.heads, self.dim), ((1 - low) * torch.sigmoid(-z)).view(T, self.heads, self.dim),
                               x[:, v:v + self.heads * self.vd].view(T, self.heads, self.vd), gate, S)
        return (o.reshape(T, -1),)

    def state_of(self, row):
        return {"S": self.g.heads_of(row.double().cpu()).transpose(1, 2)}


class HeadGated:
    """The same with gates per head: the running maximum, the key sum and the normaliser's pieces."""
    head_gates = True
    cap = 5.0

    def __init__(self, heads, dim, vd, rows, seed):
        from x0ne_engine_b200.csrc import ops
        g = torch.Generator().manual_seed(seed)
        self.ops, self.heads, self.dim, self.vd = ops, heads, dim, vd
        hd, hv = heads * dim, heads * vd
        pad = 0 if dim % 4 == 0 else 1
        self.cols = [pad, 2 * pad + hd, 2 * pad + 2 * hd, 2 * pad + 2 * hd + hv, 2 * pad + 2 * hd + hv + heads]
        self.width = -(-(self.cols[4] + heads) // 4) * 4
        self.src = torch.randn(rows, self.width, generator=g).to(DEV)
        self.src[:, self.cols[3]:self.cols[4]] *= 4.0                                 # input gates on both sides of the maximum
        self.src[:, self.cols[4]:] *= 3.0
        self.f_bias, self.i_bias = (2.0 + torch.randn(heads, generator=g)).to(DEV), torch.randn(heads, generator=g).to(DEV)
        self.g = ops.GatedState(heads, dim, vd, True)

    def run(self, state, rows, first, slots, pos0, step=False):
        ops, hd, hv = self.ops, self.heads * self.dim, self.heads * self.vd
        src = self.src[rows].contiguous()
        n = src.shape[0]
        o, nq, em = (torch.full((n, w), float("nan"), device=DEV) for w in (hv, self.heads, self.heads))
        q, k, v, i, f = self.cols
        raw = ops.gated_raw(src, q, k, v, self.f_bias, i_col=i, f_col=f, i_bias=self.i_bias, cap=self.cap, geometry=self.g, em=em,
                            seq_pos0=torch.tensor(pos0, dtype=torch.int32, device=DEV))
        if step:
            ops.gated_step(self.g, raw, o, nq, state, first, slots, len(slots))
        else:
            gates = torch.empty((n, self.heads, 2), device=DEV)
            ops.head_gates(self.g, raw, gates, state, first, slots, len(slots))
            ops.gated_scan(self.g, src[:, q:q + hd], src[:, k:k + hd], None, src[:, v:v + hv], gates, o, nq, state, first, slots, len(slots))
        return o, nq, em

    def plain(self, rows, st):
        x = self.src[rows].double().cpu()
        T, hd, H, D = x.shape[0], self.heads * self.dim, self.heads, self.dim
        q, k, v, i, f = self.cols
        ig = P.capped(x[:, i:i + H] + self.i_bias.double().cpu(), self.cap)
        fg = P.log_sigmoid(P.capped(x[:, f:f + H] + self.f_bias.double().cpu(), self.cap))
        for name, shape in (("S", (H, D, self.vd)), ("n", (H, D)), ("m", (H,))):
            st.setdefault(name, torch.zeros(*shape, dtype=torch.float64))
        o, nq, em = [], [], []
        for t in range(T):                     # one token at a time, so that the pieces of the normaliser can be looked at
            qt = x[t:t + 1, q:q + hd].view(1, H, D)
            P.mlstm_scan(qt, x[t:t + 1, k:k + hd].view(1, H, D), x[t:t + 1, v:v + H * self.vd].view(1, H, self.vd), ig[t:t + 1], fg[t:t + 1],
                         st["S"], st["n"], st["m"])
            o.append((st["S"] * qt[0][:, :, None]).sum(1).reshape(-1))
            nq.append((st["n"] * qt[0]).sum(-1))
            em.append(torch.exp(-st["m"]))
        return torch.stack(o), torch.stack(nq), torch.stack(em)

    def state_of(self, row):
        S = self.g.heads_of(row.double().cpu())
        return {"S": S[:, :self.vd].transpose(1, 2), "n": S[:, self.vd]}


@pytest.mark.parametrize("kind", [ChannelGated, HeadGated])
@pytest.mark.parametrize("heads,dim,vd", SCAN_SIZES)
def test_scan_over_unequal_sequences_and_again_from_the_state(heads, dim, vd, kind):
    """Three sequences of unequal length side by side in one launch, then a second launch that carries two of them on from
    their states beside a fresh one; a slot of -1 writes nothing; unused slots keep what they hold."""
    m = kind(heads, dim, vd, 140, seed=dim)
    state = torch.zeros((6, m.g.floats), device=DEV)
    state[1] = 5.0
    carry = [{}, {}, {}, {}]

    def close(got, want, what):
        for a, b in zip(got, want):
            assert torch.isfinite(a).all() and (a.double().cpu() - b).abs().max() <= 3e-5 * max(1e-3, float(b.abs().max())), what

    first, slots = tables([1, 50, 17], [4, 0, 2])
    got = m.run(state, slice(0, 68), first, slots, [0, 0, 0])
    for k, (a, b) in enumerate(((0, 1), (1, 51), (51, 68))):
        close([x[a:b] for x in got], m.plain(slice(a, b), carry[k]), f"sequence {k}")
    first, slots = tables([33, 2, 30, 7], [0, 4, 5, -1])
    before = state.clone()
    got = m.run(state, slice(68, 140), first, slots, [50, 1, 0, 0])
    for k, c, a, b in ((0, 1, 0, 33), (1, 0, 33, 35), (2, 3, 35, 65)):
        close([x[a:b] for x in got], m.plain(slice(68 + a, 68 + b), carry[c]), f"carried on {k}")
    for slot, c in ((0, 1), (4, 0), (5, 3), (2, 2)):
        for name, s in m.state_of(state[slot]).items():
            assert (s - carry[c][name]).abs().max() <= 3e-5 * max(1e-3, float(carry[c][name].abs().max())), (slot, name)
    for slot in (1, 2, 3):
        assert torch.equal(state[slot], before[slot])


@pytest.mark.parametrize("kind", [ChannelGated, HeadGated])
@pytest.mark.parametrize("heads,dim,vd", [s for s in SCAN_SIZES if s[1] <= 256])
def test_one_token_steps_and_other_cuts_give_the_bits_of_the_scan_over_all_rows(heads, dim, vd, kind):
    m = kind(heads, dim, vd, 45, seed=3 + vd)
    whole_state, cut_state = (torch.zeros((3, m.g.floats), device=DEV) for _ in range(2))
    first, slots = tables([45], [1])
    base = m.run(whole_state, slice(0, 45), first, slots, [0])
    at, parts = 0, []
    for n in (1, 1, 3, 18, 1, 2, 17, 1, 1):
        first, slots = tables([n], [1])
        parts.append(m.run(cut_state, slice(at, at + n), first, slots, [at], step=n == 1))
        at += n
    assert at == 45
    for x, b in zip(zip(*parts), base):
        assert torch.equal(torch.cat(x), b)
    off = m.g.m_off
    assert torch.equal(whole_state[:, :off], cut_state[:, :off])


def test_channel_gates_near_one_keep_their_small_writes():
    """A gate within 1e-7 of one writes its complement with full relative precision, and a token written by it is still there
    hundreds of rows later."""
    from x0ne_engine_b200.csrc import ops
    hd = 4
    src = torch.zeros((1, 3 * hd), device=DEV)
    src[0, hd:2 * hd] = torch.tensor([16.0, -16.0, 3.0, 40.0])
    lower = torch.tensor([0.5, 0.0, 0.999, 0.0], device=DEV)
    out = torch.empty((1, 3 * hd), device=DEV)
    ops.channel_gates(ops.gated_raw(src, 0, hd, 2 * hd, torch.zeros(hd, device=DEV), lower=lower), out, 1, hd)
    z, low = src[0, hd:2 * hd].double().cpu(), lower.double().cpu()
    want_k, want_f = (1 - low) * torch.sigmoid(-z), low + (1 - low) * torch.sigmoid(z)
    k, f = out[0, hd:2 * hd].double().cpu(), out[0, 2 * hd:].double().cpu()
    assert ((k - want_k).abs() <= 1e-6 * want_k).all() and ((f - want_f).abs() <= 1e-6 * want_f).all()


@pytest.mark.parametrize("kind", [ChannelGated, HeadGated])
def test_state_keeps_a_token_hundreds_of_rows_back(kind):
    """The first token alone writes into the state (the others' values are zero); with gates that hardly forget its value is
    read 600 rows later, whole and cut."""
    m = kind(1, 6, 3, 601, seed=1)
    if kind is ChannelGated:
        q, f, v = m.cols
        m.f_bias.fill_(12.0)
        m.src[0, f:f + 6] = -14.0                                # the first token writes
        m.src[1:, v:v + 3] = 0.0
    else:
        q, k, v, i, f = m.cols
        m.f_bias.fill_(40.0)
        m.src[:, f] = 0.0
        m.src[:, i] = 0.0
        m.src[1:, v:v + 3] = 0.0
    want = [x[-1] for x in m.plain(slice(0, 601), {})]
    assert float(want[0].abs().max()) > 1e-3
    for cuts in ([601], [1, 600], [300, 301], [64] * 9 + [25]):
        state, at = torch.zeros((1, m.g.floats), device=DEV), 0
        for n in cuts:
            first, slots = tables([n], [0])
            got = m.run(state, slice(at, at + n), first, slots, [at], step=n == 1)
            at += n
        for a, b in zip(got, want):
            assert (a[-1].double().cpu() - b).abs().max() <= 1e-4 * b.abs().max(), cuts


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,vd", [(4, 20), (3, 7), (2, 64), (1, 136), (2, 300)])
def test_scan_heads_normalised_normed_and_gated(dtype, heads, vd):
    from x0ne_engine_b200.csrc import ops
    g = torch.Generator().manual_seed(9)
    rows, eps, hv = 9, 1e-5, heads * vd
    o = torch.randn(rows, heads, vd, generator=g)
    o[:, 0] *= 50.0                                         # one head far larger: a norm over the whole row would show
    o[3] = 0.0                                              # eps alone under the root
    nq, em = torch.randn(rows, heads, generator=g), torch.exp(torch.randn(rows, heads, generator=g))
    nq[5], em[6] = 0.0, 1e-4
    wide = 2 * torch.randn(rows, hv + 4, generator=g)       # the gate lies inside wider rows
    wv, wh = 1 + 0.3 * torch.randn(vd, generator=g), 1 + 0.3 * torch.randn(hv, generator=g)
    out = torch.full((rows, hv + 12), 7.0, dtype=TORCH[dtype], device=DEV)
    d = lambda t: t.to(DEV)
    tol = 3e-6 if dtype == "float32" else 2 ** -8
    # shared weight, no gate
    ops.scan_head_norm(d(o.view(rows, -1)), d(wv), out, 8, rows, heads, vd, eps, post=1.3)
    want = (P.unit_rms(o.double(), eps) * wv.double() * 1.3).reshape(rows, -1)
    assert (out[:, 8:8 + hv].double().cpu() - want).abs().max() <= tol * want.abs().max()
    assert (out[:, :8] == 7.0).all() and (out[:, 8 + hv:] == 7.0).all()
    # normalised first (a large eps makes the normaliser's size matter), a weight per value, gated
    gate = d(wide)[:, 4:]
    ops.scan_head_norm(d(o.view(rows, -1)), d(wh), out, 8, rows, heads, vd, 0.3, nq=d(nq), em=d(em), q_scale=0.25, tiny=0.01, gate=gate, post=0.7)
    y = 0.25 * o.double() / (torch.maximum((0.25 * nq.double()).abs(), em.double()) + 0.01)[:, :, None]
    want = (P.unit_rms(y, 0.3).reshape(rows, -1) * wh.double() * torch.sigmoid(wide[:, 4:].double())) * 0.7
    assert (out[:, 8:8 + hv].double().cpu() - want).abs().max() <= tol * want.abs().max()


# ------------------------------------------------------------------------------------------ row-wise kernels
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width,taps", [(72, 3), (40, 1), (64, 2), (8, 5), (37, 3), (24, 6), (16, 17), (1040, 4)])
def test_input_convolution_over_unequal_sequences_and_again_from_the_state(dtype, width, taps):
    from x0ne_engine_b200.csrc import ops
    g = torch.Generator().manual_seed(width + taps)
    dt = TORCH[dtype]
    h = torch.randn(120, width, generator=g).to(dt)
    w = 0.5 * torch.randn(width, taps, generator=g)
    wt = w.t().contiguous().to(DEV)
    state = torch.zeros((5, max(4, -(-(taps - 1) * width // 4) * 4)), device=DEV) if taps > 1 else None
    tol = 1e-6 if dtype == "float32" else 2 ** -8
    kept = {}

    def run(rows, lengths, slots):
        first, sl = tables(lengths, slots)
        out = torch.zeros((sum(lengths), width), dtype=dt, device=DEV)
        ops.input_conv(h[rows].contiguous().to(DEV), wt, state, out, first, sl, len(slots), max(lengths) + 3)
        at = 0
        for n, s in zip(lengths, slots):
            x = h[rows][at:at + n].double()
            if s >= 0:
                want, kept[s] = P.input_conv(x, w.double(), kept.get(s))
                assert (out[at:at + n].double().cpu() - want).abs().max() <= tol * want.abs().max(), (lengths, s)
                if taps > 1:
                    assert torch.equal(state[s, :(taps - 1) * width].view(taps - 1, width).double().cpu(), kept[s])
            else:
                assert (out[at:at + n] == 0).all()
            at += n

    run(slice(0, 75), [1, 40, 33, 1], [3, 0, 4, -1])
    run(slice(75, 103), [2, 1, 25], [3, 0, 1])             # two tokens, one token and a fresh sequence
    run(slice(103, 120), [1, 16], [0, 3])


@pytest.mark.parametrize("with_delta", [False, True])
@pytest.mark.parametrize("width,taps", [(72, 3), (64, 1), (512, 5), (4104, 2), (9000, 3)])
def test_norm_and_convolution_of_one_row_in_one_launch(width, taps, with_delta):
    from x0ne_engine_b200.csrc import ops
    g = torch.Generator().manual_seed(width)
    rows, eps = 5, 1e-5
    r = lambda *s: torch.randn(*s, generator=g).to(DEV)
    resid, delta, bias, wd, w, conv = r(rows, width), r(rows, width).bfloat16(), r(width), 1 + 0.2 * r(width), 1 + 0.2 * r(width), 0.5 * r(taps, width)
    slots = torch.tensor([3, 0, -1, 5, 1], dtype=torch.int32, device=DEV)
    state = r(7, max(4, (taps - 1) * width)).bfloat16().float() if taps > 1 else None
    a = (resid.clone(), None if state is None else state.clone(), torch.empty((rows, width), dtype=torch.bfloat16, device=DEV))
    pending = (delta, bias, wd, 0.01) if with_delta else (None, None, None, 0.0)
    ops.norm_conv_step(a[0], *pending, w, eps, conv, a[1], a[2], slots, rows)
    x = resid.double()
    if with_delta:
        x = x + P.unit_rms(delta.double() + bias.double(), 0.01) * wd.double()
    assert (a[0].double() - x).abs().max() <= 2e-6 * x.abs().max()
    h = (P.unit_rms(x, eps) * w.double())
    for k, s in enumerate(slots.tolist()):
        before = torch.zeros(taps - 1, width, dtype=torch.float64) if s < 0 or taps == 1 else state[s].view(taps - 1, width).double().cpu()
        want, tail = P.input_conv(h[k:k + 1].cpu(), conv.t().double().cpu(), before)
        assert (a[2][k].double().cpu() - want[0]).abs().max() <= 2 ** -7 * want.abs().max(), k
        if s >= 0 and taps > 1:
            got = a[1][s].view(taps - 1, width).double().cpu()
            assert torch.equal(got[:-1], tail[:-1]) and (got[-1] - tail[-1]).abs().max() <= 2 ** -8 * tail[-1].abs().max()
    if taps > 1:
        for s in (2, 4, 6):
            assert torch.equal(a[1][s], state[s])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [72, 37])
def test_embedding_sum_takes_the_previous_token_over_passes(dtype, width):
    from x0ne_engine_b200.csrc import ops
    g = torch.Generator().manual_seed(4)
    dt, vocab, n_pos = TORCH[dtype], 5000, 300
    buckets, mp, mc = 97, 2_000_003, 1_500_007                          # products beyond 32 bits
    table, pairs, pos_t = (torch.randn(n, width, generator=g).to(dt).to(DEV) for n in (vocab, buckets + 1, n_pos))
    ids = {s: [int(x) for x in torch.randint(vocab - 5, vocab, (60,), generator=g)] for s in (0, 2, 3)}
    last = torch.zeros((4, 1), device=DEV)
    cfg = {"embedding": {"bigram": {"buckets": buckets, "mul_prev": mp, "mul_cur": mc}}}
    t = {"embed": table.cpu(), "bigram": pairs.cpu(), "pos": pos_t.cpu()}
    at = {s: 0 for s in ids}
    for cut in ([(2, 5), (0, 1), (3, 2)], [(0, 1), (3, 30), (2, 1)], [(3, 1)], [(2, 54), (3, 2), (0, 58)]):
        tok, slot, pos = [], [], []
        for s, n in cut:
            tok += ids[s][at[s]:at[s] + n]
            slot += [s] * n
            pos += range(at[s], at[s] + n)
        first, _ = tables([n for _, n in cut], [s for s, _ in cut])
        tok, slot, pos = tok + [0, 0], slot + [-1, -1], pos + [0, 0]                         # padding rows
        i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=DEV)
        out, copy = (torch.full((len(tok), width), float("nan"), device=DEV) for _ in range(2))
        ops.embed_sum(table, pairs, pos_t, i32(tok), out, copy, last, mp, mc, i32(slot), i32(pos), first, len(cut), len(tok))
        assert torch.equal(out, copy) and torch.isfinite(out).all()
        row = 0
        for s, n in cut:
            want = P.embed(t, cfg, ids[s][at[s]:at[s] + n], at[s], ids[s][at[s] - 1] if at[s] else None)
            assert (out[row:row + n].double().cpu() - want).abs().max() <= 1e-6 * want.abs().max(), (cut, s)
            row += n
            at[s] += n


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [72, 37, 1030])
def test_rows_concatenated_with_the_embedding_output(dtype, width):
    from x0ne_engine_b200.csrc import ops
    g = torch.Generator().manual_seed(5)
    dt, rows = TORCH[dtype], 7
    r = lambda *s: torch.randn(*s, generator=g).to(DEV)
    resid, x0, delta, bias, w = r(rows, width), r(rows, width), r(rows, width).to(dt), r(width), r(width)
    keep = resid.clone()
    for d, b, wd in ((None, None, None), (delta, None, None), (delta, None, w), (delta, bias, w)):
        out = torch.empty((rows, 2 * width), dtype=dt, device=DEV)
        ops.concat_rows(resid, d, b, wd, 0.02, x0, out, rows)
        x = resid.double()
        if d is not None:
            y = d.double() if b is None else d.double() + b.double()
            x = x + (y if wd is None else P.unit_rms(y, 0.02) * wd.double())
        want = torch.cat([x, x0.double()], dim=1)
        assert (out.double() - want).abs().max() <= (1e-6 if dtype == "float32" else 2 ** -8) * want.abs().max()
    assert torch.equal(resid, keep)


@pytest.mark.parametrize("m", [1, 8, 12, 40, 64, 300, 1000])
@pytest.mark.parametrize("inter,width", [(176, 128), (1000, 512), (8192, 256)])
def test_gated_unit_with_biases_in_every_product(m, inter, width):
    """The biases of the gate and of the up branch meet the sums wherever the activation is: in the products' epilogues and
    behind them."""
    from x0ne_engine_b200.csrc import ops
    g = torch.Generator().manual_seed(m + inter)
    x = torch.randn(m, width, generator=g).bfloat16().to(DEV)
    w = (torch.randn(2 * inter, width, generator=g) * width ** -0.5).bfloat16().to(DEV)
    b = (2.0 * torch.randn(2 * inter, generator=g)).to(DEV)
    z = x.double() @ w.double().T + b.double()
    want = P.silu(z[:, :inter]) * z[:, inter:]
    kinds = [k for k, ok in (("smallm", ops.gemm_smallm_takes(w, m, True)), ("skinny", ops.gemm_skinny_tc_takes(w, m)),
                             ("tc_pair", m >= 300), ("tc", m >= 300), ("behind", True)) if ok]
    for kind in kinds:
        out = torch.zeros((m, inter), dtype=torch.bfloat16, device=DEV)
        if kind == "smallm":
            ops.gemm_bf16_smallm(x, w, out, m, swiglu=True, bias=b)
        elif kind == "skinny":
            ops.gemm_bf16_skinny_tcgen05(x, w, out, m, swiglu=True, bias=b)
        elif kind in ("tc", "tc_pair"):
            ops.gemm_bf16_tcgen05(x, w, out, m, swiglu=True, pair=kind == "tc_pair", bias=b)
        else:
            gu = (x.float() @ w.float().T).bfloat16().contiguous()
            ops.swiglu(gu, out, m, b)
        ops.check_tc_status(x.device)
        err = (out.double() - want).abs().max() / want.abs().max()
        assert err <= (2 ** -6 if kind == "behind" else 2 ** -8), (kind, float(err))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H_,G,D,V,chunk", [(6, 2, 20, 12, 37), (3, 1, 9, 7, 11), (4, 4, 64, 64, 64), (20, 1, 16, 80, 70), (2, 2, 32, 136, 0), (4, 2, 128, 128, 200)])
def test_sigmoid_attention_alone_at_chunk_and_page_edges(dtype, H_, G, D, V, chunk):
    """Norm with a weight, rotation, cache write and attention over scattered pages, as a prompt, in pieces and decoded row by
    row, against the plain equations: every row of 210, sharp scores, results scaled into wider rows."""
    from x0ne_engine_b200.cache import SequenceCache
    from x0ne_engine_b200.csrc import ops
    from x0ne_engine_b200.engine.engine import StepContext
    from x0ne_engine_b200.engine.workspace import Workspace
    from x0ne_engine_b200.parts import CacheNeed
    from x0ne_engine_b200.parts.attention import run_attention_ex
    g = torch.Generator().manual_seed(D)
    dt, T, rot, eps, scale = TORCH[dtype], 210, D // 4 * 2, 1e-5, 3.0 / D ** 0.5
    cols = [0, -(-H_ * D // 8) * 8, 0]
    cols[2] = cols[1] + -(-G * D // 8) * 8
    width = cols[2] + -(-G * V // 8) * 8
    src = torch.randn(T, width, generator=g).to(DEV)
    qn, kn = 1 + 0.2 * torch.randn(D, generator=g), 1 + 0.2 * torch.randn(D, generator=g)
    bias = -3.0 * torch.rand(H_, generator=g)
    freq = torch.tensor([50.0 ** (-2.0 * i / rot) for i in range(rot // 2)], dtype=torch.float32) if rot else None
    pos = torch.arange(T)
    s = src.double().cpu()
    q = P.rotate_half(P.unit_rms(s[:, :H_ * D].view(T, H_, D), eps) * qn.double(), pos, rot, 50.0)
    k = P.rotate_half(P.unit_rms(s[:, cols[1]:cols[1] + G * D].view(T, G, D), eps) * kn.double(), pos, rot, 50.0)
    want = 0.6 * P.sigmoid_attention(q, k, s[:, cols[2]:cols[2] + G * V].view(T, G, V), scale, bias.double(), pos, chunk).reshape(T, -1)
    cache = SequenceCache([CacheNeed("kv", G, D, None, v_dim=None if V == D else V)], [None], 1280, 640, dt, DEV)
    cache.acquire(64)                                      # (the pages of the sequence do not lie in order)
    slot = cache.acquire(64)
    cache.ensure(0, 128)
    for t in (100, 192, T):
        cache.ensure(slot, t)
        cache.ensure(0, min(640, 2 * t))
    view, ws = cache.kv_view(0), Workspace(T, DEV)
    d = lambda t: None if t is None else t.to(DEV)
    dev = dict(qn=d(qn), kn=d(kn), freq=d(freq), bias=d(bias))
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=DEV)
    # a bfloat16 run rounds queries, keys and values: allow each weight's change and the values' rounding
    tol = 2e-6 * T if dtype == "float32" else 0.02
    for cuts in ([T], [63, 1, 2, 60, 84], [150] + [1] * 60):
        got, at = [], 0
        for n in cuts:
            rows, first, n_tiles = i32(range(at, at + n)), i32([0, n]), -(-n // 128)
            ctx = StepContext(n_rows=n, tokens=rows, row_slot=i32([slot] * n), row_pos=rows, dtype=dt, ws=ws, cache=cache, decode=n == 1, n_seqs=1,
                              max_seq_rows=n, max_context=at + n, seq_first_row=first, seq_slot=i32([slot]), seq_pos0=i32([at]), n_tiles=n_tiles,
                              tile_seq=i32([0] * n_tiles), tile_row0=i32([128 * x for x in range(n_tiles)]), sm_count=148)
            qo = torch.empty((n, H_ * D), dtype=dt, device=DEV)
            out = torch.full((n, H_ * V + 9), 7.0, dtype=dt, device=DEV)
            ops.head_norm_rope_kv_write(src[at:at + n].contiguous(), *cols, dev["qn"], dev["kn"], eps, dev["freq"], None, rot, qo, H_, view,
                                        ctx.row_slot, ctx.row_pos, n)
            extra = ops.attn_extra(chunk=chunk, sig_bias=dev["bias"], out_ld=H_ * V + 9, out_col=5, out_scale=0.6)
            run_attention_ex(ctx, qo, out, view, n, H_, scale, 0, extra)
            assert (out[:, :5] == 7.0).all() and (out[:, 5 + H_ * V:] == 7.0).all()
            got.append(out[:, 5:5 + H_ * V].double().cpu())
            at += n
        err = (torch.cat(got) - want).abs().max() / want.abs().max()
        assert err <= tol, (cuts[:4], float(err))


# ------------------------------------------------------------------------------------------ whole models
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name,lengths", [("hgrn2_only", [1, 2, 40]), ("parallel_only", [1, 2, 37, 38, 130]), ("glu_only", [1, 3, 70]), ("loop_only", [1, 30]),
                                          ("mixed", [1, 2, 37, 38, 65, 150]), ("even", [64, 131, 300]), ("wide", [5, 71, 141]), ("odd", [1, 12, 90]),
                                          ("plain", [1, 100]), ("served", [7, 300, 1000])])
def test_each_request_alone_and_whole(name, lengths, dtype):
    eng, cfg, t = engine(name, dtype)
    for k, n in enumerate(lengths):
        ids = H.random_ids(cfg, n, seed=k)
        check(dtype, whole(eng, ids), H.plain_logits(cfg, t, ids), f"{name} len {n}")


def test_residual_stream_after_every_layer_run():
    """The float32 residual after each run of a layer (the pending result normed and added by hand) against the plain one: a
    repeated layer counts each time, and what opens the next pass is not yet in it."""
    eng, cfg, t = engine("mixed", "float32", pass_graphs=False)
    ids = H.random_ids(cfg, 90, seed=3)
    seen = []
    for b in eng.model.blocks:
        def wrapped(ctx, entry, resid, delta, cache_entry=None, write_cache=True, _f=b.forward):
            out = _f(ctx, entry, resid, delta, cache_entry=cache_entry, write_cache=write_cache)
            d = out.delta[:ctx.n_rows].double() + (0.0 if out.bias is None else out.bias.double())
            seen.append((resid[:ctx.n_rows].double() + P.unit_rms(d, out.norm.eps) * out.norm.weight.double()).cpu())
            return out
        b.forward = wrapped
    try:
        whole(eng, ids)
    finally:
        for b in eng.model.blocks:
            del b.forward
    want = []
    H.plain_logits(cfg, t, ids, layers_out=want)
    assert len(seen) == len(want) == 6
    for i, (a, b) in enumerate(zip(seen, want)):
        assert (a - b.double()).abs().max() <= 1e-4 * b.abs().max(), f"layer run {i}"


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name,n,tail", [("mixed", 120, 60), ("wide", 100, 40), ("even", 160, 40), ("odd", 70, 30), ("plain", 90, 50), ("served", 330, 140)])
def test_prefill_against_token_by_token(name, n, tail, dtype):
    eng, cfg, t = engine(name, dtype)
    ids = H.random_ids(cfg, n, seed=5)
    got = in_pieces(eng, ids, [n - tail] + [1] * tail)
    same_cut(dtype, got, whole(eng, ids), f"{name}: last {tail} one by one")
    check(dtype, got, H.plain_logits(cfg, t, ids), f"{name} decoded")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mixed", "even", "odd"])
def test_prompt_in_portions_down_to_two_tokens(name, dtype):
    eng, cfg, t = engine(name, dtype)
    ids = H.random_ids(cfg, 170, seed=6)
    base = whole(eng, ids)
    for cuts in ([2] * 30, [64, 64], [63, 2, 1, 64], [37, 37, 37, 37], [3, 125, 2], [129]):
        same_cut(dtype, in_pieces(eng, ids, cuts), base, f"{name} cut {cuts[:4]}")
    check(dtype, base, H.plain_logits(cfg, t, ids), name)


def test_a_step_cut_into_passes_inside_prompts():
    eng, cfg, t = engine("mixed", "float32", max_step_tokens=64)
    ids = H.random_ids(cfg, 150, seed=7)
    assert np.array_equal(whole(eng, ids), whole(engine("mixed", "float32")[0], ids))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mixed", "wide"])
def test_unequal_batches_against_each_alone_with_slots_used_again(name, dtype):
    eng, cfg, t = engine(name, dtype)
    for round_ in range(3):                      # the second and third rounds get slots, pages and states that were used
        lengths, steps = [[1, 30, 77, 140], [66, 2, 129], [140, 5]][round_], [3, 9, 1, 6]
        full = [H.random_ids(cfg, n + steps[k], seed=10 * round_ + k) for k, n in enumerate(lengths)]
        slots = [eng.new_sequence() for _ in lengths]
        got = [[] for _ in lengths]
        first = eng.step(slots, [f[:n] for f, n in zip(full, lengths)], [list(range(n)) for n in lengths]).cpu().numpy()
        at = 0
        for k, n in enumerate(lengths):
            got[k].append(first[at:at + n])
            at += n
        live = list(range(len(lengths)))
        for step in range(max(steps)):
            live = [k for k in live if step < steps[k]]         # the shorter requests end earlier
            out = eng.step([slots[k] for k in live], [[full[k][lengths[k] + step]] for k in live]).cpu().numpy()
            for j, k in enumerate(live):
                got[k].append(out[j:j + 1])
        for s in slots:
            eng.free_sequence(s)
        for k in range(len(lengths)):
            alone = whole(eng, full[k])
            same_cut(dtype, np.concatenate(got[k]), alone, f"{name} round {round_} request {k}")
            if round_ == 0:
                check(dtype, alone, H.plain_logits(cfg, t, full[k]), f"{name} request {k}")


# ------------------------------------------------------------------------------------------ edges, far keys
@pytest.mark.parametrize("dtype", DTYPES)
def test_chunk_edges_that_decide(dtype):
    """Sharp queries make single keys decide a row, so a chunk whose edge is one off, or a page read wrongly, changes the
    logits by far more than the tolerance.  Chunks of 37 and 50 positions against pages of 64; every position of a 260-token
    sequence is checked, in a prompt and decoded alone."""
    eng, cfg, t = engine("sharp", dtype, seed=3)
    ids = H.random_ids(cfg, 260, seed=8)
    want = H.plain_logits(cfg, t, ids)

    def moved(by):
        layers = [dict(l, mixer=dict(l["mixer"], left=dict(l["mixer"]["left"], mask={"size": l["mixer"]["left"]["mask"]["size"] + by})))
                  if l["type"] == "parallel" else l for l in cfg["layers"]]
        diff = np.abs(H.plain_logits({**cfg, "layers": layers}, t, ids) - want).max(-1) / np.abs(want).max(-1)
        return (diff > 0.1).sum()
    assert moved(1) > 8 and moved(-1) > 8                  # the test sees what it is for
    check(dtype, whole(eng, ids), want, "prompt")
    check(dtype, in_pieces(eng, ids, [30] + [1] * 230), want, "decoded across chunk edges and page borders")


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_key_far_back(dtype):
    """Attention without chunks over 700 positions, every weight near zero but the last query's on the first token's key (one
    embedding feature that only the first token has feeds one key channel, another that only the last token has feeds the
    same query channel): the last logits hang on a key eleven pages back, read in a prompt and in decoding."""
    from x0ne_engine_b200 import Engine
    cfg = H.config([H.layer("parallel", H.parallel(H.attn(heads=4, kv_heads=2, rot=(4, 50.0), chunk=None), None, 3.0, 0.2), None), H.layer("hgrn2", H.hgrn2())],
                   taps=1)
    t = H.make_tensors(cfg, seed=4)
    special, late, d = 7, 11, cfg["layers"][0]["mixer"]["left"]["dim"]
    for name in ("embed", "bigram", "pos"):
        t[name][:, :2] = 0.0
    t["embed"][special, 0] = t["embed"][late, 1] = 12.0
    t["l0.canon1"].zero_()
    kr, qr = d + d - 1, 3 * d + d - 1                       # kv head 1 / query head 3, the last channel (not rotated)
    t["l0.mix.left.k"][kr], t["l0.mix.left.q"][qr] = 0.0, 0.0
    t["l0.mix.left.k"][kr, 0], t["l0.mix.left.q"][qr, 1] = 4.0, 4.0
    t["l0.mix.left.pb"].fill_(-9.0)
    t["l0.mix.left.v"] *= 4.0
    cfg["layers"][0]["mixer"]["left"]["scale"] = 0.6
    t = {k: v.bfloat16().float() for k, v in t.items()}
    folder = H.write_folder(cfg, t, "x0ne_rvp_far_")
    ids = [12 + x % (cfg["vocab"] - 12) for x in H.random_ids(cfg, 700, 9)]
    ids[0], ids[-1] = special, late
    eng = Engine.from_folder(folder, dtype=dtype, max_tokens=1024, max_seq_len=1024)
    want = H.plain_logits(cfg, t, ids)
    cut = H.plain_logits(cfg, t, [13] + ids[1:])[-1]        # another first token: the far key is gone
    assert np.abs(cut - want[-1]).max() > 0.1 * np.abs(want[-1]).max()
    check(dtype, whole(eng, ids)[-3:], want[-3:], "far key in a prompt")
    check(dtype, in_pieces(eng, ids, [697, 1, 1])[-3:], want[-3:], "far key decoded")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mixed", "wide"])
def test_first_tokens_of_a_sequence(name, dtype):
    eng, cfg, t = engine(name, dtype)
    ids = H.random_ids(cfg, 8, seed=11)
    want = H.plain_logits(cfg, t, ids)
    for cuts in ([1] * 8, [2, 2, 2], [1, 3], [3, 1, 1]):
        check(dtype, in_pieces(eng, ids, cuts), want, f"first tokens as {cuts}")


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding(dtype):
    eng, cfg, t = engine("even", dtype)
    ids = H.random_ids(cfg, 420, seed=12)
    check(dtype, in_pieces(eng, ids, [20] + [1] * 400), H.plain_logits(cfg, t, ids), "400 decoded tokens")


def test_positions_past_the_learned_rows_are_refused():
    from x0ne_engine_b200 import Engine
    folder, cfg, _ = H.folder("odd")
    eng = Engine.from_folder(folder, dtype="float32", max_tokens=1024)
    assert eng.max_seq_len == cfg["max_positions"] == 700
    slot = eng.new_sequence()
    with pytest.raises(ValueError, match="700"):
        eng.step([slot], [H.random_ids(cfg, 701)])
    eng.free_sequence(slot)


# ------------------------------------------------------------------------------------------ generation
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("decode", ["graph", "eager"])
def test_greedy_generation_through_the_entry_point(decode, dtype):
    from x0ne_engine_b200 import Model
    folder, cfg, t = H.folder("mixed")
    prompts = [H.random_ids(cfg, n, seed=20 + n) for n in (1, 7, 36, 64)]
    n_new = 14
    m = Model.from_folder(folder, dtype=dtype, max_batch=3, max_ctx=256, decode=decode)
    out = m.generate(prompts, max_tokens=n_new, stop_token_ids=())
    assert out.finish_reasons == ["length"] * len(prompts)
    for p, got in zip(prompts, out.tokens):
        carry, ids = {}, list(p)
        for tok in got:
            row = P.forward(cfg, t, ids, carry=carry)[-1].numpy()
            if tok != int(np.argmax(row)):                  # the two part only at a close call
                tol = 1e-4 if dtype == "float32" else 2 * 0.05
                assert np.sort(row)[-1] - row[tok] <= tol * np.abs(row).max(), "a token left a clear argmax"
                break
            ids = [tok]
    assert m.generate(prompts, max_tokens=n_new, stop_token_ids=()).tokens == out.tokens


def test_random_model_from_a_configuration_generates():
    from x0ne_engine_b200 import Model
    from x0ne_engine_b200.config import config_from_dict
    m = Model.random(config_from_dict(H.CONFIGS["even"]()), seed=1, max_batch=2, max_ctx=128, norm_jitter=0.1)
    out = m.generate([[1, 2, 3], [4]], max_tokens=5, stop_token_ids=())
    assert [len(x) for x in out.tokens] == [5, 5] and all(0 <= x < 256 for row in out.tokens for x in row)


def test_short_prompt_passes_replayed_from_graphs_give_the_same_bits():
    eng, cfg, t = engine("mixed", "bfloat16", pass_graphs=True)
    base, _, _ = engine("mixed", "bfloat16", pass_graphs=False)
    assert eng.replayable and eng.pass_graphs and not base.pass_graphs
    before = eng.pass_graph_replays
    for k, lengths in enumerate([[100], [120], [70], [126], [20], [30], [5], [5], [100, 20], [90, 30], [100]]):
        prompts = [H.random_ids(cfg, n, 100 + 7 * k + j) for j, n in enumerate(lengths)]
        got = []
        for e in (eng, base):
            slots = [e.new_sequence() for _ in lengths]
            first = e.step(slots, prompts).cpu().numpy()
            nxt = e.step(slots, [[int(np.argmax(r))] for r in first]).cpu().numpy()
            for s in slots:
                e.free_sequence(s)
            got.append((first, nxt))
        assert np.array_equal(got[0][0], got[1][0]) and np.array_equal(got[0][1], got[1][1]), lengths
    assert eng.pass_graph_replays - before >= 4
