"""Tarudra on the GPU against the plain implementation (tests/tarudra_plain.py), in float32 and bfloat16: every mechanism
alone, whole prompts, token-by-token decoding, portions down to two tokens, unequal batches with slots, pages and states used
again, every window's edge in prompts and in decoding (also of layers that read another layer's keys), far keys and a far token
in the delta state, the first tokens, long decoding, odd sizes and values a configuration may leave out or make equal, and greedy
generation through the entry point."""
import numpy as np
import pytest
import torch

import tarudra_helpers as H
import tarudra_plain as P
from helpers import BF16_KL_TOL, BF16_LOGIT_TOL, BF16_SELF_TOL, assert_close_f32, first_difference, kl_rows

pytestmark = pytest.mark.gpu

DTYPES = ["float32", "bfloat16"]
TORCH = {"float32": torch.float32, "bfloat16": torch.bfloat16}
DEV = "cuda:0"
_engines = {}


def engine(name, dtype, seed=0, max_tokens=1024, **kw):
    from x0ne_engine_b200 import Engine
    key = (name, dtype, seed, max_tokens, tuple(sorted(kw.items())))
    if key not in _engines:
        folder, cfg, tensors = H.folder(name, seed)
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


def i32(x):
    return torch.tensor(list(x), dtype=torch.int32, device=DEV)


# ------------------------------------------------------------------------------------------ the delta rule
class Delta:
    """Random projections of several sequences, run through the kernels in any cut and through the plain equations."""

    def __init__(self, heads, kv, dim, vd, taps, seed, decay=(-6.0, 0.0)):
        from x0ne_engine_b200.csrc import ops
        g = torch.Generator().manual_seed(seed)
        self.ops, self.g = ops, ops.DeltaState(heads, kv, dim, vd, taps)
        sizes = (kv * dim, kv * dim, heads * vd, heads, heads, heads * vd)
        self.cols, at = [], 0
        for n in sizes:
            self.cols.append(at)
            at += -(-n // 4) * 4 if dim % 4 == 0 else n + 1                     # (not aligned on purpose where a row is added)
        self.width, self.gen = at + 3 if dim % 4 else at, g
        self.conv = torch.randn(self.g.channels, taps, generator=g)
        self.A, self.dt = torch.exp(torch.rand(heads, generator=g) * 3.0 - 2.0), decay[0] + (decay[1] - decay[0]) * torch.rand(heads, generator=g)
        self.norm, self.eps = 1.0 + 0.2 * torch.randn(vd, generator=g), 1e-5
        self.dev = [t.to(DEV) for t in (self.conv, self.A, self.dt, self.norm)]
        self.state = torch.zeros(6, self.g.floats, device=DEV)
        self.seqs = {}                   # slot -> projection rows so far

    def rows(self, n):
        return torch.randn(n, self.width, generator=self.gen)

    def run(self, cut, dtype=torch.float32, step=False, chunks=False):
        """`cut`: (slot, rows) of one pass, slots of -1 being no sequence's; returns the gated heads.  `chunks`: by the scan that takes
        several tokens together."""
        ops, g = self.ops, self.g
        slots, pos0, pos, row_slot = [], [], [], []
        for s, x in cut:
            p = self.seqs[s].shape[0] if s in self.seqs else 0
            slots.append(s)
            pos0.append(p)
            pos += range(p, p + x.shape[0])
            row_slot += [s] * x.shape[0]
            if s >= 0:
                self.seqs[s] = torch.cat([self.seqs[s], x]) if s in self.seqs else x
        src = torch.cat([x for _, x in cut]).to(DEV)
        n, first = src.shape[0], i32(np.concatenate([[0], np.cumsum([x.shape[0] for _, x in cut])]))
        out = torch.full((n, g.heads * g.v_dim), float("nan"), dtype=dtype, device=DEV)
        many = {} if step else dict(planes=torch.full((n, g.plane_floats), float("nan"), device=DEV), gates=torch.empty((n, 4 * g.heads), device=DEV),
                                    o=torch.zeros((n, g.heads * g.v_dim), device=DEV))
        tabs = [i32(row_slot), i32(pos), first, i32(slots), i32(pos0)]
        a = ops.delta_arg(g, src, self.cols, *self.dev, g.dim ** -0.5, self.eps, self.state, *tabs, n, **many)
        if step:
            ops.delta_step(a, out, len(slots))
        else:
            ops.delta_prepare(a)
            if chunks:
                ops.delta_chunk_scan(a, torch.full((n, ops.DELTA_COEF * g.heads), float("nan"), device=DEV), len(slots), max(x.shape[0] for _, x in cut))
            else:
                ops.delta_scan(a, len(slots))
            ops.delta_head_norm(a, out)
        torch.cuda.synchronize()
        return out

    def plain(self, x):
        """(gated heads [T, heads * values], state [heads, channels, values], the convolutions' last inputs) of a sequence."""
        g, x, T = self.g, x.double(), x.shape[0]
        c = [x[:, at:at + n] for at, n in zip(self.cols, (g.kv_heads * g.dim,) * 2 + (g.heads * g.v_dim, g.heads, g.heads, g.heads * g.v_dim))]
        y, tail = P.causal_conv(torch.cat(c[:3], dim=1), self.conv.double())
        y = P.silu(y)
        hd = g.kv_heads * g.dim
        spread = torch.arange(g.heads) // (g.heads // g.kv_heads)
        q = P.unit_vector(y[:, :hd].reshape(T, g.kv_heads, g.dim))[:, spread] * g.dim ** -0.5
        k = P.unit_vector(y[:, hd:2 * hd].reshape(T, g.kv_heads, g.dim))[:, spread]
        gate = torch.exp(-self.A.double() * P.softplus(c[3] + self.dt.double()))
        S = torch.zeros(g.heads, g.dim, g.v_dim, dtype=torch.float64)
        o = P.delta_scan(q, k, y[:, 2 * hd:].reshape(T, g.heads, g.v_dim), torch.sigmoid(c[4]), gate, S)
        o = P.unit_rms(o, self.eps) * self.norm.double() * P.silu(c[5]).reshape(T, g.heads, g.v_dim)
        return o.reshape(T, -1), S, tail

    def check_states(self):
        for s, x in self.seqs.items():
            _, S, tail = self.plain(x)
            g, row = self.g, self.state[s].double().cpu()
            got = row[:g.heads * g.v_dim * g.dim].reshape(g.heads, g.v_dim, g.dim).transpose(1, 2)
            assert (got - S).abs().max() <= 2e-5 * S.abs().max()
            ring = row[g.ring_off:g.ring_off + g.taps * g.channels].reshape(-1, g.channels) if g.taps > 1 else None
            for back in range(min(g.taps - 1, x.shape[0])):
                assert torch.equal(ring[(x.shape[0] - 1 - back) % g.taps], tail[-1 - back])


DELTA_SIZES = [(4, 2, 12, 20, 3), (3, 1, 5, 7, 2), (2, 2, 16, 48, 1), (2, 1, 64, 16, 4), (2, 2, 33, 17, 5), (4, 2, 100, 40, 4), (2, 1, 128, 128, 4),
               (3, 3, 130, 9, 6), (1, 1, 256, 300, 3), (2, 1, 300, 10, 2)]


def close_rows(got, want, what, tol=2e-4):
    """Per row (a head's result may be the remainder of a cancellation that its norm brings back to unit size)."""
    err = (got - want).abs().amax(-1) / want.abs().amax(-1)
    assert err.max() <= tol, f"{what}: {float(err.max()):.2e}"


@pytest.mark.parametrize("chunks", [False, True])
@pytest.mark.parametrize("heads,kv,dim,vd,taps", DELTA_SIZES)
def test_delta_rule_over_unequal_sequences_and_again_from_the_state(heads, kv, dim, vd, taps, chunks):
    if chunks and dim > 256:
        pytest.skip("the scan by chunks takes heads of up to 256 channels")
    d = Delta(heads, kv, dim, vd, taps, seed=dim + taps)
    got = {}
    for cut in ([(3, 1), (0, 40), (4, 33), (-1, 2)], [(3, 2), (0, 1), (1, 25)], [(1, 1), (0, 16), (3, 70)]):
        rows = [(s, d.rows(n)) for s, n in cut]
        out, at = d.run(rows, chunks=chunks).double().cpu(), 0
        for s, x in rows:
            if s >= 0:
                got.setdefault(s, []).append(out[at:at + x.shape[0]])
            at += x.shape[0]
    for s, parts in got.items():
        close_rows(torch.cat(parts), d.plain(d.seqs[s])[0], f"slot {s}")
    d.check_states()
    assert not d.state[2].any() and not d.state[5].any()               # nobody else's state


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,kv,dim,vd,taps", [s for s in DELTA_SIZES if s[2] <= 256])
def test_one_token_steps_give_the_bits_of_the_scan(heads, kv, dim, vd, taps, dtype):
    a, b, c = (Delta(heads, kv, dim, vd, taps, seed=7) for _ in range(3))
    rows = {s: a.rows(n) for s, n in ((2, 21), (0, 21), (5, 21))}
    want = a.run([(s, x) for s, x in rows.items()], TORCH[dtype])
    cut = b.run([(s, x[:2]) for s, x in rows.items()], TORCH[dtype])
    steps = [[], [], []]
    for k in range(3):
        steps[k].append(cut[2 * k:2 * k + 2])
    for t in range(2, 21):
        one = b.run([(s, x[t:t + 1]) for s, x in rows.items()], TORCH[dtype], step=True)
        for k in range(3):
            steps[k].append(one[k:k + 1])
    assert torch.equal(torch.cat([torch.cat(s) for s in steps]), want) and torch.equal(a.state, b.state)
    first = [c.run([(s, x[t:t + 1]) for s, x in rows.items()], TORCH[dtype], step=True) for t in range(3)]        # from a sequence's first token on
    for k in range(3):
        assert torch.equal(torch.cat([f[k:k + 1] for f in first]), want[21 * k:21 * k + 3])


def test_other_cuts_of_the_scan_give_the_same_bits():
    a = Delta(4, 2, 64, 48, 4, seed=9)
    x = a.rows(1500)
    want = a.run([(1, x)])                                            # (long passes walk stretches of rows)
    for cuts in ([700, 800], [1] * 20 + [3, 1477], [64] * 23 + [28]):
        b, at, got = Delta(4, 2, 64, 48, 4, seed=9), 0, []
        for n in cuts:
            got.append(b.run([(1, x[at:at + n])]))
            at += n
        assert torch.equal(torch.cat(got), want) and torch.equal(a.state, b.state), cuts[:3]


@pytest.mark.parametrize("chunks", [False, True])
def test_a_token_read_from_the_state_600_rows_later(chunks):
    """Hardly any decay; token 0 alone writes one direction that no later key touches, and the last query asks for it."""
    d = Delta(1, 1, 32, 16, 1, seed=3, decay=(-14.0, -13.0))
    x = d.rows(601)
    q, k, v, a, b, g = d.cols
    d.conv.fill_(1.0)
    d.dev[0].fill_(1.0)
    x[:, k:k + 16] = -40.0                       # silu(-40) = 0: later keys leave the first half of the channels alone
    x[:, a] = 0.0
    x[0, k:k + 32] = -40.0
    x[0, k + 5] = 9.0
    x[0, b] = 12.0
    x[-1, q:q + 32] = -40.0
    x[-1, q + 5] = 9.0
    for cut in ([601], [1, 599, 1]):
        d.state.zero_()
        d.seqs.clear()
        at = 0
        for n in cut:
            out = d.run([(0, x[at:at + n])], chunks=chunks)
            at += n
        want = d.plain(x)[0]
        close_rows(out[-1:].double().cpu(), want[-1:], "far token", 1e-4)
        y = x.clone()
        y[0, v:v + 16] += 1.0
        assert (d.plain(y)[0][-1] - want[-1]).abs().max() > 0.1 * want[-1].abs().max()


@pytest.mark.parametrize("chunks", [False, True])
def test_a_decay_close_to_one_keeps_its_digits(chunks):
    d = Delta(2, 1, 16, 8, 2, seed=4, decay=(-15.5, -14.0))
    x = d.rows(1000)
    got = d.run([(0, x)], chunks=chunks).double().cpu()
    close_rows(got[-50:], d.plain(x)[0][-50:], "1,000 tokens")
    d.check_states()


def test_decays_that_forget_at_once_and_writes_of_full_strength():
    """Decays down to nothing and write strengths near one inside the chunks: no product of decays may be divided by."""
    d = Delta(2, 1, 24, 16, 2, seed=5, decay=(2.0, 60.0))
    d.A.fill_(3.0)
    d.dev[1].fill_(3.0)
    x = d.rows(75)
    x[::7, d.cols[3]:d.cols[3] + 2] -= 80.0                # every seventh token keeps everything
    x[:, d.cols[4]:d.cols[4] + 2] += 6.0
    close_rows(d.run([(0, x)], chunks=True).double().cpu(), d.plain(x)[0], "sharp decays")
    d.check_states()


# ------------------------------------------------------------------------------------------ norms
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [72, 37, 1000, 4096, 8200, 20000])
def test_norms_that_subtract_the_mean(width, dtype):
    """Add and norm in every combination: with and without a pending result, its bias and its own norm (centred or not), source
    rows gathered, rows whose mean is far larger than what is left without it."""
    from x0ne_engine_b200.csrc import ops
    g = torch.Generator().manual_seed(width)
    dt, n = TORCH[dtype], 6
    r = lambda *s: torch.randn(*s, generator=g)
    resid, delta = r(n, width) + 30.0 * r(n, 1), (r(n, width) + 3.0).to(dt)
    w, wd, bias = 1 + 0.2 * r(width), 1 + 0.2 * r(width), r(width)

    def plain(x, weight, eps, centred):
        return P.layer_norm(x, weight, eps) if centred else P.unit_rms(x, eps) * weight
    for centred in (True, False):
        for pending in (None, "plain", "centred", "rms", "biased"):
            for rows in (None, [4, 0, 5]):
                base = resid.to(DEV)
                take = list(range(n)) if rows is None else rows
                out = torch.empty((len(take), width), dtype=dt, device=DEV)
                kw = {}
                x = resid.double()
                if pending:
                    y = delta.double() + (bias.double() if pending == "biased" else 0.0)
                    if pending == "biased":
                        kw["delta_bias"] = bias.to(DEV)
                    if pending != "plain":
                        kw.update(delta_weight=wd.to(DEV), delta_eps=0.03, delta_centred=pending != "rms")
                        y = plain(y, wd.double(), 0.03, pending != "rms")
                    x = x + y
                ops.add_norm(base, delta.to(DEV) if pending else None, w.to(DEV), out, len(take), 1e-5, centred, None if rows is None else i32(rows), **kw)
                want = plain(x[take], w.double(), 1e-5, centred)
                tol = 3e-5 if dtype == "float32" else 2 ** -8
                assert (out.double().cpu() - want).abs().max() <= tol * want.abs().max(), (centred, pending, rows)
                assert (base.double().cpu()[take] - x[take]).abs().max() <= 1e-6 * x.abs().max()


# ------------------------------------------------------------------------------------------ attention preparation
def paged(dt, kv, hd, vd, rows, reserve=640):
    from x0ne_engine_b200.cache import SequenceCache
    from x0ne_engine_b200.parts import CacheNeed
    cache = SequenceCache([CacheNeed("kv", kv, hd, None, v_dim=None if vd == hd else vd)], [None], 1280, reserve, dt, DEV)
    cache.acquire(64)                                      # (the pages of the sequence do not lie in order)
    slot = cache.acquire(64)
    for t in (100, 192, rows):
        cache.ensure(slot, t)
        cache.ensure(0, min(reserve, 2 * t))
    return cache, slot


def context(cache, slot, dt, ws, n, at):
    from x0ne_engine_b200.engine.engine import StepContext
    rows, n_tiles = i32(range(at, at + n)), -(-n // 128)
    return StepContext(n_rows=n, tokens=rows, row_slot=i32([slot] * n), row_pos=rows, dtype=dt, ws=ws, cache=cache, decode=n == 1, n_seqs=1,
                       max_seq_rows=n, max_context=at + n, seq_first_row=i32([0, n]), seq_slot=i32([slot]), seq_pos0=i32([at]), n_tiles=n_tiles,
                       tile_seq=i32([0] * n_tiles), tile_row0=i32([128 * x for x in range(n_tiles)]), sm_count=148)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("table", [True, False])
@pytest.mark.parametrize("H_,G,D,V,rot,window", [(6, 2, 20, 12, 8, 37), (3, 1, 9, 7, 6, 11), (4, 4, 64, 64, 64, 64), (20, 1, 16, 80, 16, 70), (4, 2, 96, 32, 48, 100),
                                                 (2, 2, 32, 32, 0, 5)])
def test_biased_windowed_attention_alone_at_window_and_page_edges(H_, G, D, V, rot, window, table, dtype):
    """Biases, scaled rotation of pairs, cache write and attention over scattered pages with the extra denominator term: as a
    prompt, in pieces and row by row, then by a reader with a window of its own; every row of 210, sharp scores."""
    from x0ne_engine_b200.csrc import ops
    from x0ne_engine_b200.engine.workspace import Workspace
    from x0ne_engine_b200.parts.attention import run_attention_ex
    g = torch.Generator().manual_seed(D + window)
    dt, T, scale = TORCH[dtype], 210, 2.5 / D ** 0.5
    width = H_ * D + G * (D + V)
    src, bias = torch.randn(T, width, generator=g).to(dt), 0.5 * torch.randn(width, generator=g)
    pos, spec = torch.arange(T), {"dims": rot, "base": 50.0, "scaling": H.YARN}
    freq, mag = P.yarn(rot, 50.0, H.YARN) if rot else ([], 1.0)
    x = src.double() + bias.double()
    q = P.rotate(x[:, :H_ * D].view(T, H_, D), pos, spec, "interleaved")
    k = P.rotate(x[:, H_ * D:(H_ + G) * D].view(T, G, D), pos, spec, "interleaved")
    v = x[:, (H_ + G) * D:].view(T, G, V)
    fr = torch.tensor(freq, dtype=torch.float32, device=DEV) if rot else None
    tab = None
    if rot and table:
        ang = pos.double()[:, None] * torch.tensor(freq, dtype=torch.float64)[None]
        tab = (mag * torch.cat([torch.cos(ang), torch.sin(ang)], dim=1)).float().to(DEV).contiguous()
    cache, slot = paged(dt, G, D, V, T)
    view, ws = cache.kv_view(0), Workspace(T, DEV)
    sink = torch.zeros(H_, device=DEV)
    tol = 2e-5 if dtype == "float32" else 0.03
    for cuts in ([T], [63, 1, 2, 60, 84], [150] + [1] * 60):
        for win, own in ((window, True), (window + 23, False)):
            want = P.windowed_attention(q, k, v, scale, pos, win, True).reshape(T, -1)
            got, at = [], 0
            for n in cuts:
                ctx = context(cache, slot, dt, ws, n, at)
                part = src[at:at + n] if own else src[at:at + n, :H_ * D]
                b = bias if own else bias[:H_ * D]
                qo = torch.empty((n, H_ * D), dtype=dt, device=DEV)
                out = torch.full((n, H_ * V), 7.0, dtype=dt, device=DEV)
                ops.rope_pairs_kv_write(part.contiguous().to(DEV), H_ * D, (H_ + G) * D, fr, tab, rot, 1, D, None, qo, H_, False, view, ctx.row_slot, ctx.row_pos, n,
                                        own, bias=b.contiguous().to(DEV), mag=mag)
                run_attention_ex(ctx, qo, out, view, n, H_, scale, win, ops.attn_extra(sink=sink))
                got.append(out.double().cpu())
                at += n
            err = (torch.cat(got) - want).abs().max() / want.abs().max()
            assert err <= tol, (cuts[:4], own, float(err))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("half", [True, False])
@pytest.mark.parametrize("heads,dim,rank,q_rank,rot", [(5, 10, 22, 13, 6), (4, 16, 64, 48, 32), (3, 8, 200, 0, 16), (2, 7, 11, 5, 2)])
def test_latent_rows_and_queries_alone(heads, dim, rank, q_rank, rot, half, dtype):
    from x0ne_engine_b200.csrc import ops
    g = torch.Generator().manual_seed(rank)
    dt, T, eps = TORCH[dtype], 150, 1e-5
    cols = [0, -(-max(q_rank, 1) // 8) * 8]
    width = cols[1] + -(-(rank + rot) // 8) * 8
    src, q = torch.randn(T, width, generator=g).to(dt), torch.randn(T, heads * (dim + rot), generator=g).to(dt)
    q_abs = torch.randn(heads, T, rank, generator=g).to(dt)
    nq, nkv = 1 + 0.2 * torch.randn(max(q_rank, 1), generator=g), 1 + 0.2 * torch.randn(rank, generator=g)
    pos, layout, spec = torch.arange(T), "half" if half else "interleaved", {"dims": rot, "base": 70.0}
    freq = torch.tensor(P.yarn(rot, 70.0, None)[0], dtype=torch.float32, device=DEV)
    cache, slot = paged(dt, 1, rank + rot, 0, T)
    view = cache.kv_view(0)
    row_slot, row_pos = i32([slot] * T), i32(range(T))
    turn = ops.latent_turn(freq, None, 1.0, rot, half)
    cq = torch.empty((T, q_rank), dtype=dt, device=DEV) if q_rank else None
    ops.latent_rows(src.to(DEV), cols[0], q_rank, nq.to(DEV) if q_rank else None, cq, cols[1], rank, nkv.to(DEV), eps, turn, view, row_slot, row_pos, T)
    qo = torch.empty((T, heads * (rank + rot)), dtype=dt, device=DEV)
    ops.latent_queries(q.to(DEV), q.shape[1], q_abs.to(DEV), turn, row_pos, qo, heads, dim, rank, T)
    tol = 1e-5 if dtype == "float32" else 2 ** -7

    def close(a, b):
        assert (a.double().cpu() - b).abs().max() <= tol * b.abs().max()
    s = src.double()
    if q_rank:
        close(cq, P.unit_rms(s[:, :q_rank], eps) * nq.double())
    pages = cache.groups[0].table_host[slot]
    store = cache.groups[0].storage[0].reshape(cache.groups[0].n_pages, 64, rank + rot)
    rows = torch.stack([store[pages[t // 64], t % 64] for t in range(T)])
    close(rows[:, :rank], P.unit_rms(s[:, cols[1]:cols[1] + rank], eps) * nkv.double())
    close(rows[:, rank:], P.rotate(s[:, None, cols[1] + rank:cols[1] + rank + rot], pos, spec, layout)[:, 0])
    qv = qo.view(T, heads, rank + rot)
    assert torch.equal(qv[:, :, :rank].cpu(), q_abs.transpose(0, 1))
    close(qv[:, :, rank:], P.rotate(q.double().view(T, heads, dim + rot)[..., dim:].contiguous(), pos, spec, layout))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,vd", [(5, 14), (4, 64), (3, 7)])
def test_heads_side_by_side_times_their_gate(heads, vd, dtype):
    from x0ne_engine_b200.csrc import ops
    g = torch.Generator().manual_seed(vd)
    dt, T = TORCH[dtype], 33
    x, wide = torch.randn(heads, T, vd, generator=g).to(dt).to(DEV), torch.randn(T, heads * vd + 16, generator=g).to(dt).to(DEV)
    out = torch.empty((T, heads * vd), dtype=dt, device=DEV)
    ops.heads_gate(x, wide[0, 8:], heads * vd + 16, out, T)
    want = x.double().transpose(0, 1).reshape(T, -1) * torch.sigmoid(wide.double()[:, 8:8 + heads * vd])
    assert (out.double() - want).abs().max() <= (1e-6 if dtype == "float32" else 2 ** -8) * want.abs().max()


@pytest.mark.parametrize("rows", [1, 5, 8, 9, 32])
@pytest.mark.parametrize("heads,k,n,rot,half", [(5, 12, 22, 8, True), (3, 128, 70, 32, False), (2, 200, 33, 0, True), (4, 260, 128, 16, True), (1, 1000, 5, 0, False)])
def test_products_per_head_of_few_rows(heads, k, n, rot, half, rows):
    from x0ne_engine_b200.csrc import ops
    g = torch.Generator().manual_seed(k + rows)
    r = lambda *s: torch.randn(*s, generator=g).bfloat16()
    x, w, gate = r(rows, heads * (k + rot) + 4), r(heads, n, k), r(rows, heads * n + 9)
    pos = [7 + 13 * i for i in range(rows)]
    xh = x[:, :heads * (k + rot)].double().view(rows, heads, k + rot)
    y = torch.einsum("hnk,rhk->rhn", w.double(), xh[..., :k])
    xd, wd, gd = x.to(DEV), w.to(DEV), gate.to(DEV)
    assert ops.head_products_take(xd, x.shape[1], k + rot, wd, rows)
    out = torch.full((rows, heads * n), 7.0, dtype=torch.bfloat16, device=DEV)
    ops.head_products(xd, x.shape[1], k + rot, wd, out, n, rows, gate=gd[0, 3:], gate_ld=heads * n + 9)
    want = y.reshape(rows, -1) * torch.sigmoid(gate[:, 3:3 + heads * n].double())
    assert (out.double().cpu() - want).abs().max() <= 2 ** -8 * want.abs().max()
    freq = torch.tensor(P.yarn(rot, 70.0, None)[0], dtype=torch.float32, device=DEV) if rot else None
    out = torch.full((rows, heads * (n + rot)), 7.0, dtype=torch.bfloat16, device=DEV)
    ops.head_products(xd, x.shape[1], k + rot, wd, out, n + rot, rows, turn=ops.latent_turn(freq, None, 1.25, rot, half), row_pos=i32(pos))
    tail = xh[..., k:].contiguous()
    if rot:
        tail = 1.25 * P.rotate(tail, torch.tensor(pos), {"dims": rot, "base": 70.0}, "half" if half else "interleaved")
    want = torch.cat([y, tail], dim=-1).reshape(rows, -1)
    assert (out.double().cpu() - want).abs().max() <= 2 ** -7 * want.abs().max()


# ------------------------------------------------------------------------------------------ activations in the products
@pytest.mark.parametrize("m", [1, 8, 12, 40, 64, 300, 1000])
@pytest.mark.parametrize("n,k", [(176, 128), (1000, 512), (8192, 256)])
def test_activations_in_every_products_epilogue(n, k, m):
    from x0ne_engine_b200.csrc import ops
    g = torch.Generator().manual_seed(m + n)
    x = torch.randn(m, k, generator=g).bfloat16().to(DEV)
    w = (torch.randn(n, k, generator=g) * k ** -0.5).bfloat16().to(DEV)
    z = x.double() @ w.double().T
    kinds = [kind for kind, ok in (("smallm", ops.gemm_smallm_takes(w, m)), ("skinny", ops.gemm_skinny_tc_takes(w, m)), ("tc_pair", m >= 300), ("tc", m >= 300)) if ok]
    for dt, act, want in ((torch.bfloat16, (ops.OUT_RELU2, 0.0), P.relu_squared(z)), (torch.float32, (ops.OUT_SOFT_CAP, 1.5), P.soft_cap(z, 1.5))):
        for kind in kinds:
            out = torch.zeros((m, n), dtype=dt, device=DEV)
            if kind == "smallm":
                ops.gemm_bf16_smallm(x, w, out, m, act=act)
            elif kind == "skinny":
                ops.gemm_bf16_skinny_tcgen05(x, w, out, m, act=act)
            else:
                ops.gemm_bf16_tcgen05(x, w, out, m, pair=kind == "tc_pair", act=act)
            ops.check_tc_status(x.device)
            err = (out.double() - want).abs().max() / want.abs().max()
            assert err <= (2 ** -8 if dt == torch.bfloat16 else 2e-5), (kind, float(err))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("m", [1, 20, 200, 900])
def test_a_linear_with_an_activation_wherever_it_runs(m, dtype):
    from x0ne_engine_b200.csrc import ops
    from x0ne_engine_b200.parts import Linear
    g = torch.Generator().manual_seed(m)
    dt = TORCH[dtype]
    x, w = torch.randn(m, 64, generator=g).to(dt).to(DEV), (torch.randn(210, 64, generator=g) / 8).to(dt).to(DEV)
    z = x.double() @ w.double().T
    out = torch.empty((m, 210), dtype=dt, device=DEV)
    Linear(w)(x, out, m, act=(ops.OUT_RELU2, 0.0))
    assert (out.double() - P.relu_squared(z)).abs().max() <= (1e-5 if dtype == "float32" else 2 ** -6) * P.relu_squared(z).max()
    logits = torch.empty((m, 210), device=DEV)
    Linear(w)(x, logits, m, act=(ops.OUT_SOFT_CAP, 2.0))
    assert (logits.double() - P.soft_cap(z, 2.0)).abs().max() <= 2e-5


# ------------------------------------------------------------------------------------------ whole models
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name,lengths", [("latent_only", [1, 2, 45, 46, 130]), ("attn_only", [1, 2, 37, 38, 130]), ("delta_only", [1, 2, 3, 40]), ("mlp_only", [1, 3, 70]),
                                          ("reader_only", [1, 6, 130]), ("mixed", [1, 2, 38, 65, 150]), ("even", [64, 131, 300]), ("wide", [5, 71, 141]),
                                          ("odd", [1, 12, 90]), ("plain", [1, 100]), ("served", [7, 300, 1000])])
def test_each_request_alone_and_whole(name, lengths, dtype):
    eng, cfg, t = engine(name, dtype)
    for k, n in enumerate(lengths):
        ids = H.random_ids(cfg, n, seed=k)
        check(dtype, whole(eng, ids), H.plain_logits(cfg, t, ids), f"{name} len {n}")


def test_residual_stream_after_every_layer():
    """The float32 residual after each layer (the pending result biased, normed, scaled and added by hand) against the plain one."""
    eng, cfg, t = engine("mixed", "float32", pass_graphs=False)
    ids = H.random_ids(cfg, 90, seed=3)
    seen = []
    for b in eng.model.blocks:
        def wrapped(ctx, entry, resid, delta, cache_entry=None, write_cache=True, _f=b.forward):
            out = _f(ctx, entry, resid, delta, cache_entry=cache_entry, write_cache=write_cache)
            d = out.delta[:ctx.n_rows].double() + (0.0 if out.bias is None else out.bias.double())
            seen.append((resid[:ctx.n_rows].double() + P.layer_norm(d, out.norm.weight.double(), out.norm.eps)).cpu())
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
        assert (a - b.double()).abs().max() <= 1e-4 * b.abs().max(), f"layer {i}"


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
@pytest.mark.parametrize("name", ["mixed", "wide", "plain"])
def test_unequal_batches_against_each_alone_with_slots_used_again(name, dtype):
    eng, cfg, t = engine(name, dtype)
    for turn in range(3):                      # the second and third turns get slots, pages and states that were used
        lengths, steps = [[1, 30, 77, 140], [66, 2, 129], [140, 5]][turn], [3, 9, 1, 6]
        full = [H.random_ids(cfg, n + steps[k], seed=10 * turn + k) for k, n in enumerate(lengths)]
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
            same_cut(dtype, np.concatenate(got[k]), alone, f"{name} turn {turn} request {k}")
            if turn == 0:
                check(dtype, alone, H.plain_logits(cfg, t, full[k]), f"{name} request {k}")


@pytest.mark.parametrize("dtype", DTYPES)
def test_prompts_and_single_tokens_in_one_pass(dtype):
    """A sequence that goes on by one token beside one that brings a prompt: the kernels for many tokens take the one too."""
    eng, cfg, t = engine("mixed", dtype)
    a, b = H.random_ids(cfg, 91, seed=31), H.random_ids(cfg, 70, seed=32)
    sa, sb = eng.new_sequence(), eng.new_sequence()
    eng.step([sa], [a[:90]])
    out = eng.step([sa, sb], [a[90:], b], [[0], list(range(70))]).cpu().numpy()
    for s in (sa, sb):
        eng.free_sequence(s)
    same_cut(dtype, out[:1], whole(eng, a)[-1:], "the token")
    same_cut(dtype, out[1:], whole(eng, b), "the prompt")


# ------------------------------------------------------------------------------------------ edges, far keys
@pytest.mark.parametrize("dtype", DTYPES)
def test_window_edges_that_decide(dtype):
    """Sharp queries make single keys decide a row, so a window whose edge is one off, or a page read wrongly, changes the
    logits by far more than the tolerance.  Windows of 45, 50 and (a reader's) 70 positions against pages of 64; every position
    of a 260-token sequence is checked, in a prompt and decoded alone."""
    eng, cfg, t = engine("sharp", dtype, seed=3)
    ids = H.random_ids(cfg, 260, seed=8)
    want = H.plain_logits(cfg, t, ids)
    for which in range(3):
        for by in (1, -1):
            layers = [dict(l, mixer=dict(l["mixer"], mask={"size": l["mixer"]["mask"]["size"] + (by if i == which else 0)})) for i, l in enumerate(cfg["layers"])]
            diff = np.abs(H.plain_logits({**cfg, "layers": layers}, t, ids) - want).max(-1) / np.abs(want).max(-1)
            assert (diff > 0.1).sum() > 4, (which, by)                  # the test sees what it is for
    check(dtype, whole(eng, ids), want, "prompt")
    check(dtype, in_pieces(eng, ids, [30] + [1] * 230), want, "decoded across window edges and page borders")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind,window", [("attention", None), ("attention", 699), ("latent_attention", None), ("latent_attention", 699), ("attention", 400)])
def test_a_key_far_back(kind, window, dtype):
    """Attention over 700 positions in which the last query answers one early key alone (one embedding feature that only that
    token has feeds one key channel, another that only the last token has feeds the same query channel): the last logits
    hang on a key many pages back, just inside the window, read in a prompt and in decoding."""
    from x0ne_engine_b200 import Engine
    m = H.attn(heads=4, kv_heads=2, rot=(4, 50.0), window=window, scale=0.4) if kind == "attention" else H.latent(heads=3, window=window, scale=0.4)
    cfg = H.config([H.layer(kind, m, None), H.layer("delta", H.delta())])
    t = H.make_tensors(cfg, seed=4)
    special, late = 7, 11
    t["embed"][:, :2] = 0.0
    t["embed"][special, 0] = t["embed"][late, 1] = 14.0
    if kind == "attention":
        d = m["dim"]
        kr, qr = d + d - 1, 3 * d + d - 1                   # kv head 1 / query head 3, the last channel (not rotated)
        for name, row, feature in (("l0.mix.k", kr, 0), ("l0.mix.q", qr, 1)):
            t[name][row], t[name + ".b"][row] = 0.0, 0.0
            t[name][row, feature] = 5.0
        t["l0.mix.v"] *= 3.0
    else:
        t["l0.mix.dkv"][3], t["l0.mix.dq"][2] = 0.0, 0.0     # one value of each latent, which one head's key and query read
        t["l0.mix.dkv"][3, 0] = t["l0.mix.dq"][2, 1] = 9.0
        row = (m["dim"] + m["rot_dim"]) + 4                  # head 1, channel 4
        t["l0.mix.uq"][row], t["l0.mix.uk"][m["dim"] + 4] = 0.0, 0.0
        t["l0.mix.uq"][row, 2] = t["l0.mix.uk"][m["dim"] + 4, 3] = 4.0
    t = {k: v.bfloat16().float() for k, v in t.items()}
    folder = H.write_folder(cfg, t, "x0ne_trd_far_")
    ids = [12 + x % (cfg["vocab"] - 12) for x in H.random_ids(cfg, 700, 9)]
    at = 0 if window is None else 700 - window               # the first key the last query still sees
    ids[at], ids[-1] = special, late
    eng = Engine.from_folder(folder, dtype=dtype, max_tokens=1024, max_seq_len=1024)
    want = H.plain_logits(cfg, t, ids)
    other = list(ids)
    other[at] = 13                                           # another token in its place: the far key is gone
    gone = np.abs(H.plain_logits(cfg, t, other)[-1] - want[-1]).max()
    assert gone > 0.1 * np.abs(want[-1]).max()
    if window is not None:                                   # one position further back the key is out of sight
        moved = list(ids)
        moved[at], moved[at - 1] = 13, special
        near = H.plain_logits(cfg, t, moved)
        assert np.abs(near[-1] - want[-1]).max() > 0.1 * np.abs(want[-1]).max()
        check(dtype, whole(eng, moved)[-3:], near[-3:], "a key just outside the window")
        check(dtype, in_pieces(eng, moved, [697, 1, 1])[-3:], near[-3:], "the same decoded")
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


def test_the_extra_denominator_term_shows():
    """One key in sight and a score of zero: half the weight goes to the term that has no value."""
    eng, cfg, t = engine("attn_only", "float32")
    ids = H.random_ids(cfg, 1, seed=2)
    want = H.plain_logits(cfg, t, ids)
    keep = P.windowed_attention
    P.windowed_attention = lambda q, k, v, s, p, w, extra: keep(q, k, v, s, p, w, False)
    try:
        without = H.plain_logits(cfg, t, ids)
    finally:
        P.windowed_attention = keep
    assert np.abs(without - want).max() > 0.02 * np.abs(want).max()
    check("float32", whole(eng, ids), want, "one token")


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding(dtype):
    eng, cfg, t = engine("even", dtype)
    ids = H.random_ids(cfg, 420, seed=12)
    check(dtype, in_pieces(eng, ids, [20] + [1] * 400), H.plain_logits(cfg, t, ids), "400 decoded tokens")


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
