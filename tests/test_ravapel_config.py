"""Ravapel on the CPU: the reader of config.json, its refusals, the model as data (parts, tensor names, run order, what
every layer run keeps per sequence), and properties of the plain implementation itself."""
import copy

import numpy as np
import pytest
import torch

import ravapel_helpers as H
import ravapel_plain as P
from x0ne_engine_b200.config import ConfigError, config_from_dict, detect
from x0ne_engine_b200.config.ravapel import RavapelConfig
from x0ne_engine_b200.engine.model import CausalLM, cache_needs_of_layer, step_bytes_of_spec, tensor_needs_of_spec


def test_config_is_read_and_written_back():
    for name, make in H.CONFIGS.items():
        d = make()
        assert detect(d) == "Ravapel"
        c = config_from_dict(d)
        assert isinstance(c, RavapelConfig) and c.to_dict() == d, name
        assert config_from_dict(c.to_dict()) == c
        assert c.to_spec().max_position_embeddings == d["max_positions"]


@pytest.mark.parametrize("change,word", [
    (lambda d: d["layers"][0]["mixer"].update(extra=1), "extra"),
    (lambda d: d["layers"][1]["mixer"].update(middle=1), "middle"),
    (lambda d: d["layers"][1]["mixer"]["left"].update(sink=1), "sink"),
    (lambda d: d["layers"][1]["mixer"]["left"]["mask"].update(left=1), "left"),
    (lambda d: d["layers"][1]["mixer"]["left"].update(heads=5), "multiple"),
    (lambda d: d["layers"][1]["mixer"]["left"]["rot"].update(dims=22), "rot.dims"),
    (lambda d: d["layers"][1]["mixer"]["left"]["rot"].update(dims=7), "rot.dims"),
    (lambda d: d["layers"][1]["mixer"]["left"].pop("scale"), "scale"),
    (lambda d: d["layers"][1]["mixer"].pop("right_scale"), "right_scale"),
    (lambda d: d["layers"][1]["mixer"]["right"].pop("gate_cap"), "gate_cap"),
    (lambda d: d["layers"][1]["mixer"]["right"].update(gate_cap=0.0), "gate_cap"),
    (lambda d: d["layers"][0]["mixer"].update(dim=0), "dim"),
    (lambda d: d["layers"][0].update(type="hgrn"), "hgrn"),
    (lambda d: d["layers"][0]["mlp"].update(kind="moe"), "moe"),
    (lambda d: d["layers"][0]["mlp"].pop("ff"), "ff"),
    (lambda d: d["norm"].pop("eps"), "eps"),
    (lambda d: d["canon"].update(taps=0), "taps"),
    (lambda d: d.pop("canon"), "canon"),
    (lambda d: d["embedding"]["bigram"].update(buckets=0), "buckets"),
    (lambda d: d["embedding"]["bigram"].update(mul_prev=-3), "mul_prev"),
    (lambda d: d["embedding"].update(scale=2.0), "scale"),
    (lambda d: d.pop("max_positions"), "max_positions"),
    (lambda d: d["loop"].update(stop=9), "loop"),
    (lambda d: d["loop"].update(start=3), "loop"),
    (lambda d: d["loop"].update(times=0), "times"),
])
def test_refusals_name_the_key(change, word):
    d = copy.deepcopy(H.CONFIGS["mixed"]())
    change(d)
    with pytest.raises(ConfigError) as e:
        config_from_dict(d)
    assert word in str(e.value)


def test_run_order_repeats_the_stretch_and_opens_every_pass():
    d = H.CONFIGS["mixed"]()
    c = config_from_dict(d)
    assert [i for i, _ in c.run_layers()] == [0, 1, 2, 1, 2, 3] == [i for i, _ in P.run_order(d)]
    assert [o for _, o in c.run_layers()] == [o for _, o in P.run_order(d)]
    spec = c.to_spec()
    assert [k for k, e in enumerate(spec.run_order) if e.before is not None] == [1, 3]        # the first pass opens too
    assert all(e.reads_cache_of is None for e in spec.run_order)           # every pass keeps caches and states of its own
    assert spec.embedding["keep"]                                          # the openers read the embedding output again
    even = config_from_dict(H.CONFIGS["even"]()).to_spec()
    assert [e.layer for e in even.run_order] == [0, 1, 0, 1, 0, 1, 2]
    assert [k for k, e in enumerate(even.run_order) if e.before is not None] == [0, 2, 4]
    once = config_from_dict(H.CONFIGS["wide"]()).to_spec()
    assert [e.before is not None for e in once.run_order] == [True, False, False, False]
    none = config_from_dict(H.CONFIGS["plain"]()).to_spec()
    assert all(e.before is None for e in none.run_order) and not none.embedding["keep"]


def test_tensor_names_and_shapes_are_the_checkpoints():
    for name, make in H.CONFIGS.items():
        d = make()
        needs = {n.name: tuple(n.shape) for n in tensor_needs_of_spec(config_from_dict(d).to_spec())}
        have = {k: tuple(v.shape) for k, v in H.make_tensors(d, 0).items()}
        assert needs == have, (name, sorted(set(needs) ^ set(have)))


def test_parts_carry_every_constant_of_the_layer():
    d = H.CONFIGS["mixed"]()
    spec = config_from_dict(d).to_spec()
    e, b = spec.embedding, d["embedding"]["bigram"]
    assert e.kind == "sum_embedding" and (e["buckets"], e["mul_prev"], e["mul_cur"], e["positions"]) == (
        b["buckets"], b["mul_prev"], b["mul_cur"], d["max_positions"])
    m = d["layers"][1]["mixer"]
    pair = spec.layers[1].part("mixer")
    assert pair.kind == "side_by_side" and (pair["left_scale"], pair["right_scale"]) == (m["left_scale"], m["right_scale"])
    a, x = pair["left"], m["left"]
    assert a.kind == "sigmoid_attention" and a["chunk"] == x["mask"]["size"] and a["scale"] == x["scale"] and a["qk_norm_eps"] == d["norm"]["eps"]
    assert (a["q_heads"], a["kv_heads"], a["head_dim"], a["v_dim"]) == (x["heads"], x["kv_heads"], x["dim"], x["vdim"])
    rot = spec.positions[a["position"]]
    assert rot.kind == "rope" and rot["rotary_dim"] == x["rot"]["dims"] and rot["theta"] == x["rot"]["base"]
    r, y = pair["right"], m["right"]
    assert r.kind == "matrix_memory" and (r["heads"], r["head_dim"], r["v_dim"], r["gate_cap"]) == (y["heads"], y["dim"], y["vdim"], y["gate_cap"])
    h, z = spec.layers[0].part("mixer"), d["layers"][0]["mixer"]
    assert h.kind == "channel_gated_recurrence" and (h["heads"], h["head_dim"], h["v_dim"]) == (z["heads"], z["dim"], z["vdim"])
    assert spec.layers[0].block == "sandwich" and spec.layers[0].part("mixer_input")["taps"] == d["canon"]["taps"]
    assert spec.layers[0].part("ffn").kind == "swiglu" and spec.layers[0].part("ffn")["bias"] and "ffn" not in spec.layers[2].parts
    assert all(spec.layers[0].part(s)["one_plus"] for s in ("mixer_norm", "mixer_post_norm", "ffn_norm", "ffn_post_norm")) and spec.final_norm["one_plus"]
    # layers whose rotations have the same constants share one table; others get their own; none where nothing rotates
    assert len(spec.positions) == 2 and config_from_dict(H.CONFIGS["plain"]()).to_spec().positions == {}


def test_what_a_layer_run_keeps():
    d = H.CONFIGS["mixed"]()
    spec = config_from_dict(d).to_spec()
    needs = [{(n.kind, n.tag): n for n in cache_needs_of_layer(l)} for l in spec.layers]
    assert sorted(needs[0]) == [("state", ""), ("state", "input conv")]
    assert needs[0][("state", "")].state_shape == (3 * 12 * 20,) and needs[0][("state", "input conv")].state_shape == (2 * 72,)
    assert sorted(needs[1]) == [("kv", ""), ("state", "input conv"), ("state", "right")]
    kv = needs[1][("kv", "")]
    assert (kv.kv_heads, kv.head_dim, kv.v_dim, kv.window) == (2, 20, 12, None)
    assert needs[1][("state", "right")].state_shape == (2 * 15 * 10 + 4,)          # the key sum as a column more, two maxima per head
    _, per_token = step_bytes_of_spec(spec)
    assert per_token == 2 * (2 * 2 * (20 + 12) + 4 * (16 + 16))                  # two runs of layer 1, one of layer 3
    from x0ne_engine_b200.parts import EMBEDDINGS
    (prev,) = EMBEDDINGS.get("sum_embedding").cache_needs(spec.embedding)
    assert prev.kind == "state" and prev.state_shape == (1,)
    # one tap keeps nothing
    plain = config_from_dict(H.CONFIGS["plain"]()).to_spec()
    assert not any(n.tag == "input conv" for n in cache_needs_of_layer(plain.layers[0]))


def test_cache_of_entries_that_keep_several_things():
    from x0ne_engine_b200.cache import SequenceCache
    spec = config_from_dict(H.CONFIGS["mixed"]()).to_spec()
    needs = [cache_needs_of_layer(spec.layers[e.layer]) for e in spec.run_order]
    from x0ne_engine_b200.parts import CacheNeed
    c = SequenceCache(needs, [None] * len(needs), 512, 512, torch.float32, "cpu", max_slots=3, model_needs=[CacheNeed("state", state_shape=(1,), tag="t")])
    assert len(c.groups) == 2 and [g.entries for g in c.groups] == [[1, 3], [5]]     # every pass has a cache of its own
    a = c.acquire(10)
    for s in (c.state(0), c.state(0, "input conv"), c.state(1, "right"), c.state(3, "right"), c.model_state("t")):
        s[a] = 7.0
    assert c.state(1, "right").data_ptr() != c.state(3, "right").data_ptr()
    idx, saved = c.snapshot_states(torch.tensor([a]))
    assert len(saved) == 6 + 6 + 1                                           # six runs: a convolution and a recurrence each; the model's
    c.release(a)
    b = c.acquire(10)                                                        # the slot comes back clean
    assert b == a and all(float(s[b].abs().sum()) == 0.0 for s in c.states.values())
    with pytest.raises(ValueError, match="two states"):
        SequenceCache([[CacheNeed("state", state_shape=(1,)), CacheNeed("state", state_shape=(2,))]], [None], 64, 64, torch.float32, "cpu")
    with pytest.raises(ValueError, match="twice"):
        SequenceCache([[CacheNeed("kv", 1, 8), CacheNeed("kv", 2, 8)]], [None], 64, 64, torch.float32, "cpu")


def test_two_mixers_that_both_keep_keys_are_refused():
    from x0ne_engine_b200.config.spec import LayerSpec, PartSpec
    spec = config_from_dict(H.CONFIGS["parallel_only"]()).to_spec()
    pair = spec.layers[0].part("mixer")
    twice = spec.layers[0].with_part("mixer", PartSpec("side_by_side", {**pair.params, "right": pair["left"]}))
    assert isinstance(twice, LayerSpec)
    with pytest.raises(ConfigError, match="both keep keys"):
        cache_needs_of_layer(twice)


def test_packed_projections_start_at_aligned_columns():
    from x0ne_engine_b200.parts.side_by_side import pack_rows
    parts = [torch.randn(n, 6) for n in (5, 8, 3, 16)]
    w, cols = pack_rows(parts)
    assert cols == [0, 8, 16, 24] and w.shape == (40, 6)
    for p, c in zip(parts, cols):
        assert torch.equal(w[c:c + p.shape[0]], p)
    assert float(w[5:8].abs().sum()) == 0.0 and float(w[19:24].abs().sum()) == 0.0


def test_parts_of_every_configuration_can_be_built():
    for make in H.CONFIGS.values():
        m = CausalLM(config_from_dict(make()).to_spec(), torch.float32, "cpu", max_positions=32)
        assert m.replayable()
        m.bind({n.name: torch.zeros(n.shape) for n in tensor_needs_of_spec(m.spec)})


# ------------------------------------------------------------------------------------------ the plain implementation
def test_plain_bigram_rows():
    assert P.bigram_row(None, 5, 97, 31, 11) == 97                           # a sequence's first token: the last row
    assert P.bigram_row(0, 0, 97, 31, 11) == 0
    assert P.bigram_row(200, 100, 97, 31, 11) == (200 * 31 + 100 * 11) % 97
    assert P.bigram_row(100, 200, 97, 31, 11) != P.bigram_row(200, 100, 97, 31, 11)


def test_plain_convolution_looks_back_and_adds_to_its_input():
    h = torch.randn(9, 2, dtype=torch.float64)
    w = torch.tensor([[0.0, 0.0, 0.5], [2.0, 0.0, 0.0]], dtype=torch.float64)
    y, tail = P.input_conv(h, w)
    assert torch.allclose(y[:, 0], 1.5 * h[:, 0]) and torch.allclose(y[2:, 1], h[2:, 1] + 2 * h[:-2, 1]) and torch.equal(y[:2, 1], h[:2, 1])
    assert torch.equal(tail, h[-2:])


def test_plain_rotation_turns_halves_and_leaves_the_rest():
    x = torch.randn(5, 2, 10, dtype=torch.float64)
    pos = torch.tensor([0, 1, 2, 50, 1000])
    y = P.rotate_half(x, pos, 6, 100.0)
    assert torch.equal(y[..., 6:], x[..., 6:]) and torch.equal(y[0], x[0])
    a = 50 * 100.0 ** (-2 / 6)
    u, v = x[3, 1, 1], x[3, 1, 4]
    assert abs(float(y[3, 1, 1]) - float(u * np.cos(a) - v * np.sin(a))) < 1e-12 and abs(float(y[3, 1, 4]) - float(v * np.cos(a) + u * np.sin(a))) < 1e-12


def test_plain_sigmoid_attention_counts_keys_one_by_one():
    g = torch.Generator().manual_seed(0)
    q, k, v = (torch.randn(20, 2, 4, generator=g, dtype=torch.float64) for _ in range(3))
    pos, b = torch.arange(20), torch.tensor([-0.3, 0.8], dtype=torch.float64)
    o = P.sigmoid_attention(q, k, v, 0.7, b, pos, chunk=8)
    s = float((q[8, 1] * k[8, 1]).sum() * 0.7 + 0.8)
    assert torch.allclose(o[8, 1], v[8, 1] / (1 + np.exp(-s)))               # position 8 opens a chunk: it sees itself alone
    w = torch.sigmoid((q[7, 0] @ k[:8, 0].T) * 0.7 - 0.3)
    assert torch.allclose(o[7, 0], w @ v[:8, 0])                             # position 7 closes the chunk before


def test_plain_memory_starts_its_maximum_at_zero():
    """One token whose input gate is far below zero: the running maximum stays near zero, so the write is exp(i - m), small,
    and the normaliser is exp(-m); a maximum that started at minus infinity would write with strength one."""
    S, n, m = torch.zeros(1, 2, 2, dtype=torch.float64), torch.zeros(1, 2, dtype=torch.float64), torch.zeros(1, dtype=torch.float64)
    q = k = torch.tensor([[[1.0, 0.0]]], dtype=torch.float64)
    v = torch.tensor([[[3.0, -1.0]]], dtype=torch.float64)
    i, f = torch.tensor([[-5.0]], dtype=torch.float64), torch.tensor([[-0.1]], dtype=torch.float64)
    o = P.mlstm_scan(q, k, v, i, f, S, n, m)
    assert float(m) == -0.1
    write = np.exp(-4.9)
    assert torch.allclose(o[0, 0], v[0, 0] * write / (np.exp(0.1) + 1e-6))


@pytest.mark.parametrize("name", ["mixed", "odd", "plain"])
def test_plain_model_in_pieces_is_the_model(name):
    cfg = H.CONFIGS[name]()
    t = H.make_tensors(cfg, 2)
    ids = H.random_ids(cfg, 50, 4)
    whole = P.forward(cfg, t, ids)
    carry, out, at = {}, [], 0
    for n in (3, 1, 1, 35, 10):
        out.append(P.forward(cfg, t, ids[at:at + n], carry=carry))
        at += n
    assert torch.allclose(torch.cat(out), whole, rtol=0, atol=1e-9)
