"""Tarudra on the CPU: the reader of config.json, its refusals, the model as data (parts, tensor names, run order, what every
layer keeps per sequence), and properties of the plain implementation itself."""
import copy

import numpy as np
import pytest
import torch

import tarudra_helpers as H
import tarudra_plain as P
from x0ne_engine_b200.config import ConfigError, config_from_dict, detect
from x0ne_engine_b200.config.tarudra import TarudraConfig
from x0ne_engine_b200.engine.model import CausalLM, cache_needs_of_layer, step_bytes_of_spec, tensor_needs_of_spec


def test_config_is_read_and_written_back():
    for name, make in H.CONFIGS.items():
        d = make()
        assert detect(d) == "Tarudra"
        c = config_from_dict(d)
        assert isinstance(c, TarudraConfig) and c.to_dict() == d, name
        assert config_from_dict(c.to_dict()) == c


@pytest.mark.parametrize("change,word", [
    (lambda d: d.update(loop={}), "loop"),
    (lambda d: d["layers"][0]["mixer"].update(sink=1), "sink"),
    (lambda d: d["layers"][0]["mixer"].pop("q_rank"), "q_rank"),
    (lambda d: d["layers"][0]["mixer"].pop("rot"), "rot"),
    (lambda d: d["layers"][0]["mixer"]["rot"].update(dims=4), "rot_dim"),
    (lambda d: d["layers"][0]["mixer"].update(kv_rank=0), "kv_rank"),
    (lambda d: d["layers"][1]["mixer"].update(heads=5), "multiple"),
    (lambda d: d["layers"][1]["mixer"]["mask"].update(keep_first=1), "keep_first"),
    (lambda d: d["layers"][1]["mixer"]["mask"].update(size=0), "size"),
    (lambda d: d["layers"][1]["mixer"]["rot"].update(dims=22), "dims"),
    (lambda d: d["layers"][1]["mixer"]["rot"].update(dims=7), "dims"),
    (lambda d: d["layers"][1]["mixer"]["rot"]["scaling"].pop("slow"), "slow"),
    (lambda d: d["layers"][1]["mixer"]["rot"]["scaling"].update(beta=1), "beta"),
    (lambda d: d["layers"][1]["mixer"].pop("scale"), "scale"),
    (lambda d: d["layers"][3]["mixer"].update(kv_from=3), "kv_from"),
    (lambda d: d["layers"][3]["mixer"].update(kv_from=0), "kv_from"),
    (lambda d: d["layers"][5]["mixer"].update(kv_from=3), "kv_from"),
    (lambda d: d["layers"][3]["mixer"].update(kv_heads=1), "kv_heads"),
    (lambda d: d["layers"][3]["mixer"].update(vdim=13), "vdim"),
    (lambda d: d["layers"][3]["mixer"]["rot"].update(base=7.0), "rotation"),
    (lambda d: d["layers"][2]["mixer"].update(scale=1.0), "scale"),
    (lambda d: d["layers"][2]["mixer"].update(conv=0), "conv"),
    (lambda d: d["layers"][2]["mixer"].update(kv_heads=4), "multiple"),
    (lambda d: d["layers"][2].update(type="mamba"), "mamba"),
    (lambda d: d["layers"][0]["mlp"].update(kind="moe"), "moe"),
    (lambda d: d["layers"][0]["mlp"].pop("ff"), "ff"),
    (lambda d: d["norm"].pop("eps"), "eps"),
    (lambda d: d.update(logit_softcap=-1.0), "logit_softcap"),
    (lambda d: d.update(layers=[]), "layers"),
])
def test_refusals_name_the_key(change, word):
    d = copy.deepcopy(H.CONFIGS["mixed"]())
    change(d)
    with pytest.raises(ConfigError) as e:
        config_from_dict(d)
    assert word in str(e.value)


@pytest.mark.parametrize("name", sorted(H.CONFIGS))
def test_spec_reads_exactly_the_tensors_of_the_design(name):
    cfg = H.CONFIGS[name]()
    tensors = H.make_tensors(cfg, 0)
    needs = {n.name: tuple(n.shape) for n in tensor_needs_of_spec(config_from_dict(cfg).to_spec())}
    assert needs == {k: tuple(v.shape) for k, v in tensors.items()}


def test_what_the_layers_are_made_of_and_keep():
    spec = config_from_dict(H.CONFIGS["mixed"]()).to_spec()
    assert [l.part("mixer").kind for l in spec.layers] == ["latent_attention", "masked_attention", "gated_delta_rule", "masked_attention", "gated_delta_rule", "masked_attention"]
    assert [e.reads_cache_of for e in spec.run_order] == [None, None, None, 1, None, 1]
    assert "ffn" not in spec.layers[4].parts and spec.layers[5].part("mixer")["own_kv"] is False
    kept = [cache_needs_of_layer(l) for l in spec.layers]
    assert all(len(k) == 1 for k in kept)
    assert (kept[0][0].kind, kept[0][0].kv_heads, kept[0][0].head_dim, kept[0][0].v_dim, kept[0][0].window) == ("kv", 1, 22 + 6, 0, None)
    assert (kept[1][0].kv_heads, kept[1][0].head_dim, kept[1][0].v_dim, kept[1][0].window) == (2, 20, 12, None)
    # heads x values x channels, then a ring of as many rows as taps of q, k and v
    assert kept[2][0].kind == "state" and kept[2][0].state_shape[0] == 6 * 20 * 12 + 3 * (2 * 3 * 12 + 6 * 20)
    m = CausalLM(spec, torch.bfloat16, "cpu")
    assert m.replayable() and m.head.act[1] == 17.0
    assert CausalLM(config_from_dict(H.CONFIGS["plain"]()).to_spec(), torch.bfloat16, "cpu").head.act is None
    weights, per_token = step_bytes_of_spec(spec)
    assert weights > 0 and per_token == 2 * (28 + 2 * (20 + 12))          # one latent row and one layer's keys and values


def test_layers_with_one_rotation_share_its_table():
    spec = config_from_dict(H.CONFIGS["mixed"]()).to_spec()
    assert len(spec.positions) == 2                            # the latent's, and one for the layer with keys and its readers
    spec = config_from_dict(H.config([H.layer("attention", H.attn(rot=(8, 300.0, H.YARN))), H.layer("attention", H.attn(rot=(8, 300.0))),
                                      H.layer("attention", H.attn(rot=(8, 300.0, {**H.YARN, "factor": 2.0})))])).to_spec()
    assert len(spec.positions) == 3


def test_packed_projections_and_folded_scales_on_the_cpu():
    cfg = H.CONFIGS["mixed"]()
    t = H.make_tensors(cfg, 0)
    m = CausalLM(config_from_dict(cfg).to_spec(), torch.float32, "cpu")
    m.bind(t)
    b = m.blocks[0]
    assert torch.equal(b.mixer_post_norm.weight, t["l0.norm1b"] * t["l0.ls1"]) and torch.equal(b.ffn_post_norm.weight, t["l0.norm2b"] * t["l0.ls2"])
    assert torch.equal(b.mixer_norm.weight, t["l0.norm1"])
    lat = b.mixer
    assert [c % 8 for c in lat.cols] == [0, 0, 0] and torch.equal(lat.proj.weight[lat.cols[2]:lat.cols[2] + 70], t["l0.mix.g"])
    att, reader = m.blocks[1].mixer, m.blocks[3].mixer
    assert torch.equal(att.result_bias, t["l1.mix.o.b"]) and torch.equal(att.qkv_bias[120:160], t["l1.mix.k.b"])
    assert reader.qkv.weight.shape == (80, 72) and torch.equal(reader.qkv_bias, t["l3.mix.q.b"])
    d = m.blocks[2].mixer
    assert torch.equal(d.conv[36:72], t["l2.mix.k.conv"]) and torch.allclose(d.A, torch.exp(t["l2.mix.A_log"]))
    w = d.in_weight
    assert torch.equal(w[d.cols[3]:d.cols[3] + 6], t["l2.mix.a"]) and torch.equal(w[d.cols[5]:d.cols[5] + 120], t["l2.mix.g"])


# ------------------------------------------------------------------------------------------ the plain implementation itself
@pytest.mark.parametrize("name", ["mixed", "odd", "plain"])
def test_plain_pieces_against_the_whole(name):
    _, cfg, t = H.folder(name)
    ids = H.random_ids(cfg, 60, 1)
    want = H.plain_logits(cfg, t, ids)
    for cuts in ([1] * 60, [7, 1, 2, 50], [59, 1]):
        carry, got, at = {}, [], 0
        for n in cuts:
            got.append(P.forward(cfg, t, ids[at:at + n], carry=carry).numpy())
            at += n
        assert np.abs(np.concatenate(got) - want).max() <= 1e-9 * np.abs(want).max()


def test_plain_delta_rule_answers_what_was_written_last():
    """With beta one and no decay a key's stored value is replaced: reading it back gives the last value written."""
    q = torch.eye(4, dtype=torch.float64)[None, :3].transpose(0, 1).repeat(2, 1, 1)      # keys 0, 1, 2, then again
    v = torch.randn(6, 1, 5, dtype=torch.float64)
    one = torch.ones(6, 1, dtype=torch.float64)
    S = torch.zeros(1, 4, 5, dtype=torch.float64)
    o = P.delta_scan(q, q, v, one, one, S)
    assert torch.allclose(o, v) and torch.allclose(S[0, :3], v[3:, 0])
    half = P.delta_scan(q[:1], q[:1], v[:1], 0.25 * one[:1], 0.5 * one[:1], torch.ones(1, 4, 5, dtype=torch.float64))
    assert torch.allclose(half[0, 0], 0.5 + 0.25 * (v[0, 0] - 0.5))


def test_plain_yarn_leaves_fast_pairs_and_divides_slow_ones():
    freq, mag = P.yarn(64, 10000.0, {"factor": 8.0, "original": 256, "fast": 32.0, "slow": 1.0})
    raw, one = P.yarn(64, 10000.0, None)
    assert one == 1.0 and abs(mag - (0.1 * np.log(8.0) + 1.0)) < 1e-12
    assert freq[0] == raw[0] and abs(freq[-1] - raw[-1] / 8.0) < 1e-15
    from x0ne_engine_b200.parts import yarn_frequencies
    got, m = yarn_frequencies(64, 10000.0, {"factor": 8.0, "original": 256, "fast": 32.0, "slow": 1.0})
    assert np.allclose(got, freq, rtol=1e-13) and m == mag


def test_plain_window_and_extra_term():
    T = 9
    q = torch.zeros(T, 1, 4, dtype=torch.float64)
    v = torch.arange(T, dtype=torch.float64)[:, None, None].expand(T, 1, 2)
    pos = torch.arange(T)
    o = P.windowed_attention(q, q, v, 1.0, pos, 3, False)[:, 0, 0]
    assert torch.allclose(o[2:], pos[2:].double() - 1.0) and o[0] == 0 and o[1] == 0.5
    o1 = P.windowed_attention(q, q, v, 1.0, pos, 3, True)[:, 0, 0]
    assert torch.allclose(o1[2:], (3.0 * pos[2:].double() - 3.0) / 4.0)
