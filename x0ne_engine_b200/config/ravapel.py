"""Ravapel: the typed configuration, read strictly from config.json, and its ModelSpec.

A Ravapel model's embedding is a sum: the token's row, a row for the pair of the previous and the current token (hashed
into `embedding.bigram.buckets`; one row more for a sequence's first token), and a learned row of the position.  It runs a
list of layers with a norm before and after each sublayer, `x += norm1b(mixer(c(norm1(x))))` then (unless the layer has no
feed-forward) `x += norm2b(ff(norm2(x)))`; the norms' weights are stored centred on zero, and c is a short causal
convolution per channel that is added to its input.  A stretch of the list (`loop.start` .. `loop.stop` - 1) runs
`loop.times` times in a row with the same weights and caches and states of its own per pass; right before the first layer of
every pass, the first too, the residual becomes W [x; x0], x0 being the embedding output.

The mixer of a layer is one of

  * `hgrn2`: a recurrence with a matrix state per head and a forget gate per channel (`parts/gated_recurrence.py`);
  * `parallel`: two mixers over the same rows (`parts/side_by_side.py`), scaled and summed: on the left grouped-query
    attention with sigmoid weights over chunks of `mask.size` positions (`parts/sigmoid_attention.py`), on the right the matrix
    memory of xLSTM (`parts/gated_recurrence.py`).

The feed-forward is a SiLU-gated unit whose projections have biases.

Every size and constant comes from config.json (`embedding.bigram`, `canon.taps`, `layers[i].mixer`, `layers[i].mlp`, `loop`,
`max_positions`, `norm.eps`, `vocab`, `width`).  Tensor names: `embed`, `bigram`, `pos`, `loop.in`,
`l<i>.norm1|norm1b|norm2|norm2b|canon1`, `l<i>.mix.*` (a parallel layer's `l<i>.mix.left.*` and `l<i>.mix.right.*`), `l<i>.mlp.*`,
`final.norm`, `head`.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Dict, List, Mapping, Optional, Tuple

from .rovurax import _get, _num, _only, _pint, _plain
from .spec import ConfigError, LayerSpec, ModelSpec, PartSpec, RunEntry

ARCHITECTURE = "Ravapel"
MODEL_TYPE = "ravapel"

MIXERS = ("hgrn2", "parallel")


@dataclass(frozen=True)
class RavapelLayer:
    type: str                       # one of MIXERS
    mixer: Mapping[str, Any]
    mlp: Optional[Mapping[str, Any]]


@dataclass(frozen=True)
class RavapelLoop:
    start: int
    stop: int
    times: int


@dataclass(frozen=True)
class RavapelBigram:
    buckets: int
    mul_prev: int
    mul_cur: int


def _count(d: Mapping[str, Any], key: str, where: str) -> int:
    v = _get(d, key, where)
    if isinstance(v, bool) or not isinstance(v, int) or not 0 <= v < 1 << 31:
        raise ConfigError(f"config.json: {where}.{key} is not a whole number from 0 to 2^31 - 1")
    return v


def _check_attention(m: Mapping[str, Any], where: str) -> None:
    _only(m, ("dim", "heads", "kv_heads", "mask", "rot", "scale", "vdim"), where)
    dim, heads = _pint(m, "dim", where), _pint(m, "heads", where)
    kv = _pint(m, "kv_heads", where) if m.get("kv_heads") is not None else heads
    if m.get("vdim") is not None:
        _pint(m, "vdim", where)
    if heads % kv:
        raise ConfigError(f"config.json: {where}: heads are not a multiple of kv_heads")
    _num(m, "scale", where)
    if m.get("mask") is not None:
        _only(m["mask"], ("size",), where + ".mask")
        _pint(m["mask"], "size", where + ".mask")
    if m.get("rot") is not None:
        _only(m["rot"], ("base", "dims"), where + ".rot")
        dims = _count(m["rot"], "dims", where + ".rot")
        if dims % 2 or dims > dim:
            raise ConfigError(f"config.json: {where}.rot.dims is not an even count of at most dim = {dim} values")
        _num(m["rot"], "base", where + ".rot")


def _check_heads(m: Mapping[str, Any], keys: Tuple[str, ...], where: str) -> None:
    _only(m, ("dim", "heads", "vdim") + keys, where)
    _pint(m, "dim", where)
    _pint(m, "heads", where)
    if m.get("vdim") is not None:
        _pint(m, "vdim", where)


@dataclass(frozen=True)
class RavapelConfig:
    vocab: int
    width: int
    norm_eps: float
    max_positions: int
    layers: Tuple[RavapelLayer, ...]
    taps: int = 1
    bigram: Optional[RavapelBigram] = None
    loop: Optional[RavapelLoop] = None
    dtype: str = "bfloat16"
    eos_token_ids: tuple = ()
    raw: Mapping[str, Any] = field(default_factory=dict, compare=False, repr=False)

    @property
    def max_position_embeddings(self) -> int:
        return self.max_positions

    # ---- reading
    @classmethod
    def from_dict(cls, d: Mapping[str, Any]) -> "RavapelConfig":
        if not isinstance(d, Mapping):
            raise ConfigError("config.json: not a JSON object")
        _only(d, ("architecture", "architectures", "model_type", "canon", "embedding", "layers", "loop", "max_positions", "norm", "vocab",
                  "width", "dtype", "eos_token_id"), "the model")
        norm, canon = _get(d, "norm", "the model"), _get(d, "canon", "the model")
        _only(norm, ("eps",), "norm")
        _only(canon, ("taps",), "canon")
        bigram = None
        if d.get("embedding") is not None:
            _only(d["embedding"], ("bigram",), "embedding")
            b = d["embedding"].get("bigram")
            if b is not None:
                where = "embedding.bigram"
                _only(b, ("buckets", "mul_cur", "mul_prev"), where)
                bigram = RavapelBigram(_pint(b, "buckets", where), _count(b, "mul_prev", where), _count(b, "mul_cur", where))
        raw_layers = _get(d, "layers", "the model")
        if not isinstance(raw_layers, list) or not raw_layers:
            raise ConfigError("config.json: layers is not a list of at least one layer")
        layers: List[RavapelLayer] = []
        for i, l in enumerate(raw_layers):
            where = f"layers[{i}]"
            _only(l, ("type", "mixer", "mlp"), where)
            kind, mixer, mw = _get(l, "type", where), _get(l, "mixer", where), where + ".mixer"
            if kind == "hgrn2":
                _check_heads(mixer, (), mw)
            elif kind == "parallel":
                _only(mixer, ("left", "left_scale", "right", "right_scale"), mw)
                _check_attention(_get(mixer, "left", mw), mw + ".left")
                right = _get(mixer, "right", mw)
                _check_heads(right, ("gate_cap",), mw + ".right")
                _num(right, "gate_cap", mw + ".right")
                _num(mixer, "left_scale", mw, positive=False)
                _num(mixer, "right_scale", mw, positive=False)
            else:
                raise ConfigError(f"config.json: {where}.type {kind!r} is not a mixer of this architecture; it has {list(MIXERS)}")
            mlp = l.get("mlp")
            if mlp is not None:
                _only(mlp, ("ff", "kind"), where + ".mlp")
                if _get(mlp, "kind", where + ".mlp") != "dense":
                    raise ConfigError(f"config.json: {where}.mlp.kind {mlp['kind']!r} is not a feed-forward of this architecture; it has 'dense'")
                _pint(mlp, "ff", where + ".mlp")
            layers.append(RavapelLayer(kind, mixer, mlp))
        loop = None
        if d.get("loop") is not None:
            lp = d["loop"]
            _only(lp, ("start", "stop", "times"), "loop")
            start, stop, times = _get(lp, "start", "loop"), _pint(lp, "stop", "loop"), _pint(lp, "times", "loop")
            if isinstance(start, bool) or not isinstance(start, int) or not 0 <= start < stop <= len(layers):
                raise ConfigError(f"config.json: loop runs layers {start!r} .. {stop} - 1 of {len(layers)}")
            loop = RavapelLoop(start, stop, times)
        dtype = d.get("dtype") or "bfloat16"
        if dtype not in ("bfloat16", "float32"):
            raise ConfigError(f"config.json: dtype {dtype!r}; bfloat16 and float32 checkpoints are served")
        eos = d.get("eos_token_id")
        eos_ids = () if eos is None else ((eos,) if isinstance(eos, int) else tuple(eos))
        return cls(vocab=_pint(d, "vocab", "the model"), width=_pint(d, "width", "the model"), norm_eps=_num(norm, "eps", "norm"),
                   max_positions=_pint(d, "max_positions", "the model"), layers=tuple(layers), taps=_pint(canon, "taps", "canon"),
                   bigram=bigram, loop=loop, dtype=dtype, eos_token_ids=eos_ids, raw=dict(d))

    def to_dict(self) -> dict:
        """The config.json this configuration is read back from."""
        d: Dict[str, Any] = {"architecture": ARCHITECTURE, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
                             "canon": {"taps": self.taps}, "max_positions": self.max_positions,
                             "layers": [{"type": l.type, "mixer": _plain(l.mixer), "mlp": _plain(l.mlp)} for l in self.layers]}
        if self.bigram is not None:
            d["embedding"] = {"bigram": {"buckets": self.bigram.buckets, "mul_prev": self.bigram.mul_prev, "mul_cur": self.bigram.mul_cur}}
        if self.loop is not None:
            d["loop"] = {"start": self.loop.start, "stop": self.loop.stop, "times": self.loop.times}
        if self.dtype != "bfloat16":
            d["dtype"] = self.dtype
        if self.eos_token_ids:
            d["eos_token_id"] = list(self.eos_token_ids)
        return d

    # ---- the model as data
    def run_layers(self) -> List[Tuple[int, bool]]:
        """(layer, whether a pass of the repeated stretch opens with it) for every layer run, in order."""
        n = len(self.layers)
        if self.loop is None:
            return [(i, False) for i in range(n)]
        lp = self.loop
        order = [(i, False) for i in range(lp.start)]
        for _ in range(lp.times):
            order += [(i, i == lp.start) for i in range(lp.start, lp.stop)]
        return order + [(i, False) for i in range(lp.stop, n)]

    def to_spec(self) -> ModelSpec:
        w, eps = self.width, self.norm_eps

        def norm(name: str) -> PartSpec:
            return PartSpec("rmsnorm", dict(size=w, eps=eps, one_plus=True, names=dict(weight=name)))

        positions: Dict[str, PartSpec] = {}

        def position(m: Mapping[str, Any]) -> Optional[str]:
            """The name of the rotary encoding a mixer's `rot` asks for; mixers with the same constants share one."""
            rot = m.get("rot")
            if rot is None or not rot["dims"]:
                return None
            name = f"rot{rot['dims']}@{float(rot['base'])!r}"
            positions.setdefault(name, PartSpec("rope", dict(head_dim=rot["dims"], rotary_dim=rot["dims"], theta=float(rot["base"]),
                                                             freq_in_double=True)))
            return name

        def attention(p: str, m: Mapping[str, Any]) -> PartSpec:
            return PartSpec("sigmoid_attention", dict(
                hidden_size=w, q_heads=m["heads"], kv_heads=m.get("kv_heads") or m["heads"], head_dim=m["dim"], v_dim=m.get("vdim") or m["dim"],
                scale=float(m["scale"]), chunk=(m.get("mask") or {}).get("size"), window=None, qk_norm_eps=eps, position=position(m),
                names=dict(q=f"{p}.q", k=f"{p}.k", v=f"{p}.v", o=f"{p}.o", q_norm=f"{p}.q.norm", k_norm=f"{p}.k.norm", score_bias=f"{p}.pb")))

        def memory(p: str, m: Mapping[str, Any]) -> PartSpec:
            return PartSpec("matrix_memory", dict(
                hidden_size=w, heads=m["heads"], head_dim=m["dim"], v_dim=m.get("vdim") or m["dim"], gate_cap=float(m["gate_cap"]), eps=eps,
                names=dict(q=f"{p}.q", k=f"{p}.k", v=f"{p}.v", g=f"{p}.g", o=f"{p}.o", norm=f"{p}.norm", i=f"{p}.i", i_bias=f"{p}.i.b",
                           f=f"{p}.f", f_bias=f"{p}.f.b")))

        layers = []
        for i, l in enumerate(self.layers):
            p, m = f"l{i}", l.mixer
            if l.type == "hgrn2":
                mixer = PartSpec("channel_gated_recurrence", dict(
                    hidden_size=w, heads=m["heads"], head_dim=m["dim"], v_dim=m.get("vdim") or m["dim"], eps=eps,
                    names=dict(q=f"{p}.mix.q", f=f"{p}.mix.f", f_bias=f"{p}.mix.f.b", lower=f"{p}.mix.lower", v=f"{p}.mix.v",
                               norm=f"{p}.mix.norm", o=f"{p}.mix.o")))
            else:
                mixer = PartSpec("side_by_side", dict(hidden_size=w, left=attention(f"{p}.mix.left", m["left"]), left_scale=float(m["left_scale"]),
                                                      right=memory(f"{p}.mix.right", m["right"]), right_scale=float(m["right_scale"])))
            parts = dict(mixer_norm=norm(f"{p}.norm1"),
                         mixer_input=PartSpec("causal_input_conv", dict(hidden_size=w, taps=self.taps, names=dict(weight=f"{p}.canon1"))),
                         mixer=mixer, mixer_post_norm=norm(f"{p}.norm1b"))
            if l.mlp is not None:
                parts.update(ffn_norm=norm(f"{p}.norm2"), ffn_post_norm=norm(f"{p}.norm2b"), ffn=PartSpec("swiglu", dict(
                    hidden_size=w, intermediate_size=l.mlp["ff"], bias=True,
                    names={s + b: f"{p}.mlp.{s}{t}" for s in ("gate", "up", "down") for b, t in (("", ""), ("_bias", ".b"))})))
            layers.append(LayerSpec(block="sandwich", parts=parts))
        opener = PartSpec("concat_opener", dict(hidden_size=w, names=dict(weight="loop.in")))
        b = self.bigram
        embedding = dict(vocab_size=self.vocab, hidden_size=w, positions=self.max_positions, keep=self.loop is not None,
                         names=dict(weight="embed", pairs="bigram", positions="pos"))
        if b is not None:
            embedding.update(buckets=b.buckets, mul_prev=b.mul_prev, mul_cur=b.mul_cur)
        spec = ModelSpec(
            architecture=ARCHITECTURE, vocab_size=self.vocab, hidden_size=w, max_position_embeddings=self.max_positions,
            embedding=PartSpec("sum_embedding", embedding), positions=positions, layers=tuple(layers),
            run_order=tuple(RunEntry(i, before=opener if opens else None) for i, opens in self.run_layers()), final_norm=norm("final.norm"),
            head=PartSpec("lm_head", dict(vocab_size=self.vocab, hidden_size=w, tied=False, names=dict(weight="head"))),
            stop_token_ids=tuple(self.eos_token_ids), checkpoint_dtype=self.dtype)
        spec.validate()
        return spec
