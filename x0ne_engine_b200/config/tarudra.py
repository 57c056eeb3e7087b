"""Tarudra: the typed configuration, read strictly from config.json, and its ModelSpec.

A Tarudra model is a list of layers with a layer norm (weight, no bias) before and after each sublayer and a layer scale on what
joins the residual, `x += ls1 * norm1b(mixer(norm1(x)))` then (unless the layer has no feed-forward) `x += ls2 *
norm2b(ff(norm2(x)))`.  The mixer of a layer is one of

  * `attention`: grouped-query attention over a sliding window, with biased projections, interleaved rotary pairs with
    YaRN-scaled frequencies, and one more term of score zero in the softmax denominator; a layer may have no keys and values of its
    own and read an earlier layer's (`kv_from`);
  * `latent_attention`: attention over one cached latent row per position, queries through a latent of their own, rotate-half
    positions on a part of every head, a sliding window and an output gate per value;
  * `delta`: the gated delta rule behind short convolutions.

The feed-forward is two products around a squared ReLU; the logits may be soft-capped.

Every size and constant comes from config.json (`layers[i].mixer`, `layers[i].mlp`, `logit_softcap`, `norm.eps`, `vocab`,
`width`); the layer list may have any order and length.  Tensor names: `embed`, `l<i>.norm1|norm1b|norm2|norm2b|ls1|ls2`,
`l<i>.mix.*`, `l<i>.mlp.*`, `final.norm`, `head`.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Dict, List, Mapping, Optional, Tuple

from .rovurax import UNBOUNDED_POSITIONS, _get, _num, _only, _pint, _plain
from .spec import ConfigError, LayerSpec, ModelSpec, PartSpec, RunEntry

ARCHITECTURE = "Tarudra"
MODEL_TYPE = "tarudra"

MIXERS = ("attention", "latent_attention", "delta")


@dataclass(frozen=True)
class TarudraLayer:
    type: str                       # one of MIXERS
    mixer: Mapping[str, Any]
    mlp: Optional[Mapping[str, Any]]


def _check_rotation(rot: Optional[Mapping[str, Any]], width: int, where: str) -> None:
    if rot is None:
        return
    _only(rot, ("base", "dims", "scaling"), where)
    base, dims = _num(rot, "base", where), _get(rot, "dims", where)
    if isinstance(dims, bool) or not isinstance(dims, int) or dims < 0 or dims % 2 or dims > width:
        raise ConfigError(f"config.json: {where}.dims is not an even count of at most {width} values")
    if rot.get("scaling") is not None:
        _only(rot["scaling"], ("factor", "fast", "original", "slow"), where + ".scaling")
        for k in ("factor", "fast", "original", "slow"):
            _num(rot["scaling"], k, where + ".scaling")
        if base == 1.0:
            raise ConfigError(f"config.json: {where}.base 1 has no frequencies to scale")


def _check_mask(m: Mapping[str, Any], where: str) -> None:
    if m.get("mask") is not None:
        _only(m["mask"], ("size",), where + ".mask")
        _pint(m["mask"], "size", where + ".mask")


def _kv_heads(m: Mapping[str, Any]) -> int:
    return m.get("kv_heads") or m["heads"]


def _vdim(m: Mapping[str, Any]) -> int:
    return m.get("vdim") or m["dim"]


def _check_heads(m: Mapping[str, Any], where: str) -> None:
    _pint(m, "dim", where)
    _pint(m, "heads", where)
    for k in ("kv_heads", "vdim"):
        if m.get(k) is not None:
            _pint(m, k, where)
    if m["heads"] % _kv_heads(m):
        raise ConfigError(f"config.json: {where}: heads are not a multiple of kv_heads")


def _check_attention(m: Mapping[str, Any], i: int, layers: List[TarudraLayer], where: str) -> None:
    _only(m, ("dim", "heads", "kv_from", "kv_heads", "mask", "rot", "scale", "vdim"), where)
    _check_heads(m, where)
    _num(m, "scale", where)
    _check_mask(m, where)
    _check_rotation(m.get("rot"), m["dim"], where + ".rot")
    src = m.get("kv_from")
    if src is None:
        return
    if isinstance(src, bool) or not isinstance(src, int) or not 0 <= src < i:
        raise ConfigError(f"config.json: {where}.kv_from must name an earlier layer")
    other = layers[src]
    if other.type != "attention" or other.mixer.get("kv_from") is not None:
        raise ConfigError(f"config.json: {where}.kv_from names layer {src}, which has no keys and values of its own")
    for what, a, b in (("kv_heads", _kv_heads(other.mixer), _kv_heads(m)), ("dim", other.mixer["dim"], m["dim"]), ("vdim", _vdim(other.mixer), _vdim(m))):
        if a != b:
            raise ConfigError(f"config.json: {where}.kv_from names layer {src}, whose {what} {a} differs from {b}")
    if _plain(other.mixer.get("rot")) != _plain(m.get("rot")):
        raise ConfigError(f"config.json: {where}.kv_from names layer {src}, whose rotation differs")


def _check_latent(m: Mapping[str, Any], where: str) -> None:
    _only(m, ("dim", "heads", "kv_rank", "mask", "q_rank", "rot", "rot_dim", "scale", "vdim"), where)
    for k in ("dim", "heads", "kv_rank", "q_rank", "rot_dim", "vdim"):
        _pint(m, k, where)
    _num(m, "scale", where)
    _check_mask(m, where)
    rot = _get(m, "rot", where)
    _check_rotation(rot, m["rot_dim"], where + ".rot")
    if rot is None or rot["dims"] != m["rot_dim"]:
        raise ConfigError(f"config.json: {where}.rot does not turn the rot_dim = {m['rot_dim']} values of the rotated part")


def _check_delta(m: Mapping[str, Any], where: str) -> None:
    _only(m, ("conv", "dim", "heads", "kv_heads", "vdim"), where)
    _check_heads(m, where)
    if _pint(m, "conv", where) > 64:
        raise ConfigError(f"config.json: {where}.conv {m['conv']} taps; at most 64 are served")


@dataclass(frozen=True)
class TarudraConfig:
    vocab: int
    width: int
    norm_eps: float
    layers: Tuple[TarudraLayer, ...]
    logit_softcap: Optional[float] = None
    dtype: str = "bfloat16"
    eos_token_ids: tuple = ()
    max_position_embeddings: int = UNBOUNDED_POSITIONS
    raw: Mapping[str, Any] = field(default_factory=dict, compare=False, repr=False)

    # ---- reading
    @classmethod
    def from_dict(cls, d: Mapping[str, Any]) -> "TarudraConfig":
        if not isinstance(d, Mapping):
            raise ConfigError("config.json: not a JSON object")
        _only(d, ("architecture", "architectures", "model_type", "layers", "logit_softcap", "norm", "vocab", "width", "dtype", "eos_token_id"), "the model")
        norm = _get(d, "norm", "the model")
        _only(norm, ("eps",), "norm")
        raw_layers = _get(d, "layers", "the model")
        if not isinstance(raw_layers, list) or not raw_layers:
            raise ConfigError("config.json: layers is not a list of at least one layer")
        layers: List[TarudraLayer] = []
        for i, l in enumerate(raw_layers):
            where = f"layers[{i}]"
            _only(l, ("type", "mixer", "mlp"), where)
            kind, mixer, mw = _get(l, "type", where), _get(l, "mixer", where), where + ".mixer"
            if kind == "attention":
                _check_attention(mixer, i, layers, mw)
            elif kind == "latent_attention":
                _check_latent(mixer, mw)
            elif kind == "delta":
                _check_delta(mixer, mw)
            else:
                raise ConfigError(f"config.json: {where}.type {kind!r} is not a mixer of this architecture; it has {list(MIXERS)}")
            mlp = l.get("mlp")
            if mlp is not None:
                _only(mlp, ("ff", "kind"), where + ".mlp")
                if _get(mlp, "kind", where + ".mlp") != "dense":
                    raise ConfigError(f"config.json: {where}.mlp.kind {mlp['kind']!r} is not a feed-forward of this architecture; it has 'dense'")
                _pint(mlp, "ff", where + ".mlp")
            layers.append(TarudraLayer(kind, mixer, mlp))
        dtype = d.get("dtype") or "bfloat16"
        if dtype not in ("bfloat16", "float32"):
            raise ConfigError(f"config.json: dtype {dtype!r}; bfloat16 and float32 checkpoints are served")
        eos = d.get("eos_token_id")
        eos_ids = () if eos is None else ((eos,) if isinstance(eos, int) else tuple(eos))
        cap = _num(d, "logit_softcap", "the model") if d.get("logit_softcap") is not None else None
        return cls(vocab=_pint(d, "vocab", "the model"), width=_pint(d, "width", "the model"), norm_eps=_num(norm, "eps", "norm"), layers=tuple(layers),
                   logit_softcap=cap, dtype=dtype, eos_token_ids=eos_ids, raw=dict(d))

    def to_dict(self) -> dict:
        """The config.json this configuration is read back from."""
        d: Dict[str, Any] = {"architecture": ARCHITECTURE, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
                             "layers": [{"type": l.type, "mixer": _plain(l.mixer), "mlp": _plain(l.mlp)} for l in self.layers]}
        if self.logit_softcap is not None:
            d["logit_softcap"] = self.logit_softcap
        if self.dtype != "bfloat16":
            d["dtype"] = self.dtype
        if self.eos_token_ids:
            d["eos_token_id"] = list(self.eos_token_ids)
        return d

    # ---- the model as data
    def to_spec(self) -> ModelSpec:
        w, eps = self.width, self.norm_eps

        def norm(name: str, scale: Optional[str] = None) -> PartSpec:
            names = dict(weight=name) if scale is None else dict(weight=name, scale=scale)
            return PartSpec("layernorm", dict(size=w, eps=eps, names=names))

        positions: Dict[str, PartSpec] = {}

        def position(rot: Optional[Mapping[str, Any]], layout: str) -> Optional[str]:
            """The name of the rotary encoding a mixer's `rot` asks for; mixers with the same constants share one."""
            if rot is None or not rot["dims"]:
                return None
            scaling = {k: float(v) for k, v in sorted(rot["scaling"].items())} if rot.get("scaling") is not None else None
            name = f"{layout}.{rot['dims']}@{float(rot['base'])!r}" + ("" if scaling is None else "*" + ",".join(repr(v) for v in scaling.values()))
            positions.setdefault(name, PartSpec("yarn_rope", dict(rotary_dim=rot["dims"], theta=float(rot["base"]), scaling=scaling, layout=layout)))
            return name

        layers, order = [], []
        for i, l in enumerate(self.layers):
            p, m = f"l{i}", l.mixer
            window, src = (m.get("mask") or {}).get("size"), None
            if l.type == "attention":
                src = m.get("kv_from")
                read = ("q", "k", "v", "o") if src is None else ("q", "o")
                # (the pages keep every position: a layer that reads these keys has a window of its own)
                mixer = PartSpec("masked_attention", dict(
                    hidden_size=w, q_heads=m["heads"], kv_heads=_kv_heads(m), head_dim=m["dim"], v_dim=_vdim(m), scale=float(m["scale"]), window=window,
                    ring=False, bias=True, own_kv=src is None, sink_zero=True, position=position(m.get("rot"), "interleaved"),
                    names={s + b: f"{p}.mix.{s}{t}" for s in read for b, t in (("", ""), ("_bias", ".b"))}))
            elif l.type == "latent_attention":
                mixer = PartSpec("latent_attention", dict(
                    hidden_size=w, heads=m["heads"], head_dim=m["dim"], rot_dim=m["rot_dim"], v_dim=m["vdim"], kv_rank=m["kv_rank"], q_rank=m["q_rank"],
                    scale=float(m["scale"]), norm_eps=eps, window=window, gate=True, gate_wide=True, position=position(m["rot"], "half"),
                    names=dict(dq=f"{p}.mix.dq", dq_norm=f"{p}.mix.dq.norm", q=f"{p}.mix.uq", dkv=f"{p}.mix.dkv", dkv_norm=f"{p}.mix.dkv.norm",
                               uk=f"{p}.mix.uk", uv=f"{p}.mix.uv", gate=f"{p}.mix.g", o=f"{p}.mix.o")))
            else:
                names = {s: f"{p}.mix.{s}" for s in ("q", "k", "v", "a", "b", "A_log", "dt_bias", "norm", "g", "o")}
                names.update({s + "_conv": f"{p}.mix.{s}.conv" for s in ("q", "k", "v")})
                mixer = PartSpec("gated_delta_rule", dict(hidden_size=w, heads=m["heads"], kv_heads=_kv_heads(m), head_dim=m["dim"], v_dim=_vdim(m),
                                                          taps=m["conv"], eps=eps, names=names))
            parts = dict(mixer_norm=norm(f"{p}.norm1"), mixer=mixer, mixer_post_norm=norm(f"{p}.norm1b", f"{p}.ls1"))
            if l.mlp is not None:
                parts.update(ffn_norm=norm(f"{p}.norm2"), ffn_post_norm=norm(f"{p}.norm2b", f"{p}.ls2"), ffn=PartSpec("squared_relu_mlp", dict(
                    hidden_size=w, intermediate_size=l.mlp["ff"], names=dict(up=f"{p}.mlp.up", down=f"{p}.mlp.down"))))
            layers.append(LayerSpec(block="sandwich", parts=parts))
            order.append(RunEntry(i, reads_cache_of=src))
        spec = ModelSpec(
            architecture=ARCHITECTURE, vocab_size=self.vocab, hidden_size=w, max_position_embeddings=self.max_position_embeddings,
            embedding=PartSpec("token_embedding", dict(vocab_size=self.vocab, hidden_size=w, names=dict(weight="embed"))),
            positions=positions, layers=tuple(layers), run_order=tuple(order), final_norm=norm("final.norm"),
            head=PartSpec("lm_head", dict(vocab_size=self.vocab, hidden_size=w, tied=False, softcap=self.logit_softcap, names=dict(weight="head"))),
            stop_token_ids=tuple(self.eos_token_ids), checkpoint_dtype=self.dtype)
        spec.validate()
        return spec
