"""Typed configuration of the Ravelorn decoder, read from config.json.

A Ravelorn model is an embedding plus a learned position vector, a list of layers that each name their mixer with its own
sizes and an optional routed feed-forward, a final layer norm, a head of its own and a soft cap on the logits.  A layer
normalises its sublayers' results only: x <- x + m norm1(mixer(x)), x <- x + m norm2(ff(x)), layer norms with weight and bias,
m = ``residual_mult``; the sublayers read x itself.  Two mixers:

* ``channel_delta``: the gated delta rule with a decay per head and key channel (a narrow product) and a sigmoid gate (another
  narrow product) after a norm per head.
* ``parallel``: softmax attention (left) and the gated delta rule with a decay per head and a silu gate (right) side by side,
  left_scale * left + right_scale * right.  The attention has no rotation: queries and keys are divided by their root mean
  square, queries multiplied by a temperature that grows with the position, and the softmax's denominator has a
  learned term per head.

The feed-forward is a mixture of experts (silu) with softmax scores over all experts, a correction on the scores for the
choice only, and identity experts at the end of the list.

Keys read (every size and every constant that differs between models comes from here)::

    architecture        "Ravelorn"
    vocab, width, max_positions, residual_mult, logit_softcap (optional)
    norm.eps
    layers[i].type      "channel_delta" | "parallel"
    layers[i].mixer     channel_delta: heads, kv_heads, dim, vdim, conv
                        parallel: left_scale, right_scale,
                                  left: heads, kv_heads, dim, vdim, scale, q_temp: {coef, every} (optional)
                                  right: heads, kv_heads, dim, vdim, conv
    layers[i].mlp       null | {kind: "moe", expert: {ff}, router: {experts, top, identity (optional)}}

The inner sizes of the narrow products are not among the keys: they are read from the tensors' shapes when a folder is
loaded (``with_tensor_shapes``), or given as ``decay_rank`` and ``gate_rank`` in a ``channel_delta`` mixer.

Tensor names: ``embed``, ``pos``, ``l<i>.norm1``, ``l<i>.norm2`` (+ ``.b``), ``l<i>.mix.<q|k|v|q.conv|k.conv|v.conv|b|a1|a2|A_log|dt_bias|
g1|g2|norm|o>``, ``l<i>.mix.left.<q|k|v|sink|o>``, ``l<i>.mix.right.<q|k|v|q.conv|k.conv|v.conv|b|a|A_log|dt_bias|g|norm|o>``,
``l<i>.mlp.<router|correction>``, ``l<i>.mlp.e<j>.<gate|up|down>``, ``final.norm`` (+ ``.b``), ``head``; no ``.weight`` suffix.
"""
from __future__ import annotations

from dataclasses import dataclass, replace
from typing import Any, Callable, Mapping, Optional, Tuple, Union

from ..errors import ConfigError
from .pipilix import _get, _int, _num
from .specs import FeedForwardSpec, LayerSpec, MixerSpec, ModelSpec, NormSpec, PositionSpec, ScheduleEntry, _frozen_params

ARCHITECTURE = "Ravelorn"

UNIT_EPS = 1e-6            # under the root of a unit vector's length

_MIXERS = ("channel_delta", "parallel")

_DELTA_NAMES = {"q": "q", "k": "k", "v": "v", "o": "o", "q_conv": "q.conv", "k_conv": "k.conv", "v_conv": "v.conv", "beta": "b",
                "decay": "a", "decay_in": "a1", "decay_out": "a2", "a_log": "A_log", "dt_bias": "dt_bias", "gate": "g", "gate_in": "g1",
                "gate_out": "g2", "norm": "norm"}


def _heads(d, where):
    heads, kv = _int(d, "heads", where), _int(d, "kv_heads", where)
    if heads % kv:
        raise ConfigError(f"config.json: {where}heads {heads} is no multiple of kv_heads {kv}")
    return heads, kv


@dataclass(frozen=True)
class DeltaConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int
    decay_rank: Optional[int] = None       # inner sizes of the narrow products (channel_delta only); None: not known yet
    gate_rank: Optional[int] = None

    @staticmethod
    def from_dict(d, where) -> "DeltaConfig":
        heads, kv = _heads(d, where)
        ranks = {k: (_int(d, k, where) if d.get(k) is not None else None) for k in ("decay_rank", "gate_rank")}
        return DeltaConfig(heads=heads, kv_heads=kv, dim=_int(d, "dim", where), vdim=_int(d, "vdim", where), conv=_int(d, "conv", where), **ranks)

    def to_dict(self) -> dict:
        d = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "conv": self.conv}
        for k in ("decay_rank", "gate_rank"):
            if getattr(self, k) is not None:
                d[k] = getattr(self, k)
        return d


@dataclass(frozen=True)
class SinkAttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    q_temp: Optional[Tuple[float, float]]       # (coef, every)

    @staticmethod
    def from_dict(d, where) -> "SinkAttentionConfig":
        heads, kv = _heads(d, where)
        temp = d.get("q_temp")
        if temp is not None:
            temp = (_num(temp, "coef", where + "q_temp."), _num(temp, "every", where + "q_temp."))
            if not temp[1] > 0:
                raise ConfigError(f"config.json: {where}q_temp.every must be positive, found {temp[1]}")
        return SinkAttentionConfig(heads=heads, kv_heads=kv, dim=_int(d, "dim", where), vdim=_int(d, "vdim", where),
                                   scale=_num(d, "scale", where), q_temp=temp)

    def to_dict(self) -> dict:
        d = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "scale": self.scale}
        if self.q_temp is not None:
            d["q_temp"] = {"coef": self.q_temp[0], "every": int(self.q_temp[1]) if self.q_temp[1] == int(self.q_temp[1]) else self.q_temp[1]}
        return d


@dataclass(frozen=True)
class ParallelConfig:
    left: SinkAttentionConfig
    right: DeltaConfig
    left_scale: float
    right_scale: float

    @staticmethod
    def from_dict(d, where) -> "ParallelConfig":
        return ParallelConfig(left=SinkAttentionConfig.from_dict(_get(d, "left", where), where + "left."),
                              right=DeltaConfig.from_dict(_get(d, "right", where), where + "right."),
                              left_scale=_num(d, "left_scale", where), right_scale=_num(d, "right_scale", where))

    def to_dict(self) -> dict:
        return {"left": self.left.to_dict(), "right": self.right.to_dict(), "left_scale": self.left_scale, "right_scale": self.right_scale}


@dataclass(frozen=True)
class ExpertsConfig:
    experts: int
    top: int
    ff: int
    identity: int

    @staticmethod
    def from_dict(d, where) -> "ExpertsConfig":
        if _get(d, "kind", where) != "moe":
            raise ConfigError(f"config.json: {where}kind {d['kind']!r} is unknown (known: moe)")
        r = _get(d, "router", where)
        cfg = ExpertsConfig(experts=_int(r, "experts", where + "router."), top=_int(r, "top", where + "router."),
                            ff=_int(_get(d, "expert", where), "ff", where + "expert."),
                            identity=_int(r, "identity", where + "router.", 0) if r.get("identity") is not None else 0)
        if cfg.top > cfg.experts + cfg.identity:
            raise ConfigError(f"config.json: {where}router.top {cfg.top} exceeds the {cfg.experts} + {cfg.identity} experts")
        return cfg

    def to_dict(self) -> dict:
        return {"kind": "moe", "expert": {"ff": self.ff}, "router": {"experts": self.experts, "identity": self.identity, "top": self.top}}


_MIXER_CONFIGS = {"channel_delta": DeltaConfig, "parallel": ParallelConfig}


@dataclass(frozen=True)
class RavelornLayer:
    mixer_type: str
    mixer: Union[DeltaConfig, ParallelConfig]
    mlp: Optional[ExpertsConfig]


@dataclass(frozen=True)
class RavelornConfig:
    vocab: int
    width: int
    max_positions: int
    norm_eps: float
    residual_mult: float
    logit_softcap: Optional[float]
    layers: Tuple[RavelornLayer, ...]

    def __post_init__(self):
        if not self.layers:
            raise ConfigError("config.json: 'layers' is empty")
        if not self.norm_eps > 0:
            raise ConfigError(f"config.json: norm.eps must be positive, found {self.norm_eps}")
        if self.logit_softcap is not None and not self.logit_softcap > 0:
            raise ConfigError(f"config.json: logit_softcap must be positive, found {self.logit_softcap}")

    @staticmethod
    def from_dict(d: Mapping[str, Any]) -> "RavelornConfig":
        layers = _get(d, "layers", "")
        if not isinstance(layers, (list, tuple)):
            raise ConfigError("config.json: 'layers' must be a list")
        out = []
        for i, L in enumerate(layers):
            where = f"layers[{i}]."
            kind = _get(L, "type", where)
            if kind not in _MIXERS:
                raise ConfigError(f"config.json: {where}type {kind!r} is unknown (known: {', '.join(_MIXERS)})")
            mixer = _MIXER_CONFIGS[kind].from_dict(_get(L, "mixer", where), where + "mixer.")
            mlp = L.get("mlp")
            out.append(RavelornLayer(kind, mixer, None if mlp is None else ExpertsConfig.from_dict(mlp, where + "mlp.")))
        return RavelornConfig(vocab=_int(d, "vocab", ""), width=_int(d, "width", ""), max_positions=_int(d, "max_positions", ""),
                              norm_eps=_num(_get(d, "norm", ""), "eps", "norm."), residual_mult=_num(d, "residual_mult", ""),
                              logit_softcap=_num(d, "logit_softcap", "") if d.get("logit_softcap") is not None else None,
                              layers=tuple(out))

    def to_dict(self) -> dict:
        d = {
            "architecture": ARCHITECTURE,
            "layers": [{"type": L.mixer_type, "mixer": L.mixer.to_dict(), "mlp": None if L.mlp is None else L.mlp.to_dict()}
                       for L in self.layers],
            "max_positions": self.max_positions,
            "norm": {"eps": self.norm_eps},
            "residual_mult": self.residual_mult,
            "vocab": self.vocab,
            "width": self.width,
        }
        if self.logit_softcap is not None:
            d["logit_softcap"] = self.logit_softcap
        return d

    def with_tensor_shapes(self, shape_of: Callable[[str], Optional[tuple]]) -> "RavelornConfig":
        """The same configuration with the sizes that only the tensors tell: a channel_delta layer's inner ranks.  ``shape_of``
        gives a tensor's shape by its name in the files, or None."""
        def rank(name):
            shape = shape_of(name)
            return int(shape[0]) if shape is not None and len(shape) == 2 else None
        layers = []
        for i, L in enumerate(self.layers):
            if L.mixer_type == "channel_delta":
                m = L.mixer
                L = replace(L, mixer=replace(m, decay_rank=m.decay_rank or rank(f"l{i}.mix.a1"), gate_rank=m.gate_rank or rank(f"l{i}.mix.g1")))
            layers.append(L)
        return replace(self, layers=tuple(layers))

    # ---- the architecture, spelled as parts ------------------------------------------------------
    def _delta_spec(self, m: DeltaConfig, where: str, per_channel: bool) -> MixerSpec:
        extra = {}
        if per_channel:
            for k in ("decay_rank", "gate_rank"):
                if getattr(m, k) is None:
                    raise ConfigError(f"config.json: {where}{k} is not given, and no tensor of a model folder tells it")
                extra[k] = getattr(m, k)
        return MixerSpec.make(
            "gated_delta", None, n_heads=m.heads, n_kv_heads=m.kv_heads, head_dim=m.dim, v_head_dim=m.vdim, conv_taps=m.conv,
            decay="per_channel" if per_channel else "per_head", gate="sigmoid_low_rank" if per_channel else "silu",
            out_norm_eps=self.norm_eps, unit_eps=UNIT_EPS, names=_DELTA_NAMES, **extra)

    def _mixer_spec(self, i: int, L: RavelornLayer) -> MixerSpec:
        where = f"layers[{i}].mixer."
        if L.mixer_type == "channel_delta":
            return self._delta_spec(L.mixer, where, True)
        a = L.mixer.left
        left = dict(n_heads=a.heads, n_kv_heads=a.kv_heads, head_dim=a.dim, v_head_dim=a.vdim, scale=a.scale, qk_unit_norm=True,
                    qk_norm_eps=self.norm_eps, sink="per_head", names={"q": "q", "k": "k", "v": "v", "o": "o", "sink": "sink"})
        if a.q_temp is not None:
            left["q_temperature"] = {"coef": a.q_temp[0], "every": a.q_temp[1]}
        return MixerSpec.make(
            "side_by_side", None, left=MixerSpec.make("attention", None, **left), right=self._delta_spec(L.mixer.right, where + "right.", False),
            left_scale=L.mixer.left_scale, right_scale=L.mixer.right_scale, prefixes={"left": "left.", "right": "right."})

    def to_model_spec(self) -> ModelSpec:
        norm = NormSpec("layernorm", self.norm_eps)
        layers = []
        for i, L in enumerate(self.layers):
            ff = None if L.mlp is None else FeedForwardSpec.make(
                "routed_mlp", experts=L.mlp.experts, identity=L.mlp.identity, top=L.mlp.top, intermediate=L.mlp.ff, activation="silu",
                score="softmax", choice_bias=True, renormalize=False,
                names={"router": "router", "choice_bias": "correction", "expert": "e{e}.", "gate": "gate", "up": "up", "down": "down"})
            layers.append(LayerSpec(
                prefix=f"l{i}", mixer=self._mixer_spec(i, L), feed_forward=ff, mixer_norm=norm, ff_norm=norm, arrangement="output_norm",
                mixer_norm_name="norm1", ff_norm_name="norm2", mixer_name="mix.", ff_name="mlp.",
                arrangement_items=_frozen_params({"multiplier": self.residual_mult})))
        return ModelSpec(
            architecture=ARCHITECTURE, hidden=self.width, vocab=self.vocab, max_position=self.max_positions, layers=tuple(layers),
            schedule=tuple(ScheduleEntry(i) for i in range(len(layers))), final_norm=norm, tie_embeddings=False,
            embedding_name="embed.weight", final_norm_name="final.norm.weight", head_name="head.weight", weight_suffix="",
            bias_suffix=".b", input_position=PositionSpec("learned", params_items=_frozen_params({"rows": self.max_positions})),
            input_position_name="pos.weight", logit_softcap=self.logit_softcap)
