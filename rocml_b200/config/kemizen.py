"""Typed configuration of the Kemizen decoder, read from config.json.

A Kemizen model is an embedding times a constant, a list of layers that each name their mixer with its own sizes and an optional dense
feed-forward, a final norm and a head of its own.  A layer normalises its sublayers' results only: x <- x + norm1(mixer(x)),
x <- x + norm2(ff(x)), RMS norms with weights stored around zero; the sublayers read x itself.  Three mixers:

* ``mlstm``: a matrix memory with exponential gates under a running maximum (xLSTM), a norm per head and a sigmoid gate.
* ``attention``: differential attention (two maps a head over the same values, their difference normalised per head) with a norm and a
  rotation per map, a soft cap on the scores and a sliding window; a layer may use an earlier layer's keys and values (``kv_from``).
* ``parallel``: causal attention behind short convolutions with a norm over the whole projections and a gate for every value (left), and
  Griffin's recurrent block (right), side by side; half the sum of the two results, each normalised with a weight of its own.

The feed-forward is dense, without a gate, with the exact gelu.

Keys read (every size and every constant that differs between models comes from here)::

    architecture        "Kemizen"
    vocab, width, embedding.scale, norm.eps
    layers[i].type      "mlstm" | "attention" | "parallel"
    layers[i].mixer     mlstm: heads, dim, vdim, gate_cap
                        attention: heads, kv_heads, dim, vdim, scale, diff, softcap (optional), mask: {size} (optional), kv_from (optional),
                                   rot: {base, dims, scaling: {factor, original, fast, slow} (optional)}
                        parallel: left: heads, kv_heads, dim, vdim, scale, conv, rot
                                  right: width, blocks, conv
    layers[i].mlp       null | {kind: "dense", ff}

``max_positions`` (optional; default 131072) is the longest sequence the engine plans for; nothing in the model depends on it.

Tensor names: ``embed``, ``l<i>.norm1``, ``l<i>.norm2``, ``l<i>.mix.<q|k|v|g|i|f|o|norm>`` (+ ``i.b``, ``f.b``) for mlstm,
``l<i>.mix.<q|k|v|o|q.norm|k.norm|lq1|lk1|lq2|lk2>`` for attention (without k, v and k.norm where ``kv_from`` is given),
``l<i>.mix.left.<q|k|v|g|o>`` with ``.b`` on all but g, ``.conv`` on q, k and v and ``.norm`` on q and k, ``l<i>.mix.right.<y|x|conv|ra|ri>``
(+ ``.b``), ``l<i>.mix.right.<lam|o>``, ``l<i>.mix.<left|right>.out``, ``l<i>.mlp.<up|down>``, ``final.norm``, ``head``; no ``.weight`` suffix.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Mapping, Optional, Tuple, Union

from ..errors import ConfigError
from .pipilix import _get, _int, _num
from .specs import FeedForwardSpec, LayerSpec, MixerSpec, ModelSpec, NormSpec, PositionSpec, ScheduleEntry, _frozen_params

ARCHITECTURE = "Kemizen"

MAX_POSITIONS = 131072         # the longest sequence planned for when config.json does not say
RESULT_FACTOR = 0.5            # of the sum of a parallel mixer's two normalised results

_MLSTM_NAMES = {"q": "q", "k": "k", "v": "v", "gate": "g", "i": "i", "f": "f", "o": "o", "out_norm": "norm"}
_ATTENTION_NAMES = {"q": "q", "k": "k", "v": "v", "o": "o", "q_norm": "q.norm", "k_norm": "k.norm", "lq1": "lq1", "lk1": "lk1", "lq2": "lq2",
                    "lk2": "lk2"}
_LEFT_NAMES = {"q": "q", "k": "k", "v": "v", "o": "o", "gate": "g", "q_norm": "q.norm", "k_norm": "k.norm", "q_conv": "q.conv",
               "k_conv": "k.conv", "v_conv": "v.conv"}
_RIGHT_NAMES = {"y": "y", "x": "x", "conv": "conv", "ra": "ra", "ri": "ri", "lam": "lam", "o": "o"}


def _plain(x: float):
    """A number as config.json would hold it."""
    return int(x) if float(x) == int(x) else x


@dataclass(frozen=True)
class RotationConfig:
    base: float
    dims: int
    scaling: Optional[Tuple[float, float, float, float]]        # (factor, original, fast, slow)

    @staticmethod
    def from_dict(d, where, dim) -> "RotationConfig":
        dims = _int(d, "dims", where)
        if dims % 2 or dims > dim:
            raise ConfigError(f"config.json: {where}dims {dims} must be even and at most the head size {dim}")
        sc = d.get("scaling")
        if sc is not None:
            sc = tuple(_num(sc, k, where + "scaling.") for k in ("factor", "original", "fast", "slow"))
        return RotationConfig(base=_num(d, "base", where), dims=dims, scaling=sc)

    def to_dict(self) -> dict:
        d = {"base": self.base, "dims": self.dims}
        if self.scaling is not None:
            d["scaling"] = {k: _plain(v) for k, v in zip(("factor", "original", "fast", "slow"), self.scaling)}
        return d

    def spec(self) -> PositionSpec:
        params = {}
        if self.scaling is not None:
            params["ramp_scaling"] = dict(zip(("factor", "original", "fast", "slow"), self.scaling))
        return PositionSpec("rope_neox", theta=self.base, rot_dim=self.dims, params_items=_frozen_params(params))


def _heads(d, where):
    heads, kv = _int(d, "heads", where), _int(d, "kv_heads", where)
    if heads % kv:
        raise ConfigError(f"config.json: {where}heads {heads} is no multiple of kv_heads {kv}")
    return heads, kv


def _rotation(d, where, dim) -> Optional[RotationConfig]:
    return None if d.get("rot") is None else RotationConfig.from_dict(d["rot"], where + "rot.", dim)


def _position(rot: Optional[RotationConfig]) -> Optional[PositionSpec]:
    return None if rot is None or rot.dims == 0 else rot.spec()


@dataclass(frozen=True)
class MemoryConfig:
    heads: int
    dim: int
    vdim: int
    gate_cap: float

    @staticmethod
    def from_dict(d, where) -> "MemoryConfig":
        cap = _num(d, "gate_cap", where)
        if not cap > 0:
            raise ConfigError(f"config.json: {where}gate_cap must be positive, found {cap}")
        return MemoryConfig(heads=_int(d, "heads", where), dim=_int(d, "dim", where), vdim=_int(d, "vdim", where), gate_cap=cap)

    def to_dict(self) -> dict:
        return {"heads": self.heads, "dim": self.dim, "vdim": self.vdim, "gate_cap": self.gate_cap}

    def spec(self, eps: float) -> MixerSpec:
        return MixerSpec.make("mlstm", None, n_heads=self.heads, head_dim=self.dim, v_head_dim=self.vdim, gate_cap=self.gate_cap,
                              out_norm_eps=eps, names=_MLSTM_NAMES)


@dataclass(frozen=True)
class DifferentialConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    diff: float
    softcap: Optional[float]
    window: Optional[int]
    rot: Optional[RotationConfig]
    kv_from: Optional[int]

    @staticmethod
    def from_dict(d, where) -> "DifferentialConfig":
        heads, kv = _heads(d, where)
        cap = _num(d, "softcap", where) if d.get("softcap") is not None else None
        if cap is not None and not cap > 0:
            raise ConfigError(f"config.json: {where}softcap must be positive, found {cap}")
        window = _int(d["mask"], "size", where + "mask.") if d.get("mask") is not None else None
        dim = _int(d, "dim", where)
        source = d.get("kv_from")
        if source is not None and (isinstance(source, bool) or not isinstance(source, int) or source < 0):
            raise ConfigError(f"config.json: {where}kv_from must name a layer, found {source!r}")
        return DifferentialConfig(heads=heads, kv_heads=kv, dim=dim, vdim=_int(d, "vdim", where), scale=_num(d, "scale", where),
                                  diff=_num(d, "diff", where), softcap=cap, window=window, rot=_rotation(d, where, dim), kv_from=source)

    def to_dict(self) -> dict:
        d = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "scale": self.scale, "diff": self.diff}
        if self.softcap is not None:
            d["softcap"] = self.softcap
        if self.window is not None:
            d["mask"] = {"size": self.window}
        if self.rot is not None:
            d["rot"] = self.rot.to_dict()
        if self.kv_from is not None:
            d["kv_from"] = self.kv_from
        return d

    def spec(self, eps: float) -> MixerSpec:
        params = dict(n_heads=self.heads, n_kv_heads=self.kv_heads, head_dim=self.dim, v_head_dim=self.vdim, scale=self.scale, qk_norm=True,
                      qk_norm_eps=eps, difference=self.diff, names=_ATTENTION_NAMES)
        if self.window is not None:
            params["window"] = self.window
        if self.softcap is not None:
            params["softcap"] = self.softcap
        return MixerSpec.make("attention", _position(self.rot), **params)


@dataclass(frozen=True)
class ConvAttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    conv: int
    rot: Optional[RotationConfig]

    @staticmethod
    def from_dict(d, where) -> "ConvAttentionConfig":
        heads, kv = _heads(d, where)
        dim = _int(d, "dim", where)
        return ConvAttentionConfig(heads=heads, kv_heads=kv, dim=dim, vdim=_int(d, "vdim", where), scale=_num(d, "scale", where),
                                   conv=_int(d, "conv", where), rot=_rotation(d, where, dim))

    def to_dict(self) -> dict:
        d = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "scale": self.scale, "conv": self.conv}
        if self.rot is not None:
            d["rot"] = self.rot.to_dict()
        return d

    def spec(self, eps: float) -> MixerSpec:
        return MixerSpec.make("attention", _position(self.rot), n_heads=self.heads, n_kv_heads=self.kv_heads, head_dim=self.dim,
                              v_head_dim=self.vdim, scale=self.scale, qk_norm="whole", qk_norm_eps=eps, conv_taps=self.conv, gated="per_value",
                              bias=("q", "k", "v", "o"), names=_LEFT_NAMES)


@dataclass(frozen=True)
class RecurrentConfig:
    width: int
    blocks: int
    conv: int

    @staticmethod
    def from_dict(d, where) -> "RecurrentConfig":
        width, blocks = _int(d, "width", where), _int(d, "blocks", where)
        if width % blocks:
            raise ConfigError(f"config.json: {where}width {width} does not split in {blocks} equal blocks")
        return RecurrentConfig(width=width, blocks=blocks, conv=_int(d, "conv", where))

    def to_dict(self) -> dict:
        return {"width": self.width, "blocks": self.blocks, "conv": self.conv}

    def spec(self, eps: float) -> MixerSpec:
        return MixerSpec.make("rg_lru", None, width=self.width, blocks=self.blocks, conv_taps=self.conv, names=_RIGHT_NAMES)


@dataclass(frozen=True)
class ParallelConfig:
    left: ConvAttentionConfig
    right: RecurrentConfig

    @staticmethod
    def from_dict(d, where) -> "ParallelConfig":
        return ParallelConfig(left=ConvAttentionConfig.from_dict(_get(d, "left", where), where + "left."),
                              right=RecurrentConfig.from_dict(_get(d, "right", where), where + "right."))

    def to_dict(self) -> dict:
        return {"left": self.left.to_dict(), "right": self.right.to_dict()}

    def spec(self, eps: float) -> MixerSpec:
        return MixerSpec.make("side_by_side", None, left=self.left.spec(eps), right=self.right.spec(eps), out_norms=True, out_norm_eps=eps,
                              out_factor=RESULT_FACTOR, prefixes={"left": "left.", "right": "right."})


_MIXERS = {"mlstm": MemoryConfig, "attention": DifferentialConfig, "parallel": ParallelConfig}


@dataclass(frozen=True)
class KemizenLayer:
    mixer_type: str
    mixer: Union[MemoryConfig, DifferentialConfig, ParallelConfig]
    ff: Optional[int]

    @property
    def kv_from(self) -> Optional[int]:
        return getattr(self.mixer, "kv_from", None)


@dataclass(frozen=True)
class KemizenConfig:
    vocab: int
    width: int
    embedding_scale: float
    norm_eps: float
    layers: Tuple[KemizenLayer, ...]
    max_positions: int = MAX_POSITIONS

    def __post_init__(self):
        if not self.layers:
            raise ConfigError("config.json: 'layers' is empty")
        if not self.norm_eps > 0:
            raise ConfigError(f"config.json: norm.eps must be positive, found {self.norm_eps}")
        for i, L in enumerate(self.layers):
            j = L.kv_from
            if j is None:
                continue
            if not j < i or self.layers[j].mixer_type != "attention" or self.layers[j].kv_from is not None:
                raise ConfigError(f"config.json: layers[{i}].mixer.kv_from {j} must be an earlier attention layer with keys and values of its own")
            a, b = L.mixer, self.layers[j].mixer
            if (a.heads, a.kv_heads, a.dim, a.vdim, a.rot) != (b.heads, b.kv_heads, b.dim, b.vdim, b.rot):
                raise ConfigError(f"config.json: layers[{i}] uses the keys and values of layer {j}, whose heads, sizes or rotation differ")

    @staticmethod
    def from_dict(d: Mapping[str, Any]) -> "KemizenConfig":
        layers = _get(d, "layers", "")
        if not isinstance(layers, (list, tuple)):
            raise ConfigError("config.json: 'layers' must be a list")
        out = []
        for i, L in enumerate(layers):
            where = f"layers[{i}]."
            kind = _get(L, "type", where)
            if kind not in _MIXERS:
                raise ConfigError(f"config.json: {where}type {kind!r} is unknown (known: {', '.join(_MIXERS)})")
            mixer = _MIXERS[kind].from_dict(_get(L, "mixer", where), where + "mixer.")
            mlp, ff = L.get("mlp"), None
            if mlp is not None:
                if _get(mlp, "kind", where + "mlp.") != "dense":
                    raise ConfigError(f"config.json: {where}mlp.kind {mlp['kind']!r} is unknown (known: dense)")
                ff = _int(mlp, "ff", where + "mlp.")
            out.append(KemizenLayer(kind, mixer, ff))
        scale = _num(d["embedding"], "scale", "embedding.") if d.get("embedding") is not None else 1.0
        return KemizenConfig(vocab=_int(d, "vocab", ""), width=_int(d, "width", ""), embedding_scale=scale,
                             norm_eps=_num(_get(d, "norm", ""), "eps", "norm."), layers=tuple(out),
                             max_positions=_int(d, "max_positions", "") if d.get("max_positions") is not None else MAX_POSITIONS)

    def to_dict(self) -> dict:
        d = {
            "architecture": ARCHITECTURE,
            "embedding": {"scale": self.embedding_scale},
            "layers": [{"type": L.mixer_type, "mixer": L.mixer.to_dict(), "mlp": None if L.ff is None else {"kind": "dense", "ff": L.ff}}
                       for L in self.layers],
            "norm": {"eps": self.norm_eps},
            "vocab": self.vocab,
            "width": self.width,
        }
        if self.max_positions != MAX_POSITIONS:
            d["max_positions"] = self.max_positions
        return d

    # ---- the architecture, spelled as parts ------------------------------------------------------
    def to_model_spec(self) -> ModelSpec:
        norm = NormSpec("rmsnorm", self.norm_eps, weight_offset=1.0)
        layers = []
        for i, L in enumerate(self.layers):
            ff = None if L.ff is None else FeedForwardSpec.make("dense_mlp", intermediate=L.ff, activation="gelu",
                                                                names={"up": "up", "down": "down"})
            layers.append(LayerSpec(prefix=f"l{i}", mixer=L.mixer.spec(self.norm_eps), feed_forward=ff, mixer_norm=norm, ff_norm=norm,
                                    arrangement="output_norm", mixer_norm_name="norm1", ff_norm_name="norm2", mixer_name="mix.", ff_name="mlp."))
        return ModelSpec(
            architecture=ARCHITECTURE, hidden=self.width, vocab=self.vocab, max_position=self.max_positions, layers=tuple(layers),
            schedule=tuple(ScheduleEntry(i, reads_cache_of=L.kv_from) for i, L in enumerate(self.layers)), final_norm=norm,
            tie_embeddings=False, embedding_name="embed.weight", final_norm_name="final.norm.weight", head_name="head.weight",
            weight_suffix="", bias_suffix=".b", embedding_scale=self.embedding_scale)
