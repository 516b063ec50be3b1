"""Typed configuration of the Kakirax decoder.

Its ``config.json`` names the model under ``architecture`` and describes every layer on its own
(``layers``: a list of ``{"type", "mixer", "mlp"}`` and, optionally, ``"weights_of"``: the index of the layer
whose tensors this one runs, with a cache or state of its own; the rest of such an entry equals that
layer's).  Top-level keys: ``vocab``, ``width``, ``norm.eps``, ``embedding.scale`` (default 1) and
``logit_softcap`` (optional).

Mixer type ``attention``: ``heads``, ``kv_heads``, ``dim``, ``vdim``, ``scale``, ``rot`` (``base``, ``dims``,
optionally ``scaling`` with ``factor``, ``low``, ``high``, ``original``; ``rot`` itself may be absent).
Mixer type ``gla``: ``heads``, ``dim``, ``vdim``, ``tau``.  The number of rows of its decay's inner projection is
not in the file as such: it is the first size of the tensor ``l<i>.mix.a1``.  For a model without a checkpoint
(random weights) it is the optional key ``decay_rank``, default 16.

``mlp`` is ``null`` or ``{"kind": "dense", "ff"}``.

The file gives no limit on positions; ``max_positions`` (not a key of the design) bounds the
engine's block tables and defaults to 2**20.
"""
from __future__ import annotations

import dataclasses
from dataclasses import dataclass
from typing import Any, Mapping, Optional, Tuple, Union

from .base import ConfigReader, InvalidValue, ModelConfig, UnsupportedField, WrongType

DEFAULT_MAX_POSITIONS = 1 << 20
DEFAULT_DECAY_RANK = 16
MIXER_TYPES = ("attention", "gla")


@dataclass(frozen=True)
class WavelengthScaling:
    factor: float
    low: float
    high: float
    original: float

    def to_json(self):
        return {"factor": self.factor, "low": self.low, "high": self.high, "original": self.original}


@dataclass(frozen=True)
class AttentionMixer:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot_base: float
    rot_dims: int                # 0: no rotation
    rot_scaling: Optional[WavelengthScaling]

    def to_json(self):
        out = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "scale": self.scale}
        if self.rot_dims:
            out["rot"] = {"base": self.rot_base, "dims": self.rot_dims}
            if self.rot_scaling is not None:
                out["rot"]["scaling"] = self.rot_scaling.to_json()
        return out


@dataclass(frozen=True)
class GlaMixer:
    heads: int
    dim: int
    vdim: int
    tau: float
    decay_rank: Optional[int]    # None: the checkpoint's tensors say it

    def to_json(self):
        out = {"heads": self.heads, "dim": self.dim, "vdim": self.vdim, "tau": self.tau}
        if self.decay_rank is not None:
            out["decay_rank"] = self.decay_rank
        return out


@dataclass(frozen=True)
class DenseMlp:
    ff: int

    def to_json(self):
        return {"kind": "dense", "ff": self.ff}


@dataclass(frozen=True)
class KakiraxLayer:
    type: str
    mixer: Union[AttentionMixer, GlaMixer]
    mlp: Optional[DenseMlp]
    weights_of: Optional[int]    # None: tensors of its own

    def to_json(self):
        out = {"type": self.type, "mixer": self.mixer.to_json(), "mlp": None if self.mlp is None else self.mlp.to_json()}
        if self.weights_of is not None:
            out["weights_of"] = self.weights_of
        return out


def _read_attention(r: ConfigReader) -> AttentionMixer:
    heads, kv_heads, dim = r.positive_int("heads"), r.positive_int("kv_heads"), r.positive_int("dim")
    if heads % kv_heads:
        raise InvalidValue(f"{r.where}: 'heads' ({heads}) must be a multiple of 'kv_heads' ({kv_heads})")
    base, dims, scaling = 10000.0, 0, None
    rot = r.section("rot", optional=True)
    if rot is not None:
        base, dims = rot.positive_float("base"), rot.positive_int("dims")
        if dims % 2 or dims > dim:
            raise InvalidValue(f"{rot.where}: 'dims' ({dims}) must be even and at most dim ({dim})")
        sc = rot.section("scaling", optional=True)
        if sc is not None:
            scaling = WavelengthScaling(sc.positive_float("factor"), sc.positive_float("low"), sc.positive_float("high"),
                                        sc.positive_float("original"))
            if scaling.high < scaling.low:
                raise InvalidValue(f"{sc.where}: 'high' ({scaling.high}) must not be below 'low' ({scaling.low})")
    return AttentionMixer(heads, kv_heads, dim, r.positive_int("vdim"), r.number("scale"), base, dims, scaling)


def _read_gla(r: ConfigReader) -> GlaMixer:
    return GlaMixer(r.positive_int("heads"), r.positive_int("dim"), r.positive_int("vdim"), r.positive_float("tau"),
                    r.positive_int("decay_rank", None))


def _read_mlp(r: Optional[ConfigReader]) -> Optional[DenseMlp]:
    if r is None:
        return None
    kind = r.string("kind")
    if kind != "dense":
        raise UnsupportedField(f"{r.where}: mlp kind '{kind}' is not supported (dense)")
    return DenseMlp(r.positive_int("ff"))


@dataclass(frozen=True)
class KakiraxConfig(ModelConfig):
    vocab: int = 0
    width: int = 0
    norm_eps: float = 0.0
    embedding_scale: float = 1.0
    logit_softcap: float = 0.0   # 0: no cap
    layers: Tuple[KakiraxLayer, ...] = ()
    max_positions: int = DEFAULT_MAX_POSITIONS

    ARCHITECTURE = "Kakirax"

    def source_layer(self, i: int) -> int:
        """The layer whose tensors layer ``i`` runs (itself, if it has its own)."""
        while self.layers[i].weights_of is not None:
            i = self.layers[i].weights_of
        return i

    def needs_tensor_shapes(self) -> bool:
        return any(isinstance(layer.mixer, GlaMixer) and layer.mixer.decay_rank is None for layer in self.layers)

    def with_tensor_shapes(self, shapes: Mapping[str, Tuple[int, ...]]) -> "KakiraxConfig":
        layers = []
        for i, layer in enumerate(self.layers):
            shape = shapes.get(f"l{self.source_layer(i)}.mix.a1")
            if isinstance(layer.mixer, GlaMixer) and layer.mixer.decay_rank is None and shape is not None and \
                    len(shape) == 2 and shape[0] > 0:
                layer = dataclasses.replace(layer, mixer=dataclasses.replace(layer.mixer, decay_rank=int(shape[0])))
            layers.append(layer)
        return dataclasses.replace(self, layers=tuple(layers))

    def to_json_dict(self) -> dict:
        out = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width,
               "norm": {"eps": self.norm_eps}, "layers": [layer.to_json() for layer in self.layers]}
        if self.embedding_scale != 1.0:
            out["embedding"] = {"scale": self.embedding_scale}
        if self.logit_softcap:
            out["logit_softcap"] = self.logit_softcap
        if self.max_positions != DEFAULT_MAX_POSITIONS:
            out["max_positions"] = self.max_positions
        return out

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any]) -> "KakiraxConfig":
        r = ConfigReader(raw)
        layers_raw = raw.get("layers")
        if not isinstance(layers_raw, list) or not layers_raw:
            raise WrongType("config.json: 'layers' must be a non-empty list of layer descriptions")
        layers = []
        for i, entry in enumerate(layers_raw):
            lr = ConfigReader(entry, f"config.json: layers[{i}]")
            kind = lr.string("type")
            if kind not in MIXER_TYPES:
                raise UnsupportedField(f"{lr.where}: mixer type '{kind}' is not supported ({', '.join(MIXER_TYPES)})")
            mixer = _read_attention(lr.section("mixer")) if kind == "attention" else _read_gla(lr.section("mixer"))
            layers.append(KakiraxLayer(kind, mixer, _read_mlp(lr.section("mlp", optional=True)), lr.optional_int("weights_of")))
        for i, layer in enumerate(layers):
            j, seen = i, {i}
            while layers[j].weights_of is not None:
                j = layers[j].weights_of
                if not 0 <= j < len(layers) or j in seen:
                    raise InvalidValue(f"config.json: layers[{i}]: 'weights_of' does not lead to a layer with tensors of its own")
                seen.add(j)
            if (layer.type, layer.mixer, layer.mlp) != (layers[j].type, layers[j].mixer, layers[j].mlp):
                raise InvalidValue(f"config.json: layers[{i}] runs layer {j}'s tensors but is not described as that layer is")
        emb = r.section("embedding", optional=True)
        cap = r.number("logit_softcap", 0.0)
        if cap < 0:
            raise InvalidValue(f"config.json: 'logit_softcap' ({cap}) must not be negative")
        return cls(architecture=cls.ARCHITECTURE, vocab=r.positive_int("vocab"), width=r.positive_int("width"),
                   norm_eps=r.section("norm").positive_float("eps"),
                   embedding_scale=1.0 if emb is None else emb.number("scale", 1.0), logit_softcap=float(cap),
                   layers=tuple(layers), max_positions=r.positive_int("max_positions", DEFAULT_MAX_POSITIONS))
