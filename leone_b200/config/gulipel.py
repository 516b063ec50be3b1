"""Typed configuration of the Gulipel decoder.

Its ``config.json`` names the model under ``architecture`` and describes every layer on its own
(``layers``: a list of ``{"type", "mixer", "mlp"}``).  Top-level keys: ``vocab``, ``width``, ``max_positions`` (rows of
the table of learned positions; the tensor's shape gives it where the key is absent), ``norm.eps``, and, optionally,
``embedding`` (``scale``; ``bigram`` with ``buckets``, ``mul_prev``, ``mul_cur``), ``token_side.dim`` (the width of every
layer's slice of the second token table) and ``logit_softcap``.

A layer's ``type`` is ``parallel`` or ``mamba2``, or one of these with a number behind it (``mamba2_2``), which names the
same kind of mixer with sizes of its own:

``parallel``: ``left`` (attention: ``heads``, ``kv_heads``, ``dim``, ``vdim``, ``scale``, ``q_temp`` (``coef``, ``every``;
optional)) and ``right`` (delta rule with a decay per key channel: ``heads``, ``kv_heads``, ``dim``, ``vdim``, ``conv`` taps).
``mamba2``: ``heads``, ``vdim``, ``state``, ``groups``, ``norm_groups``, ``conv`` taps.

``mlp`` is ``null`` or ``{"kind": "dense", "ff"}``.

The inner widths of the delta rule's decay and gate are not in the file as such: they are the first sizes of the
tensors ``l<i>.mix.right.a1`` and ``l<i>.mix.right.g1``.  For a model without a checkpoint (random weights) they are the
optional keys ``decay_rank`` and ``gate_rank`` of ``right``, default 16.
"""
from __future__ import annotations

import dataclasses
import re
from dataclasses import dataclass
from typing import Any, Mapping, Optional, Tuple, Union

from .base import ConfigReader, InvalidValue, ModelConfig, UnsupportedField, WrongType

DEFAULT_MAX_POSITIONS = 1 << 14
DEFAULT_RANK = 16
MIXER_KINDS = ("parallel", "mamba2")


def mixer_kind(layer_type: str) -> Optional[str]:
    """The kind of mixer a layer's type names (``None``: no such kind)."""
    m = re.fullmatch(r"(.+?)(?:_\d+)?", layer_type)
    return m.group(1) if m and m.group(1) in MIXER_KINDS else None


@dataclass(frozen=True)
class Bigram:
    buckets: int
    mul_prev: int
    mul_cur: int

    def to_json(self):
        return {"buckets": self.buckets, "mul_prev": self.mul_prev, "mul_cur": self.mul_cur}


@dataclass(frozen=True)
class QueryTemp:
    coef: float
    every: int

    def to_json(self):
        return {"coef": self.coef, "every": self.every}


@dataclass(frozen=True)
class LeftMixer:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    q_temp: Optional[QueryTemp]

    def to_json(self):
        out = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "scale": self.scale}
        if self.q_temp is not None:
            out["q_temp"] = self.q_temp.to_json()
        return out


@dataclass(frozen=True)
class RightMixer:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int                    # taps of the convolution on q, k and v; 0: none
    decay_rank: Optional[int]    # None: the checkpoint's tensors say it
    gate_rank: Optional[int]

    def to_json(self):
        out = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim}
        for key, value in (("conv", self.conv), ("decay_rank", self.decay_rank), ("gate_rank", self.gate_rank)):
            if value:
                out[key] = value
        return out


@dataclass(frozen=True)
class ParallelMixer:
    left: LeftMixer
    right: RightMixer

    def to_json(self):
        return {"left": self.left.to_json(), "right": self.right.to_json()}


@dataclass(frozen=True)
class MambaMixer:
    heads: int
    vdim: int
    state: int
    groups: int
    norm_groups: int
    conv: int

    def to_json(self):
        return {"heads": self.heads, "vdim": self.vdim, "state": self.state, "groups": self.groups,
                "norm_groups": self.norm_groups, "conv": self.conv}


@dataclass(frozen=True)
class DenseMlp:
    ff: int

    def to_json(self):
        return {"kind": "dense", "ff": self.ff}


@dataclass(frozen=True)
class GulipelLayer:
    type: str
    mixer: Union[ParallelMixer, MambaMixer]
    mlp: Optional[DenseMlp]

    def to_json(self):
        return {"type": self.type, "mixer": self.mixer.to_json(), "mlp": None if self.mlp is None else self.mlp.to_json()}


def _heads(r: ConfigReader):
    heads, kv_heads = r.positive_int("heads"), r.positive_int("kv_heads")
    if heads % kv_heads:
        raise InvalidValue(f"{r.where}: 'heads' ({heads}) must be a multiple of 'kv_heads' ({kv_heads})")
    return heads, kv_heads


def _taps(r: ConfigReader, least: int) -> int:
    conv = r.optional_int("conv") or 0
    if not least <= conv <= 16:
        raise InvalidValue(f"{r.where}: 'conv' ({conv}) must be between {least} and 16 taps")
    return conv


def _read_parallel(r: ConfigReader) -> ParallelMixer:
    lr, rr = r.section("left"), r.section("right")
    heads, kv_heads = _heads(lr)
    temp = lr.section("q_temp", optional=True)
    left = LeftMixer(heads, kv_heads, lr.positive_int("dim"), lr.positive_int("vdim"), lr.number("scale"),
                     None if temp is None else QueryTemp(temp.number("coef"), temp.positive_int("every")))
    rheads, rkv = _heads(rr)
    right = RightMixer(rheads, rkv, rr.positive_int("dim"), rr.positive_int("vdim"), _taps(rr, 0),
                       rr.positive_int("decay_rank", None), rr.positive_int("gate_rank", None))
    return ParallelMixer(left, right)


def _read_mamba(r: ConfigReader) -> MambaMixer:
    m = MambaMixer(r.positive_int("heads"), r.positive_int("vdim"), r.positive_int("state"), r.positive_int("groups"),
                   r.positive_int("norm_groups"), _taps(r, 1))
    if m.heads % m.groups:
        raise InvalidValue(f"{r.where}: 'heads' ({m.heads}) must be a multiple of 'groups' ({m.groups})")
    if m.heads * m.vdim % m.norm_groups:
        raise InvalidValue(f"{r.where}: heads * vdim ({m.heads * m.vdim}) must be a multiple of 'norm_groups' ({m.norm_groups})")
    return m


def _read_mlp(r: Optional[ConfigReader]) -> Optional[DenseMlp]:
    if r is None:
        return None
    kind = r.string("kind")
    if kind != "dense":
        raise UnsupportedField(f"{r.where}: mlp kind '{kind}' is not supported (dense)")
    return DenseMlp(r.positive_int("ff"))


@dataclass(frozen=True)
class GulipelConfig(ModelConfig):
    vocab: int = 0
    width: int = 0
    max_positions: int = DEFAULT_MAX_POSITIONS
    norm_eps: float = 0.0
    embedding_scale: float = 1.0
    bigram: Optional[Bigram] = None
    side_dim: int = 0            # 0: no per-layer token input
    logit_softcap: float = 0.0   # 0: no cap
    layers: Tuple[GulipelLayer, ...] = ()
    positions_given: bool = True

    ARCHITECTURE = "Gulipel"

    def needs_tensor_shapes(self) -> bool:
        return not self.positions_given or any(
            isinstance(layer.mixer, ParallelMixer) and None in (layer.mixer.right.decay_rank, layer.mixer.right.gate_rank)
            for layer in self.layers)

    def with_tensor_shapes(self, shapes: Mapping[str, Tuple[int, ...]]) -> "GulipelConfig":
        def rows(name, known):
            shape = shapes.get(name)
            return int(shape[0]) if known is None and shape is not None and len(shape) == 2 and shape[0] > 0 else known
        layers = []
        for i, layer in enumerate(self.layers):
            if isinstance(layer.mixer, ParallelMixer):
                r = layer.mixer.right
                r = dataclasses.replace(r, decay_rank=rows(f"l{i}.mix.right.a1", r.decay_rank),
                                        gate_rank=rows(f"l{i}.mix.right.g1", r.gate_rank))
                layer = dataclasses.replace(layer, mixer=dataclasses.replace(layer.mixer, right=r))
            layers.append(layer)
        positions = self.max_positions if self.positions_given else rows("pos", None) or self.max_positions
        return dataclasses.replace(self, layers=tuple(layers), max_positions=positions)

    def to_json_dict(self) -> dict:
        out = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width,
               "max_positions": self.max_positions, "norm": {"eps": self.norm_eps},
               "layers": [layer.to_json() for layer in self.layers]}
        emb = {}
        if self.embedding_scale != 1.0:
            emb["scale"] = self.embedding_scale
        if self.bigram is not None:
            emb["bigram"] = self.bigram.to_json()
        if emb:
            out["embedding"] = emb
        if self.side_dim:
            out["token_side"] = {"dim": self.side_dim}
        if self.logit_softcap:
            out["logit_softcap"] = self.logit_softcap
        return out

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any]) -> "GulipelConfig":
        r = ConfigReader(raw)
        layers_raw = raw.get("layers")
        if not isinstance(layers_raw, list) or not layers_raw:
            raise WrongType("config.json: 'layers' must be a non-empty list of layer descriptions")
        layers = []
        for i, entry in enumerate(layers_raw):
            lr = ConfigReader(entry, f"config.json: layers[{i}]")
            name = lr.string("type")
            kind = mixer_kind(name)
            if kind is None:
                raise UnsupportedField(f"{lr.where}: mixer type '{name}' is not supported ({', '.join(MIXER_KINDS)})")
            mixer = _read_parallel(lr.section("mixer")) if kind == "parallel" else _read_mamba(lr.section("mixer"))
            layers.append(GulipelLayer(name, mixer, _read_mlp(lr.section("mlp", optional=True))))
        emb = r.section("embedding", optional=True)
        bigram = None if emb is None else emb.section("bigram", optional=True)
        if bigram is not None:
            muls = [bigram.optional_int(k) for k in ("mul_prev", "mul_cur")]
            if any(m is None or m < 0 for m in muls):
                raise InvalidValue(f"{bigram.where}: 'mul_prev' and 'mul_cur' must be integers of at least 0")
            bigram = Bigram(bigram.positive_int("buckets"), *muls)
        side = r.section("token_side", optional=True)
        cap = r.number("logit_softcap", 0.0)
        if cap < 0:
            raise InvalidValue(f"config.json: 'logit_softcap' ({cap}) must not be negative")
        return cls(architecture=cls.ARCHITECTURE, vocab=r.positive_int("vocab"), width=r.positive_int("width"),
                   max_positions=r.positive_int("max_positions", DEFAULT_MAX_POSITIONS),
                   positions_given=r.has("max_positions"), norm_eps=r.section("norm").positive_float("eps"),
                   embedding_scale=1.0 if emb is None else emb.number("scale", 1.0), bigram=bigram,
                   side_dim=0 if side is None else side.positive_int("dim"), logit_softcap=float(cap), layers=tuple(layers))
