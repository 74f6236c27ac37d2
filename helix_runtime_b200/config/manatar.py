"""Typed configuration of the Manatar decoder, read from its ``config.json``.

The document is nested: ``vocab`` and ``width`` at the top, ``norm.eps``, ``residual_mult`` (the
factor on every sublayer's normed result), ``embedding.bigram`` (``buckets``, ``mul_prev``,
``mul_cur``; may be left out: no second table), and a list ``layers`` whose entries name the mixer
(``type``: ``attention`` or ``mlstm``), its sizes (``mixer``) and the feed-forward (``mlp``, null
for none; ``kind`` ``dense`` with ``ff`` and ``limit``, or ``moe`` with ``expert.ff``,
``router.{experts, top}`` and an optional ``shared.ff``).  Every size and constant is read from the
document; layers may differ from one another in every one of them.
"""
from __future__ import annotations

import dataclasses
from typing import Any, Dict, Mapping, Optional, Tuple

from .errors import ConfigError
from .keys import COUNT, REAL, TEXT, Key, Kind, read_keys
from .rekasun import FACTOR, _object, _whole
from .rorovik import RotaryScalingConfig, _optional_object

ARCHITECTURE = "Manatar"
DEFAULT_MAX_POSITIONS = 1 << 17

INTEGER = Kind(lambda value: isinstance(value, int) and not isinstance(value, bool)
               and abs(value) < 1 << 31, int, "must be an integer below 2^31")


@dataclasses.dataclass(frozen=True)
class PairTableConfig:
    """Which row of the second table a pair of neighbouring tokens picks."""
    buckets: int
    mul_prev: int
    mul_cur: int

    KEYS = (Key("buckets", COUNT), Key("mul_prev", INTEGER), Key("mul_cur", INTEGER))


@dataclasses.dataclass(frozen=True)
class DifferentialAttentionConfig:
    heads: int
    kv_heads: int            # query head h reads key/value head h // (heads / kv_heads)
    dim: int                 # of one map of a query / key head
    vdim: int                # of a value head
    scale: float
    conv: int                # taps of the causal filter on q, k and v
    diff: float              # the constant of the maps' balance
    rot_base: float
    rot_dims: int            # leading coordinates of each map that turn
    scaling: Optional[RotaryScalingConfig]
    kv_from: Optional[int]   # the layer whose keys and values this one uses

    KEYS = (Key("heads", COUNT), Key("kv_heads", COUNT, default=None), Key("dim", COUNT),
            Key("vdim", COUNT, default=None), Key("scale", REAL), Key("conv", COUNT, default=1),
            Key("diff", FACTOR))

    @classmethod
    def from_dict(cls, document: Mapping[str, Any], where: str) -> "DifferentialAttentionConfig":
        values = read_keys(document, cls.KEYS, where)
        values["kv_heads"] = values["kv_heads"] or values["heads"]
        values["vdim"] = values["vdim"] or values["dim"]
        if values["heads"] % values["kv_heads"]:
            raise ConfigError(f"config field '{where}heads' must be a multiple of "
                              f"'{where}kv_heads'")
        rot = _object(document, "rot", where)
        base = read_keys(rot, (Key("base", REAL),), where + "rot.")["base"]
        dims = rot.get("dims", values["dim"])
        if not (_whole(dims) and dims % 2 == 0 and dims <= values["dim"]):
            raise ConfigError(f"config field '{where}rot.dims' must be even and at most "
                              f"{values['dim']}")
        scaling = _optional_object(rot, "scaling", where + "rot.")
        if scaling is not None:
            scaling = RotaryScalingConfig(**read_keys(scaling, RotaryScalingConfig.KEYS,
                                                      where + "rot.scaling."))
            if base <= 1.0:
                raise ConfigError(f"config field '{where}rot.base' must exceed 1 with scaling")
        kv_from = document.get("kv_from")
        if kv_from is not None and not _whole(kv_from):
            raise ConfigError(f"config field '{where}kv_from' must name a layer")
        return cls(rot_base=base, rot_dims=int(dims), scaling=scaling, kv_from=kv_from, **values)

    def to_dict(self) -> Dict[str, Any]:
        rot: Dict[str, Any] = {"base": self.rot_base, "dims": self.rot_dims}
        if self.scaling is not None:
            rot["scaling"] = dataclasses.asdict(self.scaling)
        document = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim,
                    "vdim": self.vdim, "scale": self.scale, "conv": self.conv, "diff": self.diff,
                    "rot": rot}
        if self.kv_from is not None:
            document["kv_from"] = self.kv_from
        return document


@dataclasses.dataclass(frozen=True)
class MatrixLstmConfig:
    heads: int
    dim: int                 # rows of a head's matrix
    vdim: int                # its columns
    gate_cap: float          # level that both gates' logarithms run into

    KEYS = (Key("heads", COUNT), Key("dim", COUNT), Key("vdim", COUNT, default=None),
            Key("gate_cap", REAL))

    @classmethod
    def from_dict(cls, document: Mapping[str, Any], where: str) -> "MatrixLstmConfig":
        values = read_keys(document, cls.KEYS, where)
        values["vdim"] = values["vdim"] or values["dim"]
        return cls(**values)

    def to_dict(self) -> Dict[str, Any]:
        return dataclasses.asdict(self)


# one configuration class per value of a layer's ``type``
MIXER_CONFIGS = {"attention": DifferentialAttentionConfig, "mlstm": MatrixLstmConfig}


@dataclasses.dataclass(frozen=True)
class FeedForwardConfig:
    kind: str                # dense | moe
    ff: int                  # of the dense layer, or of one expert
    limit: float = 0.0       # the dense layer's clamp
    experts: int = 0
    top: int = 0
    shared_ff: int = 0       # of the expert every token uses (0: none)

    @classmethod
    def from_dict(cls, document: Mapping[str, Any], where: str) -> "FeedForwardConfig":
        kind = read_keys(document, (Key("kind", TEXT),), where)["kind"]
        if kind == "dense":
            return cls(kind=kind, **read_keys(document, (Key("ff", COUNT), Key("limit", REAL)), where))
        if kind != "moe":
            raise ConfigError(f"config field '{where}kind' is {kind!r}; known: dense, moe")
        ff = read_keys(_object(document, "expert", where), (Key("ff", COUNT),), where + "expert.")["ff"]
        counts = read_keys(_object(document, "router", where),
                           (Key("experts", COUNT), Key("top", COUNT)), where + "router.")
        if counts["top"] > counts["experts"]:
            raise ConfigError(f"config field '{where}router.top' is more than the experts")
        shared = _optional_object(document, "shared", where)
        shared_ff = 0 if shared is None else \
            read_keys(shared, (Key("ff", COUNT),), where + "shared.")["ff"]
        return cls(kind=kind, ff=ff, shared_ff=shared_ff, **counts)

    def to_dict(self) -> Dict[str, Any]:
        if self.kind == "dense":
            return {"kind": "dense", "ff": self.ff, "limit": self.limit}
        document = {"kind": "moe", "expert": {"ff": self.ff},
                    "router": {"experts": self.experts, "top": self.top}}
        if self.shared_ff:
            document["shared"] = {"ff": self.shared_ff}
        return document


@dataclasses.dataclass(frozen=True)
class ManatarLayerConfig:
    type: str
    mixer: Any
    mlp: Optional[FeedForwardConfig]

    @classmethod
    def from_dict(cls, document: Any, index: int) -> "ManatarLayerConfig":
        where = f"layers[{index}]."
        if not isinstance(document, dict):
            raise ConfigError(f"config field 'layers[{index}]' must be an object")
        kind = document.get("type")
        if kind not in MIXER_CONFIGS:
            raise ConfigError(f"config field '{where}type' is {kind!r}; known: "
                              + ", ".join(sorted(MIXER_CONFIGS)))
        mixer = MIXER_CONFIGS[kind].from_dict(_object(document, "mixer", where), where + "mixer.")
        mlp = _optional_object(document, "mlp", where)
        return cls(kind, mixer,
                   None if mlp is None else FeedForwardConfig.from_dict(mlp, where + "mlp."))

    def to_dict(self) -> Dict[str, Any]:
        return {"type": self.type, "mixer": self.mixer.to_dict(),
                "mlp": None if self.mlp is None else self.mlp.to_dict()}


@dataclasses.dataclass(frozen=True)
class ManatarConfig:
    vocab: int
    width: int
    norm_eps: float
    residual_mult: float
    pairs: Optional[PairTableConfig]     # None: no second table
    layers: Tuple[ManatarLayerConfig, ...]
    max_positions: int = DEFAULT_MAX_POSITIONS

    architecture = ARCHITECTURE

    def __post_init__(self) -> None:
        if not self.layers:
            raise ConfigError("config field 'layers' must name at least one layer")
        for index, layer in enumerate(self.layers):
            source = getattr(layer.mixer, "kv_from", None)
            if source is None:
                continue
            label = f"config field 'layers[{index}].mixer.kv_from'"
            if not source < index or self.layers[source].type != "attention" \
                    or self.layers[source].mixer.kv_from is not None:
                raise ConfigError(f"{label} must name an earlier attention layer with keys and values "
                                  "of its own")
            other = self.layers[source].mixer
            if (other.kv_heads, other.dim, other.vdim) != (layer.mixer.kv_heads, layer.mixer.dim,
                                                           layer.mixer.vdim):
                raise ConfigError(f"{label} names a layer whose heads have another shape")

    @classmethod
    def from_dict(cls, document: Mapping[str, Any]) -> "ManatarConfig":
        values = read_keys(document, (Key("vocab", COUNT), Key("width", COUNT),
                                      Key("residual_mult", FACTOR, default=1.0),
                                      Key("max_positions", COUNT, default=DEFAULT_MAX_POSITIONS)))
        eps = read_keys(_object(document, "norm"), (Key("eps", REAL),), "norm.")["eps"]
        embedding = _optional_object(document, "embedding", "") or {}
        pairs = _optional_object(embedding, "bigram", "embedding.")
        if pairs is not None:
            pairs = PairTableConfig(**read_keys(pairs, PairTableConfig.KEYS, "embedding.bigram."))
        layers = document.get("layers")
        if not isinstance(layers, list) or not layers:
            raise ConfigError("config field 'layers' must be a list of layers")
        return cls(vocab=values["vocab"], width=values["width"], norm_eps=eps,
                   residual_mult=values["residual_mult"], pairs=pairs,
                   max_positions=values["max_positions"],
                   layers=tuple(ManatarLayerConfig.from_dict(layer, index)
                                for index, layer in enumerate(layers)))

    def to_dict(self) -> Dict[str, Any]:
        document: Dict[str, Any] = {
            "architecture": self.architecture, "vocab": self.vocab, "width": self.width,
            "norm": {"eps": self.norm_eps}, "residual_mult": self.residual_mult,
            "layers": [layer.to_dict() for layer in self.layers],
        }
        if self.pairs is not None:
            document["embedding"] = {"bigram": dataclasses.asdict(self.pairs)}
        if self.max_positions != DEFAULT_MAX_POSITIONS:
            document["max_positions"] = self.max_positions
        return document

    @staticmethod
    def random_scale(name: str, shape: Tuple[int, ...]):
        """What a model with random weights holds in its vectors (None: ones): biases are zero, the
        vectors of the maps' balance small."""
        leaf = name.rsplit(".", 1)[-1]
        if leaf == "b":
            return 0.0
        if leaf in ("lq1", "lk1", "lq2", "lk2"):
            return 0.1
        return None
