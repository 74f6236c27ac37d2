"""Typed configuration of the Pizilix decoder, read from its ``config.json``.

The document is nested: ``vocab`` and ``width`` at the top, ``norm.eps``, ``logit_softcap`` (left
out: the logits as they are), a list ``layers`` whose entries name the mixer (``type``:
``attention`` or ``rglru``), its sizes (``mixer``) and the feed-forward (``mlp``, null for none),
and an optional ``loop`` (``start``, ``stop``, ``times``): layers ``start`` to ``stop - 1`` run
``times`` times in a row with the same weights, every run with its own cache and state.  Every size
and constant is read from the document; layers may differ from one another in every one of them.
"""
from __future__ import annotations

import dataclasses
from typing import Any, Dict, Mapping, Optional, Tuple

from .errors import ConfigError
from .keys import COUNT, REAL, Key, read_keys
from .rekasun import FACTOR, DenseMlpConfig, LoopConfig, _object, _whole
from .rorovik import RotaryScalingConfig, _optional_object

ARCHITECTURE = "Pizilix"
DEFAULT_MAX_POSITIONS = 1 << 17


@dataclasses.dataclass(frozen=True)
class ChunkedAttentionConfig:
    heads: int
    kv_heads: int                # query head h reads key/value head h // (heads / kv_heads)
    dim: int                     # size of a query / key head; the values are the keys
    scale: float
    softcap: Optional[float]     # the level the scores run into
    chunk: Optional[int]         # positions see each other inside chunks of this many
    rot_base: float
    rot_dims: int                # leading coordinates of a head that turn, in neighbouring pairs
    scaling: Optional[RotaryScalingConfig]

    KEYS = (Key("heads", COUNT), Key("kv_heads", COUNT, default=None), Key("dim", COUNT),
            Key("vdim", COUNT, default=None), Key("scale", FACTOR),
            Key("softcap", REAL, default=None))

    @classmethod
    def from_dict(cls, document: Mapping[str, Any], where: str) -> "ChunkedAttentionConfig":
        values = read_keys(document, cls.KEYS, where)
        values["kv_heads"] = values["kv_heads"] or values["heads"]
        if values["heads"] % values["kv_heads"]:
            raise ConfigError(f"config field '{where}heads' must be a multiple of "
                              f"'{where}kv_heads'")
        if values.pop("vdim") not in (None, values["dim"]):
            raise ConfigError(f"config field '{where}vdim' must be '{where}dim': the values are the "
                              "keys")
        mask = _optional_object(document, "mask", where)
        chunk = None
        if mask is not None:
            chunk = read_keys(mask, (Key("size", COUNT),), where + "mask.")["size"]
        rot = _object(document, "rot", where)
        base = read_keys(rot, (Key("base", REAL),), where + "rot.")["base"]
        dims = rot.get("dims", values["dim"])
        if not (_whole(dims) and dims % 2 == 0 and dims <= values["dim"]):
            raise ConfigError(f"config field '{where}rot.dims' must be even and at most "
                              f"'{where}dim'")
        scaling = _optional_object(rot, "scaling", where + "rot.")
        if scaling is not None:
            scaling = RotaryScalingConfig(**read_keys(scaling, RotaryScalingConfig.KEYS,
                                                      where + "rot.scaling."))
            if base <= 1.0:
                raise ConfigError(f"config field '{where}rot.base' must exceed 1 with scaling")
        return cls(chunk=chunk, rot_base=base, rot_dims=int(dims), scaling=scaling, **values)

    def to_dict(self) -> Dict[str, Any]:
        rot: Dict[str, Any] = {"base": self.rot_base, "dims": self.rot_dims}
        if self.scaling is not None:
            rot["scaling"] = dataclasses.asdict(self.scaling)
        document: Dict[str, Any] = {
            "heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.dim,
            "scale": self.scale, "rot": rot}
        if self.softcap is not None:
            document["softcap"] = self.softcap
        if self.chunk is not None:
            document["mask"] = {"size": self.chunk}
        return document


@dataclasses.dataclass(frozen=True)
class GatedRecurrenceConfig:
    width: int               # channels of either branch
    blocks: int              # equal parts of the channels, each with its own gate matrices
    conv: int                # taps of the causal filter on the recurrent branch

    KEYS = (Key("width", COUNT), Key("blocks", COUNT, default=1), Key("conv", COUNT, default=1))

    @classmethod
    def from_dict(cls, document: Mapping[str, Any], where: str) -> "GatedRecurrenceConfig":
        values = read_keys(document, cls.KEYS, where)
        if values["width"] % values["blocks"]:
            raise ConfigError(f"config field '{where}width' must be a multiple of "
                              f"'{where}blocks'")
        return cls(**values)

    def to_dict(self) -> Dict[str, Any]:
        return dataclasses.asdict(self)


# one configuration class per value of a layer's ``type``
MIXER_CONFIGS = {"attention": ChunkedAttentionConfig, "rglru": GatedRecurrenceConfig}


@dataclasses.dataclass(frozen=True)
class PizilixLayerConfig:
    type: str
    mixer: Any
    mlp: Optional[DenseMlpConfig]

    @classmethod
    def from_dict(cls, document: Any, index: int) -> "PizilixLayerConfig":
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
                   None if mlp is None else DenseMlpConfig.from_dict(mlp, where + "mlp."))

    def to_dict(self) -> Dict[str, Any]:
        return {"type": self.type, "mixer": self.mixer.to_dict(),
                "mlp": None if self.mlp is None else self.mlp.to_dict()}


@dataclasses.dataclass(frozen=True)
class PizilixConfig:
    vocab: int
    width: int
    norm_eps: float
    layers: Tuple[PizilixLayerConfig, ...]
    logit_softcap: Optional[float] = None     # the level the logits run into
    loop: Optional[LoopConfig] = None
    max_positions: int = DEFAULT_MAX_POSITIONS

    architecture = ARCHITECTURE

    def __post_init__(self) -> None:
        if not self.layers:
            raise ConfigError("config field 'layers' must name at least one layer")
        if self.loop is not None:
            loop = self.loop
            if not 0 <= loop.start < loop.stop <= len(self.layers) or loop.times < 1:
                raise ConfigError(f"config field 'loop' ({loop.start}, {loop.stop}, {loop.times}) "
                                  f"does not fit {len(self.layers)} layers")

    @classmethod
    def from_dict(cls, document: Mapping[str, Any]) -> "PizilixConfig":
        values = read_keys(document, (Key("vocab", COUNT), Key("width", COUNT),
                                      Key("logit_softcap", REAL, default=None),
                                      Key("max_positions", COUNT, default=DEFAULT_MAX_POSITIONS)))
        eps = read_keys(_object(document, "norm"), (Key("eps", REAL),), "norm.")["eps"]
        layers = document.get("layers")
        if not isinstance(layers, list) or not layers:
            raise ConfigError("config field 'layers' must be a list of layers")
        loop = document.get("loop")
        if loop is not None:
            if not isinstance(loop, dict) or not all(_whole(loop.get(k)) for k in ("start", "stop", "times")):
                raise ConfigError("config field 'loop' must give whole numbers start, stop, times")
            loop = LoopConfig(int(loop["start"]), int(loop["stop"]), int(loop["times"]))
        return cls(vocab=values["vocab"], width=values["width"], norm_eps=eps,
                   logit_softcap=values["logit_softcap"], loop=loop,
                   max_positions=values["max_positions"],
                   layers=tuple(PizilixLayerConfig.from_dict(layer, index)
                                for index, layer in enumerate(layers)))

    def to_dict(self) -> Dict[str, Any]:
        document: Dict[str, Any] = {
            "architecture": self.architecture, "vocab": self.vocab, "width": self.width,
            "norm": {"eps": self.norm_eps},
            "layers": [layer.to_dict() for layer in self.layers],
        }
        if self.logit_softcap is not None:
            document["logit_softcap"] = self.logit_softcap
        if self.loop is not None:
            document["loop"] = dataclasses.asdict(self.loop)
        if self.max_positions != DEFAULT_MAX_POSITIONS:
            document["max_positions"] = self.max_positions
        return document

    @staticmethod
    def random_scale(name: str, shape: Tuple[int, ...]):
        """What a model with random weights holds in its vectors (None: ones): norm weights are
        stored around zero, biases are zero, the filter takes mostly the token itself, and with
        its gate half open a channel keeps between 90 and 99.9 percent of its state per token."""
        import math

        import torch
        leaf = name.rsplit(".", 1)[-1]
        if leaf in ("norm1", "norm2", "b") or name == "final.norm":
            return 0.0
        if leaf == "conv":
            taps = torch.full(shape, 0.1)
            taps[:, -1] = 1.0
            return taps
        if leaf == "lam":
            kept = torch.linspace(math.log(0.9), math.log(0.999), shape[0], dtype=torch.float64)
            return torch.log(torch.expm1(-kept / 4.0)).to(torch.float32)
        return None

    def layer_runs(self) -> Tuple[Tuple[int, bool], ...]:
        """The layers in the order they run, as ``(layer, starts_a_repeat)``: the second is
        true for the first layer of every pass through the loop but the first pass."""
        count = len(self.layers)
        if self.loop is None:
            return tuple((layer, False) for layer in range(count))
        loop = self.loop
        runs = [(layer, False) for layer in range(loop.start)]
        for turn in range(loop.times):
            runs.extend((layer, turn > 0 and layer == loop.start)
                        for layer in range(loop.start, loop.stop))
        runs.extend((layer, False) for layer in range(loop.stop, count))
        return tuple(runs)
