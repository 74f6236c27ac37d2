"""The Pizilix decoder as a list of parts.

A layer is pre-norm (RMS norm, weight stored around zero): ``x += mixer(norm1(x))``, then, unless
the layer has none, ``x += ff(norm2(x))`` with a silu-gated feed-forward.  Mixers: ``attention``
(grouped key/value heads whose values are the keys as projected, before the rotation; rotary
positions on neighbouring pairs of the first coordinates with frequencies stretched for long
contexts; scores that run into a level; positions see each other inside chunks counted from
position 0; one added to the softmax's denominator) and ``rglru`` (a causal filter and a
real-gated linear recurrence on one branch, gelu_tanh on the other, their product through the
output matrix).  A stretch of layers may run several times with the same weights (``loop``);
every run owns its cache and state, and the embedding's output is added to the residual before
every repeat.  The model ends with the same norm, the embedding table as its head, and logits that
run into a level.

Tensor names: ``embed``; per layer ``l<i>.norm1``, ``l<i>.norm2``; ``l<i>.mix.{q,k,o}``
(attention); ``l<i>.mix.{y,x}`` with ``.b``, ``l<i>.mix.conv`` with ``.b``, ``l<i>.mix.{ra,ri}`` with
``.b``, ``l<i>.mix.{lam,o}`` (rglru); ``l<i>.mlp.{gate,up,down}``; ``final.norm``.
"""
from __future__ import annotations

from typing import Callable, Dict

from ..config.pizilix import (ARCHITECTURE, ChunkedAttentionConfig, GatedRecurrenceConfig,
                              PizilixConfig)
from ..config.registry import register_architecture
from ..config.spec import BlockSpec, ModelSpec, PartSpec, ScheduleEntry

SINK_SCORE = 0.0        # one more term of the softmax's denominator: exp(0)
DECAY_RATE = 8.0        # log a = -DECAY_RATE * r * softplus(lam)


def _attention(prefix: str, mixer: ChunkedAttentionConfig, config: PizilixConfig) -> PartSpec:
    rotary = {"theta": mixer.rot_base, "exact_theta": True, "head_dim": mixer.dim,
              "rotary_dim": mixer.rot_dims, "pairing": "adjacent",
              "max_positions": config.max_positions}
    if mixer.scaling is not None:
        rotary["scaling"] = {"factor": mixer.scaling.factor, "original": mixer.scaling.original,
                             "fast": mixer.scaling.fast, "slow": mixer.scaling.slow}
    return PartSpec("paged_attention", {
        "num_heads": mixer.heads, "num_kv_heads": mixer.kv_heads, "head_dim": mixer.dim,
        "scale": mixer.scale, "chunk": mixer.chunk, "softcap": mixer.softcap,
        "sinks": SINK_SCORE, "values": "keys", "position": PartSpec("rotary", rotary),
    }, {name: f"{prefix}.mix.{name}" for name in ("q", "k", "o")})


def _gated_recurrence(prefix: str, mixer: GatedRecurrenceConfig, config: PizilixConfig) -> PartSpec:
    roles = {"y": "y", "y_bias": "y.b", "x": "x", "x_bias": "x.b", "filter": "conv",
             "filter_bias": "conv.b", "r": "ra", "r_bias": "ra.b", "i": "ri", "i_bias": "ri.b",
             "decay": "lam", "o": "o"}
    return PartSpec("gated_recurrence", {
        "width": mixer.width, "blocks": mixer.blocks, "filter_taps": mixer.conv,
        "decay_rate": DECAY_RATE,
    }, {role: f"{prefix}.mix.{name}" for role, name in roles.items()})


# one builder per value of a layer's ``type``
MIXER_SPECS: Dict[str, Callable[[str, object, PizilixConfig], PartSpec]] = {
    "attention": _attention, "rglru": _gated_recurrence}


def build_pizilix_spec(config: PizilixConfig) -> ModelSpec:
    def norm(name: str) -> PartSpec:
        return PartSpec("rms", {"eps": config.norm_eps, "one_plus": True}, {"weight": name})

    blocks = []
    for index, layer in enumerate(config.layers):
        prefix = f"l{index}"
        has_mlp = layer.mlp is not None
        blocks.append(BlockSpec(
            arrangement="pre_norm",
            mixer_norm=norm(f"{prefix}.norm1"),
            mixer=MIXER_SPECS[layer.type](prefix, layer.mixer, config),
            feed_forward_norm=norm(f"{prefix}.norm2") if has_mlp else None,
            feed_forward=PartSpec("gated_mlp", {"intermediate_size": layer.mlp.ff,
                                                "activation": "silu"},
                                  {name: f"{prefix}.mlp.{name}" for name in ("gate", "up", "down")})
            if has_mlp else None,
        ))
    return ModelSpec(
        architecture=config.architecture,
        hidden_size=config.width,
        vocab_size=config.vocab,
        max_positions=config.max_positions,
        embedding=PartSpec("token_table", {"vocab_size": config.vocab}, {"weight": "embed"}),
        blocks=tuple(blocks),
        schedule=tuple(ScheduleEntry(block=layer, add_embedding=repeat)
                       for layer, repeat in config.layer_runs()),
        final_norm=norm("final.norm"),
        lm_head=PartSpec("linear", {"vocab_size": config.vocab, "tied": True,
                                    "softcap": config.logit_softcap}, {"weight": "embed"}),
    )


register_architecture(ARCHITECTURE, PizilixConfig.from_dict, build_pizilix_spec,
                      aliases=("pizilix",))
