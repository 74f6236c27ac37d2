"""The Manatar decoder as a list of parts.

The residual starts as the token's row of the table plus a row of a second table that the previous
token and the token pick together.  Sublayers read the residual itself; what they add passes an RMS
norm (plain weight) and a constant: ``x += c N1(mixer(x))``, then, unless the layer has none, ``x +=
c N2(ff(x))``.  Mixers: ``attention`` (two score maps per head over the same values, the second
taken off the first; biases, a causal filter over time on q, k and v, a norm per map of a query or
key head, rotary positions on neighbouring pairs with frequencies stretched for long contexts, a
norm per head and a sigmoid gate behind the maps; a layer may use an earlier layer's keys and
values) and ``mlstm`` (a matrix per head with exponential input and sigmoid forget gates, kept in
the scale of a running maximum).  The feed-forward is dense with a clamped gate, or a mixture of
experts (silu) whose router is a softmax over the chosen logits, beside an expert every token uses.
The model ends with the same kind of norm and an untied head.

Tensor names: ``embed``, ``bigram``; per layer ``l<i>.norm1``, ``l<i>.norm2``;
``l<i>.mix.{q,k,v}`` with ``.b`` and ``.conv``, ``l<i>.mix.{q,k}.norm``,
``l<i>.mix.{lq1,lk1,lq2,lk2,g,o,o.b}`` (attention); ``l<i>.mix.{q,k,v,g,o,norm}``,
``l<i>.mix.{i,f}`` with ``.b`` (mlstm); ``l<i>.mlp.{gate,up,down}`` (dense);
``l<i>.mlp.{router,router.b}``, ``l<i>.mlp.{e<j>,shared}.{gate,up,down}`` (experts); ``final.norm``,
``head``.
"""
from __future__ import annotations

import dataclasses
from typing import Callable, Dict

from ..config.manatar import (ARCHITECTURE, DifferentialAttentionConfig, FeedForwardConfig,
                              ManatarConfig, MatrixLstmConfig)
from ..config.registry import register_architecture
from ..config.spec import BlockSpec, ModelSpec, PartSpec, ScheduleEntry

LSTM_FLOOR = 1e-6        # added to the divisor of the matrix memory's output


def _attention(prefix: str, mixer: DifferentialAttentionConfig, config: ManatarConfig) -> PartSpec:
    rotary = {"theta": mixer.rot_base, "dims": mixer.rot_dims, "max_positions": config.max_positions}
    if mixer.scaling is not None:
        rotary["scaling"] = dataclasses.asdict(mixer.scaling)
    roles = {name: name for name in ("q", "k", "v", "g", "o", "lq1", "lk1", "lq2", "lk2")}
    roles.update({f"{name}_bias": f"{name}.b" for name in ("q", "k", "v", "o")})
    roles.update({f"{name}_conv": f"{name}.conv" for name in ("q", "k", "v")})
    roles.update({f"{name}_norm": f"{name}.norm" for name in ("q", "k")})
    return PartSpec("differential_attention", {
        "num_heads": mixer.heads, "num_kv_heads": mixer.kv_heads, "head_dim": mixer.dim,
        "value_dim": mixer.vdim, "scale": mixer.scale, "short_conv": mixer.conv, "bias": True,
        "qk_norm": {"eps": config.norm_eps}, "rotary": rotary, "diff": mixer.diff,
        "eps": config.norm_eps, "output_gate": "sigmoid", "shared_cache": mixer.kv_from is not None,
    }, {role: f"{prefix}.mix.{name}" for role, name in roles.items()})


def _matrix_lstm(prefix: str, mixer: MatrixLstmConfig, config: ManatarConfig) -> PartSpec:
    roles = {name: name for name in ("q", "k", "v", "g", "i", "f", "norm", "o")}
    roles.update(i_bias="i.b", f_bias="f.b")
    return PartSpec("matrix_lstm", {
        "heads": mixer.heads, "head_dim": mixer.dim, "value_dim": mixer.vdim,
        "gate_cap": mixer.gate_cap, "q_scale": mixer.dim ** -0.5, "floor": LSTM_FLOOR,
        "eps": config.norm_eps,
    }, {role: f"{prefix}.mix.{name}" for role, name in roles.items()})


# one builder per value of a layer's ``type``
MIXER_SPECS: Dict[str, Callable[[str, object, ManatarConfig], PartSpec]] = {
    "attention": _attention, "mlstm": _matrix_lstm}


def _gated(prefix: str, ff: int, **params) -> PartSpec:
    return PartSpec("gated_mlp", {"intermediate_size": ff, **params},
                    {name: f"{prefix}.{name}" for name in ("gate", "up", "down")})


def _feed_forward(prefix: str, mlp: FeedForwardConfig) -> PartSpec:
    if mlp.kind == "dense":
        return _gated(prefix, mlp.ff, activation="clamped_sigmoid", limit=mlp.limit)
    names = {"router": f"{prefix}.router", "router_bias": f"{prefix}.router.b"}
    for expert in range(mlp.experts):
        for role in ("gate", "up", "down"):
            names[f"{role}.{expert}"] = f"{prefix}.e{expert}.{role}"
    params = {"experts": mlp.experts, "top": mlp.top, "intermediate_size": mlp.ff,
              "score": "chosen_softmax", "router_bias": True, "activation": "silu"}
    if mlp.shared_ff:
        params["shared"] = _gated(f"{prefix}.shared", mlp.shared_ff, activation="silu")
    return PartSpec("routed_experts", params, names)


def build_manatar_spec(config: ManatarConfig) -> ModelSpec:
    def joined(name: str) -> PartSpec:
        return PartSpec("post_norm", {"eps": config.norm_eps, "scale": config.residual_mult},
                        {"weight": name})

    blocks, schedule = [], []
    for index, layer in enumerate(config.layers):
        prefix = f"l{index}"
        has_mlp = layer.mlp is not None
        blocks.append(BlockSpec(
            arrangement="output_norm",
            mixer_norm=None,
            mixer=MIXER_SPECS[layer.type](prefix, layer.mixer, config),
            feed_forward=_feed_forward(f"{prefix}.mlp", layer.mlp) if has_mlp else None,
            mixer_connection=joined(f"{prefix}.norm1"),
            feed_forward_connection=joined(f"{prefix}.norm2") if has_mlp else None,
        ))
        schedule.append(ScheduleEntry(block=index, cache_from=getattr(layer.mixer, "kv_from", None)))
    embedding = {"vocab_size": config.vocab}
    tables = {"weight": "embed"}
    if config.pairs is not None:
        embedding["pairs"] = dataclasses.asdict(config.pairs)
        tables["pairs"] = "bigram"
    return ModelSpec(
        architecture=config.architecture,
        hidden_size=config.width,
        vocab_size=config.vocab,
        max_positions=config.max_positions,
        embedding=PartSpec("token_table", embedding, tables),
        blocks=tuple(blocks),
        schedule=tuple(schedule),
        final_norm=PartSpec("rms", {"eps": config.norm_eps}, {"weight": "final.norm"}),
        lm_head=PartSpec("linear", {"vocab_size": config.vocab, "tied": False}, {"weight": "head"}),
    )


register_architecture(ARCHITECTURE, ManatarConfig.from_dict, build_manatar_spec,
                      aliases=("manatar",))
