"""Dozotar: from its typed configuration to the architecture-neutral model specification.

This is the only place that knows how Dozotar arranges its parts and names its tensors.  Every layer normalises the output
of each sub-layer with a norm whose weight is one number, and lets the sub-layers read the stream as it is
(``output_norm``); its mixer is ``gqa_attention`` in the form with convolved and wholly normalised projections, chunks and a
bias by distance, ``retention``, or ``state_space_duality``; its feed-forward, where it has one, is ``gelu_glu`` or
``routed_experts`` with softmax scores, groups and a gated shared expert.

Tensors: ``embed``, ``head``, ``final.norm``; layer i: ``l<i>.norm1`` (behind the mixer), ``l<i>.norm2`` (behind the
feed-forward), ``l<i>.mix.*``, ``l<i>.mlp.gate`` / ``.up`` / ``.down``, or ``l<i>.mlp.router``, ``l<i>.mlp.e<j>.*`` and
``l<i>.mlp.shared.*``.
"""
from __future__ import annotations

from ..config.dozotar import DozotarConfig
from ..config.registry import register_architecture
from ..config.spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry

ATTENTION_NAMES = (("q", "q"), ("k", "k"), ("v", "v"), ("o", "o"), ("q_norm", "q.norm"), ("k_norm", "k.norm"), ("rel", "rel"))


def _position_of(mixer: dict, positions: dict):
    """Name of the position encoding this mixer uses (made on first use; equal constants share one)."""
    rot = mixer.get("rot")
    if not rot:
        return None
    part = PartSpec.of("rotary", head_dim=int(mixer["dim"]), theta=float(rot["base"]), rotary_dim=int(rot["dims"]))
    for name, known in positions.items():
        if known == part:
            return name
    name = f"rot{len(positions)}"
    positions[name] = part
    return name


def _mixer_of(kind: str, mixer: dict, config: DozotarConfig) -> PartSpec:
    if kind == "attention":
        size = (mixer.get("mask") or {}).get("size")
        # the number of buckets is the bias table's number of rows; a configuration may name it ("buckets") for models
        # whose weights are made rather than read
        buckets = int(mixer["buckets"]) if mixer.get("buckets") else None
        return PartSpec.of("gqa_attention", hidden=config.width, heads=int(mixer["heads"]), kv_heads=int(mixer["kv_heads"]),
                           head_dim=int(mixer["dim"]), value_dim=int(mixer["vdim"]), scale=float(mixer["scale"]),
                           qk_norm="projection", eps=config.norm_eps, conv=int(mixer["conv"]), chunk=int(size) if size else None,
                           distance_bias=(buckets, float(mixer["bias_max"])), precise_weights=True, names=ATTENTION_NAMES)
    if kind == "retention":
        return PartSpec.of("retention", hidden=config.width, heads=int(mixer["heads"]), dim=int(mixer["dim"]),
                           value_dim=int(mixer["vdim"]), decay=tuple(float(value) for value in mixer["decay"]), eps=config.norm_eps)
    return PartSpec.of("state_space_duality", hidden=config.width, heads=int(mixer["heads"]), value_dim=int(mixer["vdim"]),
                       state=int(mixer["state"]), groups=int(mixer["groups"]), conv=int(mixer["conv"]),
                       norm_groups=int(mixer["norm_groups"]), eps=config.norm_eps)


def _feed_forward_of(mlp, config: DozotarConfig):
    if mlp is None:
        return None
    if mlp["kind"] == "dense":
        return PartSpec.of("gelu_glu", hidden=config.width, intermediate=int(mlp["ff"]))
    router, groups, shared = mlp["router"], mlp["router"].get("groups"), mlp.get("shared")
    return PartSpec.of("routed_experts", hidden=config.width, experts=int(router["experts"]), top=int(router["top"]),
                       intermediate=int(mlp["expert"]["ff"]), activation="silu", correction=False, route_scale=1.0,
                       scores="softmax", groups=(int(groups["count"]), int(groups["keep"])) if groups else None, renormalise=True,
                       shared_intermediate=int(shared["ff"]) if shared else None, shared_gate=bool(shared))


def dozotar_spec(config: DozotarConfig) -> ModelSpec:
    def norm():
        return PartSpec.of("rmsnorm", width=config.width, eps=config.norm_eps, tensor="", scalar=True)

    positions, layers = {}, []
    for index, layer in enumerate(config.layers):
        feed_forward = _feed_forward_of(layer.mlp, config)
        block = PartSpec.of("output_norm", feed_forward=feed_forward is not None, mixer_prefix="mix.", feed_forward_prefix="mlp.",
                            mixer_out_norm_prefix="norm1", feed_forward_out_norm_prefix="norm2")
        extra = (("mixer_out_norm", norm()),) + ((("feed_forward_out_norm", norm()),) if feed_forward is not None else ())
        layers.append(LayerSpec(prefix=f"l{index}.", block=block, mixer=_mixer_of(layer.type, layer.mixer, config),
                                feed_forward=feed_forward, extra=extra,
                                position=_position_of(layer.mixer, positions) if layer.type == "retention" else None))
    schedule = [ScheduleEntry(index) for index in range(len(layers))]
    return ModelSpec(architecture=config.architecture, vocab_size=config.vocab, hidden_size=config.width, layers=layers,
                     schedule=schedule, positions=positions, final_norm=norm(), embedding_name="embed",
                     final_norm_prefix="final.norm", head_name="head", tie_head=False, eos_token_ids=config.eos_token_id)


register_architecture("Dozotar", DozotarConfig, dozotar_spec)
