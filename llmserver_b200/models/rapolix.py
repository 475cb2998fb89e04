"""Rapolix: from its typed configuration to the architecture-neutral model specification.

This is the only place that knows how Rapolix arranges its parts and names its tensors.  Every layer is a
``hyper_connections`` block over several residual streams with a layer norm in front of each sub-layer; its mixer is
``parallel_mixers`` with normalised branches: ``gqa_attention`` in the form with a window, kept first tokens and an output gate,
and ``gated_linear_recurrent_unit``; its feed-forward, where it has one, is ``biased_glu`` or ``routed_experts`` with squared-ReLU
experts, identity outputs, a correction of the choice and renormalised softmax scores.  Sinusoids join the embedding, the final
norm reads the sum of the streams and the logits are capped.

Tensors: ``embed``, ``head``, ``final.norm``; layer i: ``l<i>.norm1`` / ``.norm2``, ``l<i>.hc1.*`` / ``.hc2.*`` (in, out, mix),
``l<i>.mix.left.*``, ``l<i>.mix.right.*`` (each branch's norm is its ``.out``), ``l<i>.mlp.gate`` / ``.up`` / ``.down`` with ``.b``, or
``l<i>.mlp.router``, ``.correction``, ``.e<j>.*`` and ``.shared.*``.
"""
from __future__ import annotations

from ..config.rapolix import RapolixConfig
from ..config.registry import register_architecture
from ..config.spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry

ATTENTION_NAMES = (("q", "q"), ("k", "k"), ("v", "v"), ("o", "o"), ("g", "g"))


def _mixer_of(mixer: dict, config: RapolixConfig) -> PartSpec:
    left, right = mixer["left"], mixer["right"]
    mask = left.get("mask") or {}
    size = int(mask["size"]) if mask.get("size") else None
    attention = PartSpec.of("gqa_attention", hidden=config.width, heads=int(left["heads"]), kv_heads=int(left["kv_heads"]),
                            head_dim=int(left["dim"]), value_dim=int(left["vdim"]), scale=float(left["scale"]), window=size,
                            keep_first=int(mask.get("keep_first") or 0) if size else 0, gate=True, precise_weights=True, names=ATTENTION_NAMES)
    recurrent = PartSpec.of("gated_linear_recurrent_unit", hidden=config.width, width=int(right["width"]), blocks=int(right["blocks"]),
                            conv=int(right["conv"]))
    return PartSpec.of("parallel_mixers", width=config.width, norm_eps=config.norm_eps,
                       branches=(("left", attention, 0.5, False), ("right", recurrent, 0.5, False)))


def _feed_forward_of(mlp, config: RapolixConfig):
    if mlp is None:
        return None
    if mlp["kind"] == "dense":
        return PartSpec.of("biased_glu", hidden=config.width, intermediate=int(mlp["ff"]), activation="silu")
    router, groups, shared = mlp["router"], mlp["router"].get("groups"), mlp.get("shared")
    return PartSpec.of("routed_experts", hidden=config.width, experts=int(router["experts"]), identity=int(router.get("identity") or 0),
                       top=int(router["top"]), intermediate=int(mlp["expert"]["ff"]), activation="squared_relu", correction=True,
                       route_scale=1.0, scores="softmax", groups=(int(groups["count"]), int(groups["keep"])) if groups else None,
                       renormalise=True, shared_intermediate=int(shared["ff"]) if shared else None)


def rapolix_spec(config: RapolixConfig) -> ModelSpec:
    def norm():
        return PartSpec.of("layernorm", width=config.width, eps=config.norm_eps, tensor="")

    layers = []
    for index, layer in enumerate(config.layers):
        feed_forward = _feed_forward_of(layer.mlp, config)
        block = PartSpec.of("hyper_connections", streams=config.streams, feed_forward=feed_forward is not None, mixer_prefix="mix.",
                            feed_forward_prefix="mlp.", mixer_norm_prefix="norm1", feed_forward_norm_prefix="norm2",
                            mixer_connections="hc1.", feed_forward_connections="hc2.")
        layers.append(LayerSpec(prefix=f"l{index}.", block=block, mixer=_mixer_of(layer.mixer, config), feed_forward=feed_forward,
                                mixer_norm=norm(), feed_forward_norm=norm() if feed_forward is not None else None))
    schedule = [ScheduleEntry(index) for index in range(len(layers))]
    return ModelSpec(architecture=config.architecture, vocab_size=config.vocab, hidden_size=config.width, layers=layers,
                     schedule=schedule, positions={"sinusoids": PartSpec.of("sinusoidal", width=config.width)}, final_norm=norm(),
                     embedding_name="embed", final_norm_prefix="final.norm", head_name="head", tie_head=False, streams=config.streams,
                     logit_softcap=config.logit_softcap, eos_token_ids=config.eos_token_id)


register_architecture("Rapolix", RapolixConfig, rapolix_spec)
