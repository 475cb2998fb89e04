"""Typed configuration of the Rapolix decoder, read from its own config.json keys.

Rapolix lists its layers one by one.  A layer's mixer is two mixers side by side ("parallel"): on the left grouped-query
attention over a sliding window that keeps a sequence's first tokens, with an output gate and without rotation; on the right a
recurrent block with a real-gated linear recurrent unit.  Its feed-forward, where it has one, is a dense gated layer with
biases or routed experts without gates, with identity outputs and a shared expert beside them.  A token carries several residual
streams, and sinusoids join the embedding.  Nothing is assumed equal between layers.

    vocab, width, streams, norm.eps, logit_softcap (absent or null: the logits are not capped)
    layers[i].type     "parallel"
    layers[i].mixer    left:  heads, kv_heads, dim, vdim, scale, mask: {size, keep_first} | null
                       right: width, blocks, conv
    layers[i].mlp      null | {kind: "dense", ff}
                       | {kind: "moe", router: {experts, top, groups: {count, keep} | null, identity}, expert: {ff}, shared: {ff} | null}
"""
from __future__ import annotations

import copy
import json
import os
from dataclasses import dataclass, field
from typing import Optional, Tuple

from .errors import UnsupportedModelError

LEFT_KEYS = ("heads", "kv_heads", "dim", "vdim", "scale")
RIGHT_KEYS = ("width", "blocks", "conv")
FEED_FORWARD_KINDS = ("dense", "moe")


def _need(where: str, raw, *keys):
    if not isinstance(raw, dict):
        raise UnsupportedModelError(f"Rapolix config: {where} must be an object")
    missing = [key for key in keys if raw.get(key) is None]
    if missing:
        raise UnsupportedModelError(f"Rapolix config: {where} lacks {', '.join(missing)}")


def _positive(where: str, raw: dict, *keys):
    for key in keys:
        if raw.get(key) is not None and int(raw[key]) <= 0:
            raise UnsupportedModelError(f"Rapolix config: {where}.{key} must be positive")


def _check_mixer(where: str, mixer) -> None:
    _need(where, mixer, "left", "right")
    left, right = mixer["left"], mixer["right"]
    _need(where + ".left", left, *LEFT_KEYS)
    _positive(where + ".left", left, "heads", "kv_heads", "dim", "vdim")
    if int(left["heads"]) % int(left["kv_heads"]):
        raise UnsupportedModelError(f"Rapolix config: {where}.left: {left['heads']} heads are no multiple of {left['kv_heads']} kv_heads")
    if not float(left["scale"]) > 0.0:
        raise UnsupportedModelError(f"Rapolix config: {where}.left.scale must be positive")
    if left.get("rot"):
        raise UnsupportedModelError(f"Rapolix config: {where}.left does not rotate")
    mask = left.get("mask")
    if mask:
        _need(where + ".left.mask", mask, "size")
        _positive(where + ".left.mask", mask, "size")
        if int(mask.get("keep_first") or 0) < 0:
            raise UnsupportedModelError(f"Rapolix config: {where}.left.mask.keep_first must not be negative")
    _need(where + ".right", right, *RIGHT_KEYS)
    _positive(where + ".right", right, *RIGHT_KEYS)
    if int(right["width"]) % int(right["blocks"]):
        raise UnsupportedModelError(f"Rapolix config: {where}.right: {right['width']} channels do not divide into {right['blocks']} blocks")


def _check_mlp(where: str, mlp) -> None:
    _need(where, mlp, "kind")
    if mlp["kind"] not in FEED_FORWARD_KINDS:
        raise UnsupportedModelError(f"Rapolix config: {where} has the unknown kind {mlp['kind']!r} (known: {', '.join(FEED_FORWARD_KINDS)})")
    if mlp["kind"] == "dense":
        _need(where, mlp, "ff")
        _positive(where, mlp, "ff")
        return
    _need(where, mlp, "router", "expert")
    router = mlp["router"]
    _need(where + ".router", router, "experts", "top")
    _positive(where + ".router", router, "experts", "top")
    _need(where + ".expert", mlp["expert"], "ff")
    _positive(where + ".expert", mlp["expert"], "ff")
    identity = int(router.get("identity") or 0)
    outputs, top = int(router["experts"]) + identity, int(router["top"])
    if identity < 0 or top > outputs:
        raise UnsupportedModelError(f"Rapolix config: {where}: {top} of {outputs} router outputs cannot be chosen")
    groups = router.get("groups")
    if groups:
        _need(where + ".router.groups", groups, "count", "keep")
        count, keep = int(groups["count"]), int(groups["keep"])
        if count <= 0 or outputs % count or not 0 < keep <= count or top > keep * (outputs // count):
            raise UnsupportedModelError(f"Rapolix config: {where}: {outputs} router outputs in {count} equal groups of which {keep} are "
                                        f"kept cannot give {top} choices")
    if mlp.get("shared"):
        _need(where + ".shared", mlp["shared"], "ff")
        _positive(where + ".shared", mlp["shared"], "ff")


@dataclass(frozen=True)
class RapolixLayer:
    type: str
    mixer: dict
    mlp: Optional[dict]


@dataclass(frozen=True)
class RapolixConfig:
    vocab: int
    width: int
    streams: int
    norm_eps: float
    layers: Tuple[RapolixLayer, ...]
    logit_softcap: float = 0.0
    eos_token_id: Tuple[int, ...] = ()
    architecture: str = "Rapolix"
    extra: dict = field(default_factory=dict, compare=False)

    @property
    def vocab_size(self) -> int:
        return self.vocab

    @property
    def hidden_size(self) -> int:
        return self.width

    # ---------------------------------------------------------------- parsing
    @classmethod
    def from_dict(cls, raw: dict) -> "RapolixConfig":
        _need("config.json", raw, "vocab", "width", "streams", "layers", "norm")
        _need("norm", raw["norm"], "eps")
        _positive("config.json", raw, "vocab", "width", "streams")
        softcap = float(raw.get("logit_softcap") or 0.0)
        if softcap < 0.0:
            raise UnsupportedModelError("Rapolix config: logit_softcap must not be negative")
        if not isinstance(raw["layers"], list) or not raw["layers"]:
            raise UnsupportedModelError("Rapolix config: layers must be a non-empty list")
        layers = []
        for index, entry in enumerate(raw["layers"]):
            where = f"layers[{index}]"
            _need(where, entry, "type", "mixer")
            if entry["type"] != "parallel":
                raise UnsupportedModelError(f"Rapolix config: {where} has the unknown mixer type {entry['type']!r} (known: parallel)")
            _check_mixer(where + ".mixer", entry["mixer"])
            if entry.get("mlp") is not None:
                _check_mlp(where + ".mlp", entry["mlp"])
            layers.append(RapolixLayer(entry["type"], copy.deepcopy(entry["mixer"]), copy.deepcopy(entry.get("mlp"))))
        eos = raw.get("eos_token_id")
        eos = () if eos is None else ((int(eos),) if isinstance(eos, int) else tuple(int(e) for e in eos))
        known = {"architecture", "architectures", "vocab", "width", "streams", "norm", "layers", "logit_softcap", "eos_token_id"}
        return cls(vocab=int(raw["vocab"]), width=int(raw["width"]), streams=int(raw["streams"]), norm_eps=float(raw["norm"]["eps"]),
                   layers=tuple(layers), logit_softcap=softcap, eos_token_id=eos,
                   extra={key: value for key, value in raw.items() if key not in known})

    @classmethod
    def from_json_file(cls, path: str) -> "RapolixConfig":
        if os.path.isdir(path):
            path = os.path.join(path, "config.json")
        with open(path) as handle:
            return cls.from_dict(json.load(handle))

    def to_dict(self) -> dict:
        """config.json form (round-trips through ``from_dict``)."""
        layers = [{"type": layer.type, "mixer": copy.deepcopy(layer.mixer), "mlp": copy.deepcopy(layer.mlp)} for layer in self.layers]
        out = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "streams": self.streams,
               "norm": {"eps": self.norm_eps}, "logit_softcap": self.logit_softcap or None, "layers": layers}
        if self.eos_token_id:
            out["eos_token_id"] = list(self.eos_token_id)
        return out
