"""Typed configuration of the Dozotar decoder, read from its own config.json keys.

Dozotar lists its layers one by one.  A layer's mixer is grouped-query attention inside chunks of positions, whose
projections pass a short convolution and a norm over the whole projection and whose scores get a learned bias by distance
("attention"); retention, a matrix-valued state with a fixed decay per head ("retention"); or the state-space form whose
decay comes from each token ("mamba2").  Its feed-forward, where it has one, is a dense gated layer or routed experts with
a shared one beside them.  Nothing is assumed equal between layers.

    vocab, width, norm.eps
    layers[i].type     "attention" | "retention" | "mamba2"
    layers[i].mixer    attention:  heads, kv_heads, dim, vdim, conv, scale, bias_max, mask: {size} | null
                                   (buckets: optional, else the bias table's rows say)
                       retention:  heads, dim, vdim, decay: [one per head], rot: {base, dims} | null
                       mamba2:     heads, vdim, state, groups, conv, norm_groups
    layers[i].mlp      null | {kind: "dense", ff}
                       | {kind: "moe", router: {experts, top, groups: {count, keep} | null}, expert: {ff}, shared: {ff} | null}
"""
from __future__ import annotations

import copy
import json
import os
from dataclasses import dataclass, field
from typing import Optional, Tuple

from .errors import UnsupportedModelError

MIXER_KEYS = {
    "attention": ("heads", "kv_heads", "dim", "vdim", "conv", "scale", "bias_max"),
    "retention": ("heads", "dim", "vdim", "decay"),
    "mamba2": ("heads", "vdim", "state", "groups", "conv", "norm_groups"),
}
POSITIVE_KEYS = ("heads", "kv_heads", "dim", "vdim", "conv", "state", "groups", "norm_groups")
FEED_FORWARD_KINDS = ("dense", "moe")


def _need(where: str, raw, *keys):
    if not isinstance(raw, dict):
        raise UnsupportedModelError(f"Dozotar config: {where} must be an object")
    missing = [key for key in keys if raw.get(key) is None]
    if missing:
        raise UnsupportedModelError(f"Dozotar config: {where} lacks {', '.join(missing)}")


def _positive(where: str, raw: dict, *keys):
    for key in keys:
        if raw.get(key) is not None and int(raw[key]) <= 0:
            raise UnsupportedModelError(f"Dozotar config: {where}.{key} must be positive")


def _check_mixer(where: str, kind: str, mixer) -> None:
    _need(where, mixer, *MIXER_KEYS[kind])
    _positive(where, mixer, *(key for key in POSITIVE_KEYS if key in MIXER_KEYS[kind]))
    if kind == "attention":
        if int(mixer["heads"]) % int(mixer["kv_heads"]):
            raise UnsupportedModelError(f"Dozotar config: {where}: {mixer['heads']} heads are no multiple of {mixer['kv_heads']} kv_heads")
        if mixer.get("mask"):
            _need(where + ".mask", mixer["mask"], "size")
            _positive(where + ".mask", mixer["mask"], "size")
        if mixer.get("rot"):
            raise UnsupportedModelError(f"Dozotar config: {where}: an attention layer does not rotate")
    elif kind == "retention":
        if not isinstance(mixer["decay"], (list, tuple)) or len(mixer["decay"]) != int(mixer["heads"]):
            raise UnsupportedModelError(f"Dozotar config: {where}.decay must list one number per head ({mixer['heads']})")
        rot = mixer.get("rot")
        if rot:
            _need(where + ".rot", rot, "base", "dims")
            if int(rot["dims"]) % 2 or not 0 < int(rot["dims"]) <= int(mixer["dim"]):
                raise UnsupportedModelError(f"Dozotar config: {where}: rot.dims must be even and at most dim")
    else:
        if int(mixer["heads"]) % int(mixer["groups"]):
            raise UnsupportedModelError(f"Dozotar config: {where}: {mixer['heads']} heads are no multiple of {mixer['groups']} groups")
        if int(mixer["heads"]) * int(mixer["vdim"]) % int(mixer["norm_groups"]):
            raise UnsupportedModelError(f"Dozotar config: {where}: the channels do not divide into {mixer['norm_groups']} norm_groups")


def _check_mlp(where: str, mlp) -> None:
    _need(where, mlp, "kind")
    if mlp["kind"] not in FEED_FORWARD_KINDS:
        raise UnsupportedModelError(f"Dozotar config: {where} has the unknown kind {mlp['kind']!r} (known: {', '.join(FEED_FORWARD_KINDS)})")
    if mlp["kind"] == "dense":
        _need(where, mlp, "ff")
        _positive(where, mlp, "ff")
        return
    _need(where, mlp, "router", "expert")
    router = mlp["router"]
    _need(where + ".router", router, "experts", "top")
    _need(where + ".expert", mlp["expert"], "ff")
    _positive(where + ".expert", mlp["expert"], "ff")
    experts, top = int(router["experts"]), int(router["top"])
    if not 0 < top <= experts:
        raise UnsupportedModelError(f"Dozotar config: {where}: top must lie in 1..experts")
    groups = router.get("groups")
    if groups:
        _need(where + ".router.groups", groups, "count", "keep")
        count, keep = int(groups["count"]), int(groups["keep"])
        if count <= 0 or experts % count or not 0 < keep <= count or top > keep * (experts // count):
            raise UnsupportedModelError(f"Dozotar config: {where}: {experts} experts in {count} equal groups of which {keep} are kept "
                                        f"cannot give {top} choices")
    if mlp.get("shared"):
        _need(where + ".shared", mlp["shared"], "ff")
        _positive(where + ".shared", mlp["shared"], "ff")


@dataclass(frozen=True)
class DozotarLayer:
    type: str
    mixer: dict
    mlp: Optional[dict]


@dataclass(frozen=True)
class DozotarConfig:
    vocab: int
    width: int
    norm_eps: float
    layers: Tuple[DozotarLayer, ...]
    eos_token_id: Tuple[int, ...] = ()
    architecture: str = "Dozotar"
    extra: dict = field(default_factory=dict, compare=False)

    @property
    def vocab_size(self) -> int:
        return self.vocab

    @property
    def hidden_size(self) -> int:
        return self.width

    # ---------------------------------------------------------------- parsing
    @classmethod
    def from_dict(cls, raw: dict) -> "DozotarConfig":
        _need("config.json", raw, "vocab", "width", "layers", "norm")
        _need("norm", raw["norm"], "eps")
        _positive("config.json", raw, "vocab", "width")
        if not isinstance(raw["layers"], list) or not raw["layers"]:
            raise UnsupportedModelError("Dozotar config: layers must be a non-empty list")
        layers = []
        for index, entry in enumerate(raw["layers"]):
            where = f"layers[{index}]"
            _need(where, entry, "type", "mixer")
            kind = entry["type"]
            if kind not in MIXER_KEYS:
                raise UnsupportedModelError(f"Dozotar config: {where} has the unknown mixer type {kind!r} "
                                            f"(known: {', '.join(sorted(MIXER_KEYS))})")
            _check_mixer(where + ".mixer", kind, entry["mixer"])
            if entry.get("mlp") is not None:
                _check_mlp(where + ".mlp", entry["mlp"])
            layers.append(DozotarLayer(kind, copy.deepcopy(entry["mixer"]), copy.deepcopy(entry.get("mlp"))))
        eos = raw.get("eos_token_id")
        eos = () if eos is None else ((int(eos),) if isinstance(eos, int) else tuple(int(e) for e in eos))
        known = {"architecture", "architectures", "vocab", "width", "norm", "layers", "eos_token_id"}
        return cls(vocab=int(raw["vocab"]), width=int(raw["width"]), norm_eps=float(raw["norm"]["eps"]), layers=tuple(layers),
                   eos_token_id=eos, extra={key: value for key, value in raw.items() if key not in known})

    @classmethod
    def from_json_file(cls, path: str) -> "DozotarConfig":
        if os.path.isdir(path):
            path = os.path.join(path, "config.json")
        with open(path) as handle:
            return cls.from_dict(json.load(handle))

    def to_dict(self) -> dict:
        """config.json form (round-trips through ``from_dict``)."""
        layers = [{"type": layer.type, "mixer": copy.deepcopy(layer.mixer), "mlp": copy.deepcopy(layer.mlp)} for layer in self.layers]
        out = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
               "layers": layers}
        if self.eos_token_id:
            out["eos_token_id"] = list(self.eos_token_id)
        return out
