"""Grouped-query attention over the paged cache, with optional per-head Q/K RMSNorm, rotary
positions and a sliding window."""
from __future__ import annotations

import functools
import math

import torch

from .. import ops
from ..cache.manager import KVPagesNeed, StateNeed
from ..weights.declare import NORM, WIDE, WeightDecl
from .base import Mixer
from .registry import MIXERS


def distance_buckets(count: int, largest: float, distances: int) -> list:
    """The bucket of each distance 0 .. distances - 1 among ``count`` buckets: with half = count / 2, distance n < half has a
    bucket of its own, and farther ones share buckets whose borders grow geometrically up to ``largest``,

        half + floor(ln(n / half) / ln(largest / half) * (count - half)),  at most count - 1."""
    half = count // 2
    if count < 2 or largest <= half:
        raise ValueError(f"{count} buckets need a largest distance above {half}, got {largest}")
    found = []
    for n in range(distances):
        if n < half:
            found.append(n)
        else:
            found.append(min(count - 1, half + int(math.floor(math.log(n / half) / math.log(largest / half) * (count - half)))))
    return found


@MIXERS.register("gqa_attention")
class GQAttention(Mixer):
    """Q, K, V = x Wq^T, x Wk^T, x Wv^T as one fused product (utils/attention.py:54-66,118-128); each Q
    and K head RMS-normalised with a shared [D] weight before the rotation (utils/attention.py:38-39,
    143-158); K stored after norm and rotation, V raw (utils/attention.py:172-176); softmax(Q K^T *
    scale) V over the request's cached tokens, query head h reading kv head h // group
    (utils/attention.py:186-198); output through Wo (utils/attention.py:299-300).

    Parameters: ``hidden``, ``heads``, ``kv_heads``, ``head_dim``, ``scale``, ``qk_norm`` (bool),
    ``eps`` (of the Q/K norms), ``window`` (None = all keys; else a query at position p reads keys
    p - window + 1 .. p).  ``bias`` and ``softcap`` are known and must be off: the kernels have neither a bias
    epilogue nor score capping, and say so instead of computing without them.  ``value_dim``: the size of a value
    head where it differs from ``head_dim`` (the output projection then reads heads * value_dim columns).  ``sinks``
    (bool): a learned number per query head joins each softmax's denominator as exp(sink), without a key or a value,
    neither scaled nor masked.  ``precise_weights`` (bool): the design wants its attention weights in 32-bit, so the
    bfloat16 kernels may not round them to 8 bits for the P V product.  ``values_are_keys`` (bool): there is no value
    projection, a head's key as projected (and normalised and rotated, where the layer does that) is also its value; the
    cache then keeps keys alone.  ``unit_sink`` (bool): every softmax denominator holds one more 1 (a sink whose score is
    0, without a learned number).  ``query_temperature`` = (coef, every): the query at position p is multiplied by
    1 + coef * ln(floor((p + 1) / every) + 1).  ``conv`` (taps): q, k and v pass a causal convolution over time per channel
    right behind their projections (weights: the projection's name with ".conv" added, [channels, taps], the last column
    the current token's); the last taps - 1 projected rows of every request are kept in its state slot.  ``qk_norm``
    "projection": one RMS norm over all of q and one over all of k, weights as long as they, in place of the norms per
    head.  ``chunk``: a query at position p reads keys floor(p / chunk) * chunk .. p.  ``keep_first``: with a window, every query also reads
    the sequence's first ``keep_first`` keys, at their true distances.  ``gate`` (bool): the concatenated heads are multiplied by
    sigmoid(W_g x) (role g, [heads * value_dim, hidden], part of the fused product) in front of the output projection.  ``distance_bias`` = (buckets, largest):
    a learned number per head and bucket of the distance between query and key (``rel`` [buckets, heads]; see
    ``distance_buckets``; buckets None: as many as the tensor has rows) is added to the scaled score.  ``names``: pairs (role, tensor name behind the prefix) for checkpoints that call the
    tensors otherwise; roles are q, k, v, o, g, q_norm, k_norm, sinks, rel.

    How positions are encoded comes from the position encoding the layer names (``attach``): its inverse
    frequencies, how many elements of a head rotate (``rotary_dim``, at most head_dim) and how they pair
    ("halves" or "interleaved").  An encoding that scales the rotated values (``attention_factor`` other than 1) is
    goes through the rotation kernel that takes a magnitude, which has no per-head norm: with ``qk_norm`` it is
    refused.  The same kernel serves heads whose values have another size than their keys; with ``qk_norm`` as well,
    such heads go through the kernel for heads made of units (pairing "halves" only)."""

    KNOWN_PARAMS = ("hidden", "heads", "kv_heads", "head_dim", "scale", "qk_norm", "eps", "window", "bias", "softcap",
                    "value_dim", "sinks", "names", "precise_weights", "values_are_keys", "unit_sink", "query_temperature",
                    "conv", "chunk", "distance_bias", "keep_first", "gate")
    NAMES = {"q": "q_proj.weight", "k": "k_proj.weight", "v": "v_proj.weight", "o": "o_proj.weight",
             "g": "g_proj.weight", "q_norm": "q_norm.weight", "k_norm": "k_norm.weight", "sinks": "sinks", "rel": "rel"}

    @classmethod
    def names(cls, params) -> dict:
        given = dict(params.get("names") or ())
        unknown = sorted(set(given) - set(cls.NAMES))
        if unknown:
            raise ValueError(f"gqa_attention has no tensor in the role(s) {', '.join(unknown)}")
        return {**cls.NAMES, **given}

    @classmethod
    def check_params(cls, params):
        super().check_params(params)
        if params.get("bias"):
            raise ValueError("gqa_attention has no biases in its projections (bias must be absent or false)")
        if params.get("softcap"):
            raise ValueError("gqa_attention does not cap attention scores (softcap must be absent or 0)")
        if params.get("values_are_keys") and params.get("value_dim") and int(params["value_dim"]) != int(params["head_dim"]):
            raise ValueError("gqa_attention: values that are the keys have the keys' size")
        if params.get("unit_sink") and params.get("sinks"):
            raise ValueError("gqa_attention: a softmax has learned sinks or the unit sink, not both")
        temperature = params.get("query_temperature")
        if temperature and (len(temperature) != 2 or int(temperature[1]) <= 0):
            raise ValueError("gqa_attention: query_temperature is (coef, every) with a positive period")
        if params.get("qk_norm") not in (None, True, False, "projection"):
            raise ValueError(f"gqa_attention: qk_norm is a truth value or 'projection', not {params['qk_norm']!r}")
        if cls.by_rows(params) and (params.get("values_are_keys") or params.get("query_temperature")):
            raise ValueError("gqa_attention: convolutions and norms over whole projections come with a value projection and "
                             "without a query temperature")
        if params.get("chunk") and (int(params["chunk"]) <= 0 or params.get("window")):
            raise ValueError("gqa_attention: keys are bounded by a window or by chunks of a positive size, not by both")
        if int(params.get("keep_first") or 0) < 0 or (params.get("keep_first") and params.get("chunk")):
            raise ValueError("gqa_attention: first keys are kept beside a window, and not a negative number of them")
        if params.get("gate") and (cls.by_rows(params) or params.get("values_are_keys")):
            raise ValueError("gqa_attention: an output gate comes with a value projection and heads normalised one by one")
        if params.get("distance_bias") and params["distance_bias"][0] is not None:
            distance_buckets(int(params["distance_bias"][0]), float(params["distance_bias"][1]), 1)

    @classmethod
    def by_rows(cls, params) -> bool:
        """Whether whole rows of the projection are convolved or normalised before they become heads."""
        return bool(params.get("conv")) or params.get("qk_norm") == "projection"

    @classmethod
    def declare_weights(cls, params):
        hidden, heads, kv_heads, dim = params["hidden"], params["heads"], params["kv_heads"], params["head_dim"]
        value_dim = params.get("value_dim") or dim
        name = cls.names(params)
        wanted = {name["q"]: WeightDecl((heads * dim, hidden)),
                  name["k"]: WeightDecl((kv_heads * dim, hidden)),
                  name["v"]: WeightDecl((kv_heads * value_dim, hidden)),
                  name["o"]: WeightDecl((hidden, heads * value_dim))}
        if params.get("values_are_keys"):
            del wanted[name["v"]]
        if params.get("gate"):
            wanted[name["g"]] = WeightDecl((heads * value_dim, hidden))
        if params.get("qk_norm"):
            whole = params["qk_norm"] == "projection"
            wanted[name["q_norm"]] = WeightDecl((heads * dim if whole else dim,), NORM)
            wanted[name["k_norm"]] = WeightDecl((kv_heads * dim if whole else dim,), NORM)
        if params.get("conv"):
            for role in ("q", "k", "v"):
                wanted[name[role] + ".conv"] = WeightDecl((wanted[name[role]].shape[0], int(params["conv"])), WIDE)
        if params.get("distance_bias"):
            wanted[name["rel"]] = WeightDecl((int(params["distance_bias"][0]) if params["distance_bias"][0] else -1, heads), WIDE)
        if params.get("sinks"):
            wanted[name["sinks"]] = WeightDecl((heads,), WIDE)
        return wanted

    @classmethod
    def cache_need(cls, params):
        if params.get("values_are_keys"):
            return KVPagesNeed(int(params["kv_heads"]), int(params["head_dim"]), params.get("window"), None, keys_only=True)
        pages = KVPagesNeed(int(params["kv_heads"]), int(params["head_dim"]), params.get("window"),
                            int(params["value_dim"]) if params.get("value_dim") else None,
                            chunk=int(params["chunk"]) if params.get("chunk") else None,
                            keep_first=int(params.get("keep_first") or 0))
        if int(params.get("conv") or 1) == 1:
            return pages
        kv_heads, dim = int(params["kv_heads"]), int(params["head_dim"])
        channels = (int(params["heads"]) + kv_heads) * dim + kv_heads * int(params.get("value_dim") or dim)
        return (pages, StateNeed((int(params["conv"]) - 1, channels), "float32"))

    def __init__(self, params, weights, runtime):
        super().__init__(params, weights, runtime)
        self.heads, self.kv_heads, self.head_dim = int(params["heads"]), int(params["kv_heads"]), int(params["head_dim"])
        if self.heads % self.kv_heads:
            raise ValueError(f"{self.heads} query heads are no multiple of {self.kv_heads} kv heads")
        self.scale = float(params["scale"])
        self.window = int(params["window"]) if params.get("window") else 0
        self.eps = float(params.get("eps", 0.0))
        self.value_dim = int(params.get("value_dim") or self.head_dim)
        # keys and values of different sizes are rotated and cached by the kernel for split sizes
        self.split = self.value_dim != self.head_dim
        name = self.names(params)
        self.values_are_keys = bool(params.get("values_are_keys"))
        self.temperature = tuple(params["query_temperature"]) if params.get("query_temperature") else None
        rows = [weights[name["q"]], weights[name["k"]]] + ([] if self.values_are_keys else [weights[name["v"]]])
        self.keep_first = int(params.get("keep_first") or 0) if self.window else 0
        self.gate_column = None
        if params.get("gate"):
            # the gate's rows lie behind the values', everything at whole 16-byte pieces of the packed row
            def fill():
                ragged = -sum(int(row.shape[0]) for row in rows) % 8
                if ragged:
                    rows.append(torch.zeros((ragged, rows[0].shape[1]), dtype=rows[0].dtype, device=rows[0].device))
            fill()
            self.gate_column = sum(int(row.shape[0]) for row in rows)
            rows.append(weights[name["g"]])
            fill()
        self.qkv = torch.cat(rows, dim=0).contiguous()
        self.out = weights[name["o"]].contiguous()
        self.q_norm = weights[name["q_norm"]].contiguous() if params.get("qk_norm") else None
        self.k_norm = weights[name["k_norm"]].contiguous() if params.get("qk_norm") else None
        self.sinks = weights[name["sinks"]].to(torch.float32).contiguous() if params.get("sinks") else None
        if params.get("unit_sink"):
            self.sinks = torch.zeros(self.heads, dtype=torch.float32, device=runtime.device)      # exp(0): a one in every denominator
        # keys that are their own values and queries with a temperature go through the kernel for heads made of units
        # (as do packed rows with a gate behind their values: that kernel takes longer rows)
        self.by_units = self.values_are_keys or self.temperature is not None or self.gate_column is not None
        self.inv_freq, self.rotary_dim, self.interleaved, self.magnitude = None, self.head_dim, False, 1.0
        self.rows_first = self.by_rows(params)
        self.taps = None
        if params.get("conv"):
            self.taps = torch.cat([weights[name[role] + ".conv"].to(torch.float32) for role in ("q", "k", "v")], dim=0).t().contiguous()
        self.chunk = int(params.get("chunk") or 0)
        self.bias = self.bias_log2 = None
        if params.get("distance_bias"):
            # the table by distance, made once: a chunk or the window bounds the distances, and from the largest one on
            # every distance falls into the last bucket
            table = weights[name["rel"]].to(torch.float32)
            count, largest = table.shape[0], float(params["distance_bias"][1])
            reach = math.ceil(largest) + 1
            for bound in (self.chunk, self.window):
                reach = min(reach, bound) if bound else reach
            buckets = torch.tensor(distance_buckets(count, largest, reach), dtype=torch.long, device=table.device)
            self.bias = table[buckets].t().contiguous()
            self.bias_log2 = (self.bias * ops.LOG2E).contiguous()

    def attach(self, position):
        """``position``: None (no rotation) or an encoding with ``inv_freq`` (float32 [rotary_dim / 2] on the device)
        and, optionally, ``rotary_dim``, ``pairing`` ("halves" | "interleaved") and ``attention_factor``."""
        if position is None:
            return
        if self.rows_first:
            raise ValueError("gqa_attention: the kernel that convolves and normalises whole projections does not rotate heads")
        inv_freq = getattr(position, "inv_freq", None)
        if inv_freq is None:
            raise ValueError(f"gqa_attention rotates queries and keys: the position encoding {type(position).__name__} "
                             "gives no inv_freq (an encoding that acts on the embedding is not named by a layer)")
        rotary_dim = int(getattr(position, "rotary_dim", 2 * inv_freq.numel()))
        if rotary_dim != 2 * inv_freq.numel() or rotary_dim > self.head_dim or rotary_dim % 2:
            raise ValueError(f"the position encoding rotates {rotary_dim} elements with {inv_freq.numel()} frequencies; "
                             f"gqa_attention needs an even rotary_dim of at most head_dim {self.head_dim} and half as many frequencies")
        pairing = getattr(position, "pairing", "halves")
        if pairing not in ("halves", "interleaved"):
            raise ValueError(f"gqa_attention pairs rotated elements as 'halves' or 'interleaved', not {pairing!r}")
        self.magnitude = float(getattr(position, "attention_factor", 1.0))
        if self.magnitude != 1.0:
            if self.by_units:
                raise ValueError("gqa_attention: the kernel for heads made of units does not scale the rotated values, and the "
                                 f"position encoding's attention_factor is {self.magnitude}")
            if self.q_norm is not None:
                raise ValueError("gqa_attention: the rotation kernel that applies per-head Q/K norms does not scale the rotated "
                                 f"values, and the position encoding's attention_factor is {self.magnitude}")
            self.split = True
        self.inv_freq, self.rotary_dim, self.interleaved = inv_freq, rotary_dim, pairing == "interleaved"
        if self.interleaved and self.split and self.q_norm is not None and not self.by_units:
            raise ValueError("gqa_attention: per-head Q/K norms with values of another size than the keys rotate in halves only")

    feeds_stream = True

    @functools.cached_property
    def takes_unscaled(self):
        return not self.split and not self.by_units and not self.rows_first and ops.unscaled_rows_supported(self.qkv)

    def forward(self, x, batch, cache, sink=None):
        if self.rows_first:
            pages, history = cache, None
            if cache.parts:
                pages, history = cache.parts[0], cache.parts[1].state
            tables = batch.block_tables[pages.group]
            queries = ops.conv_norm_kv(ops.linear(x, self.qkv), self.taps, history, batch, tables, pages.k_pages, pages.v_pages,
                                       self.heads, self.kv_heads, self.head_dim, self.value_dim, self.q_norm, self.k_norm, self.eps,
                                       write_cache=pages.writes)
            return ops.linear(self._attend(queries, batch, tables, pages, queries.shape[1]), self.out, sink=sink)
        tables = batch.block_tables[cache.group]
        if self.by_units:
            # one unit per head: norms, temperature, rotation and the cache write in one kernel; without a value projection
            # the packed row ends behind the keys and the V pages are the K pages
            qkv = ops.linear(x, self.qkv)
            rotating = self.rotary_dim if self.inv_freq is not None else 0
            ops.norm_rope_units(qkv, batch.positions, batch.seq_of_token, tables, cache.k_pages,
                                None if self.values_are_keys else cache.v_pages, self.heads, self.kv_heads, 1, self.head_dim,
                                self.head_dim, 0 if self.values_are_keys else self.value_dim, batch.error_flag,
                                q_weight=self.q_norm, k_weight=self.k_norm, eps=self.eps, inv_freq=self.inv_freq,
                                rotary_dim=rotating, write_cache=cache.writes, interleaved=self.interleaved,
                                q_temp=self.temperature)
            return ops.linear(self._attend(qkv, batch, tables, cache, qkv.shape[1]), self.out, sink=sink)
        if self.split and self.q_norm is not None:
            # heads with a norm whose values have another size than their keys: the kernel for heads made of units, one
            # unit per head
            qkv = ops.linear(x, self.qkv)
            ops.norm_rope_units(qkv, batch.positions, batch.seq_of_token, tables, cache.k_pages, cache.v_pages, self.heads,
                                self.kv_heads, 1, self.head_dim, self.head_dim, self.value_dim, batch.error_flag,
                                q_weight=self.q_norm, k_weight=self.k_norm, eps=self.eps, inv_freq=self.inv_freq,
                                rotary_dim=self.rotary_dim if self.inv_freq is not None else 0, write_cache=cache.writes)
        elif self.split:
            qkv = ops.linear(x, self.qkv)
            ops.rope_kv_write_split(qkv, self.inv_freq, self.magnitude, batch.positions, batch.seq_of_token, tables,
                                    cache.k_pages, cache.v_pages, self.heads, self.kv_heads, self.head_dim, self.value_dim,
                                    cache.writes, batch.error_flag, self.rotary_dim if self.inv_freq is not None else 0,
                                    self.interleaved)
        else:
            qkv = ops.qkv_projection(x, self.qkv, self.q_norm, self.k_norm, self.inv_freq, batch.positions, batch.seq_of_token,
                                     tables, cache.k_pages, cache.v_pages, self.heads, self.kv_heads, self.head_dim, self.eps,
                                     cache.writes, batch.error_flag, self.rotary_dim, self.interleaved)
        return ops.linear(self._attend(qkv, batch, tables, cache), self.out, sink=sink)

    def _attend(self, queries, batch, tables, pages, q_stride=None):
        return ops.attention(queries, batch, tables, pages.k_pages, pages.v_pages, self.heads, self.kv_heads, self.head_dim,
                             self.scale, self.window, value_dim=self.value_dim, sinks=self.sinks,
                             precise=bool(self.params.get("precise_weights")), q_stride=q_stride, chunk=self.chunk, bias=self.bias,
                             bias_log2=self.bias_log2, keep=self.keep_first, gate=queries if self.gate_column is not None else None,
                             gate_column=self.gate_column or 0)
