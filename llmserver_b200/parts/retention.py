"""Linear attention with one decay per head: retention, whose decays are constants of the heads, and the state-space form,
whose decay comes from each token."""
from __future__ import annotations

import torch

from .. import ops
from ..cache.manager import StateNeed
from ..weights.declare import NORM, WIDE, WeightDecl
from .base import Mixer
from .registry import MIXERS


def _names(cls, params) -> dict:
    given = dict(params.get("names") or ())
    unknown = sorted(set(given) - set(cls.NAMES))
    if unknown:
        raise ValueError(f"{cls.KIND} has no tensor in the role(s) {', '.join(unknown)}")
    return {**cls.NAMES, **given}


@MIXERS.register("retention")
class Retention(Mixer):
    """Per head, with S in R^(dim x value_dim) starting at zero for every request (the recurrence of Sun et al., "Retentive
    Network: A Successor to Transformer for Large Language Models"):

        q = R_p W_q x,  k = R_p W_k x * dim^(-1/2),  v = W_v x          R_p: the rotation the layer's position encoding gives
        S_t = decay_h S_(t-1) + k_t v_t^T,   o_t = S_t^T q_t
        y = W_o (concat_h(o_h / rms(o_h)) * silu(W_g x))

    The state is float32 [heads, dim, value_dim] in the request's state slot; rotation, recurrence and head norm are 32-bit
    in either path, the projections run in the activation type.  The position encoding (optional) rotates the first
    ``rotary_dim`` elements of a head, paired as halves.  Parameters: ``hidden``, ``heads``, ``dim``, ``value_dim``, ``decay``
    (one number per head), ``eps``; ``names``: pairs (role, tensor name behind the prefix) for q, k, v, g, o."""

    KIND = "retention"
    KNOWN_PARAMS = ("hidden", "heads", "dim", "value_dim", "decay", "eps", "names")
    NAMES = {"q": "q", "k": "k", "v": "v", "g": "g", "o": "o"}

    @classmethod
    def check_params(cls, params):
        super().check_params(params)
        if len(params["decay"]) != int(params["heads"]):
            raise ValueError(f"retention: {len(params['decay'])} decays for {params['heads']} heads")

    @classmethod
    def declare_weights(cls, params):
        hidden, heads = int(params["hidden"]), int(params["heads"])
        keys, values = heads * int(params["dim"]), heads * int(params["value_dim"])
        name = _names(cls, params)
        return {name["q"]: WeightDecl((keys, hidden)), name["k"]: WeightDecl((keys, hidden)), name["v"]: WeightDecl((values, hidden)),
                name["g"]: WeightDecl((values, hidden)), name["o"]: WeightDecl((hidden, values))}

    @classmethod
    def cache_need(cls, params):
        return StateNeed((int(params["heads"]), int(params["dim"]), int(params["value_dim"])), "float32")

    def __init__(self, params, weights, runtime):
        super().__init__(params, weights, runtime)
        self.heads, self.dim, self.value_dim = int(params["heads"]), int(params["dim"]), int(params["value_dim"])
        self.eps = float(params["eps"])
        if not ops.decay_recurrence_supported(self.dim, self.value_dim):
            raise ValueError(f"retention: no kernel for heads of {self.dim} key and {self.value_dim} value channels")
        name = _names(type(self), params)
        self.fused = torch.cat([weights[name[role]] for role in ("q", "k", "v", "g")], dim=0).contiguous()
        keys, values = self.heads * self.dim, self.heads * self.value_dim
        self.columns = (0, keys, 2 * keys, 2 * keys + values)
        self.decay = torch.tensor([float(value) for value in params["decay"]], dtype=torch.float32, device=runtime.device)
        self.out = weights[name["o"]].contiguous()
        self.inv_freq = None

    def attach(self, position):
        if position is None:
            return
        inv_freq = getattr(position, "inv_freq", None)
        if inv_freq is None or 2 * inv_freq.numel() > self.dim:
            raise ValueError(f"retention rotates up to {self.dim} elements of a head by inverse frequencies, which "
                             f"{type(position).__name__} does not give")
        if getattr(position, "pairing", "halves") != "halves" or float(getattr(position, "attention_factor", 1.0)) != 1.0:
            raise ValueError("retention pairs rotated elements as halves and does not scale them")
        self.inv_freq = inv_freq

    def forward(self, x, batch, cache):
        proj = ops.linear(x, self.fused)
        mixed = ops.retention_recurrent(proj, *self.columns, self.decay, self.inv_freq, cache.state, batch, self.heads, self.dim,
                                        self.value_dim, self.dim ** -0.5, self.eps)
        return ops.linear(mixed, self.out)


@MIXERS.register("state_space_duality")
class StateSpaceDuality(Mixer):
    """Per head, with S in R^(state x value_dim) starting at zero for every request (the recurrence of Dao and Gu,
    "Transformers are SSMs: Generalized Models and Efficient Algorithms Through Structured State Space Duality"):

        [z | x | B | C | dt] = W_in u                  z, x: heads * value_dim rows; B, C: groups * state; dt: heads
        x, B, C <- silu(conv(x, B, C) + bias)           a short causal convolution per channel
        dt <- softplus(dt + dt_bias)
        S_t = exp(-exp(A) dt) S_(t-1) + dt B_t x_t^T,   y_t = S_t^T C_t + D x_t
        out = W_o (groupnorm(y * silu(z)) * norm)        root mean squares over ``norm_groups`` equal parts

    Head h reads B and C of group h // (heads / groups).  Per request the mixer keeps the state, float32 [heads, state,
    value_dim], and the last ``conv`` - 1 inputs of the convolution, float32 [conv - 1, channels].  dt from the 32-bit sums
    of its projection on, decays, recurrence and norm are 32-bit in either path.  Parameters: ``hidden``, ``heads``,
    ``value_dim``, ``state``, ``groups``, ``conv`` (taps), ``norm_groups``, ``eps``; ``names``: pairs (role, tensor name behind
    the prefix) for in, conv, conv_bias, dt_bias, A, D, norm, o."""

    KIND = "state_space_duality"
    KNOWN_PARAMS = ("hidden", "heads", "value_dim", "state", "groups", "conv", "norm_groups", "eps", "names")
    NAMES = {"in": "in", "conv": "conv", "conv_bias": "conv.b", "dt_bias": "dt_bias", "A": "A_log", "D": "D", "norm": "norm", "o": "o"}

    @classmethod
    def sizes(cls, params):
        """(heads, value_dim, state, groups, inner, channels of the convolution)"""
        heads, value_dim, state, groups = (int(params[key]) for key in ("heads", "value_dim", "state", "groups"))
        inner = heads * value_dim
        return heads, value_dim, state, groups, inner, inner + 2 * groups * state

    @classmethod
    def check_params(cls, params):
        super().check_params(params)
        heads, _, _, groups, inner, _ = cls.sizes(params)
        if heads % groups:
            raise ValueError(f"state_space_duality: {heads} heads are no multiple of {groups} groups")
        if inner % int(params["norm_groups"]):
            raise ValueError(f"state_space_duality: {inner} channels do not divide into {params['norm_groups']} equal parts")
        if int(params["conv"]) < 1:
            raise ValueError("state_space_duality: the convolution needs at least one tap")

    @classmethod
    def declare_weights(cls, params):
        hidden = int(params["hidden"])
        heads, _, _, _, inner, channels = cls.sizes(params)
        name = _names(cls, params)
        return {name["in"]: WeightDecl((inner + channels + heads, hidden)), name["conv"]: WeightDecl((channels, int(params["conv"])), WIDE),
                name["conv_bias"]: WeightDecl((channels,), WIDE), name["dt_bias"]: WeightDecl((heads,), WIDE),
                name["A"]: WeightDecl((heads,), WIDE), name["D"]: WeightDecl((heads,), WIDE), name["norm"]: WeightDecl((inner,), NORM),
                name["o"]: WeightDecl((hidden, inner))}

    @classmethod
    def cache_need(cls, params):
        heads, value_dim, state, _, _, channels = cls.sizes(params)
        return (StateNeed((heads, state, value_dim), "float32"), StateNeed((max(int(params["conv"]) - 1, 1), channels), "float32"))

    CONV_UNIT = 256      # channels a block of the convolution kernel takes

    def __init__(self, params, weights, runtime):
        super().__init__(params, weights, runtime)
        self.heads, self.value_dim, self.state, self.groups, self.inner, self.channels = self.sizes(params)
        self.norm_groups, self.eps = int(params["norm_groups"]), float(params["eps"])
        if not ops.decay_recurrence_supported(self.state, self.value_dim):
            raise ValueError(f"state_space_duality: no kernel for a state of {self.state} by {self.value_dim} channels")
        name = _names(type(self), params)
        into = weights[name["in"]]
        self.into = into[:self.inner + self.channels].contiguous()      # z | x | B | C
        self.steps = into[self.inner + self.channels:].contiguous()     # dt, whose sums stay 32-bit
        self.taps = weights[name["conv"]].to(torch.float32).contiguous()
        self.conv_bias = weights[name["conv_bias"]].to(torch.float32).contiguous()
        self.dt_bias, self.a_log, self.skip = (weights[name[role]].to(torch.float32).contiguous() for role in ("dt_bias", "A", "D"))
        self.norm = weights[name["norm"]].contiguous()
        self.out = weights[name["o"]].contiguous()

    def forward(self, x, batch, cache):
        state, history = cache.parts[0].state, cache.parts[1].state
        proj = ops.linear(x, self.into)
        steps = ops.linear_wide(x, self.steps)      # 32-bit sums: what becomes a decay or a step size is never rounded to 16 bits
        pre = ops.short_conv_units(proj, self.inner, self.taps, history, batch, 0, 0, 0, -(-self.channels // self.CONV_UNIT),
                                   self.CONV_UNIT, 0.0, 1.0, bias=self.conv_bias, channels=self.channels)
        b_column = self.inner
        mixed = ops.ssd_recurrent(proj, 0, pre, 0, b_column, b_column + self.groups * self.state, steps, self.a_log, self.dt_bias,
                                  self.skip, state, batch, self.heads, self.groups, self.state, self.value_dim)
        return ops.linear(ops.grouped_rmsnorm(mixed, self.norm, self.norm_groups, self.eps, self.runtime.dtype), self.out)
