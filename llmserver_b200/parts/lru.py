"""The recurrent block around a real-gated linear recurrent unit: one number of state per channel, decayed and fed by gates
that come from each token."""
from __future__ import annotations

import torch

from .. import ops
from ..cache.manager import StateNeed
from ..weights.declare import WIDE, WeightDecl
from .base import Mixer
from .registry import MIXERS


@MIXERS.register("gated_linear_recurrent_unit")
class GatedLinearRecurrentUnit(Mixer):
    """Two branches of ``width`` channels, the state S in R^width starting at zero for every request (the recurrent block of De et
    al., "Griffin: Mixing Gated Linear Recurrences with Local Attention for Efficient Language Models"):

        y = gelu_tanh(W_y x + b_y);   u = conv(W_x x + b_x) + b_c          a short causal convolution per channel, no activation
        r = sigmoid(R u + b_r),  i = sigmoid(I u + b_i)                    R, I: block-diagonal, ``blocks`` square matrices each
        log a = -rate * r * softplus(lam);   S_t = a S_(t-1) + sqrt(1 - a^2) i u_t
        out = W_o (S * y)

    Per request the mixer keeps the state, float32 [width], and the last ``conv`` - 1 inputs of the convolution (with their bias;
    zeros in front of a sequence), float32 [conv - 1, width].  The gates (from the 32-bit sums of their products on), decays, the
    recurrence and the product with y are 32-bit in either path; the projections and the convolution's result are in the
    activation type.  Parameters: ``hidden``, ``width``, ``blocks``, ``conv`` (taps), ``rate`` (default 8); ``names``: pairs (role,
    tensor name behind the prefix) for y, y_bias, x, x_bias, conv, conv_bias, r, r_bias, i, i_bias, lam, o."""

    KNOWN_PARAMS = ("hidden", "width", "blocks", "conv", "rate", "names")
    NAMES = {"y": "y", "y_bias": "y.b", "x": "x", "x_bias": "x.b", "conv": "conv", "conv_bias": "conv.b", "r": "ra", "r_bias": "ra.b",
             "i": "ri", "i_bias": "ri.b", "lam": "lam", "o": "o"}
    CONV_UNIT = 256      # channels a block of the convolution kernel takes
    ALIGN = 8            # both branches begin at whole 16-byte pieces of the packed projection

    @classmethod
    def names(cls, params) -> dict:
        given = dict(params.get("names") or ())
        unknown = sorted(set(given) - set(cls.NAMES))
        if unknown:
            raise ValueError(f"gated_linear_recurrent_unit has no tensor in the role(s) {', '.join(unknown)}")
        return {**cls.NAMES, **given}

    @classmethod
    def check_params(cls, params):
        super().check_params(params)
        if int(params["blocks"]) < 1 or int(params["width"]) % int(params["blocks"]):
            raise ValueError(f"gated_linear_recurrent_unit: {params['width']} channels do not divide into {params['blocks']} equal parts")
        if int(params["conv"]) < 1:
            raise ValueError("gated_linear_recurrent_unit: the convolution needs at least one tap")

    @classmethod
    def declare_weights(cls, params):
        hidden, width, blocks = int(params["hidden"]), int(params["width"]), int(params["blocks"])
        size = width // blocks
        name = cls.names(params)
        return {name["y"]: WeightDecl((width, hidden)), name["y_bias"]: WeightDecl((width,), WIDE),
                name["x"]: WeightDecl((width, hidden)), name["x_bias"]: WeightDecl((width,), WIDE),
                name["conv"]: WeightDecl((width, int(params["conv"])), WIDE), name["conv_bias"]: WeightDecl((width,), WIDE),
                name["r"]: WeightDecl((blocks, size, size)), name["r_bias"]: WeightDecl((blocks, size), WIDE),
                name["i"]: WeightDecl((blocks, size, size)), name["i_bias"]: WeightDecl((blocks, size), WIDE),
                name["lam"]: WeightDecl((width,), WIDE), name["o"]: WeightDecl((hidden, width))}

    @classmethod
    def cache_need(cls, params):
        width = int(params["width"])
        return (StateNeed((width,), "float32"), StateNeed((max(int(params["conv"]) - 1, 1), width), "float32"))

    def __init__(self, params, weights, runtime):
        super().__init__(params, weights, runtime)
        self.width = int(params["width"])
        name = self.names(params)
        wide = {role: weights[name[role]].to(torch.float32).contiguous() for role in ("y_bias", "x_bias", "conv", "conv_bias")}
        self.y_bias, self.x_bias, self.taps, self.conv_bias = wide["y_bias"], wide["x_bias"], wide["conv"], wide["conv_bias"]
        rows, ragged = [weights[name["y"]], weights[name["x"]]], -self.width % self.ALIGN
        if ragged:
            fill = torch.zeros((ragged, rows[0].shape[1]), dtype=rows[0].dtype, device=rows[0].device)
            rows = [rows[0], fill, rows[1], fill]
        self.x_column = self.width + ragged
        self.into = torch.cat(rows, dim=0).contiguous()
        # a block's recurrence gates, then its input gates
        self.gates = torch.cat([weights[name["r"]], weights[name["i"]]], dim=1).contiguous()
        self.gate_bias = torch.cat([weights[name["r_bias"]].to(torch.float32), weights[name["i_bias"]].to(torch.float32)], dim=1).contiguous()
        lam = weights[name["lam"]].to(torch.float64)
        self.rate = (-float(params.get("rate", 8.0)) * torch.nn.functional.softplus(lam, threshold=100.0)).to(torch.float32).contiguous()
        self.out = weights[name["o"]].contiguous()

    def forward(self, x, batch, cache):
        state, history = cache.parts[0].state, cache.parts[1].state
        proj = ops.linear(x, self.into)
        u = ops.short_conv_units(proj, self.x_column, self.taps, history, batch, 0, 0, 0, -(-self.width // self.CONV_UNIT), self.CONV_UNIT,
                                 0.0, 1.0, bias=self.conv_bias, channels=self.width, in_bias=self.x_bias, silu=False, out_dtype=self.runtime.dtype)
        mixed = ops.gated_scan(ops.unit_linear_wide(u, self.gates), u, self.gate_bias, self.rate, proj, 0, self.y_bias, state, batch)
        return ops.linear(mixed, self.out)
