"""A routed feed-forward: many small experts of which each token uses a few, and an optional shared one."""
from __future__ import annotations

import torch

from .. import ops
from ..weights.declare import WIDE, WeightDecl
from .base import FeedForward
from .registry import FEED_FORWARDS


@FEED_FORWARDS.register("routed_experts")
class RoutedExperts(FeedForward):
    """y = sum over the chosen experts e of w_e * expert_e(x)  (+ shared(x)).

    Router: z = W_r x in 32-bit, s = sigmoid(z).  The ``top`` experts with the largest s + correction are chosen (the
    correction, a learned number per expert, only steers the choice; ties go to the lower index); their weights are
    s * ``route_scale``, not renormalised.  An expert is a gated feed-forward without biases:

        g = min(W_gate x, limit),  u = clamp(W_up x, -limit, limit),  expert(x) = W_down (g * sigmoid(alpha * g) * (u + 1))

    and the shared expert, which every token uses with weight 1, has the same form with sizes and a limit of its own.
    With ``activation`` "silu" an expert is the plain gated layer expert(x) = W_down (silu(W_gate x) * (W_up x)), nothing
    clamped (``limit`` and ``alpha`` are then not given).  With ``weight_on`` "input" a routing weight multiplies what goes
    into its expert instead of what comes out, y = sum_e expert_e(w_e * x): the pair's row is scaled as the first product
    reads it, and the experts' outputs are summed as they are.

    ``scores`` "softmax": s = softmax(z) over all experts.  ``groups`` = (count, keep): the experts form ``count`` equal groups
    of neighbours and only those of the ``keep`` best groups can be chosen, a group's score being the largest in it.
    ``renormalise``: the chosen experts' weights are divided by their sum (+ 1e-20).  ``shared_gate``: the shared expert's
    output is multiplied by sigmoid(W_sg x), one number per token; W_sg is one more row of the router's product.

    ``activation`` "squared_relu": experts without a gate, expert(x) = W_down (max(W_up x, 0)^2), the shared one likewise (there are
    no gate tensors).  ``identity``: the router has that many more outputs behind the experts', whose "expert" is the input
    itself; scores, correction, groups and choice run over all outputs.

    Parameters: ``hidden``, ``experts``, ``top``, ``intermediate``, ``limit``, ``route_scale``; ``alpha`` (default
    1.702); ``correction`` (default True: the router has one); ``shared_intermediate`` and ``shared_limit`` (absent: no
    shared expert).  Tensors behind the part's prefix: ``e<i>.gate``, ``e<i>.up`` [intermediate, hidden], ``e<i>.down``
    [hidden, intermediate], ``router`` [experts, hidden], ``correction`` [experts], ``shared.gate`` / ``.up`` /
    ``.down``, ``shared.sg`` [1, hidden].  Router and correction are held in float32 in either path."""

    KNOWN_PARAMS = ("hidden", "experts", "top", "intermediate", "limit", "route_scale", "alpha", "correction",
                    "shared_intermediate", "shared_limit", "activation", "weight_on", "scores", "groups", "renormalise", "shared_gate",
                    "identity")
    ACTIVATIONS = ("clamped_swish", "silu", "squared_relu")

    @classmethod
    def outputs(cls, params) -> int:
        """Outputs of the router: the experts and, behind them, the identities."""
        return int(params["experts"]) + int(params.get("identity") or 0)

    @classmethod
    def check_params(cls, params):
        super().check_params(params)
        outputs = cls.outputs(params)
        if int(params.get("identity") or 0) < 0 or not 0 < int(params["top"]) <= outputs:
            raise ValueError(f"routed_experts: top {params['top']} must lie in 1..the router's outputs ({outputs})")
        activation = params.get("activation", "clamped_swish")
        if activation not in cls.ACTIVATIONS:
            raise ValueError(f"routed_experts: unknown activation {activation!r} (known: {', '.join(cls.ACTIVATIONS)})")
        if activation != "clamped_swish" and (params.get("limit") is not None or params.get("alpha") is not None or params.get("shared_limit") is not None):
            raise ValueError(f"routed_experts: the {activation} activation takes no limit or alpha")
        if activation == "clamped_swish" and params.get("limit") is None:
            raise ValueError("routed_experts: the clamped activation needs its limit")
        if params.get("weight_on", "output") not in ("output", "input"):
            raise ValueError(f"routed_experts: weight_on is 'output' or 'input', not {params.get('weight_on')!r}")
        if params.get("identity") and params.get("weight_on") == "input":
            raise ValueError("routed_experts: identity outputs take their weight behind them")
        if params.get("scores", "sigmoid") not in ("sigmoid", "softmax"):
            raise ValueError(f"routed_experts: scores are 'sigmoid' or 'softmax', not {params.get('scores')!r}")
        if params.get("groups"):
            count, keep = (int(value) for value in params["groups"])
            if count <= 0 or outputs % count or not 0 < keep <= count:
                raise ValueError(f"routed_experts: {outputs} outputs do not form {count} equal groups of which {keep} are kept")
            if int(params["top"]) > keep * (outputs // count):
                raise ValueError(f"routed_experts: {keep} groups hold fewer than top {params['top']} experts")
        if params.get("shared_gate") and not params.get("shared_intermediate"):
            raise ValueError("routed_experts: a gate on the shared expert needs a shared expert")

    @classmethod
    def declare_weights(cls, params):
        hidden, inter = int(params["hidden"]), int(params["intermediate"])
        gated = params.get("activation") != "squared_relu"
        wanted = {}
        for e in range(int(params["experts"])):
            if gated:
                wanted[f"e{e}.gate"] = WeightDecl((inter, hidden))
            wanted[f"e{e}.up"] = WeightDecl((inter, hidden))
            wanted[f"e{e}.down"] = WeightDecl((hidden, inter))
        wanted["router"] = WeightDecl((cls.outputs(params), hidden), WIDE)
        if params.get("correction", True):
            wanted["correction"] = WeightDecl((cls.outputs(params),), WIDE)
        if params.get("shared_intermediate"):
            shared = int(params["shared_intermediate"])
            if gated:
                wanted["shared.gate"] = WeightDecl((shared, hidden))
            wanted["shared.up"] = WeightDecl((shared, hidden))
            wanted["shared.down"] = WeightDecl((hidden, shared))
            if params.get("shared_gate"):
                wanted["shared.sg"] = WeightDecl((1, hidden), WIDE)
        return wanted

    def __init__(self, params, weights, runtime):
        super().__init__(params, weights, runtime)
        self.experts, self.top = int(params["experts"]), int(params["top"])
        self.outputs_count, self.identity = self.outputs(params), int(params.get("identity") or 0)
        self.squared_relu = params.get("activation") == "squared_relu"
        if self.squared_relu:
            self.limit, self.alpha, self.gate = float("inf"), 1.0, None
        elif params.get("activation", "clamped_swish") == "silu":
            # the gated epilogues compute min(g, limit) * sigmoid(alpha * min(g, limit)) * (clamp(u) + shift)
            self.limit, self.alpha, self.gate = float("inf"), 1.0, (float("inf"), 1.0, 0.0)
        else:
            self.limit, self.alpha = float(params["limit"]), float(params.get("alpha", 1.702))
            self.gate = (self.limit, self.alpha)
        self.route_scale = float(params.get("route_scale", 1.0))
        self.weight_on_input = params.get("weight_on", "output") == "input"
        # one tensor per kind of matrix: [E, 2 I, H] with an expert's gate rows in front of its up rows (without gates [E, I, H]),
        # and [E, H, I]
        self.gate_up = torch.stack([weights[f"e{e}.up"] if self.squared_relu else torch.cat([weights[f"e{e}.gate"], weights[f"e{e}.up"]], dim=0)
                                    for e in range(self.experts)]).contiguous()
        self.down = torch.stack([weights[f"e{e}.down"] for e in range(self.experts)]).contiguous()
        self.router = weights["router"].to(torch.float32).contiguous()
        self.rule = {"scores": params.get("scores", "sigmoid"), "groups": tuple(params["groups"]) if params.get("groups") else None,
                     "renormalise": bool(params.get("renormalise")), "gate": bool(params.get("shared_gate"))}
        if self.rule["gate"]:
            self.router = torch.cat([self.router, weights["shared.sg"].to(torch.float32)], dim=0).contiguous()
        # A router whose weights are bfloat16 numbers (what a bfloat16 checkpoint holds) can be multiplied on the tensor
        # cores without leaving 32-bit arithmetic: products of two bfloat16 numbers are exact in 32-bit, and the sums
        # are 32-bit.  Any other router, and the 32-bit path, use the FMA kernel that makes the choice as well.
        narrow = self.router.to(torch.bfloat16)
        if narrow.shape[0] % 8:      # the library's products want rows of whole 16-byte pieces; the padding is never looked at
            narrow = torch.cat([narrow, narrow.new_zeros((8 - narrow.shape[0] % 8, narrow.shape[1]))], dim=0)
        self.router_narrow = narrow.contiguous() if runtime.dtype == torch.bfloat16 and bool((narrow[:self.router.shape[0]].float() == self.router).all()) else None
        self.correction = weights["correction"].to(torch.float32).contiguous() if params.get("correction", True) else None
        self.shared_gate_up = self.shared_down = None
        self.shared_group = 0
        if params.get("shared_intermediate") and self.squared_relu:
            self.shared_gate_up = weights["shared.up"].contiguous()
            self.shared_down = weights["shared.down"].contiguous()
        elif params.get("shared_intermediate"):
            gate, up = weights["shared.gate"], weights["shared.up"]
            # a plain silu layer in bfloat16: rows interleaved so that the product kernel for few rows applies the gate itself
            if params.get("activation") == "silu" and gate.dtype == torch.bfloat16 and gate.shape[0] % ops.GATE_UP_GROUP == 0:
                self.shared_group = ops.GATE_UP_GROUP
            self.shared_gate_up = ops.interleave_gate_up(gate, up) if self.shared_group else torch.cat([gate, up], dim=0).contiguous()
            self.shared_down = weights["shared.down"].contiguous()
            self.shared_limit = float(params.get("shared_limit", self.limit))

        # bfloat16 steps of more than a few tokens sort their (token, expert) pairs by expert and run one tiled product
        # over all experts; the 32-bit path and steps of few tokens multiply pair by pair, reading each pair's matrices
        self.grouped = (runtime.dtype == torch.bfloat16 and ops.moe_grouped_supported(self.gate_up, not self.squared_relu)
                        and ops.moe_grouped_supported(self.down, False) and self.down.shape[1] % 4 == 0
                        and self.gate_up.shape[2] % 64 == 0 and self.down.shape[2] % 64 == 0)

    GROUPED_FROM = 16     # tokens from which pairs are sorted and multiplied tile by tile

    def forward(self, x):
        tokens = x.shape[0]
        if self.router_narrow is not None:
            logits = ops.linear_wide(x, self.router_narrow)
            chosen, weights, *gate = ops.moe_select(logits, self.correction, self.top, self.route_scale, experts=self.outputs_count, **self.rule)
        else:
            chosen, weights, *gate = ops.moe_route(x, self.router, self.correction, self.top, self.route_scale, **self.rule)
        shared_gate = gate[0] if gate else None
        shared = None
        if self.shared_gate_up is not None and self.squared_relu:
            shared = ops.linear(ops.relu_squared(ops.linear(x, self.shared_gate_up)), self.shared_down)
        elif self.shared_gate_up is not None and self.params.get("activation") == "silu":
            shared = ops.linear(ops.gate_up_silu(x, self.shared_gate_up, self.shared_group), self.shared_down)
        elif self.shared_gate_up is not None:
            shared = ops.linear(ops.clamped_glu(ops.linear(x, self.shared_gate_up), self.shared_limit, self.alpha),
                                self.shared_down)
        on_input = weights.view(-1) if self.weight_on_input else None
        if self.weight_on_input:
            weights = self._ones(weights)       # the weights act on the way in; on the way out the outputs are summed
        if self.grouped and tokens >= self.GROUPED_FROM:
            plan = ops.moe_plan(chosen, self.experts)
            hidden = ops.moe_grouped(x, self.gate_up, plan, gather_div=self.top, gated=self.gate, pair_scale=on_input,
                                     squared_relu=self.squared_relu)
            down = ops.moe_grouped(hidden, self.down, plan)
            return ops.moe_combine_rows(down, plan, weights, shared, self.runtime.dtype, shared_gate, own=x if self.identity else None)
        pairs = tokens * self.top
        index = chosen.view(-1)
        hidden = ops.indexed_linear(x, self.gate_up, index, pairs, in_div=self.top, gated=self.gate, in_scale=on_input,
                                    squared_relu=self.squared_relu)
        down = ops.indexed_linear(hidden, self.down, index, pairs, out_dtype=torch.float32)
        return ops.moe_combine(down, weights, shared, self.runtime.dtype, shared_gate, own=x if self.identity else None, chosen=chosen,
                               experts=self.experts)

    def _ones(self, like):
        """Unit weights of ``like``'s shape (kept: a step's shapes repeat, and a captured step must not allocate anew)."""
        kept = getattr(self, "_unit_weights", None)
        if kept is None or kept.numel() < like.numel():
            kept = self._unit_weights = torch.ones(max(like.numel(), 4096), dtype=torch.float32, device=like.device)
        return kept[:like.numel()].view(like.shape)
