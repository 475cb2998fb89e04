"""A plain float64 implementation of the Dozotar decoder, written from the design's equations: one function per
mechanism, token-by-token recurrences, dense score matrices, no cache.  It shares nothing with the engine and serves as
the oracle of the tests.

Notation: T tokens, positions 0 .. T - 1; W x means the stored [out, in] matrix times the vector; a mixer's tensors are
looked up under its prefix.  Every mixer takes what came before the tokens it is given as explicit state (recurrent
state, convolution history), so the same code answers "whole prompt" (state absent) and "continued from a state"."""
import math

import torch

F64 = torch.float64


def rms_divide(x, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def scalar_norm(x, g, eps):
    """The block's norm: one number scales all coordinates."""
    return rms_divide(x, eps) * g


def silu(x):
    return x * torch.sigmoid(x)


def gelu_tanh(x):
    return 0.5 * x * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (x + 0.044715 * x ** 3)))


def causal_convolution(x, taps_w, bias=None, history=None):
    """x [T, C], taps_w [C, taps] (last column: the current token); history [taps - 1, C]: the inputs before x."""
    taps = taps_w.shape[1]
    if history is None:
        history = torch.zeros((taps - 1, x.shape[1]), dtype=F64)
    padded = torch.cat([history, x], dim=0)
    y = torch.zeros_like(x)
    for j in range(taps):
        y = y + padded[j:j + x.shape[0]] * taps_w[:, j]
    if bias is not None:
        y = y + bias
    return y, padded[padded.shape[0] - (taps - 1):]


# ------------------------------------------------------------------------------------------------ chunked attention
def distance_bucket(n, buckets, largest):
    """The first half of the buckets holds one distance each, the second half grows logarithmically up to ``largest``."""
    half = buckets // 2
    if n < half:
        return n
    return min(buckets - 1, half + math.floor(math.log(n / half) / math.log(largest / half) * (buckets - half)))


def chunked_attention(h, weights, prefix, m, eps, history=None, want_probabilities=False):
    """Over the whole sequence (keys have to be at hand); ``history`` only concerns the convolutions."""
    T = h.shape[0]
    H, G, D, DV = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    made = {}
    for role in ("q", "k", "v"):
        made[role], _ = causal_convolution(h @ weights[prefix + role].T, weights[prefix + role + ".conv"],
                                           history=None if history is None else history[role])
    q = (rms_divide(made["q"], eps) * weights[prefix + "q.norm"]).view(T, H, D)
    k = (rms_divide(made["k"], eps) * weights[prefix + "k.norm"]).view(T, G, D)
    v = made["v"].view(T, G, DV)
    table = weights[prefix + "rel"]
    size = (m.get("mask") or {}).get("size")
    bias = torch.zeros((H, T, T), dtype=F64)
    visible = torch.zeros((T, T), dtype=torch.bool)
    for i in range(T):
        for j in range(i + 1):
            visible[i, j] = size is None or i // int(size) == j // int(size)
    by_distance = torch.stack([table[distance_bucket(n, table.shape[0], float(m["bias_max"]))] for n in range(T)])     # [T, H]
    distance = (torch.arange(T)[:, None] - torch.arange(T)[None, :]).clamp(min=0)
    bias = by_distance[distance].permute(2, 0, 1)
    out = torch.zeros((T, H, DV), dtype=F64)
    kept = []
    for head in range(H):
        group = head // (H // G)
        scores = (q[:, head] @ k[:, group].T) * float(m["scale"]) + bias[head]
        p = torch.softmax(scores.masked_fill(~visible, -math.inf), dim=-1)
        kept.append(p)
        out[:, head] = p @ v[:, group]
    y = out.reshape(T, H * DV) @ weights[prefix + "o"].T
    return (y, kept) if want_probabilities else y


# ------------------------------------------------------------------------------------------------ retention
def rotate_heads(x, positions, rot):
    """x [T, heads, dim]: the first rot.dims elements of every head turn, element i with element i + dims / 2."""
    dims = int(rot["dims"])
    frequencies = torch.tensor([float(rot["base"]) ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=F64)
    angle = positions.to(F64)[:, None] * frequencies[None, :]
    c, s = torch.cos(angle)[:, None, :], torch.sin(angle)[:, None, :]
    a, b = x[..., :dims // 2], x[..., dims // 2:dims]
    return torch.cat([a * c - b * s, b * c + a * s, x[..., dims:]], dim=-1)


def decayed_scan(q, k, v, decay, S):
    """q, k [T, dim], v [T, vdim], decay [T]; S [dim, vdim] is advanced token by token, outputs read the new state."""
    out = torch.zeros((q.shape[0], v.shape[1]), dtype=F64)
    for t in range(q.shape[0]):
        S = decay[t] * S + torch.outer(k[t], v[t])
        out[t] = S.T @ q[t]
    return out, S


def retention(h, weights, prefix, m, eps, state=None, first_position=0):
    """state: None or S [heads, dim, vdim]; returns (y, new state)."""
    T = h.shape[0]
    H, D, DV = int(m["heads"]), int(m["dim"]), int(m["vdim"])
    S = state if state is not None else torch.zeros((H, D, DV), dtype=F64)
    q = (h @ weights[prefix + "q"].T).view(T, H, D)
    k = (h @ weights[prefix + "k"].T).view(T, H, D)
    v = (h @ weights[prefix + "v"].T).view(T, H, DV)
    positions = torch.arange(first_position, first_position + T)
    if m.get("rot"):
        q, k = rotate_heads(q, positions, m["rot"]), rotate_heads(k, positions, m["rot"])
    k = k * D ** -0.5
    out, new_S = torch.zeros((T, H, DV), dtype=F64), torch.zeros_like(S)
    for head in range(H):
        decay = torch.full((T,), float(m["decay"][head]), dtype=F64)
        out[:, head], new_S[head] = decayed_scan(q[:, head], k[:, head], v[:, head], decay, S[head])
    y = rms_divide(out, eps).reshape(T, H * DV) * silu(h @ weights[prefix + "g"].T)
    return y @ weights[prefix + "o"].T, new_S


# ------------------------------------------------------------------------------------------------ state-space duality
def ssd(h, weights, prefix, m, eps, state=None):
    """state: None or (S [heads, state, vdim], convolution history [taps - 1, C]); returns (y, new state)."""
    T = h.shape[0]
    H, DV, N, G, parts = int(m["heads"]), int(m["vdim"]), int(m["state"]), int(m["groups"]), int(m["norm_groups"])
    inner = H * DV
    S, history = state if state is not None else (torch.zeros((H, N, DV), dtype=F64), None)
    projected = h @ weights[prefix + "in"].T
    z, mixed, dt = projected[:, :inner], projected[:, inner:2 * inner + 2 * G * N], projected[:, 2 * inner + 2 * G * N:]
    convolved, new_history = causal_convolution(mixed, weights[prefix + "conv"], weights[prefix + "conv.b"], history)
    convolved = silu(convolved)
    x = convolved[:, :inner].view(T, H, DV)
    B = convolved[:, inner:inner + G * N].view(T, G, N)
    C = convolved[:, inner + G * N:].view(T, G, N)
    dt = torch.nn.functional.softplus(dt + weights[prefix + "dt_bias"])
    out, new_S = torch.zeros((T, H, DV), dtype=F64), torch.zeros_like(S)
    for head in range(H):
        group = head // (H // G)
        decay = torch.exp(-torch.exp(weights[prefix + "A_log"][head]) * dt[:, head])
        out[:, head], new_S[head] = decayed_scan(C[:, group], dt[:, head, None] * B[:, group], x[:, head], decay, S[head])
        out[:, head] = out[:, head] + weights[prefix + "D"][head] * x[:, head]
    y = out.reshape(T, inner) * silu(z)
    y = rms_divide(y.view(T, parts, inner // parts), eps).reshape(T, inner) * weights[prefix + "norm"]
    return y @ weights[prefix + "o"].T, (new_S, new_history)


# ------------------------------------------------------------------------------------------------ feed-forwards
def gated_layer(h, weights, prefix, act):
    return (act(h @ weights[prefix + "gate"].T) * (h @ weights[prefix + "up"].T)) @ weights[prefix + "down"].T


def route(z, router):
    """Chosen experts and their weights for one token's router logits z [experts]."""
    experts, top = int(router["experts"]), int(router["top"])
    s = torch.softmax(z, dim=-1)
    allowed = list(range(experts))
    if router.get("groups"):
        count, keep = int(router["groups"]["count"]), int(router["groups"]["keep"])
        size = experts // count
        best = sorted(range(count), key=lambda g: (-float(s[g * size:(g + 1) * size].max()), g))[:keep]
        allowed = [e for e in allowed if e // size in best]
    chosen = sorted(allowed, key=lambda e: (-float(s[e]), e))[:top]
    picked = s[chosen]
    return chosen, picked / (picked.sum() + 1e-20)


def routing_margin(z, router):
    """How far one token's choice is from another one, in units of the router's logits: the gap between the last expert
    chosen and the first one left out, and between the last group kept and the first one dropped."""
    experts, top = int(router["experts"]), int(router["top"])
    gaps, allowed = [], list(range(experts))
    if router.get("groups"):
        count, keep = int(router["groups"]["count"]), int(router["groups"]["keep"])
        size = experts // count
        best = sorted(((float(z[g * size:(g + 1) * size].max()), g) for g in range(count)), reverse=True)
        if keep < count:
            gaps.append(best[keep - 1][0] - best[keep][0])
        allowed = [e for e in allowed if e // size in [g for _, g in best[:keep]]]
    ranked = sorted((float(z[e]) for e in allowed), reverse=True)
    if top < len(ranked):
        gaps.append(ranked[top - 1] - ranked[top])
    return min(gaps) if gaps else math.inf


def routed_feed_forward(h, weights, prefix, mlp):
    z = h @ weights[prefix + "router"].T
    y = torch.zeros_like(h)
    for t in range(h.shape[0]):
        chosen, share = route(z[t], mlp["router"])
        for e, w in zip(chosen, share):
            y[t] = y[t] + w * gated_layer(h[t], weights, f"{prefix}e{e}.", silu)
    if mlp.get("shared"):
        gate = torch.sigmoid(h @ weights[prefix + "shared.sg"].T)
        y = y + gate * gated_layer(h, weights, prefix + "shared.", silu)
    return y


def feed_forward(h, weights, prefix, mlp):
    if mlp["kind"] == "dense":
        return gated_layer(h, weights, prefix, gelu_tanh)
    return routed_feed_forward(h, weights, prefix, mlp)


# ------------------------------------------------------------------------------------------------ the model
def mixer_output(layer, x, weights, prefix, eps, lose_state_at=None):
    """One layer's mixer over the whole sequence.  ``lose_state_at``: recurrent state and convolution history are dropped
    in front of that token (what a fault in the state manager would do)."""
    m = layer["mixer"]
    if layer["type"] == "attention":
        return chunked_attention(x, weights, prefix, m, eps)
    function = retention if layer["type"] == "retention" else ssd
    if lose_state_at is None:
        return function(x, weights, prefix, m, eps)[0]
    first = function(x[:lose_state_at], weights, prefix, m, eps)[0]
    if layer["type"] == "retention":
        return torch.cat([first, retention(x[lose_state_at:], weights, prefix, m, eps, first_position=lose_state_at)[0]], dim=0)
    return torch.cat([first, ssd(x[lose_state_at:], weights, prefix, m, eps)[0]], dim=0)


def forward(config, weights, tokens, lose_state_at=None, streams=None, margins=None):
    """float64 logits [T, vocab] of the whole sequence.  ``margins``: receives each token's smallest routing margin."""
    eps = float(config["norm"]["eps"])
    x = weights["embed"][torch.tensor(list(tokens))]
    for index, layer in enumerate(config["layers"]):
        prefix = f"l{index}."
        x = x + scalar_norm(mixer_output(layer, x, weights, prefix + "mix.", eps, lose_state_at), weights[prefix + "norm1"], eps)
        if layer.get("mlp"):
            if margins is not None and layer["mlp"]["kind"] == "moe":
                z = x @ weights[prefix + "mlp.router"].T
                found = torch.tensor([routing_margin(row, layer["mlp"]["router"]) for row in z])
                margins.append(found if not margins else torch.minimum(margins.pop(), found))
            x = x + scalar_norm(feed_forward(x, weights, prefix + "mlp.", layer["mlp"]), weights[prefix + "norm2"], eps)
        if streams is not None:
            streams.append(x.clone())
    return scalar_norm(x, weights["final.norm"], eps) @ weights["head"].T
