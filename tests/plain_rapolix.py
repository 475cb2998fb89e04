"""A plain float64 implementation of the Rapolix decoder, written from the design's equations: one function per mechanism,
token-by-token recurrence, dense score matrices, no cache.  It shares nothing with the engine and serves as the oracle of
the tests.

Notation: T tokens, positions 0 .. T - 1; W x means the stored [out, in] matrix times the vector; a mixer's tensors are
looked up under its prefix.  The recurrent branch takes what came before the tokens it is given as explicit state
(recurrent state, convolution history), so the same code answers "whole prompt" (state absent) and "continued from a state"."""
import math

import torch

F64 = torch.float64


def rms_norm(x, w, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps) * w


def layer_norm(x, w, eps):
    centred = x - x.mean(dim=-1, keepdim=True)
    return centred / torch.sqrt((centred * centred).mean(dim=-1, keepdim=True) + eps) * w


def gelu_tanh(x):
    return 0.5 * x * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (x + 0.044715 * x ** 3)))


def sinusoids(positions, width):
    """[T, width]: sines of p * 10000^(-2i/width) in the even entries, cosines in the odd ones."""
    out = torch.zeros((len(positions), width), dtype=F64)
    for e in range(width):
        i = e // 2
        angle = positions.to(F64) * 10000.0 ** (-2.0 * i / width)
        out[:, e] = torch.sin(angle) if e % 2 == 0 else torch.cos(angle)
    return out


# ------------------------------------------------------------------------------------------------ several streams
def read_streams(x, weights, prefix):
    """x [S, T, width]: what a sub-layer reads before its norm."""
    return torch.einsum("s,stw->tw", weights[prefix + "in"], x)


def write_streams(x, y, weights, prefix):
    """Every stream anew from the old ones and the sub-layer's output y [T, width]."""
    return torch.einsum("ab,atw->btw", weights[prefix + "mix"], x) + weights[prefix + "out"][:, None, None] * y


# ------------------------------------------------------------------------------------------------ attention
def visible(i, j, mask):
    if j > i:
        return False
    if not mask or not mask.get("size"):
        return True
    return i - j < int(mask["size"]) or j < int(mask.get("keep_first") or 0)


def windowed_attention(h, weights, prefix, m, want_probabilities=False):
    T = h.shape[0]
    H, G, D, DV = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    q = (h @ weights[prefix + "q"].T).view(T, H, D)
    k = (h @ weights[prefix + "k"].T).view(T, G, D)
    v = (h @ weights[prefix + "v"].T).view(T, G, DV)
    seen = torch.tensor([[visible(i, j, m.get("mask")) for j in range(T)] for i in range(T)])
    out, kept = torch.zeros((T, H, DV), dtype=F64), []
    for head in range(H):
        group = head // (H // G)
        scores = (q[:, head] @ k[:, group].T) * float(m["scale"])
        p = torch.softmax(scores.masked_fill(~seen, -math.inf), dim=-1)
        kept.append(p)
        out[:, head] = p @ v[:, group]
    y = (out.reshape(T, H * DV) * torch.sigmoid(h @ weights[prefix + "g"].T)) @ weights[prefix + "o"].T
    return (y, kept) if want_probabilities else y


# ------------------------------------------------------------------------------------------------ gated linear recurrent unit
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


def block_product(u, matrices, biases):
    """u [T, blocks * n], matrices [blocks, n, n], biases [blocks, n]: every block has a matrix of its own."""
    blocks, n, _ = matrices.shape
    return (torch.einsum("bij,tbj->tbi", matrices, u.view(-1, blocks, n)) + biases).reshape(u.shape)


def gated_scan(u, r, i, lam, S):
    """u, r, i [T, C], lam [C]; S [C] is advanced token by token.  Returns every token's state and the last one."""
    rate = -8.0 * torch.log1p(torch.exp(-lam.abs())) - 8.0 * lam.clamp(min=0)      # -8 softplus(lam)
    states = torch.zeros_like(u)
    for t in range(u.shape[0]):
        a = torch.exp(rate * r[t])
        S = a * S + torch.sqrt(1.0 - a * a) * i[t] * u[t]
        states[t] = S
    return states, S


def recurrent_block(h, weights, prefix, m, state=None):
    """state: None or (S [width], convolution history [taps - 1, width]); returns (y, new state)."""
    S, history = state if state is not None else (torch.zeros(int(m["width"]), dtype=F64), None)
    y = gelu_tanh(h @ weights[prefix + "y"].T + weights[prefix + "y.b"])
    u, new_history = causal_convolution(h @ weights[prefix + "x"].T + weights[prefix + "x.b"], weights[prefix + "conv"],
                                        weights[prefix + "conv.b"], history)
    r = torch.sigmoid(block_product(u, weights[prefix + "ra"], weights[prefix + "ra.b"]))
    i = torch.sigmoid(block_product(u, weights[prefix + "ri"], weights[prefix + "ri.b"]))
    states, S = gated_scan(u, r, i, weights[prefix + "lam"], S)
    return (states * y) @ weights[prefix + "o"].T, (S, new_history)


def parallel(h, weights, prefix, m, eps, lose_state_at=None):
    """Half the sum of both branches' normalised outputs.  ``lose_state_at``: the recurrent branch drops its state in front
    of that token (what a fault in the state manager would do)."""
    left = windowed_attention(h, weights, prefix + "left.", m["left"])
    if lose_state_at is None:
        right = recurrent_block(h, weights, prefix + "right.", m["right"])[0]
    else:
        right = torch.cat([recurrent_block(piece, weights, prefix + "right.", m["right"])[0]
                           for piece in (h[:lose_state_at], h[lose_state_at:])], dim=0)
    return 0.5 * (rms_norm(left, weights[prefix + "left.out"], eps) + rms_norm(right, weights[prefix + "right.out"], eps))


# ------------------------------------------------------------------------------------------------ feed-forwards
def biased(h, weights, name):
    return h @ weights[name].T + weights[name + ".b"]


def dense_feed_forward(h, weights, prefix):
    gate = biased(h, weights, prefix + "gate")
    return biased(gate * torch.sigmoid(gate) * biased(h, weights, prefix + "up"), weights, prefix + "down")


def squared_relu_layer(h, weights, prefix):
    return (h @ weights[prefix + "up"].T).clamp(min=0) ** 2 @ weights[prefix + "down"].T


def route(z, correction, router):
    """Chosen outputs (experts, then identities) and their weights for one token's router logits z."""
    total, top = z.shape[0], int(router["top"])
    s = torch.softmax(z, dim=-1)
    choice = s + correction
    allowed = list(range(total))
    if router.get("groups"):
        count, keep = int(router["groups"]["count"]), int(router["groups"]["keep"])
        size = total // count
        best = sorted(range(count), key=lambda g: (-float(choice[g * size:(g + 1) * size].max()), g))[:keep]
        allowed = [e for e in allowed if e // size in best]
    chosen = sorted(allowed, key=lambda e: (-float(choice[e]), e))[:top]
    picked = s[chosen]
    return chosen, picked / (picked.sum() + 1e-20)


def routing_margin(z, correction, router, matters=0.0):
    """How far one token's choice is from another one, in choice scores: the gap between the last output chosen and the
    first one left out, and between the last group kept and the first one dropped.  Calls between outputs (or groups whose
    outputs) have less than the share ``matters`` of the chosen scores are left out: either way changes little."""
    total, top = z.shape[0], int(router["top"])
    s = torch.softmax(z, dim=-1)
    choice = s + correction
    chosen, _ = route(z, correction, router)
    weight = float(s[chosen].sum())
    gaps, allowed = [], list(range(total))
    if router.get("groups"):
        count, keep = int(router["groups"]["count"]), int(router["groups"]["keep"])
        size = total // count
        best = sorted(((float(choice[g * size:(g + 1) * size].max()), g) for g in range(count)), reverse=True)
        if keep < count:
            at_stake = max(float(s[g * size:(g + 1) * size].max()) for _, g in best[keep - 1:keep + 1])
            if at_stake >= matters * weight:
                gaps.append(best[keep - 1][0] - best[keep][0])
        allowed = [e for e in allowed if e // size in [g for _, g in best[:keep]]]
    ranked = sorted(((float(choice[e]), float(s[e])) for e in allowed), reverse=True)
    if top < len(ranked) and max(ranked[top - 1][1], ranked[top][1]) >= matters * weight:
        gaps.append(ranked[top - 1][0] - ranked[top][0])
    return min(gaps) if gaps else math.inf


def routed_feed_forward(h, weights, prefix, mlp):
    experts = int(mlp["router"]["experts"])
    z = h @ weights[prefix + "router"].T
    y = torch.zeros_like(h)
    for t in range(h.shape[0]):
        chosen, share = route(z[t], weights[prefix + "correction"], mlp["router"])
        for e, w in zip(chosen, share):
            y[t] = y[t] + w * (h[t] if e >= experts else squared_relu_layer(h[t], weights, f"{prefix}e{e}."))
    if mlp.get("shared"):
        y = y + squared_relu_layer(h, weights, prefix + "shared.")
    return y


def feed_forward(h, weights, prefix, mlp):
    return dense_feed_forward(h, weights, prefix) if mlp["kind"] == "dense" else routed_feed_forward(h, weights, prefix, mlp)


# ------------------------------------------------------------------------------------------------ the model
def forward(config, weights, tokens, lose_state_at=None, streams=None, margins=None):
    """float64 logits [T, vocab] of the whole sequence.  ``streams``: receives the sum of the streams behind every layer;
    ``margins``: receives each token's smallest routing margin that matters."""
    eps = float(config["norm"]["eps"])
    embedded = weights["embed"][torch.tensor(list(tokens))] + sinusoids(torch.arange(len(tokens)), int(config["width"]))
    x = embedded.expand(int(config["streams"]), -1, -1).clone()
    for index, layer in enumerate(config["layers"]):
        prefix = f"l{index}."
        h = layer_norm(read_streams(x, weights, prefix + "hc1."), weights[prefix + "norm1"], eps)
        x = write_streams(x, parallel(h, weights, prefix + "mix.", layer["mixer"], eps, lose_state_at), weights, prefix + "hc1.")
        if layer.get("mlp"):
            h = layer_norm(read_streams(x, weights, prefix + "hc2."), weights[prefix + "norm2"], eps)
            if margins is not None and layer["mlp"]["kind"] == "moe":
                z = h @ weights[prefix + "mlp.router"].T
                found = torch.tensor([routing_margin(row, weights[prefix + "mlp.correction"], layer["mlp"]["router"], matters=0.04) for row in z])
                margins.append(found if not margins else torch.minimum(margins.pop(), found))
            x = write_streams(x, feed_forward(h, weights, prefix + "mlp.", layer["mlp"]), weights, prefix + "hc2.")
        if streams is not None:
            streams.append(x.sum(dim=0))
    logits = layer_norm(x.sum(dim=0), weights["final.norm"], eps) @ weights["head"].T
    cap = config.get("logit_softcap")
    return cap * torch.tanh(logits / cap) if cap else logits
