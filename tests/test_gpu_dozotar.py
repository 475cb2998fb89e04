"""Dozotar on the GPU against the plain implementation in plain_dozotar.py: each mechanism alone, then whole models
through the step function, the cache and the scheduler, cut and batched in different ways, in 32-bit and bfloat16."""
import copy
import json
import math
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import plain_dozotar as plain
import traces
from dozotar_configs import DOZOTAR
from helpers import tokens_for

pytestmark = pytest.mark.gpu

DEVICE = "cuda:0"
DTYPES = ["float32", "bfloat16"]
NAMES = sorted(DOZOTAR)
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
F64 = torch.float64
# Largest allowed |engine - plain| as a fraction of the row's largest |plain logit|.  float32: states that keep what they
# were given for hundreds of tokens also keep the 32-bit rounding of every update.  bfloat16: besides the activations
# between kernels, every sub-layer reads the 32-bit stream itself rounded to 8 significant bits.
ALLOWED = {"float32": 4e-5, "bfloat16": 6e-2}
CLEAR = 0.1      # routing margins from which on bfloat16 activations do not change a choice


# ------------------------------------------------------------------------------------------------ model folders
def _redraw(tensors, config, seed):
    """Weights redrawn where the generic random mode would hide a fault: norm weights of queries and keys large enough for
    peaked attention, biases by distance of the size of the scores, convolution taps and biases far from zero, decays
    that keep state for hundreds of tokens in some heads and lose it at once in others, routers sure of their first
    choices (the last expert chosen then weighs little, so that one that rounding swaps for another moves little)."""
    generator = torch.Generator().manual_seed(seed)
    for key in sorted(tensors):
        shape = tensors[key].shape

        def draw(deviation, mean=0.0):
            return (torch.randn(shape, generator=generator) * deviation + mean).to(torch.bfloat16)
        if key.endswith((".q.norm", ".k.norm")):
            tensors[key] = draw(0.4, 1.2)
        elif key.endswith((".norm1", ".norm2")):
            tensors[key] = draw(0.1, 0.8)
        elif key.endswith(".rel"):
            tensors[key] = draw(1.0)
        elif key.endswith((".conv", ".conv.b", ".D")):
            tensors[key] = draw(0.6)
        elif key.endswith((".mix.q", ".mix.k", ".mix.v", ".mix.g", ".mix.o", ".gate", ".up", ".down", ".shared.sg")):
            tensors[key] = draw(1.0 / math.sqrt(shape[1]))
        elif key.endswith(".mix.in"):
            tensors[key] = draw(0.7 / math.sqrt(shape[1]))
        elif key.endswith(".router"):
            tensors[key] = draw(2.0 / math.sqrt(shape[1]))
        elif key.endswith(".A_log"):
            tensors[key] = torch.linspace(-4.0, 0.5, shape[0]).to(torch.bfloat16)
        elif key.endswith(".dt_bias"):
            tensors[key] = draw(1.0, -1.0)
        elif key == "embed":
            tensors[key] = draw(1.0)
    return tensors


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    from safetensors.torch import load_file, save_file

    import llmserver_b200.models  # noqa: F401
    from llmserver_b200.config import DozotarConfig
    from llmserver_b200.weights import write_model_folder

    root = tmp_path_factory.mktemp("dozotar")
    made = {}
    for name, (raw, seed) in DOZOTAR.items():
        folder = write_model_folder(DozotarConfig.from_dict(raw), str(root / name), seed, torch.bfloat16)
        path = os.path.join(folder, "model.safetensors")
        save_file(_redraw(load_file(path), raw, seed), path)
        made[name] = folder
    return made


_PLAIN, _LOGITS = {}, {}


def plain_model_of(folder):
    if folder not in _PLAIN:
        from safetensors.torch import load_file
        with open(os.path.join(folder, "config.json")) as handle:
            config = json.load(handle)
        _PLAIN[folder] = (config, {key: value.to(F64) for key, value in load_file(os.path.join(folder, "model.safetensors")).items()})
    return _PLAIN[folder]


def plain_logits(folder, tokens):
    return plain_rows(folder, tokens)[0]


def plain_rows(folder, tokens):
    """The plain logits of a sequence, and of every token the smallest margin of its routing decisions."""
    key = (folder, tuple(tokens))
    if key not in _LOGITS:
        config, weights = plain_model_of(folder)
        margins = []
        logits = plain.forward(config, weights, list(tokens), margins=margins).numpy()
        _LOGITS[key] = (logits, margins[0].numpy() if margins else np.full(len(tokens), np.inf))
    return _LOGITS[key]


def run_in_process(folder, dtype, records, max_tokens, page_size=16):
    from llmserver_b200.engine.replay import TraceReplayer

    replayer = TraceReplayer(folder, dtype, max_tokens, page_size)
    out = {}
    for record in records:
        logits = replayer.run_step(record)
        if logits is not None:
            out[record["step"]] = logits
    replayer.cache.check_invariants()
    assert not replayer.cache.requests, "requests left in the cache after the trace ended"
    for group in replayer.cache.groups:
        assert group.pool.num_available == group.pool.num_pages, "pages were lost"
    return out, replayer


def compare(got, records, requests, folder, dtype, what):
    """32-bit: every row within the allowance.  bfloat16: a sub-layer's output is normalised whatever its size, so a row
    whose parts nearly cancel, or whose state holds one or two keys, amplifies rounding: up to one row in twenty (or two)
    may exceed the allowance, none may reach half the largest logit.  A token whose experts or groups are a hair apart goes
    either way once activations are rounded: rows are compared where every routing decision of the token itself is clear
    in the plain implementation (a third of the rows at least).  A fault of the cache or the state moves most rows behind
    it (``test_a_lost_state_or_a_chunk_one_token_off_would_show``)."""
    want = traces.expected_rows(records, requests, lambda name: plain_logits(folder, requests[name]))
    margin = traces.expected_rows(records, requests, lambda name: plain_rows(folder, requests[name])[1][:, None])
    assert set(got) == set(want), f"{what}: steps with logits differ"
    errors, total = [], 0
    for step in sorted(want):
        assert got[step].shape == want[step].shape and np.isfinite(got[step]).all(), f"{what} step {step}"
        scale = np.abs(want[step]).max(axis=-1)
        found = [(float(e), step, row) for row, e in enumerate(np.abs(got[step] - want[step]).max(axis=-1) / scale)]
        total += len(found)
        errors += [item for item in found if dtype == "float32" or margin[step][item[2], 0] >= CLEAR]
    assert len(errors) >= total / 3, f"{what}: only {len(errors)} of {total} rows have clear routing"
    worst, step, row = max(errors)
    over = sum(1 for error, _, _ in errors if error > ALLOWED[dtype])
    middle = sorted(error for error, _, _ in errors)[len(errors) // 2]
    hard = ALLOWED[dtype] if dtype == "float32" else 0.5
    assert worst <= hard, f"{what} step {step}: row {row} differs by {worst:.3e} of its largest logit, allowed {hard:.1e}"
    assert over <= (max(2, len(errors) // 20) if dtype == "bfloat16" else 0), f"{what}: {over} of {len(errors)} rows differ by more than {ALLOWED[dtype]:.1e}"
    assert middle <= ALLOWED[dtype] / 2, f"{what}: the middle row differs by {middle:.3e}"


def _batch(pieces, slots, tables=None):
    """A step's batch: ``pieces`` = (tokens before, tokens now) per sequence, with one block table each where pages matter."""
    from llmserver_b200.engine.batch import SequenceSlice, build_batch
    return build_batch([SequenceSlice(f"r{index}", [0] * now, before, [], [tables[index] if tables else [0]], slots[index])
                        for index, (before, now) in enumerate(pieces)], 1, DEVICE)


# ------------------------------------------------------------------------------------------------ mechanisms alone
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("width", [40, 96, 1000])
def test_norm_with_one_number(dtype, width):
    """A sub-layer's output through a norm whose weight is one number, added to the 32-bit stream; the final norm on
    selected rows."""
    from llmserver_b200.parts import NORMS, Runtime
    from llmserver_b200.parts.norm import NormedDelta, add_and_read
    generator = torch.Generator().manual_seed(width)
    g = torch.tensor(0.7265625).to(torch.bfloat16)
    norm = NORMS.get("rmsnorm")({"width": width, "eps": 1e-5, "tensor": "", "scalar": True}, {"": g.to(dtype).to(DEVICE)},
                                Runtime(dtype, torch.device(DEVICE)))
    assert norm.weight.shape == (width,) and bool((norm.weight == 0.7265625).all())
    stream = torch.randn((5, width), generator=generator)
    delta = (torch.randn((5, width), generator=generator) * 3).to(dtype)
    on_device = stream.clone().to(DEVICE)
    out = add_and_read(on_device, NormedDelta(delta.to(DEVICE), norm), dtype)
    want = stream.double() + plain.scalar_norm(delta.double(), g.double(), 1e-5)
    assert torch.allclose(on_device.cpu().double(), want, atol=3e-6, rtol=3e-6) and torch.equal(out.cpu(), on_device.cpu().to(dtype))
    rows = torch.tensor([4, 1], dtype=torch.int32, device=DEVICE)
    got = norm.add_norm(stream.clone().to(DEVICE), NormedDelta(delta.to(DEVICE), norm), rows=rows)
    tolerance = 1e-5 if dtype == torch.float32 else 1e-2
    assert torch.allclose(got.cpu().double(), plain.scalar_norm(want[[4, 1]], g.double(), 1e-5), atol=tolerance, rtol=tolerance)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("rows,inner,group", [(3, 40, 0), (1, 7, 0), (70, 128, 64), (5, 96, 0), (2, 30, 10)])
def test_gelu_gate(dtype, rows, inner, group):
    from llmserver_b200 import ops
    generator = torch.Generator().manual_seed(inner)
    gate, up = (torch.randn((rows, inner), generator=generator).mul(3).to(dtype) for _ in range(2))
    packed = torch.cat([gate, up], dim=1)
    if group:
        packed = torch.stack([gate.view(rows, -1, group), up.view(rows, -1, group)], dim=2).reshape(rows, 2 * inner)
    got = ops.gelu_mul(packed.contiguous().to(DEVICE), group=group).cpu().double()
    want = plain.gelu_tanh(gate.double()) * up.double()
    tolerance = 2e-6 if dtype == torch.float32 else 1e-2
    assert torch.allclose(got, want, atol=tolerance, rtol=tolerance)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("rows,width,parts", [(3, 30, 5), (2, 48, 4), (9, 66, 1), (40, 4096, 1), (7, 4096, 2), (5, 1500, 1), (3, 512, 8)])
def test_norm_in_parts(dtype, rows, width, parts):
    from llmserver_b200 import ops
    generator = torch.Generator().manual_seed(width + parts)
    x = torch.randn((rows, width), generator=generator) * torch.logspace(-2, 1, parts).repeat_interleave(width // parts)
    weight = (1 + 0.3 * torch.randn((width,), generator=generator)).to(dtype)
    got = ops.grouped_rmsnorm(x.to(DEVICE), weight.to(DEVICE), parts, 1e-4, dtype).cpu().double()
    want = plain.rms_divide(x.double().view(rows, parts, -1), 1e-4).reshape(rows, width) * weight.double()
    tolerance = 1e-5 if dtype == torch.float32 else 1e-2
    assert torch.allclose(got, want, atol=tolerance, rtol=tolerance)


ROUTERS = [(6, 2, None), (9, 3, (3, 2)), (8, 4, (2, 1)), (16, 5, (4, 4)), (12, 1, (12, 1)), (64, 6, (8, 3)), (72, 8, (36, 5)), (40, 40, None)]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("experts,top,groups", ROUTERS)
def test_router_choices(dtype, experts, top, groups):
    """Softmax scores, the best groups, renormalised weights and the shared expert's gate, from the kernel that makes the
    logits itself and from the one that reads a product's (padded) rows; ties go to the lower index."""
    from llmserver_b200 import ops
    generator = torch.Generator().manual_seed(experts * 10 + top)
    tokens, width = 37, 48
    x = torch.randn((tokens, width), generator=generator).to(dtype)
    router = torch.randn((experts + 1, width), generator=generator).mul(0.4).to(torch.bfloat16).float()      # the last row: the gate
    z = x.double() @ router.double().T
    rule = {"experts": experts, "top": top, "groups": {"count": groups[0], "keep": groups[1]} if groups else None}
    options = dict(scores="softmax", groups=groups, renormalise=True, gate=True)
    logits = torch.zeros((tokens, -(-(experts + 1) // 8) * 8))
    logits[:, :experts + 1] = z.float()
    for chosen, weights, gate in (ops.moe_route(x.to(DEVICE), router.to(DEVICE), None, top, 1.0, **options),
                                  ops.moe_select(logits.to(DEVICE), None, top, 1.0, experts=experts, **options)):
        assert torch.allclose(gate.cpu().double(), torch.sigmoid(z[:, experts]), atol=1e-5)
        for t in range(tokens):
            want, share = plain.route(z[t, :experts], rule)
            got = chosen[t].cpu().tolist()
            assert sorted(got) == sorted(want), f"token {t}: {got} where {want} is expected"
            by_expert = dict(zip(want, share.tolist()))
            assert all(abs(by_expert[e] - w) < 1e-5 for e, w in zip(got, weights[t].cpu().tolist()))
    tied = ops.moe_select(torch.zeros((2, experts), device=DEVICE), None, top, 1.0, scores="softmax", groups=groups, renormalise=True)[0]
    assert tied.cpu().tolist() == [list(range(top))] * 2


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("tokens", [1, 5, 40])
@pytest.mark.parametrize("width,mlp", [(48, {"router": {"experts": 9, "top": 3, "groups": {"count": 3, "keep": 2}}, "ff": 16, "shared": 20}),
                                       (40, {"router": {"experts": 8, "top": 4, "groups": {"count": 2, "keep": 1}}, "ff": 24, "shared": 0}),
                                       (128, {"router": {"experts": 10, "top": 4, "groups": {"count": 5, "keep": 3}}, "ff": 64, "shared": 128}),
                                       (64, {"router": {"experts": 5, "top": 5, "groups": None}, "ff": 128, "shared": 64})])
def test_routed_experts_with_a_gated_shared_one(dtype, tokens, width, mlp):
    """The whole feed-forward: pair by pair, and, with more tokens in bfloat16 at sizes that allow it, by sorted pairs."""
    from llmserver_b200.parts import FEED_FORWARDS, Runtime
    generator = torch.Generator().manual_seed(width + tokens)
    experts, top, ff, shared = mlp["router"]["experts"], mlp["router"]["top"], mlp["ff"], mlp["shared"]
    groups = mlp["router"]["groups"]
    params = dict(hidden=width, experts=experts, top=top, intermediate=ff, activation="silu", correction=False, route_scale=1.0,
                  scores="softmax", groups=(groups["count"], groups["keep"]) if groups else None, renormalise=True,
                  shared_intermediate=shared or None, shared_gate=bool(shared))
    cls = FEED_FORWARDS.get("routed_experts")
    weights = {}
    for name, declaration in cls.declare_weights(params).items():
        scale = 3.0 if name == "router" else 1.0
        weights[name] = (torch.randn(declaration.shape, generator=generator) * scale / math.sqrt(declaration.shape[1])).to(torch.bfloat16)
    part = cls(params, {name: (tensor.float() if name in ("router", "shared.sg") else tensor.to(dtype)).to(DEVICE) for name, tensor in weights.items()},
               Runtime(dtype, torch.device(DEVICE)))
    x = torch.randn((tokens, width), generator=generator).to(torch.bfloat16)
    got = part.forward(x.to(dtype).to(DEVICE)).cpu().double()
    config = {"router": {"experts": experts, "top": top, "groups": groups}, "shared": {"ff": shared} if shared else None}
    want = plain.routed_feed_forward(x.double(), {name: tensor.double() for name, tensor in weights.items()}, "", config)
    error = (got - want).abs().max(dim=-1).values / want.abs().max()
    assert float(error.max()) < (2e-5 if dtype == torch.float32 else 2e-2)


def _stepwise(lengths):
    """For three sequences cut into steps: per step the live (sequence, (tokens before, tokens now))."""
    for step in range(max(len(steps) for steps in lengths)):
        yield [(s, steps[step]) for s, steps in enumerate(lengths) if step < len(steps)]


SHORT_AND_LONG = [([(0, 1), (1, 2), (3, 9)], [(0, 17)], [(0, 6), (6, 1)]),
                  ([(0, 3), (3, 150), (153, 2)], [(0, 129)], [(0, 65), (65, 1)])]      # portions that several blocks share


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("taps,channels,column,row", [(4, 72, 8, 88), (2, 320, 0, 320), (3, 1032, 16, 1056), (5, 64, 0, 64), (4, 70, 3, 77),
                                                      (1, 40, 8, 48), (9, 300, 1, 301)])
@pytest.mark.parametrize("lengths", SHORT_AND_LONG)
def test_convolution_with_bias_and_history_in_slots(dtype, taps, channels, column, row, lengths):
    """Portions shorter than the convolution, longer than a block takes, single tokens; the stored inputs are compared and
    nobody's slot stays as it is."""
    from llmserver_b200 import ops
    generator = torch.Generator().manual_seed(taps * 100 + channels)
    slots = [2, 0, 3]
    x = [torch.randn((sum(now for _, now in steps), row), generator=generator).to(dtype) for steps in lengths]
    taps_w = torch.randn((channels, taps), generator=generator) * 0.6
    bias = torch.randn((channels,), generator=generator)
    state = torch.zeros((4, max(taps - 1, 1), channels), dtype=torch.float32, device=DEVICE)
    state[1] = 7.0
    got = [[] for _ in lengths]
    for live in _stepwise(lengths):
        rows = torch.cat([x[s][before:before + now] for s, (before, now) in live]).to(DEVICE)
        out = ops.short_conv_units(rows, column, taps_w.to(DEVICE), state, _batch([piece for _, piece in live], [slots[s] for s, _ in live]),
                                   0, 0, 0, -(-channels // 256), 256, 0.0, 1.0, bias=bias.to(DEVICE), channels=channels).cpu().double()
        at = 0
        for s, (_, now) in live:
            got[s].append(out[at:at + now])
            at += now
    for s in range(len(lengths)):
        y, history = plain.causal_convolution(x[s][:, column:column + channels].double(), taps_w.double(), bias.double())
        assert torch.allclose(torch.cat(got[s]), plain.silu(y), atol=2e-5, rtol=2e-5), f"sequence {s}"
        if taps > 1:
            assert torch.equal(state[slots[s]].cpu().double(), history), f"stored inputs of sequence {s}"
    assert bool((state[1] == 7.0).all())


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads,kv_heads,dim,vdim,taps,page_size", [(4, 2, 16, 16, 3, 4), (3, 3, 8, 24, 2, 16), (6, 2, 64, 32, 4, 8), (2, 1, 12, 10, 4, 4),
                                                                    (2, 2, 8, 8, 6, 8), (3, 1, 16, 8, 1, 16), (32, 8, 128, 128, 4, 16)])
@pytest.mark.parametrize("lengths", SHORT_AND_LONG)
def test_convolved_and_normalised_projections_into_the_cache(dtype, heads, kv_heads, dim, vdim, taps, page_size, lengths):
    """q, k and v convolved, q and k normalised over all of their channels, k and v on their (shuffled) pages, the stored
    rows brought up to date; pages and slots of nobody stay as they are."""
    from llmserver_b200 import ops
    generator = torch.Generator().manual_seed(taps * 10 + dim)
    slots = [2, 0, 3]
    channels = (heads + kv_heads) * dim + kv_heads * vdim
    totals = [sum(now for _, now in steps) for steps in lengths]
    x = [torch.randn((total, channels), generator=generator).to(dtype) for total in totals]
    taps_w = torch.randn((channels, taps), generator=generator) * 0.6
    q_weight, k_weight = ((1 + 0.3 * torch.randn((size,), generator=generator)).to(dtype) for size in (heads * dim, kv_heads * dim))
    state = torch.zeros((4, max(taps - 1, 1), channels), dtype=torch.float32, device=DEVICE)
    state[1] = 7.0
    blocks = [-(-total // page_size) for total in totals]
    order = torch.randperm(sum(blocks) + 1, generator=generator).tolist()
    spare = order.pop()
    tables = [[order.pop() for _ in range(count)] for count in blocks]
    k_pages = torch.zeros((sum(blocks) + 1, kv_heads, page_size, dim), dtype=dtype, device=DEVICE)
    v_pages = torch.zeros((sum(blocks) + 1, kv_heads, page_size, vdim), dtype=dtype, device=DEVICE)
    k_pages[spare], v_pages[spare] = 5.0, 5.0
    got = [[] for _ in lengths]
    for live in _stepwise(lengths):
        batch = _batch([piece for _, piece in live], [slots[s] for s, _ in live], [tables[s] for s, _ in live])
        rows = torch.cat([x[s][before:before + now] for s, (before, now) in live]).to(DEVICE)
        out = ops.conv_norm_kv(rows, taps_w.t().contiguous().to(DEVICE), state, batch, batch.block_tables[0], k_pages, v_pages, heads, kv_heads,
                               dim, vdim, q_weight.to(DEVICE), k_weight.to(DEVICE), 1e-5).cpu().double()
        assert int(batch.error_flag.item()) == 0
        at = 0
        for s, (_, now) in live:
            got[s].append(out[at:at + now])
            at += now
    tolerance = 2e-5 if dtype == torch.float32 else 2e-2
    q_end, k_end = heads * dim, (heads + kv_heads) * dim
    for s, total in enumerate(totals):
        y, history = plain.causal_convolution(x[s].double(), taps_w.double())
        q = plain.rms_divide(y[:, :q_end], 1e-5) * q_weight.double()
        k = (plain.rms_divide(y[:, q_end:k_end], 1e-5) * k_weight.double()).view(total, kv_heads, dim)
        v = y[:, k_end:].view(total, kv_heads, vdim)
        assert torch.allclose(torch.cat(got[s]), q, atol=tolerance, rtol=tolerance), f"queries of sequence {s}"
        positions = torch.arange(total)
        pages = torch.tensor(tables[s])[positions // page_size]
        assert torch.allclose(k_pages.cpu().double()[pages, :, positions % page_size], k, atol=tolerance, rtol=tolerance), f"keys of {s}"
        assert torch.allclose(v_pages.cpu().double()[pages, :, positions % page_size], v, atol=tolerance, rtol=tolerance), f"values of {s}"
        if taps > 1:
            assert torch.equal(state[slots[s]].cpu().double(), history), f"stored rows of sequence {s}"
    assert bool((state[1] == 7.0).all()) and bool((k_pages[spare] == 5.0).all()) and bool((v_pages[spare] == 5.0).all())


def _recurrence_inputs(kind, dtype, lengths, heads, groups, dim, vdim, dims, seed):
    """Inputs of the retention or state-space kernel for whole sequences, and the plain result of each."""
    from llmserver_b200 import ops
    generator = torch.Generator().manual_seed(seed)
    keys, values = heads * dim, heads * vdim

    class Case:
        pass

    case = Case()
    if kind == "retention":
        case.proj = [torch.randn((length, 2 * keys + 2 * values + 3), generator=generator).to(dtype) for length in lengths]
        decay = torch.linspace(1.0, 0.3, heads) if heads > 1 else torch.tensor([0.998])
        rot = {"base": 1000.0, "dims": dims}
        inv_freq = torch.tensor([1000.0 ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=F64).float().to(DEVICE) if dims else None
        decay_on_device = decay.to(DEVICE)

        def run(rows, batch, state, segment=None):
            proj = torch.cat([case.proj[s][r] for s, r in rows]).contiguous().to(DEVICE)
            return ops.retention_recurrent(proj, 0, keys, 2 * keys, 2 * keys + values, decay_on_device, inv_freq, state, batch, heads, dim,
                                           vdim, dim ** -0.5, 1e-5, segment=segment)

        def want(s):
            p = case.proj[s].double()
            q, k, v = p[:, :keys].view(-1, heads, dim), p[:, keys:2 * keys].view(-1, heads, dim), p[:, 2 * keys:2 * keys + values].view(-1, heads, vdim)
            positions = torch.arange(p.shape[0])
            if dims:
                q, k = plain.rotate_heads(q, positions, rot), plain.rotate_heads(k, positions, rot)
            out, S = torch.zeros_like(v), torch.zeros((heads, dim, vdim), dtype=F64)
            for head in range(heads):
                g = torch.full((p.shape[0],), float(decay[head]), dtype=F64)
                out[:, head], S[head] = plain.decayed_scan(q[:, head], k[:, head] * dim ** -0.5, v[:, head], g, S[head])
            return plain.rms_divide(out, 1e-5).reshape(-1, values) * plain.silu(p[:, 2 * keys + values:2 * (keys + values)]), S
    else:
        width = values + 2 * groups * dim
        case.proj = [torch.randn((length, values + 3), generator=generator).to(dtype) for length in lengths]      # the gate
        case.pre = [torch.randn((length, width), generator=generator) for length in lengths]
        case.wide = [torch.randn((length, heads), generator=generator) * 2 for length in lengths]
        a_log, dt_bias, skip = torch.linspace(-5.0, 0.5, heads), torch.randn((heads,), generator=generator), torch.randn((heads,), generator=generator)
        constants = [tensor.to(DEVICE) for tensor in (a_log, dt_bias, skip)]

        def run(rows, batch, state, segment=None):
            proj, pre, wide = (torch.cat([source[s][r] for s, r in rows]).contiguous().to(DEVICE) for source in (case.proj, case.pre, case.wide))
            return ops.ssd_recurrent(proj, 3, pre, 0, values, values + groups * dim, wide, *constants, state, batch, heads, groups, dim, vdim,
                                     segment=segment)

        def want(s):
            p = case.pre[s].double()
            x = p[:, :values].view(-1, heads, vdim)
            B, C = p[:, values:values + groups * dim].view(-1, groups, dim), p[:, values + groups * dim:].view(-1, groups, dim)
            dt = torch.nn.functional.softplus(case.wide[s].double() + dt_bias.double())
            out, S = torch.zeros_like(x), torch.zeros((heads, dim, vdim), dtype=F64)
            for head in range(heads):
                group = head // (heads // groups)
                g = torch.exp(-torch.exp(a_log[head].double()) * dt[:, head])
                out[:, head], S[head] = plain.decayed_scan(C[:, group], dt[:, head, None] * B[:, group], x[:, head], g, S[head])
                out[:, head] += float(skip[head]) * x[:, head]
            return out.reshape(-1, values) * plain.silu(case.proj[s][:, 3:].double()), S
    case.run, case.want = run, want
    return case


RECURRENCES = [("retention", 2, 1, 24, 40, 8), ("retention", 5, 1, 8, 16, 8), ("retention", 1, 1, 72, 33, 2), ("retention", 3, 1, 64, 128, 64),
               ("retention", 1, 1, 40, 7, 0), ("retention", 2, 1, 128, 256, 96), ("retention", 1, 1, 200, 64, 200), ("retention", 2, 1, 16, 1, 16),
               ("ssd", 4, 1, 128, 64, 0), ("ssd", 6, 3, 12, 8, 0), ("ssd", 2, 2, 70, 33, 0), ("ssd", 3, 1, 20, 10, 0), ("ssd", 4, 2, 64, 128, 0),
               ("ssd", 2, 1, 33, 48, 0), ("ssd", 1, 1, 256, 64, 0)]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("segment", [0, 5, 16])
@pytest.mark.parametrize("kind,heads,groups,dim,vdim,dims", RECURRENCES)
def test_recurrences_with_one_decay_per_head(dtype, segment, kind, heads, groups, dim, vdim, dims):
    """Three sequences in one step: one from zero, one that continues from the state that an earlier step left (in another
    slot order), a single token behind a longer past; in one pass and by segments (the last ones shorter), the states
    behind the step compared too.  Decays run from 'keeps everything' to 'forgets at once'."""
    pieces = [(0, 37), (19, 11), (45, 1)]
    case = _recurrence_inputs(kind, dtype, [before + now for before, now in pieces], heads, groups, dim, vdim, dims, dim * 7 + vdim)
    slots = [2, 0, 3]
    state = torch.zeros((4, heads, dim, vdim), dtype=torch.float32, device=DEVICE)
    state[1] = 7.0
    earlier = [(2, 45), (1, 19)]
    case.run([(s, slice(0, count)) for s, count in earlier], _batch([(0, count) for _, count in earlier], [slots[s] for s, _ in earlier]), state)
    got = case.run([(s, slice(before, None)) for s, (before, _) in enumerate(pieces)], _batch(pieces, slots), state, segment=segment).cpu().double()
    tolerance = 3e-5 if dtype == torch.float32 or kind == "ssd" else 2e-2
    at = 0
    for s, (before, now) in enumerate(pieces):
        want, last = case.want(s)
        allowed = tolerance * max(1.0, float(want.abs().max()))
        if dtype == torch.bfloat16 and kind == "ssd":
            allowed = max(allowed, 1e-4 * float(want.abs().max()))
        assert (got[at:at + now] - want[before:]).abs().max() < allowed, f"sequence {s}"
        assert (state[slots[s]].cpu().double() - last).abs().max() < 3e-5 * max(1.0, float(last.abs().max())), f"state of sequence {s}"
        at += now
    assert bool((state[1] == 7.0).all())


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("kind", ["retention", "ssd"])
def test_recurrences_keep_a_far_key_across_portions_and_segments(dtype, kind):
    """One pair of key and value is written at the third token; no later key has a part along it and nothing decays, and
    only the last token, 700 tokens on, asks for it.  The sequence comes as a long portion (walked by segments in
    bfloat16), a second one that ends in the middle of a segment, and a single token."""
    total, portions, heads, dim, vdim = 703, [(0, 300), (300, 402), (702, 1)], 1, 32, 32
    case = _recurrence_inputs(kind, dtype, [total], heads, 1, dim, vdim, 0, 5)
    columns = (slice(0, dim), slice(dim, 2 * dim)) if kind == "retention" else (slice(vdim + dim, vdim + 2 * dim), slice(vdim, vdim + dim))
    table = case.proj[0] if kind == "retention" else case.pre[0]
    q, k = table[:, columns[0]], table[:, columns[1]]
    q *= 0.3
    k *= 0.3
    k[:, 0] = 0.0
    k[2], q[-1] = 0.0, 0.0
    k[2, 0], q[-1, 0] = 40.0, 3.0
    if kind == "ssd":
        case.wide[0][:] = -9.0
        case.wide[0][2] = 3.0
    want, _ = case.want(0)
    kept = float(k[2, 0])
    k[2, 0] = 0.0
    without, _ = case.want(0)
    k[2, 0] = kept
    assert (want[-1] - without[-1]).abs().max() > 0.5
    state = torch.zeros((2, heads, dim, vdim), dtype=torch.float32, device=DEVICE)
    got = torch.cat([case.run([(0, slice(before, before + now))], _batch([(before, now)], [1]), state) for before, now in portions]).cpu().double()
    tolerance = 3e-4 if dtype == torch.float32 or kind == "ssd" else 2e-2
    assert torch.allclose(got, want, atol=tolerance * max(1.0, float(want.abs().max())), rtol=tolerance)


def _chunked_attention_case(dtype, heads, kv_heads, dim, vdim, lengths, new_tokens, page_size, chunk, bias, seed, spike):
    """Queries, paged keys and values on shuffled pages, and softmax attention of every query over its own chunk with a bias
    by distance, in float64.  ``spike`` = (query index, key position): that query and that key are made parallel and long,
    so that their score towers over the row's other scores."""
    generator = torch.Generator().manual_seed(seed)
    queries = [(s, p) for s, (length, count) in enumerate(zip(lengths, new_tokens)) for p in range(length - count, length)]
    keys = [torch.randn((length, kv_heads, dim), generator=generator).to(dtype) for length in lengths]
    values = [torch.randn((length, kv_heads, vdim), generator=generator).to(dtype) for length in lengths]
    q = torch.randn((len(queries), heads, dim), generator=generator).to(dtype)
    scale = 1.3 / math.sqrt(dim)
    if spike is not None:
        index, position = spike
        direction = torch.nn.functional.normalize(torch.randn((dim,), generator=generator), dim=0)
        size = math.sqrt(35.0 / scale)
        keys[queries[index][0]][position] = (direction * size).to(dtype)
        q[index] = (direction * size).to(dtype)
    blocks = [-(-length // page_size) for length in lengths]
    order = torch.randperm(sum(blocks), generator=generator).tolist()
    tables = torch.zeros((len(lengths), max(blocks)), dtype=torch.int32)
    k_pages = torch.zeros((sum(blocks), kv_heads, page_size, dim), dtype=dtype)
    v_pages = torch.zeros((sum(blocks), kv_heads, page_size, vdim), dtype=dtype)
    for s, length in enumerate(lengths):
        for block in range(blocks[s]):
            page = order.pop()
            tables[s, block] = page
            rows = slice(block * page_size, min(length, (block + 1) * page_size))
            k_pages[page, :, :rows.stop - rows.start] = keys[s][rows].transpose(0, 1)
            v_pages[page, :, :rows.stop - rows.start] = values[s][rows].transpose(0, 1)
    want = torch.zeros((len(queries), heads, vdim), dtype=F64)
    spike_weight = None
    group_of = torch.arange(heads) // (heads // kv_heads)
    for index, (s, p) in enumerate(queries):
        first = p // chunk * chunk if chunk else 0
        near = (p - torch.arange(first, p + 1)).clamp(max=bias.shape[1] - 1)
        scores = torch.einsum("hd,khd->hk", q[index].double(), keys[s][first:p + 1][:, group_of].double()) * scale + bias.double()[:, near]
        weights = torch.softmax(scores, dim=-1)
        want[index] = torch.einsum("hk,khv->hv", weights, values[s][first:p + 1][:, group_of].double())
        if spike is not None and index == spike[0] and spike[1] >= first:
            spike_weight = float(weights[:, spike[1] - first].min())
    return queries, q, k_pages, v_pages, tables, blocks, scale, want.reshape(len(queries), heads * vdim), spike_weight


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads,kv_heads,dim,vdim,chunk,distances,page_size", [
    (4, 2, 128, 128, 100, 91, 16), (8, 1, 128, 128, 300, 130, 16), (16, 1, 128, 128, 90, 90, 8), (3, 3, 128, 128, 0, 40, 16),
    (6, 2, 64, 64, 33, 33, 8), (4, 1, 64, 128, 64, 20, 16), (8, 2, 128, 64, 1, 1, 16), (4, 2, 64, 64, 650, 650, 16), (12, 1, 64, 64, 0, 700, 16),
    (10, 2, 128, 128, 256, 129, 16), (4, 1, 32, 48, 64, 30, 16), (3, 3, 24, 24, 1000, 9, 4)])
def test_chunk_edges_and_bias_in_prompts_and_decoding(dtype, heads, kv_heads, dim, vdim, chunk, distances, page_size):
    """Attention as a step runs it (a whole prompt, a portion behind cached tokens, single decoded tokens, one of them
    behind a long context), with one score that towers over its row: for the first key of a chunk (it must carry the row),
    for the last key of the chunk before (it must not be seen, whatever its score), for a key in the middle, the last slot
    of a page, a key near the sequence's start; biases as large as the scores, over few and many distances."""
    from llmserver_b200 import ops
    from llmserver_b200.engine.batch import SequenceSlice, build_batch
    from llmserver_b200.ops.library import check_wait_errors
    lengths = [300, 241, 1, 130, 700]
    new_tokens = [1, 241, 1, 30, 1]
    counts = [sum(new_tokens[:s]) for s in range(len(lengths))]
    bias = torch.randn((heads, distances), generator=torch.Generator().manual_seed(8)) * 2
    bias[:, -1] += 1.0
    spikes = [None]
    for index, position in ((counts[4], 699), (counts[3] + 20, 120), (counts[1] + 200, 200)):
        first = position // chunk * chunk if chunk else 0
        spikes += [(index, first), (index, (position + first) // 2)]
        if first >= 1:
            spikes.append((index, first - 1))
    spikes.append((counts[4], 699 - (699 % page_size) - 1))
    for spike in spikes:
        queries, q, k_pages, v_pages, tables, blocks, scale, want, spike_weight = _chunked_attention_case(
            dtype, heads, kv_heads, dim, vdim, lengths, new_tokens, page_size, chunk, bias, 37, spike)
        slices = [SequenceSlice(f"r{s}", [0] * count, length - count, [], [tables[s, :blocks[s]].tolist()], 0)
                  for s, (length, count) in enumerate(zip(lengths, new_tokens))]
        batch = build_batch(slices, 1, DEVICE)
        out = ops.attention(q.reshape(len(queries), heads * dim).contiguous().to(DEVICE), batch, batch.block_tables[0], k_pages.to(DEVICE),
                            v_pages.to(DEVICE), heads, kv_heads, dim, scale, value_dim=vdim, precise=True, q_stride=heads * dim, chunk=chunk,
                            bias=bias.to(DEVICE))
        torch.cuda.synchronize()
        check_wait_errors()
        error = (out.cpu().double() - want).abs().max(dim=-1).values / want.abs().max(dim=-1).values.clamp_min(0.05)
        allowed = 2e-5 if dtype == torch.float32 else 6e-3
        assert error.max() < allowed, f"spike {spike}: row {int(error.argmax())} of {len(queries)} differs by {float(error.max()):.2e}"
        if spike_weight is not None:
            assert spike_weight > 0.9       # a kernel that missed the key would be far off


# ------------------------------------------------------------------------------------------------ whole models
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_whole_prompt_and_token_by_token(folders, name, dtype):
    vocab = DOZOTAR[name][0]["vocab"]
    tokens = tokens_for(vocab, 203, 7)
    records = traces.whole("r", tokens)
    got, _ = run_in_process(folders[name], dtype, records, traces.rounded(len(tokens)))
    compare(got, records, {"r": tokens}, folders[name], dtype, f"{name} whole")
    records = traces.tail_decoded("r", tokens, 60)      # chunks end inside the decoded tokens
    got, _ = run_in_process(folders[name], dtype, records, traces.rounded(len(tokens)), page_size=8)
    compare(got, records, {"r": tokens}, folders[name], dtype, f"{name} tail decoded")
    short = tokens[:30]                                 # and from the very first token on, one by one
    records = traces.tail_decoded("r", short, 29)
    got, _ = run_in_process(folders[name], dtype, records, traces.rounded(len(short)), page_size=4)
    compare(got, records, {"r": short}, folders[name], dtype, f"{name} decoded from the start")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_portions_down_to_two_tokens(folders, name, dtype):
    vocab = DOZOTAR[name][0]["vocab"]
    tokens = tokens_for(vocab, 203, 7)
    records = traces.portions("r", tokens, [7, 2, 5, 3, 2, 16, 33, 2, 64, 1, 17])
    got, _ = run_in_process(folders[name], dtype, records, traces.rounded(len(tokens)), page_size=8)
    compare(got, records, {"r": tokens}, folders[name], dtype, f"{name} portions")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_mixed_batches_reuse_pages_and_slots(folders, name, dtype):
    vocab = DOZOTAR[name][0]["vocab"]
    lengths = {"r0": 110, "r1": 67, "r2": 40, "r3": 131, "r4": 64, "r5": 18, "r6": 99}
    requests = {key: tokens_for(vocab, length, 31 + index) for index, (key, length) in enumerate(lengths.items())}
    records, peak = traces.mixed(requests, seed=5)
    got, replayer = run_in_process(folders[name], dtype, records, peak)
    compare(got, records, requests, folders[name], dtype, f"{name} mixed")
    for group in replayer.cache.groups:
        if not group.gives_back:
            assert group.pool.allocations > group.pool.num_pages, "the trace was meant to reuse pages"
    # seven requests went through four state slots
    assert replayer.cache.slots.num_slots == 4 and len(replayer.cache.slots.free) == 4


@pytest.mark.parametrize("name", ["retention_only", "mamba_only", "tensor_core_sizes"])
def test_portions_walked_by_short_segments(folders, name, monkeypatch):
    """The recurrences walk a long portion's segments in parallel.  With segments of eight tokens every portion of sixteen
    or more goes that way, beside shorter ones and single tokens that do not; the segments' ends fall anywhere."""
    monkeypatch.setattr("llmserver_b200.ops.REC_SEGMENT", 8)
    vocab = DOZOTAR[name][0]["vocab"]
    tokens = tokens_for(vocab, 203, 7)
    records = traces.portions("r", tokens, [17, 2, 16, 3, 41, 1, 70, 15])
    got, _ = run_in_process(folders[name], "bfloat16", records, traces.rounded(len(tokens)), page_size=8)
    compare(got, records, {"r": tokens}, folders[name], "bfloat16", f"{name} portions by segments")
    lengths = {"r0": 110, "r1": 67, "r2": 40, "r3": 131}
    requests = {key: tokens_for(vocab, length, 31 + index) for index, (key, length) in enumerate(lengths.items())}
    records, peak = traces.mixed(requests, seed=6)
    got, _ = run_in_process(folders[name], "bfloat16", records, peak)
    compare(got, records, requests, folders[name], "bfloat16", f"{name} mixed by segments")


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding(folders, dtype):
    name = "all_kinds"
    vocab = DOZOTAR[name][0]["vocab"]
    tokens = tokens_for(vocab, 330, 3)
    records = traces.tail_decoded("r", tokens, tail=322)
    got, _ = run_in_process(folders[name], dtype, records, traces.rounded(len(tokens)))
    compare(got, records, {"r": tokens}, folders[name], dtype, "long decoding")


def test_a_lost_state_or_a_chunk_one_token_off_would_show(folders):
    """The plain implementation with recurrent state and convolution history dropped at a portion's start, with chunks one
    token longer or shorter, or with a bias read one distance off, gives logits far outside the allowance: the models of
    these tests do not hide such faults."""
    for name in ("attention_only", "retention_only", "mamba_only", "all_kinds"):
        config, weights = plain_model_of(folders[name])
        tokens = tokens_for(config["vocab"], 90, 13)
        want = plain_logits(folders[name], tokens)
        scale = np.abs(want).max(axis=-1)

        def far_off(logits, what, first=0):
            moved = np.abs(logits.numpy() - want).max(axis=-1)[first:] / scale[first:]
            assert moved.max() > 2 * ALLOWED["bfloat16"] and (moved > ALLOWED["bfloat16"]).mean() > 0.1, f"{name}: {what}"
        if name != "attention_only":
            far_off(plain.forward(config, weights, tokens, lose_state_at=60), "a lost state", first=60)
        if name in ("attention_only", "all_kinds"):
            for change in (1, -1):
                other = copy.deepcopy(config)
                for layer in other["layers"]:
                    mask = layer["mixer"].get("mask")
                    if mask and mask["size"] + change > 0:
                        mask["size"] += change
                far_off(plain.forward(other, weights, tokens), f"chunks {change:+d}")
            shifted = {key: (torch.cat([value[1:], value[-1:]]) if key.endswith(".rel") else value) for key, value in weights.items()}
            far_off(plain.forward(config, shifted, tokens), "a bias one distance off")


def test_float32_logits_do_not_depend_on_the_cut(folders):
    name = "all_kinds"
    vocab = DOZOTAR[name][0]["vocab"]
    tokens = tokens_for(vocab, 120, 19)
    other = tokens_for(vocab, 75, 20)
    whole, _ = run_in_process(folders[name], "float32", traces.whole("r", tokens), 128)
    pieces, _ = run_in_process(folders[name], "float32", traces.portions("r", tokens, [3, 2, 40, 1, 1, 9]), 128, page_size=4)
    assert np.array_equal(np.concatenate([pieces[step] for step in sorted(pieces)]), whole[0])
    records, peak = traces.mixed({"r": tokens, "o": other}, seed=2)
    mixed, _ = run_in_process(folders[name], "float32", records, peak)
    fed = 0
    for record in records:
        row = 0
        for entry in record["entries"]:
            for place in entry["want"]:
                if entry["id"] == "r":
                    assert np.array_equal(mixed[record["step"]][row], whole[0][fed + place])
                row += 1
            if entry["id"] == "r":
                fed += len(entry["tokens"])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_greedy_generation_through_the_engine(folders, name, dtype):
    """Requests of unequal length through the engine's own scheduler (portions, continuous batching, a pool so small
    that pages come back and are used again, fewer state slots than requests): every generated token maximises the
    plain logits of its own prefix."""
    from llmserver_b200 import Engine
    vocab = DOZOTAR[name][0]["vocab"]
    prompts = [tokens_for(vocab, length, 50 + length) for length in (5, 23, 41, 9, 30)]
    engine = Engine(folders[name], max_new_tokens=10, max_batch_size=3, max_num_batched_tokens=32, prefill_chunk_size=12,
                    kv_cache_num_blocks=40, kv_cache_block_size=4, ignore_eos=True, dtype=dtype)
    if name == "tensor_core_sizes":
        engine.warmup()      # products tuned and decode graphs captured ahead of the first request
    generated = engine.generate(prompts)
    assert all(len(tokens) == 10 for tokens in generated)
    for prompt, tokens in zip(prompts, generated):
        logits, margins = plain_rows(folders[name], list(prompt) + list(tokens))
        slack = 2 * ALLOWED[dtype] if dtype == "float32" else 4 * ALLOWED[dtype]
        for index, token in enumerate(tokens):
            row = logits[len(prompt) - 1 + index]
            if dtype == "bfloat16" and margins[len(prompt) - 1 + index] < CLEAR:
                continue
            assert row[token] >= row.max() - slack * np.abs(row).max(), f"token {index} of a prompt of {len(prompt)}"
    engine.cache.check_invariants()
    assert engine.cache.available() == engine.cache.capacity()


def test_decode_graphs_give_the_logits_of_eager_steps(folders):
    """Greedy tokens of a batch through captured decode graphs, padded rows beside real ones, equal those of eager steps
    (in 32-bit, where a row's sums do not depend on how many rows there are)."""
    from llmserver_b200 import Engine
    name = "tensor_core_sizes"
    vocab = DOZOTAR[name][0]["vocab"]
    prompts = [tokens_for(vocab, length, 90 + length) for length in (6, 75, 130)]
    generated = []
    for graphs in (True, False):
        engine = Engine(folders[name], max_new_tokens=40, max_batch_size=3, kv_cache_num_blocks=96, kv_cache_block_size=8,
                        ignore_eos=True, dtype="float32", cuda_graphs=graphs)
        generated.append(engine.generate(prompts))
        assert (engine.step_function.graph_steps > 20) == graphs
    assert generated[0] == generated[1]


def test_trace_run_program(folders, tmp_path):
    name, dtype = "all_kinds", "float32"
    vocab = DOZOTAR[name][0]["vocab"]
    requests = {"x": tokens_for(vocab, 90, 1), "y": tokens_for(vocab, 33, 2), "z": tokens_for(vocab, 130, 3)}
    records, peak = traces.mixed(requests, seed=9, max_live=2)
    out_dir = tmp_path / "out"
    process = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", folders[name],
                              "--dtype", dtype, "--out", str(out_dir), "--max-tokens", str(peak)],
                             input="\n".join(json.dumps(record) for record in records) + "\n",
                             capture_output=True, text=True, timeout=600)
    assert process.returncode == 0, process.stderr[-2000:]
    assert [line for line in process.stdout.splitlines() if line.startswith("done ")] == [f"done {r['step']}" for r in records]
    got = {}
    for record in records:
        wanted = sum(len(entry["want"]) for entry in record["entries"])
        if wanted:
            got[record["step"]] = np.fromfile(out_dir / f"{record['step']}.f32", dtype="<f4").reshape(wanted, vocab)
    compare(got, records, requests, folders[name], dtype, f"trace_run {name}")


def test_generate_command(folders):
    """The command line a user generates with: ids in, ids out, the model chosen by its config.json."""
    name = "all_kinds"
    vocab = DOZOTAR[name][0]["vocab"]
    prompts = [tokens_for(vocab, 19, 71), tokens_for(vocab, 3, 72)]
    command = [sys.executable, "-m", "llmserver_b200.cli.generate", "--model", folders[name], "--dtype", "float32",
               "--max-new-tokens", "6", "--ignore-eos", "--block-size", "8", "--json"]
    for prompt in prompts:
        command += ["--prompt-ids", ",".join(str(token) for token in prompt)]
    process = subprocess.run(command, capture_output=True, text=True, timeout=600, cwd=ROOT)
    assert process.returncode == 0, process.stderr[-2000:]
    generated = json.loads(process.stdout.strip().splitlines()[-1])["generated"]
    for prompt, tokens in zip(prompts, generated):
        assert len(tokens) == 6
        logits = plain_logits(folders[name], list(prompt) + list(tokens))
        assert tokens == [int(logits[len(prompt) - 1 + index].argmax()) for index in range(6)]
