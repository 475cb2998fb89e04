"""Rapolix on the GPU against the plain implementation in plain_rapolix.py: each mechanism alone, then whole models through
the step function, the cache and the scheduler, cut and batched in different ways, in 32-bit and bfloat16."""
import copy
import json
import math
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import plain_rapolix as plain
import traces
from helpers import tokens_for
from rapolix_configs import RAPOLIX

pytestmark = pytest.mark.gpu

DEVICE = "cuda:0"
DTYPES = ["float32", "bfloat16"]
TORCH_DTYPES = [torch.float32, torch.bfloat16]
NAMES = sorted(RAPOLIX)
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
F64 = torch.float64
# Largest allowed |engine - plain| as a fraction of the row's largest |plain logit|.
ALLOWED = {"float32": 4e-5, "bfloat16": 6e-2}
CLEAR = 0.01     # routing margins (in choice scores) from which on bfloat16 activations do not change a choice


# ------------------------------------------------------------------------------------------------ model folders
def _redraw(tensors, seed):
    """Weights redrawn where the generic random mode would hide a fault: peaked attention, streams that differ and are read and
    written with different weights (without cancelling one another, which would blow rounding up), convolution taps and biases far from zero, decays that keep state for hundreds of tokens
    in some channels and lose it at once in others, routers sure of their first choices (the last one then weighs little, so
    that one that rounding swaps for another moves little) with corrections that still steer it."""
    generator = torch.Generator().manual_seed(seed)
    for key in sorted(tensors):
        shape = tensors[key].shape

        def draw(deviation, mean=0.0):
            return (torch.randn(shape, generator=generator) * deviation + mean).to(torch.bfloat16)
        if key.endswith(("left.q", "left.k")):
            tensors[key] = draw(1.3 / math.sqrt(shape[1]))
        elif key.endswith((".left.v", ".left.g", ".left.o", ".right.y", ".right.x", ".right.o", ".gate", ".up", ".down")):
            tensors[key] = draw(1.0 / math.sqrt(shape[1]))
        elif key.endswith((".ra", ".ri")):
            tensors[key] = draw(1.5 / math.sqrt(shape[2]))
        elif key.endswith(".lam"):
            tensors[key] = torch.linspace(-9.0, 1.0, shape[0]).to(torch.bfloat16)
        elif key.endswith(".conv"):
            tensors[key] = draw(0.6)
        elif key.endswith(".b"):
            tensors[key] = draw(0.4)
        elif ".hc" in key:
            if key.endswith(".mix"):
                tensors[key] = (torch.randn(shape, generator=generator) * 0.08 + 0.1 + 0.6 * torch.eye(shape[0])).to(torch.bfloat16)
            else:
                tensors[key] = draw(0.3, 0.8)
        elif key.endswith(".router"):
            tensors[key] = draw(2.5 / math.sqrt(shape[1]))
        elif key.endswith(".correction"):
            tensors[key] = draw(0.05)
        elif key == "embed":
            tensors[key] = draw(1.0)
        elif key == "head":
            tensors[key] = draw(3.0 / math.sqrt(shape[1]))
    return tensors


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    from safetensors.torch import load_file, save_file

    import llmserver_b200.models  # noqa: F401
    from llmserver_b200.config import RapolixConfig
    from llmserver_b200.weights import write_model_folder

    root = tmp_path_factory.mktemp("rapolix")
    made = {}
    for name, (raw, seed) in RAPOLIX.items():
        folder = write_model_folder(RapolixConfig.from_dict(raw), str(root / name), seed, torch.bfloat16)
        path = os.path.join(folder, "model.safetensors")
        save_file(_redraw(load_file(path), seed), path)
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
    """32-bit: every row within the allowance.  bfloat16: rows are compared where every routing decision of the token itself is
    clear in the plain implementation (a quarter of the rows at least); up to one row in twenty (or two) may exceed the allowance
    (an earlier token's close call reaches later ones through keys and state), none may reach half the largest logit."""
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
    assert len(errors) >= total / 4, f"{what}: only {len(errors)} of {total} rows have clear routing"
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


def _close(got, want, tolerance, what=""):
    scale = max(1.0, float(want.abs().max()))
    error = float((got.cpu().double() - want).abs().max()) / scale
    assert error <= tolerance, f"{what}: {error:.2e} of the largest value, allowed {tolerance:.1e}"


# ------------------------------------------------------------------------------------------------ mechanisms alone
@pytest.mark.parametrize("dtype", TORCH_DTYPES)
@pytest.mark.parametrize("width,copies", [(48, 1), (45, 3), (1, 2), (256, 2), (10, 5)])
def test_embedding_with_sinusoids_and_copies(dtype, width, copies):
    """Positions up to a million: the angles of far positions keep their 32-bit exactness."""
    from llmserver_b200 import ops
    from llmserver_b200.parts import POSITION_ENCODINGS, Runtime
    generator = torch.Generator().manual_seed(width)
    table = torch.randn((30, width), generator=generator).to(dtype)
    ids = torch.tensor([3, 29, 0, 3, 7, 11], dtype=torch.int32)
    positions = torch.tensor([0, 1, 77, 4095, 70001, 1000003], dtype=torch.int32)
    encoding = POSITION_ENCODINGS.get("sinusoidal")({"width": width}, {}, Runtime(dtype, torch.device(DEVICE)))
    got = ops.embedding(table.to(DEVICE), ids.to(DEVICE), copies=copies, positions=positions.to(DEVICE), frequencies=encoding.frequencies)
    want = table.double()[ids.long()] + plain.sinusoids(positions, width)
    assert got.shape == ((6, width) if copies == 1 else (6, copies, width))
    for copy_index in range(copies):
        _close(got.view(6, copies, width)[:, copy_index], want, 5e-7)


@pytest.mark.parametrize("dtype", TORCH_DTYPES)
@pytest.mark.parametrize("streams,width", [(1, 40), (2, 64), (3, 96), (4, 4200), (2, 1000), (5, 64), (3, 45), (2, 16384), (9, 30)])
def test_streams_written_read_and_normalised(dtype, streams, width):
    """What is pending written into all streams from the old ones, the streams read and normalised: two outputs with norms of
    their own, one with a bias, nothing pending, selected rows (nothing is written then), and both kinds of norm."""
    from llmserver_b200 import ops
    generator = torch.Generator().manual_seed(streams * 1000 + width)

    def draw(*shape, mean=0.0, scale=1.0):
        return torch.randn(shape, generator=generator) * scale + mean
    rows, eps = 5, 1e-3
    x = draw(rows, streams, width, mean=0.7)
    a, b = (draw(rows, width, scale=s).to(dtype) for s in (3.0, 0.2))
    bias = draw(width)
    wa, wb, weight = (draw(width, mean=1.0, scale=0.3).to(dtype) for _ in range(3))
    mix, out_w, read = draw(streams, streams), draw(streams), draw(streams)
    coefficients = {"mix": mix.double(), "out": out_w.double(), "in": read.double()}
    selected = torch.tensor([4, 1, 1], dtype=torch.int32)
    tolerance = 5e-6 if dtype == torch.float32 else 1e-2
    on_device = {id(t): t.to(DEVICE) for t in (a, b, bias, wa, wb, weight, mix, out_w, read)}

    def dev(t):
        return None if t is None else on_device[id(t)]
    two = 0.5 * (plain.rms_norm(a.double(), wa.double(), 1e-5) + plain.rms_norm(b.double() + bias.double(), wb.double(), 1e-2))
    cases = [([(a, None, wa, 1e-5, 0.5), (b, bias, wb, 1e-2, 0.5)], two), ([(a, bias, None, 0.0, 1.0)], a.double() + bias.double()),
             ([(b, None, None, 0.0, 1.0), (a, None, wa, 1e-5, 2.0)], b.double() + 2.0 * plain.rms_norm(a.double(), wa.double(), 1e-5)), ([], None)]
    for parts, y in cases:
        described = [(dev(part), dev(part_bias), dev(part_weight), part_eps, scale) for part, part_bias, part_weight, part_eps, scale in parts]
        for centre in (True, False):
            old = x.double().transpose(0, 1)
            new = old if y is None else plain.write_streams(old, y, coefficients, "")
            u = plain.read_streams(new, coefficients, "")
            want = (plain.layer_norm if centre else plain.rms_norm)(u, weight.double(), eps)
            stream = x.clone().to(DEVICE)
            got = ops.streams_norm(stream, described, dev(weight), eps, centre, mix=dev(mix), out_weight=dev(out_w), read=dev(read), act_dtype=dtype)
            _close(got, want, tolerance, "normalised")
            _close(stream, new.transpose(0, 1), 3e-6, "streams")
            untouched = x.clone().to(DEVICE)
            got = ops.streams_norm(untouched, described, dev(weight), eps, centre, mix=dev(mix), out_weight=dev(out_w), read=dev(read),
                                   rows=selected.to(DEVICE), act_dtype=dtype)
            _close(got, want[selected.long()], tolerance, "selected rows")
            assert torch.equal(untouched.cpu(), x)
    # without coefficients: the sum of the streams; one stream and a plain residual add
    got = ops.streams_norm(x.clone().to(DEVICE), [], dev(weight), eps, True, act_dtype=dtype)
    _close(got, plain.layer_norm(x.double().sum(dim=1), weight.double(), eps), tolerance, "sum")
    one = x[:, 0].contiguous().to(DEVICE)
    got = ops.streams_norm(one, [(dev(a), None, None, 0.0, 1.0)], dev(weight), eps, True, act_dtype=dtype)
    _close(got, plain.layer_norm(x[:, 0].double() + a.double(), weight.double(), eps), tolerance, "one stream")
    _close(one, x[:, 0].double() + a.double(), 1e-6)


def _stepwise(lengths):
    for step in range(max(len(steps) for steps in lengths)):
        yield [(s, steps[step]) for s, steps in enumerate(lengths) if step < len(steps)]


SHORT_AND_LONG = [([(0, 1), (1, 2), (3, 9)], [(0, 17)], [(0, 6), (6, 1)]),
                  ([(0, 3), (3, 150), (153, 2)], [(0, 129)], [(0, 65), (65, 1)])]      # portions that several blocks share


@pytest.mark.parametrize("dtype", TORCH_DTYPES)
@pytest.mark.parametrize("taps,channels,column,row", [(4, 72, 8, 88), (2, 320, 0, 320), (3, 1032, 16, 1056), (5, 64, 0, 64), (4, 70, 3, 77), (1, 40, 8, 48)])
@pytest.mark.parametrize("lengths", SHORT_AND_LONG)
def test_convolution_without_activation_over_biased_inputs(dtype, taps, channels, column, row, lengths):
    """The projection's bias belongs to the inputs, also to the kept ones, but not to what stands before a sequence."""
    from llmserver_b200 import ops
    generator = torch.Generator().manual_seed(taps * 100 + channels)
    slots = [2, 0, 3]
    x = [torch.randn((sum(now for _, now in steps), row), generator=generator).to(dtype) for steps in lengths]
    taps_w = torch.randn((channels, taps), generator=generator) * 0.6
    bias, in_bias = (torch.randn((channels,), generator=generator) for _ in range(2))
    state = torch.zeros((4, max(taps - 1, 1), channels), dtype=torch.float32, device=DEVICE)
    state[1] = 7.0
    got = [[] for _ in lengths]
    for live in _stepwise(lengths):
        rows = torch.cat([x[s][before:before + now] for s, (before, now) in live]).to(DEVICE)
        out = ops.short_conv_units(rows, column, taps_w.to(DEVICE), state, _batch([piece for _, piece in live], [slots[s] for s, _ in live]),
                                   0, 0, 0, -(-channels // 256), 256, 0.0, 1.0, bias=bias.to(DEVICE), channels=channels, in_bias=in_bias.to(DEVICE),
                                   silu=False, out_dtype=dtype)
        assert out.dtype == dtype
        at = 0
        for s, (_, now) in live:
            got[s].append(out.cpu()[at:at + now])
            at += now
    for s in range(len(lengths)):
        y, history = plain.causal_convolution(x[s][:, column:column + channels].double() + in_bias.double(), taps_w.double(), bias.double())
        _close(torch.cat(got[s]), y, 2e-6 if dtype == torch.float32 else 4e-3, f"sequence {s}")
        if taps > 1:
            assert torch.allclose(state[slots[s]].cpu().double(), history, atol=1e-6), f"stored inputs of sequence {s}"
    assert bool((state[1] == 7.0).all())


@pytest.mark.parametrize("dtype", TORCH_DTYPES)
@pytest.mark.parametrize("tokens", [1, 7, 33, 70])
@pytest.mark.parametrize("units,rows,inner", [(2, 40, 20), (3, 14, 7), (1, 128, 64), (16, 256, 128)])
def test_products_with_a_matrix_per_unit(dtype, tokens, units, rows, inner):
    from llmserver_b200 import ops
    generator = torch.Generator().manual_seed(units * 10 + inner)
    x = torch.randn((tokens, units * inner), generator=generator).to(dtype)
    weight = (torch.randn((units, rows, inner), generator=generator) / math.sqrt(inner)).to(dtype)
    got = ops.unit_linear_wide(x.to(DEVICE), weight.to(DEVICE))
    assert got.dtype == torch.float32 and got.shape == (tokens, units, rows)
    _close(got, torch.einsum("tuk,urk->tur", x.double().view(tokens, units, inner), weight.double()), 3e-6)


class _Scan:
    """Inputs of the gated scan for whole sequences, the kernel on pieces of them and the plain result."""

    def __init__(self, dtype, lengths, units, size, seed, units_first=False):
        generator = torch.Generator().manual_seed(seed)
        self.dtype, self.units, self.size, self.units_first = dtype, units, size, units_first
        width = self.width = units * size
        self.z = [torch.randn((length, units, 2 * size), generator=generator) * 2 for length in lengths]
        self.u = [torch.randn((length, width), generator=generator).to(dtype) for length in lengths]
        self.y = [torch.randn((length, width + 8), generator=generator).to(dtype) for length in lengths]
        self.lam = torch.linspace(-10.0, 2.0, width)
        self.gate_bias, self.y_bias = torch.randn((units, 2 * size), generator=generator), torch.randn((width,), generator=generator)

    def run(self, rows, batch, state, segment=None):
        from llmserver_b200 import ops
        z, u, y = (torch.cat([source[s][r] for s, r in rows]).contiguous().to(DEVICE) for source in (self.z, self.u, self.y))
        if self.units_first:
            z = z.transpose(0, 1).contiguous().transpose(0, 1)
        rate = (-8.0 * torch.nn.functional.softplus(self.lam.double())).float().to(DEVICE)
        return ops.gated_scan(z, u, self.gate_bias.to(DEVICE), rate, y, 8, self.y_bias.to(DEVICE), state, batch, segment=segment)

    def want(self, s):
        z = self.z[s].double() + self.gate_bias.double()
        r = torch.sigmoid(z[:, :, :self.size]).reshape(-1, self.width)
        i = torch.sigmoid(z[:, :, self.size:]).reshape(-1, self.width)
        states, last = plain.gated_scan(self.u[s].double(), r, i, self.lam.double(), torch.zeros(self.width, dtype=F64))
        return states * plain.gelu_tanh(self.y[s][:, 8:].double() + self.y_bias.double()), last


@pytest.mark.parametrize("dtype", TORCH_DTYPES)
@pytest.mark.parametrize("segment", [0, 5, 16])
@pytest.mark.parametrize("units,size,units_first", [(2, 40, False), (3, 7, True), (1, 300, True), (5, 64, False), (9, 1, False), (4, 128, True)])
def test_gated_scan_over_slots_and_segments(dtype, segment, units, size, units_first):
    """Three sequences in one step: one from zero, one that continues from the state that an earlier step left (in another slot
    order), a single token behind a longer past; in one pass and by segments, the states behind the step compared too.  Decays
    run from 'keeps everything' to 'forgets at once'."""
    pieces = [(0, 37), (19, 11), (45, 1)]
    case = _Scan(dtype, [before + now for before, now in pieces], units, size, units * 100 + size, units_first)
    slots = [2, 0, 3]
    state = torch.zeros((4, case.width), dtype=torch.float32, device=DEVICE)
    state[1] = 7.0
    earlier = [(2, 45), (1, 19)]
    case.run([(s, slice(0, count)) for s, count in earlier], _batch([(0, count) for _, count in earlier], [slots[s] for s, _ in earlier]), state,
             segment=segment)
    got = case.run([(s, slice(before, None)) for s, (before, _) in enumerate(pieces)], _batch(pieces, slots), state, segment=segment)
    at = 0
    for s, (before, now) in enumerate(pieces):
        want, last = case.want(s)
        _close(got[at:at + now], want[before:], 5e-6 if dtype == torch.float32 else 8e-3, f"sequence {s}")
        _close(state[slots[s]], last, 1e-5, f"state of sequence {s}")
        at += now
    assert bool((state[1] == 7.0).all())


@pytest.mark.parametrize("dtype", TORCH_DTYPES)
def test_gated_scan_keeps_a_far_token_across_portions_and_segments(dtype):
    """One input enters at the third token, gates are shut for every later one and nothing decays; only the last token, 700
    tokens on, has an output gate that is open.  A long portion (walked by segments in bfloat16), a second one that ends inside
    a segment, and a single token."""
    total, portions = 703, [(0, 300), (300, 402), (702, 1)]
    case = _Scan(dtype, [total], 2, 32, 5)
    case.lam[:] = -12.0
    case.z[0][:, :, 32:] = -30.0
    case.z[0][2, :, 32:], case.u[0][2] = 30.0, 60.0
    case.y[0][:] = -30.0
    case.y[0][-1] = 3.0
    want, _ = case.want(0)
    kept = case.u[0][2].clone()
    case.u[0][2] = 0.0
    without, _ = case.want(0)
    case.u[0][2] = kept
    assert (want[-1] - without[-1]).abs().min() > 0.1
    state = torch.zeros((2, case.width), dtype=torch.float32, device=DEVICE)
    got = torch.cat([case.run([(0, slice(before, before + now))], _batch([(before, now)], [1]), state) for before, now in portions])
    _close(got, want, 3e-5 if dtype == torch.float32 else 8e-3)


@pytest.mark.parametrize("dtype", TORCH_DTYPES)
@pytest.mark.parametrize("hidden,width,blocks,taps", [(48, 40, 2, 4), (45, 63, 3, 2), (64, 128, 1, 5), (64, 20, 20, 1)])
def test_recurrent_block_as_a_mixer(dtype, hidden, width, blocks, taps):
    """The whole branch: projections, convolution, gates, recurrence and output, a prompt cut in three against the plain one."""
    from llmserver_b200.parts import MIXERS, EntryCache, Runtime
    generator = torch.Generator().manual_seed(hidden + width)
    cls = MIXERS.get("gated_linear_recurrent_unit")
    params = dict(hidden=hidden, width=width, blocks=blocks, conv=taps)
    weights = {}
    for name, declaration in cls.declare_weights(params).items():
        shape = declaration.shape
        scale = 1.0 / math.sqrt(shape[-1]) if len(shape) > 1 and name != "conv" else 0.5
        weights[name] = (torch.randn(shape, generator=generator) * scale).to(torch.bfloat16)
    weights["lam"] = torch.linspace(-8.0, 1.0, width).to(torch.bfloat16)
    wide = ("y.b", "x.b", "conv", "conv.b", "ra.b", "ri.b", "lam")
    part = cls(params, {name: (tensor.float() if name in wide else tensor.to(dtype)).to(DEVICE) for name, tensor in weights.items()},
               Runtime(dtype, torch.device(DEVICE)))
    h = torch.randn((90, hidden), generator=generator).to(torch.bfloat16)
    views = [EntryCache(state=torch.zeros((3,) + need.shape, dtype=torch.float32, device=DEVICE)) for need in cls.cache_need(params)]
    got = torch.cat([part.forward(h[before:before + now].to(dtype).to(DEVICE), _batch([(before, now)], [1]), EntryCache(parts=views))
                     for before, now in ((0, 70), (70, 3), (73, 17))])
    want, (S, history) = plain.recurrent_block(h.double(), {name: tensor.double() for name, tensor in weights.items()}, "", params)
    _close(got, want, 1e-5 if dtype == torch.float32 else 2e-2)
    _close(views[0].state[1], S, 1e-5 if dtype == torch.float32 else 2e-2, "state")
    if taps > 1:
        _close(views[1].state[1], history, 1e-5 if dtype == torch.float32 else 2e-2, "stored inputs")


def _attention_case(dtype, heads, kv_heads, dim, vdim, lengths, new_tokens, page_size, window, keep, seed, spike):
    """Queries, paged keys and values on shuffled pages (pages that a window has passed and nobody keeps hold other things), and
    gated softmax attention of every query over what it sees, in float64.  ``spike`` = (query index, key position): that query
    and that key are made parallel and long, so that their score towers over the row's other scores."""
    generator = torch.Generator().manual_seed(seed)
    queries = [(s, p) for s, (length, count) in enumerate(zip(lengths, new_tokens)) for p in range(length - count, length)]
    keys = [torch.randn((length, kv_heads, dim), generator=generator).to(dtype) for length in lengths]
    values = [torch.randn((length, kv_heads, vdim), generator=generator).to(dtype) for length in lengths]
    used = (heads + kv_heads) * dim + kv_heads * vdim
    column = -(-used // 8) * 8
    row = -(-(column + heads * vdim) // 8) * 8
    packed = torch.randn((len(queries), row), generator=generator).to(dtype)
    q = packed[:, :heads * dim].reshape(len(queries), heads, dim)
    scale = 1.3 / math.sqrt(dim)
    if spike is not None:
        index, position = spike
        direction = torch.nn.functional.normalize(torch.randn((dim,), generator=generator), dim=0)
        keys[queries[index][0]][position] = (direction * math.sqrt(35.0 / scale)).to(dtype)
        q = q.clone()
        q[index] = (direction * math.sqrt(35.0 / scale)).to(dtype)
        packed[:, :heads * dim] = q.reshape(len(queries), heads * dim)
    blocks = [-(-length // page_size) for length in lengths]
    order = torch.randperm(sum(blocks) + 1, generator=generator).tolist()
    foreign = order.pop()
    tables = [[] for _ in lengths]
    k_pages = torch.zeros((sum(blocks) + 1, kv_heads, page_size, dim), dtype=dtype)
    v_pages = torch.zeros((sum(blocks) + 1, kv_heads, page_size, vdim), dtype=dtype)
    k_pages[foreign], v_pages[foreign] = 4.0, -9.0      # what another request may have put on a page that was given back
    for s, length in enumerate(lengths):
        earliest = length - new_tokens[s]               # the first query of this step
        passed = max(0, earliest - window + 1) // page_size if window else 0
        for block in range(blocks[s]):
            page = order.pop()
            rows = slice(block * page_size, min(length, (block + 1) * page_size))
            k_pages[page, :, :rows.stop - rows.start] = keys[s][rows].transpose(0, 1)
            v_pages[page, :, :rows.stop - rows.start] = values[s][rows].transpose(0, 1)
            tables[s].append(foreign if -(-keep // page_size) <= block < passed else page)
    want = torch.zeros((len(queries), heads, vdim), dtype=F64)
    spike_weight = None
    group_of = torch.arange(heads) // (heads // kv_heads)
    mask = {"size": window, "keep_first": keep} if window else None
    for index, (s, p) in enumerate(queries):
        seen = torch.tensor([j for j in range(p + 1) if plain.visible(p, j, mask)])
        scores = torch.einsum("hd,khd->hk", q[index].double(), keys[s][seen][:, group_of].double()) * scale
        weights = torch.softmax(scores, dim=-1)
        want[index] = torch.einsum("hk,khv->hv", weights, values[s][seen][:, group_of].double())
        if spike is not None and index == spike[0] and spike[1] in seen.tolist():
            spike_weight = float(weights[:, seen.tolist().index(spike[1])].min())
    gate = torch.sigmoid(packed[:, column:column + heads * vdim].double())
    return packed, column, k_pages, v_pages, tables, scale, want.reshape(len(queries), heads * vdim) * gate, spike_weight


@pytest.mark.parametrize("dtype", TORCH_DTYPES)
@pytest.mark.parametrize("heads,kv_heads,dim,vdim,window,keep,page_size", [
    (4, 2, 128, 128, 100, 4, 16), (8, 1, 128, 128, 30, 70, 16), (16, 1, 128, 128, 90, 129, 8), (3, 3, 128, 128, 0, 5, 16),
    (6, 2, 64, 64, 33, 1, 8), (4, 1, 64, 128, 64, 64, 16), (8, 2, 128, 64, 1, 3, 16), (4, 2, 64, 64, 650, 9, 16), (12, 1, 64, 64, 50, 200, 16),
    (10, 2, 128, 128, 256, 0, 16), (4, 1, 32, 48, 64, 6, 16), (3, 3, 24, 24, 20, 33, 4), (2, 1, 9, 7, 40, 2, 8)])
def test_window_edges_and_kept_tokens_in_prompts_and_decoding(dtype, heads, kv_heads, dim, vdim, window, keep, page_size):
    """Gated attention as a step runs it (a whole prompt, a portion behind cached tokens, single decoded tokens, one of them behind a
    long context), with one score that towers over its row: for the window's first key (it must carry the row), for the key just in
    front of it (unseen, unless kept), for the first and the last kept key, for the first one that is not kept, for a key in the
    middle and the last slot of a page."""
    from llmserver_b200 import ops
    from llmserver_b200.ops.library import check_wait_errors
    lengths, new_tokens = [300, 241, 1, 130, 700], [1, 241, 1, 30, 1]
    counts = [sum(new_tokens[:s]) for s in range(len(lengths))]
    spikes = [None]
    for index, position in ((counts[4], 699), (counts[3] + 20, 120), (counts[1] + 200, 200)):
        first = max(0, position - window + 1) if window else 0
        spikes += [(index, key) for key in sorted({first, first - 1, (position + first) // 2, 0, keep - 1, keep}) if 0 <= key <= position]
    spikes.append((counts[4], 699 - (699 % page_size) - 1))
    for spike in spikes:
        packed, column, k_pages, v_pages, tables, scale, want, spike_weight = _attention_case(
            dtype, heads, kv_heads, dim, vdim, lengths, new_tokens, page_size, window, keep, 37, spike)
        batch = _batch([(length - count, count) for length, count in zip(lengths, new_tokens)], [0] * len(lengths), tables)
        on_device = packed.to(DEVICE)
        out = ops.attention(on_device, batch, batch.block_tables[0], k_pages.to(DEVICE), v_pages.to(DEVICE), heads, kv_heads, dim, scale, window,
                            value_dim=vdim, precise=True, q_stride=packed.shape[1], keep=keep, gate=on_device, gate_column=column)
        torch.cuda.synchronize()
        check_wait_errors()
        error = (out.cpu().double() - want).abs().max(dim=-1).values / want.abs().max(dim=-1).values.clamp_min(0.05)
        allowed = 2e-5 if dtype == torch.float32 else 6e-3
        assert error.max() < allowed, f"spike {spike}: row {int(error.argmax())} of {len(error)} differs by {float(error.max()):.2e}"
        if spike_weight is not None:
            assert spike_weight > 0.9       # a kernel that missed the key would be far off


@pytest.mark.parametrize("dtype", TORCH_DTYPES)
@pytest.mark.parametrize("heads,kv_heads,dim,vdim,gate", [(4, 2, 16, 24, 8), (3, 3, 128, 128, 40), (2, 1, 9, 7, 0), (6, 2, 8, 12, 4)])
def test_keys_and_values_cached_as_projected(dtype, heads, kv_heads, dim, vdim, gate):
    """Nothing is normalised or turned: keys and values go to their (shuffled) pages in 16-byte pieces where the sizes allow it; queries,
    what lies behind the values and everybody else's pages stay as they are, and so does the cache when it may not be written."""
    from llmserver_b200 import ops
    generator = torch.Generator().manual_seed(heads * dim)
    pieces, page_size = [(0, 21), (13, 5), (40, 1)], 8
    used = (heads + kv_heads) * dim + kv_heads * vdim
    packed = torch.randn((27, used + gate), generator=generator).to(dtype)
    order = torch.randperm(20, generator=generator).tolist()
    tables = [[order.pop() for _ in range(-(-(before + now) // page_size))] for before, now in pieces]
    batch = _batch(pieces, [0] * 3, tables)
    for write in (True, False):
        k_pages, v_pages = (torch.full((20, kv_heads, page_size, size), 5.0, dtype=dtype, device=DEVICE) for size in (dim, vdim))
        rows = packed.clone().to(DEVICE)
        ops.norm_rope_units(rows, batch.positions, batch.seq_of_token, batch.block_tables[0], k_pages, v_pages, heads, kv_heads, 1, dim, dim, vdim,
                            batch.error_flag, write_cache=write)
        assert torch.equal(rows.cpu(), packed) and int(batch.error_flag.item()) == 0
        want_k, want_v, at = torch.full_like(k_pages.cpu(), 5.0), torch.full_like(v_pages.cpu(), 5.0), 0
        for (before, now), table in zip(pieces, tables):
            for position in range(before, before + now):
                if write:
                    k = packed[at, heads * dim:(heads + kv_heads) * dim].view(kv_heads, dim)
                    want_k[table[position // page_size], :, position % page_size] = k
                    want_v[table[position // page_size], :, position % page_size] = packed[at, (heads + kv_heads) * dim:used].view(kv_heads, vdim)
                at += 1
        assert torch.equal(k_pages.cpu(), want_k) and torch.equal(v_pages.cpu(), want_v)


ROUTERS = [(6, 2, None, 0), (7, 3, (3, 2), 2), (8, 4, (2, 1), 0), (13, 5, (4, 4), 3), (12, 1, (14, 1), 2), (60, 6, (8, 3), 4), (33, 8, (9, 2), 3), (5, 6, None, 2)]


@pytest.mark.parametrize("dtype", TORCH_DTYPES)
@pytest.mark.parametrize("experts,top,groups,identity", ROUTERS)
def test_router_choices_with_correction_and_identities(dtype, experts, top, groups, identity):
    """Softmax scores; a correction that steers groups and outputs (also one that makes every choice score negative) and stays out
    of the weights; groups of experts and identities together; from both router kernels; ties go to the lower index."""
    from llmserver_b200 import ops
    generator = torch.Generator().manual_seed(experts * 10 + top)
    tokens, width, outputs = 37, 48, experts + identity
    x = torch.randn((tokens, width), generator=generator).to(dtype)
    router = torch.randn((outputs, width), generator=generator).mul(0.4).to(torch.bfloat16).float()
    z = x.double() @ router.double().T
    rule = {"top": top, "groups": {"count": groups[0], "keep": groups[1]} if groups else None}
    options = dict(scores="softmax", groups=groups, renormalise=True)
    logits = torch.zeros((tokens, -(-outputs // 8) * 8))
    logits[:, :outputs] = z.float()
    for mean in (0.0, -2.0):
        correction = torch.randn((outputs,), generator=generator) * 0.1 + mean
        for chosen, weights in (ops.moe_route(x.to(DEVICE), router.to(DEVICE), correction.to(DEVICE), top, 1.0, **options),
                                ops.moe_select(logits.to(DEVICE), correction.to(DEVICE), top, 1.0, experts=outputs, **options)):
            for t in range(tokens):
                if plain.routing_margin(z[t], correction.double(), rule) < 1e-5:
                    continue
                want, share = plain.route(z[t], correction.double(), rule)
                got = chosen[t].cpu().tolist()
                assert sorted(got) == sorted(want), f"token {t}: {got} where {want} is expected"
                by_output = dict(zip(want, share.tolist()))
                assert all(abs(by_output[e] - w) < 1e-5 for e, w in zip(got, weights[t].cpu().tolist()))
    tied = ops.moe_select(torch.zeros((2, outputs), device=DEVICE), torch.zeros(outputs, device=DEVICE), top, 1.0, **options)[0]
    assert tied.cpu().tolist() == [list(range(top))] * 2


@pytest.mark.parametrize("dtype", TORCH_DTYPES)
@pytest.mark.parametrize("tokens", [1, 5, 40, 150])
@pytest.mark.parametrize("width,experts,top,ff,groups,identity,shared", [(48, 7, 3, 16, (3, 2), 2, 20), (45, 8, 4, 24, (2, 1), 0, 0), (128, 9, 4, 64, (5, 3), 1, 128),
                                                                         (64, 4, 5, 128, None, 3, 64), (192, 12, 2, 320, (7, 4), 2, 64)])
def test_squared_relu_experts_with_identities(dtype, tokens, width, experts, top, ff, groups, identity, shared):
    """The whole feed-forward: pair by pair, and, with more tokens in bfloat16 at sizes that allow it, by sorted pairs; with the
    router's own choices, with identities alone and with none of them."""
    from llmserver_b200.parts import FEED_FORWARDS, Runtime
    generator = torch.Generator().manual_seed(width + tokens)
    params = dict(hidden=width, experts=experts, identity=identity, top=top, intermediate=ff, activation="squared_relu", correction=True,
                  route_scale=1.0, scores="softmax", groups=groups, renormalise=True, shared_intermediate=shared or None)
    cls = FEED_FORWARDS.get("routed_experts")
    weights = {}
    for name, declaration in cls.declare_weights(params).items():
        scale = 3.0 if name == "router" else 1.0
        weights[name] = (torch.randn(declaration.shape, generator=generator) * scale / math.sqrt(declaration.shape[-1])).to(torch.bfloat16)
    x = torch.randn((tokens, width), generator=generator).to(torch.bfloat16)
    config = {"router": {"experts": experts, "top": top, "groups": {"count": groups[0], "keep": groups[1]} if groups else None},
              "shared": {"ff": shared} if shared else None}
    corrections = [torch.randn((experts + identity,), generator=generator) * 0.1]
    corrections.append(torch.cat([torch.zeros(experts), torch.full((identity,), -5.0)]))
    corrections.append(torch.cat([torch.full((experts,), -5.0), torch.zeros(identity)]))
    for correction in corrections:
        weights["correction"] = correction.to(torch.bfloat16)
        part = cls(params, {name: (tensor.float() if name in ("router", "correction") else tensor.to(dtype)).to(DEVICE) for name, tensor in weights.items()},
                   Runtime(dtype, torch.device(DEVICE)))
        got = part.forward(x.to(dtype).to(DEVICE))
        want = plain.routed_feed_forward(x.double(), {name: tensor.double() for name, tensor in weights.items()}, "", config)
        z = x.double() @ weights["router"].double().T      # (rows whose choice hangs on the last bit of a score are left out)
        clear = torch.tensor([plain.routing_margin(row, weights["correction"].double(), config["router"]) > 1e-5 for row in z])
        assert clear.float().mean() > 0.75
        _close((got.cpu().double() / want.abs().max())[clear], (want / want.abs().max())[clear], 2e-5 if dtype == torch.float32 else 1e-2)


@pytest.mark.parametrize("dtype", TORCH_DTYPES)
@pytest.mark.parametrize("rows,width,ff", [(3, 48, 40), (1, 45, 29), (70, 128, 192), (5, 96, 64)])
@pytest.mark.parametrize("activation", ["silu", "gelu"])
def test_dense_feed_forward_with_biases(dtype, rows, width, ff, activation):
    from llmserver_b200.parts import FEED_FORWARDS, Runtime
    generator = torch.Generator().manual_seed(width + ff)
    cls = FEED_FORWARDS.get("biased_glu")
    params = dict(hidden=width, intermediate=ff, activation=activation)
    weights = {name: (torch.randn(declaration.shape, generator=generator) / math.sqrt(declaration.shape[-1] if len(declaration.shape) > 1 else 1.0)).to(torch.bfloat16)
               for name, declaration in cls.declare_weights(params).items()}
    part = cls(params, {name: (tensor.float() if name.endswith(".b") else tensor.to(dtype)).to(DEVICE) for name, tensor in weights.items()},
               Runtime(dtype, torch.device(DEVICE)))
    x = torch.randn((rows, width), generator=generator).to(torch.bfloat16)
    got = part.forward(x.to(dtype).to(DEVICE)).cpu().double() + part.output_bias.cpu().double()
    wide = {name: tensor.double() for name, tensor in weights.items()}
    if activation == "silu":
        want = plain.dense_feed_forward(x.double(), wide, "")
    else:
        want = plain.biased(plain.gelu_tanh(plain.biased(x.double(), wide, "gate")) * plain.biased(x.double(), wide, "up"), wide, "down")
    _close(got, want, 1e-5 if dtype == torch.float32 else 2e-2)


# ------------------------------------------------------------------------------------------------ whole models
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_whole_prompt_and_token_by_token(folders, name, dtype):
    vocab = RAPOLIX[name][0]["vocab"]
    tokens = tokens_for(vocab, 203, 7)
    records = traces.whole("r", tokens)
    got, _ = run_in_process(folders[name], dtype, records, traces.rounded(len(tokens)))
    compare(got, records, {"r": tokens}, folders[name], dtype, f"{name} whole")
    records = traces.tail_decoded("r", tokens, 120)      # windows pass over decoded tokens
    got, _ = run_in_process(folders[name], dtype, records, traces.rounded(len(tokens)), page_size=8)
    compare(got, records, {"r": tokens}, folders[name], dtype, f"{name} tail decoded")
    short = tokens[:30]                                  # and from the very first token on, one by one
    records = traces.tail_decoded("r", short, 29)
    got, _ = run_in_process(folders[name], dtype, records, traces.rounded(len(short)), page_size=4)
    compare(got, records, {"r": short}, folders[name], dtype, f"{name} decoded from the start")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_portions_down_to_two_tokens(folders, name, dtype):
    vocab = RAPOLIX[name][0]["vocab"]
    tokens = tokens_for(vocab, 203, 7)
    records = traces.portions("r", tokens, [7, 2, 5, 3, 2, 16, 33, 2, 64, 1, 17])
    got, _ = run_in_process(folders[name], dtype, records, traces.rounded(len(tokens)), page_size=8)
    compare(got, records, {"r": tokens}, folders[name], dtype, f"{name} portions")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_mixed_batches_reuse_pages_and_slots(folders, name, dtype):
    vocab = RAPOLIX[name][0]["vocab"]
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


@pytest.mark.parametrize("name", ["mixed_sizes", "tensor_core_sizes"])
def test_portions_walked_by_short_segments(folders, name, monkeypatch):
    """With segments of eight tokens every portion of sixteen or more is walked segment by segment, beside shorter ones and
    single tokens that are not; the segments' ends fall anywhere."""
    monkeypatch.setattr("llmserver_b200.ops.SCAN_SEGMENT", 8)
    vocab = RAPOLIX[name][0]["vocab"]
    tokens = tokens_for(vocab, 203, 7)
    records = traces.portions("r", tokens, [17, 2, 16, 3, 41, 1, 70, 15])
    got, _ = run_in_process(folders[name], "bfloat16", records, traces.rounded(len(tokens)), page_size=8)
    compare(got, records, {"r": tokens}, folders[name], "bfloat16", f"{name} portions by segments")
    requests = {key: tokens_for(vocab, length, 31 + index) for index, (key, length) in enumerate({"r0": 110, "r1": 67, "r2": 40, "r3": 131}.items())}
    records, peak = traces.mixed(requests, seed=6)
    got, _ = run_in_process(folders[name], "bfloat16", records, peak)
    compare(got, records, requests, folders[name], "bfloat16", f"{name} mixed by segments")


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding(folders, dtype):
    name = "mixed_sizes"
    tokens = tokens_for(RAPOLIX[name][0]["vocab"], 330, 3)
    records = traces.tail_decoded("r", tokens, tail=322)
    got, _ = run_in_process(folders[name], dtype, records, traces.rounded(len(tokens)))
    compare(got, records, {"r": tokens}, folders[name], dtype, "long decoding")


def test_a_lost_state_or_a_window_one_token_off_would_show(folders):
    """The plain implementation with recurrent state and convolution history dropped at a portion's start, with windows one token
    longer or shorter, with one kept token more or fewer, or with positions that start anew gives logits outside the
    allowance of either path: the models of these tests do not hide such faults."""
    for name in ("mixed_sizes", "one_stream"):
        config, weights = plain_model_of(folders[name])
        tokens = tokens_for(config["vocab"], 90, 13)
        want = plain_logits(folders[name], tokens)
        scale = np.abs(want).max(axis=-1)

        def far_off(logits, what, first=0):
            moved = np.abs(logits.numpy() - want).max(axis=-1)[first:] / scale[first:]
            assert moved.max() > 1.2 * ALLOWED["bfloat16"], f"{name}: {what}: {moved.max():.3f}"
            assert (moved > 100 * ALLOWED["float32"]).mean() > 0.2, f"{name}: {what}: {(moved > 100 * ALLOWED['float32']).mean():.2f}"
        far_off(plain.forward(config, weights, tokens, lose_state_at=60), "a lost state", first=60)
        for what, key, change in (("window +1", "size", 1), ("window -1", "size", -1), ("kept +1", "keep_first", 1), ("kept -1", "keep_first", -1)):
            other = copy.deepcopy(config)
            for layer in other["layers"]:
                mask = layer["mixer"]["left"].get("mask")
                if mask and mask[key] + change >= (1 if key == "size" else 0):
                    mask[key] += change
            far_off(plain.forward(other, weights, tokens), what)


def test_float32_logits_do_not_depend_on_the_cut(folders):
    name = "mixed_sizes"
    vocab = RAPOLIX[name][0]["vocab"]
    tokens, other = tokens_for(vocab, 120, 19), tokens_for(vocab, 75, 20)
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
    """Requests of unequal length through the engine's own scheduler (portions, continuous batching, a pool so small that pages
    come back and are used again, fewer state slots than requests): every generated token maximises the plain logits of its own
    prefix."""
    from llmserver_b200 import Engine
    vocab = RAPOLIX[name][0]["vocab"]
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
    """Greedy tokens of a batch through captured decode graphs, padded rows beside real ones, equal those of eager steps (in 32-bit,
    where a row's sums do not depend on how many rows there are)."""
    from llmserver_b200 import Engine
    name = "tensor_core_sizes"
    prompts = [tokens_for(RAPOLIX[name][0]["vocab"], length, 90 + length) for length in (6, 75, 130)]
    generated = []
    for graphs in (True, False):
        engine = Engine(folders[name], max_new_tokens=40, max_batch_size=3, kv_cache_num_blocks=96, kv_cache_block_size=8,
                        ignore_eos=True, dtype="float32", cuda_graphs=graphs)
        generated.append(engine.generate(prompts))
        assert (engine.step_function.graph_steps > 20) == graphs
    assert generated[0] == generated[1]


def test_trace_run_program(folders, tmp_path):
    name, dtype = "mixed_sizes", "float32"
    vocab = RAPOLIX[name][0]["vocab"]
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
    name = "one_stream"
    vocab = RAPOLIX[name][0]["vocab"]
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
