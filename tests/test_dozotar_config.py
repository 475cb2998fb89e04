"""Dozotar without a GPU: configuration, refusals, cache needs, chunks in the cache manager, declared tensors, the table of
distance buckets, and properties of the plain implementation that the GPU tests lean on."""
import copy
import math

import pytest
import torch

import plain_dozotar as plain
from dozotar_configs import ALL_KINDS, ATTENTION_ONLY, DOZOTAR, MAMBA_ONLY, RETENTION_ONLY

F64 = torch.float64


def _spec(raw):
    import llmserver_b200.models  # noqa: F401
    from llmserver_b200.config import DozotarConfig
    from llmserver_b200.config.registry import architecture_of
    config = DozotarConfig.from_dict(raw)
    return config, architecture_of(raw).build_spec(config)


def _needs(spec):
    from llmserver_b200.parts import BLOCKS, MIXERS
    needs = []
    for entry in spec.schedule:
        layer = spec.layers[entry.layer]
        mixer = layer.part(BLOCKS.get(layer.block.kind).mixer_role(layer.block.as_dict()))
        needs.append(MIXERS.get(mixer.kind).cache_need(mixer.as_dict()))
    return needs


@pytest.mark.parametrize("name", sorted(DOZOTAR))
def test_configuration_round_trips(name):
    from llmserver_b200.config import DozotarConfig
    raw = DOZOTAR[name][0]
    config = DozotarConfig.from_dict(raw)
    assert DozotarConfig.from_dict(config.to_dict()) == config
    assert config.vocab_size == raw["vocab"] and config.hidden_size == raw["width"] and config.norm_eps == raw["norm"]["eps"]


def test_refusals():
    from llmserver_b200.config import DozotarConfig, UnsupportedModelError

    def broken(change):
        raw = copy.deepcopy(ALL_KINDS)
        change(raw)
        with pytest.raises(UnsupportedModelError):
            DozotarConfig.from_dict(raw)
    broken(lambda raw: raw["layers"][0].update(type="wkv"))
    broken(lambda raw: raw["layers"][0]["mixer"].update(decay=[0.5]))
    broken(lambda raw: raw["layers"][0]["mixer"]["rot"].update(dims=9))
    broken(lambda raw: raw["layers"][0]["mixer"]["rot"].update(dims=18))
    broken(lambda raw: raw["layers"][1]["mixer"].update(kv_heads=3))
    broken(lambda raw: raw["layers"][1]["mixer"]["mask"].update(size=0))
    broken(lambda raw: raw["layers"][1]["mixer"].pop("bias_max"))
    broken(lambda raw: raw["layers"][1]["mixer"].update(rot={"base": 100.0, "dims": 4}))
    broken(lambda raw: raw["layers"][1]["mlp"]["router"]["groups"].update(count=4))
    broken(lambda raw: raw["layers"][1]["mlp"]["router"]["groups"].update(keep=1))       # one group of two experts cannot give three
    broken(lambda raw: raw["layers"][1]["mlp"]["router"].update(top=11))
    broken(lambda raw: raw["layers"][1]["mlp"]["shared"].update(ff=0))
    broken(lambda raw: raw["layers"][2]["mixer"].update(groups=4))
    broken(lambda raw: raw["layers"][2]["mixer"].update(norm_groups=5))
    broken(lambda raw: raw["layers"][2]["mlp"].update(kind="glu"))
    broken(lambda raw: raw.pop("norm"))


def test_specification_parts_and_constants():
    _, spec = _spec(ALL_KINDS)
    assert [layer.mixer.kind for layer in spec.layers] == ["retention", "gqa_attention", "state_space_duality", "gqa_attention",
                                                           "state_space_duality", "retention"]
    assert [layer.feed_forward.kind if layer.feed_forward else None for layer in spec.layers] == \
        ["gelu_glu", "routed_experts", "routed_experts", "gelu_glu", "routed_experts", None]
    assert not spec.tie_head and spec.final_norm.get("scalar") and all(dict(layer.extra)["mixer_out_norm"].get("scalar") for layer in spec.layers)
    assert spec.layers[0].position != spec.layers[5].position and len(spec.positions) == 2 and spec.layers[1].position is None
    attention = spec.layers[1].mixer
    assert attention.get("qk_norm") == "projection" and attention.get("chunk") == 45 and attention.get("conv") == 3
    assert attention.get("distance_bias") == (16, 60.0) and attention.get("window") is None
    routed = spec.layers[1].feed_forward
    assert routed.get("scores") == "softmax" and routed.get("groups") == (5, 2) and routed.get("renormalise") and routed.get("shared_gate")
    assert spec.layers[5].mixer.get("decay") == (0.99, 0.9, 0.97, 0.7)


def test_cache_needs_and_declared_tensors():
    from llmserver_b200.cache import CacheManager, KVPagesNeed, StateNeed
    from llmserver_b200.weights.declare import declared_weights
    _, spec = _spec(ALL_KINDS)
    needs = _needs(spec)
    assert needs[0] == StateNeed((3, 16, 24), "float32")
    assert needs[1] == (KVPagesNeed(2, 16, chunk=45), StateNeed((2, 4 * 16 + 2 * 16 + 2 * 16), "float32"))
    assert needs[2] == (StateNeed((6, 24, 16), "float32"), StateNeed((2, 6 * 16 + 2 * 2 * 24), "float32"))
    assert needs[3] == (KVPagesNeed(1, 32, None, 48, chunk=20), StateNeed((3, 2 * 32 + 32 + 48), "float32"))
    cache = CacheManager(needs, 8, 10, num_slots=2, prefix_sharing=True)
    assert len(cache.groups) == 2 and all(group.gives_back for group in cache.groups) and not cache.prefix_sharing
    names = declared_weights(spec)
    assert names["embed"].shape == names["head"].shape == (300, 96) and names["final.norm"].shape == () and names["l0.norm1"].shape == ()
    assert names["l0.mix.g"].shape == (72, 96) and "l5.norm2" not in names
    assert names["l1.mix.q.norm"].shape == (64,) and names["l1.mix.k.norm"].shape == (32,) and names["l1.mix.v.conv"].shape == (32, 3)
    assert names["l1.mix.rel"].shape == (16, 4) and names["l1.mlp.shared.sg"].shape == (1, 96) and names["l1.mlp.e9.down"].shape == (96, 32)
    assert names["l2.mix.in"].shape == (2 * 96 + 2 * 48 + 6, 96) and names["l2.mix.conv"].shape == (192, 3) and names["l2.mix.conv.b"].shape == (192,)
    assert names["l2.mix.norm"].shape == (96,) and names["l2.mix.D"].shape == (6,)
    # a layer whose convolution has one tap keeps pages alone; a bias table's rows may be left to the checkpoint
    raw = copy.deepcopy(ATTENTION_ONLY)
    del raw["layers"][0]["mixer"]["buckets"]
    _, spec = _spec(raw)
    assert _needs(spec)[2] == KVPagesNeed(1, 24, None, 40, chunk=1) and _needs(spec)[4][0] == KVPagesNeed(2, 16)
    assert declared_weights(spec)["l0.mix.rel"].shape == (-1, 3)


def test_chunks_give_pages_back_when_the_next_chunk_begins():
    from llmserver_b200.cache import CacheManager, KVPagesNeed
    from llmserver_b200.cache.manager import RELEASED
    cache = CacheManager([KVPagesNeed(1, 8, chunk=10), KVPagesNeed(1, 8)], page_size=4, num_pages=12, num_slots=2)
    cache.admit("a")
    cache.ensure("a", 9)
    assert cache.advance("a", 9) == 0                   # position 9 still sees 0 .. 9
    cache.ensure("a", 10)
    assert cache.advance("a", 10) == 2                  # position 10 sees itself: pages 0 and 1 are done, page 2 holds 8 .. 11
    assert [page == RELEASED for page in cache.table("a", 0)] == [True, True, False]
    cache.ensure("a", 30)
    assert cache.advance("a", 29) == 3                  # the chunk from 20 on: pages 2, 3 and 4 as well
    assert cache.advance("a", 30) == 2                  # the chunk from 30 on: pages 5 and 6; page 7 holds 28 .. 31
    assert cache.groups[0].pool.num_available == 12 - 1 and all(page != RELEASED for page in cache.table("a", 1))
    cache.check_invariants()
    cache.free("a")
    assert cache.available() == [12, 12]
    with pytest.raises(ValueError):
        KVPagesNeed(1, 8, window=5, chunk=10)
    with pytest.raises(ValueError):
        KVPagesNeed(1, 8, chunk=0)


def test_distance_buckets_against_their_definition():
    from llmserver_b200.parts.attention import distance_buckets
    for count, largest in ((8, 20.0), (16, 90.0), (32, 128.0), (4, 9.0), (12, 40.0), (16, 8.5)):
        found = distance_buckets(count, largest, 300)
        half = count // 2
        assert found[:half] == list(range(half)) and found[half] == half
        assert all(later >= earlier for earlier, later in zip(found, found[1:])) and found[-1] == count - 1
        assert found[math.ceil(largest):] == [count - 1] * (300 - math.ceil(largest))
        assert found == [plain.distance_bucket(n, count, largest) for n in range(300)]
    for count, largest in ((1, 5.0), (8, 4.0)):
        with pytest.raises(ValueError):
            distance_buckets(count, largest, 10)


def test_part_parameters_are_checked():
    from llmserver_b200.parts import FEED_FORWARDS, MIXERS
    attention = MIXERS.get("gqa_attention")
    base = dict(hidden=8, heads=2, kv_heads=1, head_dim=8, scale=1.0)
    for wrong in (dict(chunk=4, window=3), dict(chunk=-1), dict(qk_norm="rows"), dict(conv=3, values_are_keys=True), dict(distance_bias=(8, 3.0))):
        with pytest.raises(ValueError):
            attention.check_params({**base, **wrong})
    attention.check_params({**base, "chunk": 4, "conv": 3, "qk_norm": "projection", "distance_bias": (8, 30.0)})
    routed = FEED_FORWARDS.get("routed_experts")
    base = dict(hidden=8, experts=6, top=2, intermediate=8, activation="silu", correction=False)
    for wrong in (dict(scores="tanh"), dict(groups=(4, 2)), dict(groups=(3, 4)), dict(groups=(6, 1)), dict(shared_gate=True), dict(limit=7.0)):
        with pytest.raises(ValueError):
            routed.check_params({**base, **wrong})
    routed.check_params({**base, "scores": "softmax", "groups": (3, 1), "renormalise": True, "shared_intermediate": 8, "shared_gate": True})
    with pytest.raises(ValueError):
        MIXERS.get("retention").check_params(dict(hidden=8, heads=2, dim=8, value_dim=8, decay=(0.5,), eps=1e-6))


def test_segments_of_decaying_recurrences_fill_the_gpu_once(monkeypatch):
    """Long bfloat16 portions are cut into as many segments as fill the GPU about once, at least 64 tokens each; short
    portions, 32-bit steps and steps with enough heads to fill it anyway run in one pass; a given length is taken."""
    from types import SimpleNamespace

    from llmserver_b200 import ops
    monkeypatch.setattr(ops, "_sm_count", lambda device: 148)

    def choose(q_lens, dtype=torch.bfloat16, segment=None, heads=16, dim=64, vdim=128):
        batch = SimpleNamespace(n_seqs=len(q_lens), max_q_len=max(q_lens), q_lens=list(q_lens), scratch={})
        return ops._decay_segments(batch, torch.empty((1,), dtype=dtype), segment, heads, dim, vdim)

    segment, segments, state, move = choose([2048])
    assert (segment, segments) == (64, 32) and state.shape == (1, 32, 16, 64, 128) and move.shape == (1, 32, 16)
    assert choose([2048], heads=64, dim=128, vdim=64)[:2] == (228, 9)           # 592 blocks of 128 threads at a time
    assert choose([2048] + [1] * 7, heads=64, dim=128, vdim=64)[:2] == (228, 9)     # single tokens do not count
    assert choose([2048] * 4, heads=64, dim=128, vdim=64)[:2] == (1024, 2)
    assert choose([2048] * 16, heads=64, dim=128, vdim=64) == (0, 0, None, None)
    assert choose([2048], dtype=torch.float32) == (0, 0, None, None) and choose([127, 3]) == (0, 0, None, None)
    assert choose([100, 90], segment=7)[:2] == (7, 15) and choose([100], dtype=torch.float32, segment=7)[:2] == (7, 15)


# ------------------------------------------------------------------------------------------------ the plain implementation
def _random_weights(raw, seed):
    from llmserver_b200.weights.declare import declared_weights
    from llmserver_b200.weights.random_init import random_tensor
    _, spec = _spec(raw)
    return {name: random_tensor(name, declaration, seed).to(F64) for name, declaration in declared_weights(spec).items()}


def test_plain_recurrent_state_carries_over_portions():
    weights = _random_weights(ALL_KINDS, 1)
    h = torch.randn((19, ALL_KINDS["width"]), dtype=F64, generator=torch.Generator().manual_seed(2))
    cuts = ((0, 1), (1, 3), (3, 4), (4, 12), (12, 19))      # portions shorter than the convolution too
    mixer = ALL_KINDS["layers"][0]["mixer"]
    whole, last = plain.retention(h, weights, "l0.mix.", mixer, 1e-6)
    out, state = [], None
    for begin, end in cuts:
        piece, state = plain.retention(h[begin:end], weights, "l0.mix.", mixer, 1e-6, state=state, first_position=begin)
        out.append(piece)
    assert torch.allclose(torch.cat(out), whole, atol=1e-12) and torch.allclose(state, last, atol=1e-12)
    mixer = ALL_KINDS["layers"][2]["mixer"]
    whole, (last, history) = plain.ssd(h, weights, "l2.mix.", mixer, 1e-6)
    out, state = [], None
    for begin, end in cuts:
        piece, state = plain.ssd(h[begin:end], weights, "l2.mix.", mixer, 1e-6, state=state)
        out.append(piece)
    assert torch.allclose(torch.cat(out), whole, atol=1e-12) and torch.allclose(state[0], last, atol=1e-12)
    assert torch.allclose(state[1], history, atol=1e-12) and history.shape == (2, 192)


def test_plain_scan_against_its_unrolled_sum_and_relative_rotation():
    generator = torch.Generator().manual_seed(5)
    T, D, V = 6, 4, 3
    q, k = (torch.randn((T, D), dtype=F64, generator=generator) for _ in range(2))
    v = torch.randn((T, V), dtype=F64, generator=generator)
    decay = torch.rand(T, dtype=F64, generator=generator)
    out, _ = plain.decayed_scan(q, k, v, decay, torch.zeros((D, V), dtype=F64))
    for t in range(T):      # o_t = sum_(s<=t) (prod_(s<j<=t) g_j) (q_t . k_s) v_s
        want = sum(torch.prod(decay[s + 1:t + 1]) * (q[t] @ k[s]) * v[s] for s in range(t + 1))
        assert torch.allclose(out[t], want, atol=1e-12)
    # rotated queries and keys meet by the difference of their positions
    rot = {"base": 100.0, "dims": 4}
    x = torch.randn((2, 1, 6), dtype=F64, generator=generator)
    near = plain.rotate_heads(x, torch.tensor([3, 8]), rot)
    far = plain.rotate_heads(x, torch.tensor([40, 45]), rot)
    assert torch.allclose(near[0, 0] @ near[1, 0], far[0, 0] @ far[1, 0], atol=1e-12) and torch.equal(near[..., 4:], x[..., 4:])


def test_plain_chunks_and_bias():
    weights = _random_weights(ATTENTION_ONLY, 3)
    h = torch.randn((18, ATTENTION_ONLY["width"]), dtype=F64, generator=torch.Generator().manual_seed(4))
    mixer = ATTENTION_ONLY["layers"][0]["mixer"]          # chunks of seven positions
    _, kept = plain.chunked_attention(h, weights, "l0.mix.", mixer, 1e-5, want_probabilities=True)
    for row, first in ((6, 0), (7, 7), (13, 7), (14, 14), (17, 14)):
        p = kept[1][row]
        assert bool((p[:first] == 0).all()) and bool((p[first:row + 1] > 0).all()) and bool((p[row + 1:] == 0).all())
    alone = ATTENTION_ONLY["layers"][2]["mixer"]
    _, kept = plain.chunked_attention(h, weights, "l2.mix.", alone, 1e-5, want_probabilities=True)
    assert torch.allclose(kept[0], torch.eye(18, dtype=F64))
    # without queries only the bias decides: the logs of two weights of a row differ by what the table says
    bare = dict(weights)
    bare["l4.mix.q"] = torch.zeros_like(weights["l4.mix.q"])
    mixer = ATTENTION_ONLY["layers"][4]["mixer"]
    _, kept = plain.chunked_attention(h, bare, "l4.mix.", mixer, 1e-5, want_probabilities=True)
    rel = weights["l4.mix.rel"]
    got = torch.log(kept[1][15, 3]) - torch.log(kept[1][15, 14])
    assert torch.allclose(got, rel[plain.distance_bucket(12, 12, 40.0), 1] - rel[1, 1], atol=1e-9)


def test_plain_router_keeps_groups():
    router = {"experts": 6, "top": 2, "groups": {"count": 3, "keep": 1}}
    z = torch.tensor([1.0, 0.9, 1.1, -3.0, 0.5, 0.4], dtype=F64)
    chosen, share = plain.route(z, router)
    assert chosen == [2, 3] and abs(float(share.sum()) - 1.0) < 1e-12       # expert 2's group wins, although its other is weak
    assert plain.route(z, {"experts": 6, "top": 2})[0] == [2, 0]
    assert plain.route(z, {**router, "groups": {"count": 3, "keep": 2}})[0] == [2, 0]
    assert plain.route(torch.zeros(6, dtype=F64), router)[0] == [0, 1]


def test_plain_forward_runs_every_configuration():
    for name, (raw, seed) in DOZOTAR.items():
        weights = _random_weights(raw, seed)
        tokens = [(7 * i + 3) % raw["vocab"] for i in range(11)]
        streams = []
        logits = plain.forward(raw, weights, tokens, streams=streams)
        assert logits.shape == (11, raw["vocab"]) and len(streams) == len(raw["layers"]) and bool(torch.isfinite(logits).all())
        changed = plain.forward(raw, weights, tokens[:-1] + [(tokens[-1] + 1) % raw["vocab"]])      # causal
        assert torch.allclose(changed[:-1], logits[:-1], atol=1e-12) and not torch.allclose(changed[-1], logits[-1], atol=1e-9)


def test_norm_parts_and_groups_of_the_state_space_form():
    """Norm parts that cut heads in two, and heads that share B and C by groups, in the plain implementation."""
    weights = _random_weights(MAMBA_ONLY, 6)
    mixer = MAMBA_ONLY["layers"][1]["mixer"]              # six heads of eight in three groups; parts of twelve channels
    h = torch.randn((5, MAMBA_ONLY["width"]), dtype=F64, generator=torch.Generator().manual_seed(7))
    y, _ = plain.ssd(h, weights, "l1.mix.", mixer, 1e-5)
    scaled = dict(weights)
    scaled["l1.mix.norm"] = weights["l1.mix.norm"].clone()
    scaled["l1.mix.norm"][12:24] *= 2.0                   # one part's weights: linear in what that part contributes
    y2, _ = plain.ssd(h, scaled, "l1.mix.", mixer, 1e-5)
    only = dict(weights)
    only["l1.mix.norm"] = torch.zeros_like(weights["l1.mix.norm"])
    only["l1.mix.norm"][12:24] = weights["l1.mix.norm"][12:24]
    part, _ = plain.ssd(h, only, "l1.mix.", mixer, 1e-5)
    assert torch.allclose(y2 - y, part, atol=1e-12)
    assert RETENTION_ONLY["layers"][1]["mixer"]["decay"][0] == 1.0      # a head that forgets nothing is among the tests' models
