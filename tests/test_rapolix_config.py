"""Rapolix without a GPU: configuration, refusals, cache needs, kept pages in the cache manager, declared tensors, what parts
and blocks refuse, and properties of the plain implementation that the GPU tests lean on."""
import copy

import pytest
import torch

import plain_rapolix as plain
from rapolix_configs import MIXED_SIZES, ODD_SIZES, RAPOLIX, TENSOR_CORE_SIZES

F64 = torch.float64


def _spec(raw):
    import llmserver_b200.models  # noqa: F401
    from llmserver_b200.config import RapolixConfig
    from llmserver_b200.config.registry import architecture_of
    config = RapolixConfig.from_dict(raw)
    return config, architecture_of(raw).build_spec(config)


def _needs(spec):
    from llmserver_b200.parts import BLOCKS, MIXERS
    needs = []
    for entry in spec.schedule:
        layer = spec.layers[entry.layer]
        mixer = layer.part(BLOCKS.get(layer.block.kind).mixer_role(layer.block.as_dict()))
        needs.append(MIXERS.get(mixer.kind).cache_need(mixer.as_dict()))
    return needs


@pytest.mark.parametrize("name", sorted(RAPOLIX))
def test_configuration_round_trips(name):
    from llmserver_b200.config import RapolixConfig
    raw = RAPOLIX[name][0]
    config = RapolixConfig.from_dict(raw)
    assert RapolixConfig.from_dict(config.to_dict()) == config
    assert config.vocab_size == raw["vocab"] and config.hidden_size == raw["width"] and config.streams == raw["streams"]
    assert config.logit_softcap == (raw["logit_softcap"] or 0.0) and config.norm_eps == raw["norm"]["eps"]


def test_refusals():
    from llmserver_b200.config import RapolixConfig, UnsupportedModelError

    def broken(change):
        raw = copy.deepcopy(MIXED_SIZES)
        change(raw)
        with pytest.raises(UnsupportedModelError):
            RapolixConfig.from_dict(raw)
    broken(lambda raw: raw["layers"][0].update(type="attention"))
    broken(lambda raw: raw["layers"][0]["mixer"].pop("right"))
    broken(lambda raw: raw["layers"][1]["mixer"]["left"].update(kv_heads=4))
    broken(lambda raw: raw["layers"][1]["mixer"]["left"].update(scale=0.0))
    broken(lambda raw: raw["layers"][1]["mixer"]["left"]["mask"].update(size=0))
    broken(lambda raw: raw["layers"][1]["mixer"]["left"]["mask"].update(keep_first=-1))
    broken(lambda raw: raw["layers"][1]["mixer"]["left"].update(rot={"base": 100.0, "dims": 4}))
    broken(lambda raw: raw["layers"][1]["mixer"]["right"].update(blocks=2))
    broken(lambda raw: raw["layers"][1]["mixer"]["right"].update(conv=0))
    broken(lambda raw: raw["layers"][3]["mlp"]["router"]["groups"].update(count=4))
    broken(lambda raw: raw["layers"][3]["mlp"]["router"].update(identity=1))             # eight outputs in three groups
    broken(lambda raw: raw["layers"][3]["mlp"]["router"]["groups"].update(keep=4))
    broken(lambda raw: raw["layers"][4]["mlp"]["router"].update(top=5))                  # two groups of two outputs are kept
    broken(lambda raw: raw["layers"][3]["mlp"]["shared"].update(ff=0))
    broken(lambda raw: raw["layers"][1]["mlp"].update(kind="glu"))
    broken(lambda raw: raw.update(streams=0))
    broken(lambda raw: raw.update(logit_softcap=-1.0))
    broken(lambda raw: raw.pop("norm"))


def test_specification_parts_and_constants():
    _, spec = _spec(MIXED_SIZES)
    assert spec.streams == 3 and spec.logit_softcap == 9.0 and not spec.tie_head and spec.final_norm.kind == "layernorm"
    assert [part.kind for part in spec.positions.values()] == ["sinusoidal"] and all(layer.position is None for layer in spec.layers)
    assert all(layer.block.kind == "hyper_connections" and layer.mixer.kind == "parallel_mixers" for layer in spec.layers)
    assert [layer.feed_forward.kind if layer.feed_forward else None for layer in spec.layers] == \
        [None, "biased_glu", "routed_experts", "routed_experts", "routed_experts"]
    (left_name, left, left_scale, _), (right_name, right, right_scale, _) = spec.layers[1].mixer.get("branches")
    assert (left_name, right_name, left_scale, right_scale) == ("left", "right", 0.5, 0.5) and spec.layers[1].mixer.get("norm_eps") == 1e-5
    assert left.get("window") == 30 and left.get("keep_first") == 3 and left.get("gate") and left.get("scale") == 0.4
    assert right.kind == "gated_linear_recurrent_unit" and right.get("blocks") == 3 and right.get("conv") == 2 and right.get("width") == 63
    routed = spec.layers[3].feed_forward
    assert routed.get("identity") == 2 and routed.get("groups") == (3, 2) and routed.get("correction") and routed.get("renormalise")
    assert routed.get("activation") == "squared_relu" and routed.get("scores") == "softmax" and routed.get("shared_intermediate") == 20
    assert spec.layers[4].mixer.get("branches")[0][1].get("window") is None


def test_cache_needs_and_declared_tensors():
    from llmserver_b200.cache import CacheManager, KVPagesNeed, StateNeed
    from llmserver_b200.weights.declare import declared_weights
    _, spec = _spec(MIXED_SIZES)
    needs = _needs(spec)
    assert needs[1] == (KVPagesNeed(2, 8, 30, keep_first=3), (StateNeed((63,), "float32"), StateNeed((1, 63), "float32")))
    assert needs[3] == (KVPagesNeed(4, 12, 400, 10, keep_first=5), (StateNeed((96,), "float32"), StateNeed((5, 96), "float32")))
    assert needs[4][0] == KVPagesNeed(2, 16) and needs[4][0].keep_first == 0
    cache = CacheManager(needs, 8, 10, num_slots=2, prefix_sharing=True)
    assert len(cache.groups) == 5 and [group.gives_back for group in cache.groups] == [True] * 4 + [False] and not cache.prefix_sharing
    names = declared_weights(spec)
    assert names["l1.mix.left.g"].shape == (48, 48) and names["l3.mix.left.g"].shape == (40, 48) and names["l3.mix.left.o"].shape == (48, 40)
    assert names["l1.mix.right.ra"].shape == (3, 21, 21) and names["l1.mix.right.ri.b"].shape == (3, 21) and names["l1.mix.right.conv"].shape == (63, 2)
    assert names["l1.mix.left.out"].shape == names["l1.mix.right.out"].shape == (48,) and names["l1.hc2.mix"].shape == (3, 3)
    assert names["l1.mlp.down.b"].shape == (48,) and names["l1.mlp.gate.b"].shape == (40,)
    assert names["l3.mlp.router"].shape == (9, 48) and names["l3.mlp.correction"].shape == (9,) and "l3.mlp.e7.up" not in names
    assert "l3.mlp.e0.gate" not in names and names["l3.mlp.shared.up"].shape == (20, 48) and "l2.mlp.shared.up" not in names
    assert "l0.norm2" not in names and "l0.hc2.in" not in names and names["embed"].shape == names["head"].shape == (160, 48)


def test_kept_pages_stay_when_the_window_passes():
    from llmserver_b200.cache import CacheManager, KVPagesNeed
    from llmserver_b200.cache.manager import RELEASED
    cache = CacheManager([KVPagesNeed(1, 8, window=6, keep_first=5), KVPagesNeed(1, 8, window=6), KVPagesNeed(1, 8)], page_size=4, num_pages=12,
                         num_slots=2)
    assert [group.kept_pages for group in cache.groups] == [2, 0, 0]
    cache.admit("a")
    cache.ensure("a", 9)
    assert cache.advance("a", 9) == 1                   # position 9 sees 4 .. 9: page 0 goes where it is not kept
    assert [page == RELEASED for page in cache.table("a", 0)] == [False] * 3 and cache.table("a", 1)[0] == RELEASED
    cache.ensure("a", 24)
    assert cache.advance("a", 23) == 2 + 3              # position 23 sees 18 .. 23: pages 2 and 3; pages 1, 2 and 3
    assert [page == RELEASED for page in cache.table("a", 0)] == [False, False, True, True, False, False]
    assert cache.groups[0].pool.num_available == 12 - 4 and all(page != RELEASED for page in cache.table("a", 2))
    cache.check_invariants()
    cache.free("a")
    assert cache.available() == [12, 12, 12]
    with pytest.raises(ValueError):
        KVPagesNeed(1, 8, window=5, keep_first=-1)
    assert KVPagesNeed(1, 8, keep_first=7) == KVPagesNeed(1, 8)      # nothing to keep where nothing is given back


def test_part_parameters_are_checked():
    from llmserver_b200.parts import BLOCKS, FEED_FORWARDS, MIXERS
    attention = MIXERS.get("gqa_attention")
    base = dict(hidden=8, heads=2, kv_heads=1, head_dim=8, scale=1.0)
    for wrong in (dict(keep_first=-1), dict(chunk=4, keep_first=2), dict(gate=True, values_are_keys=True), dict(gate=True, conv=3)):
        with pytest.raises(ValueError):
            attention.check_params({**base, **wrong})
    attention.check_params({**base, "window": 4, "keep_first": 9, "gate": True, "qk_norm": True})
    routed = FEED_FORWARDS.get("routed_experts")
    base = dict(hidden=8, experts=6, top=2, intermediate=8, activation="squared_relu")
    for wrong in (dict(limit=7.0), dict(identity=-1), dict(identity=1, groups=(3, 1)), dict(top=9, identity=2), dict(identity=1, weight_on="input")):
        with pytest.raises(ValueError):
            routed.check_params({**base, **wrong})
    routed.check_params({**base, "identity": 3, "groups": (3, 1), "scores": "softmax", "top": 3})
    for wrong in (dict(width=10, blocks=3, conv=2), dict(width=10, blocks=0, conv=2), dict(width=10, blocks=2, conv=0)):
        with pytest.raises(ValueError):
            MIXERS.get("gated_linear_recurrent_unit").check_params(dict(hidden=8, **wrong))
    with pytest.raises(ValueError):
        FEED_FORWARDS.get("biased_glu").check_params(dict(hidden=8, intermediate=8, activation="relu"))
    with pytest.raises(ValueError):
        BLOCKS.get("hyper_connections").check_params(dict(streams=0))


def test_blocks_that_would_drop_a_bias_refuse_the_part():
    from types import SimpleNamespace

    from llmserver_b200.parts import BLOCKS
    part = SimpleNamespace(output_bias=torch.zeros(4), runtime=SimpleNamespace(device="cpu"), feeds_stream=False)
    plain_part = SimpleNamespace(runtime=SimpleNamespace(device="cpu"), feeds_stream=False)
    parts = {"mixer": plain_part, "feed_forward": part, "mixer_norm": plain_part, "feed_forward_norm": plain_part}
    with pytest.raises(ValueError):
        BLOCKS.get("pre_norm")({}, parts)
    weights = {prefix + name: torch.ones(shape) for prefix in ("hc1.", "hc2.") for name, shape in (("in", (2,)), ("out", (2,)), ("mix", (2, 2)))}
    BLOCKS.get("hyper_connections")({"streams": 2}, parts, weights)


def test_segments_of_the_gated_scan():
    """Long bfloat16 portions are cut into at most 128 segments of at least 32 tokens; short ones and 32-bit steps run in one
    pass; a given length is taken."""
    from llmserver_b200 import ops
    assert ops.SCAN_SEGMENT == 32 and ops.SCAN_MAX_SEGMENTS == 128
    choose = ops.scan_segment
    assert choose(torch.bfloat16, 63) == 0 and choose(torch.bfloat16, 64) == 32 and choose(torch.bfloat16, 4096) == 32
    assert choose(torch.bfloat16, 8193) == 65 and choose(torch.float32, 5000) == 0


# ------------------------------------------------------------------------------------------------ the plain implementation
def _random_weights(raw, seed):
    from llmserver_b200.weights.declare import declared_weights
    from llmserver_b200.weights.random_init import random_tensor
    _, spec = _spec(raw)
    return {name: random_tensor(name, declaration, seed).to(F64) for name, declaration in declared_weights(spec).items()}


def test_plain_recurrent_state_carries_over_portions():
    weights = _random_weights(MIXED_SIZES, 1)
    h = torch.randn((19, MIXED_SIZES["width"]), dtype=F64, generator=torch.Generator().manual_seed(2))
    for layer in (1, 2, 3):      # two, one and six taps
        mixer = MIXED_SIZES["layers"][layer]["mixer"]["right"]
        prefix = f"l{layer}.mix.right."
        whole, (last, history) = plain.recurrent_block(h, weights, prefix, mixer)
        out, state = [], None
        for begin, end in ((0, 1), (1, 3), (3, 4), (4, 12), (12, 19)):      # portions shorter than the convolution too
            piece, state = plain.recurrent_block(h[begin:end], weights, prefix, mixer, state=state)
            out.append(piece)
        assert torch.allclose(torch.cat(out), whole, atol=1e-12) and torch.allclose(state[0], last, atol=1e-12)
        assert torch.allclose(state[1], history, atol=1e-12) and history.shape == (mixer["conv"] - 1, mixer["width"])


def test_plain_scan_against_its_unrolled_sum():
    generator = torch.Generator().manual_seed(5)
    u = torch.randn((7, 3), dtype=F64, generator=generator)
    r, i = (torch.rand((7, 3), dtype=F64, generator=generator) for _ in range(2))
    lam = torch.tensor([-6.0, 0.5, 30.0], dtype=F64)
    states, last = plain.gated_scan(u, r, i, lam, torch.zeros(3, dtype=F64))
    decay = torch.exp(-8.0 * r * torch.nn.functional.softplus(lam))
    fed = torch.sqrt(1.0 - decay ** 2) * i * u
    for t in range(7):
        want = sum(torch.prod(decay[s + 1:t + 1], dim=0) * fed[s] for s in range(t + 1))
        assert torch.allclose(states[t], want, atol=1e-12)
    assert torch.equal(states[-1], last)


def test_plain_window_with_kept_tokens():
    weights = _random_weights(MIXED_SIZES, 3)
    h = torch.randn((40, MIXED_SIZES["width"]), dtype=F64, generator=torch.Generator().manual_seed(4))
    _, kept = plain.windowed_attention(h, weights, "l1.mix.left.", MIXED_SIZES["layers"][1]["mixer"]["left"], want_probabilities=True)
    p = kept[0][37]                                       # a window of 30 and three kept tokens: keys 0 .. 2 and 8 .. 37
    assert bool((p[:3] > 0).all()) and bool((p[3:8] == 0).all()) and bool((p[8:38] > 0).all()) and bool((p[38:] == 0).all())
    assert bool((kept[0][32][:33] > 0).all()) and kept[0][33][3] == 0 and kept[0][33][4] > 0      # 32 - 3 < 30, 33 - 3 is not
    _, kept = plain.windowed_attention(h, weights, "l2.mix.left.", MIXED_SIZES["layers"][2]["mixer"]["left"], want_probabilities=True)
    assert (kept[0][20] > 0).nonzero().flatten().tolist() == [0, 1, 20]


def test_plain_router_with_correction_groups_and_identities():
    z = torch.tensor([2.0, 0.0, 1.5, 1.4, 0.3, 0.2], dtype=F64)          # the last two may be identities: nothing tells them apart here
    none = torch.zeros(6, dtype=F64)
    chosen, share = plain.route(z, none, {"top": 2, "groups": {"count": 3, "keep": 1}})
    assert chosen == [0, 1] and abs(float(share.sum()) - 1.0) < 1e-12    # expert 0's group wins, although its other is weak
    assert plain.route(z, none, {"top": 2})[0] == [0, 2]
    # the correction steers experts and groups and does not enter the weights; it may make every choice score negative
    pushed = torch.tensor([-2.0, -2.0, -2.0, -2.0, -1.0, -1.5], dtype=F64)
    chosen, share = plain.route(z, pushed, {"top": 3, "groups": {"count": 3, "keep": 2}})
    assert chosen == [4, 5, 0]
    s = torch.softmax(z, dim=-1)
    assert torch.allclose(share, s[chosen] / s[chosen].sum(), atol=1e-12)
    weights = _random_weights(TENSOR_CORE_SIZES, 2)
    mlp = TENSOR_CORE_SIZES["layers"][2]["mlp"]
    only = dict(weights)
    only["l2.mlp.correction"] = torch.tensor([-9.0] * 14 + [5.0] * 4, dtype=F64)       # identities alone: the input comes back
    h = torch.randn((3, 256), dtype=F64, generator=torch.Generator().manual_seed(8))
    assert torch.allclose(plain.routed_feed_forward(h, only, "l2.mlp.", mlp), h, atol=1e-12)


def test_plain_streams_are_written_from_the_old_ones():
    generator = torch.Generator().manual_seed(9)
    x = torch.randn((3, 2, 4), dtype=F64, generator=generator)
    y = torch.randn((2, 4), dtype=F64, generator=generator)
    weights = {"hc.in": torch.randn(3, dtype=F64, generator=generator), "hc.out": torch.randn(3, dtype=F64, generator=generator),
               "hc.mix": torch.randn((3, 3), dtype=F64, generator=generator)}
    new = plain.write_streams(x, y, weights, "hc.")
    for t in range(3):
        want = weights["hc.out"][t] * y + sum(weights["hc.mix"][s, t] * x[s] for s in range(3))
        assert torch.allclose(new[t], want, atol=1e-12)
    assert torch.allclose(plain.read_streams(x, weights, "hc."), sum(weights["hc.in"][s] * x[s] for s in range(3)), atol=1e-12)
    assert torch.allclose(plain.sinusoids(torch.tensor([0]), 5)[0], torch.tensor([0.0, 1.0, 0.0, 1.0, 0.0], dtype=F64))


def test_plain_forward_runs_every_configuration():
    for name, (raw, seed) in RAPOLIX.items():
        weights = _random_weights(raw, seed)
        tokens = [(7 * i + 3) % raw["vocab"] for i in range(11)]
        streams = []
        logits = plain.forward(raw, weights, tokens, streams=streams)
        assert logits.shape == (11, raw["vocab"]) and len(streams) == len(raw["layers"]) and bool(torch.isfinite(logits).all())
        changed = plain.forward(raw, weights, tokens[:-1] + [(tokens[-1] + 1) % raw["vocab"]])      # causal
        assert torch.allclose(changed[:-1], logits[:-1], atol=1e-12) and not torch.allclose(changed[-1], logits[-1], rtol=0, atol=1e-14)
    assert ODD_SIZES["width"] % 2 == 1
