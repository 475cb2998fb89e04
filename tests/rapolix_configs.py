"""Small Rapolix configurations of the tests.  Between them they vary what a configuration may vary: one, two, three and five
residual streams, odd widths, layers with a dense, a routed and no feed-forward, grouped and ungrouped query heads, value heads
smaller and larger than key heads, windows of one position, of a few, of some pages and longer than any prompt, no window, no
kept tokens, one, a few, more than a page, more than a tile of the kernels and more than the window of them, convolutions of
one to six taps, recurrent branches narrower and wider than the model in one block and in many, of sizes with and without a
factor of four, routers with and without groups and identity outputs, whose groups mix experts and identities, with as many
outputs chosen as the kept groups hold, shared experts beside them or none, capped and uncapped logits."""


def _layer(left, right, mlp):
    heads, kv_heads, dim, vdim, scale, mask = left
    width, blocks, conv = right
    return {"type": "parallel", "mlp": mlp,
            "mixer": {"left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale,
                               "mask": {"size": mask[0], "keep_first": mask[1]} if mask else None},
                      "right": {"width": width, "blocks": blocks, "conv": conv}}}


def _dense(ff):
    return {"kind": "dense", "ff": ff}


def _moe(experts, top, ff, groups=None, identity=0, shared=None):
    return {"kind": "moe", "router": {"experts": experts, "top": top, "identity": identity,
                                      "groups": {"count": groups[0], "keep": groups[1]} if groups else None},
            "expert": {"ff": ff}, "shared": {"ff": shared} if shared else None}


MIXED_SIZES = {
    "architecture": "Rapolix", "vocab": 160, "width": 48, "streams": 3, "norm": {"eps": 1e-5}, "logit_softcap": 9.0,
    "layers": [
        _layer((3, 3, 16, 24, 0.25, (7, 0)), (40, 2, 4), None),
        _layer((6, 2, 8, 8, 0.4, (30, 3)), (63, 3, 2), _dense(40)),
        _layer((2, 1, 24, 40, 0.2, (1, 2)), (20, 1, 1), _moe(6, 2, 24)),
        _layer((4, 4, 12, 10, 0.3, (400, 5)), (96, 12, 6), _moe(7, 3, 16, (3, 2), 2, 20)),
        _layer((2, 2, 16, 16, 0.25, None), (36, 4, 3), _moe(5, 4, 20, (4, 2), 3)),
    ],
}

# an odd width, five streams: the kernels' forms without vectors
ODD_SIZES = {
    "architecture": "Rapolix", "vocab": 151, "width": 45, "streams": 5, "norm": {"eps": 1e-6}, "logit_softcap": None,
    "layers": [
        _layer((5, 1, 9, 7, 0.35, (12, 20)), (33, 3, 5), _moe(9, 5, 13, (5, 3), 1, 11)),
        _layer((3, 3, 14, 14, 0.3, (25, 1)), (54, 2, 3), _dense(29)),
        _layer((2, 2, 10, 21, 0.3, (40, 9)), (45, 9, 4), None),
    ],
}

# sizes at which the bfloat16 path takes its tensor-core kernels
TENSOR_CORE_SIZES = {
    "architecture": "Rapolix", "vocab": 384, "width": 256, "streams": 2, "norm": {"eps": 1e-6}, "logit_softcap": 20.0,
    "layers": [
        _layer((4, 2, 128, 128, 0.09, (50, 6)), (192, 3, 4), _moe(12, 3, 64, (7, 4), 2, 128)),
        _layer((8, 1, 64, 64, 0.125, (33, 70)), (128, 1, 2), _dense(192)),
        _layer((2, 2, 128, 128, 0.09, (100, 130)), (320, 5, 3), _moe(14, 4, 128, None, 4)),
        _layer((4, 1, 64, 128, 0.125, (70, 17)), (256, 4, 4), None),
        _layer((12, 2, 128, 64, 0.08, (64, 64)), (256, 2, 4), _dense(320)),
    ],
}

ONE_STREAM = {
    "architecture": "Rapolix", "vocab": 200, "width": 64, "streams": 1, "norm": {"eps": 1e-4}, "logit_softcap": 30.0,
    "layers": [
        _layer((4, 1, 16, 16, 0.3, (20, 4)), (64, 4, 4), _moe(4, 1, 32, (2, 1), 0, 32)),
        _layer((4, 2, 32, 16, 0.2, (45, 0)), (80, 5, 2), _dense(128)),
    ],
}

# name -> (config.json contents, seed of the random weights)
RAPOLIX = {"mixed_sizes": (MIXED_SIZES, 3), "odd_sizes": (ODD_SIZES, 4), "tensor_core_sizes": (TENSOR_CORE_SIZES, 5), "one_stream": (ONE_STREAM, 6)}
