"""Small Dozotar configurations of the tests.  Between them they vary what a configuration may vary: the order of the three
kinds of layers, layers with a dense, a routed and no feed-forward, grouped and ungrouped query heads, value heads smaller
and larger than key heads, chunks of one position, of a few, of some pages and longer than any prompt, no chunks, few and
many distance buckets whose last one is reached early, late or never, convolutions of one to six taps, all or a part of a
retention head rotating or nothing of it, decays of one and below it (a head that forgets at once
reads little but its own token, and its sign is all that the division by its root mean square leaves of q . k: rounding
would decide it), state-space groups of one and of several heads,
norm parts smaller and larger than a head and ones that cut heads in two, routers whose groups are all kept, half kept or
absent, as many experts chosen as the kept groups hold, and shared experts beside them or none."""


def _attention(heads, kv_heads, dim, vdim, conv, scale, bias_max, buckets, size, mlp):
    return {"type": "attention", "mlp": mlp,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv, "scale": scale, "bias_max": bias_max,
                      "buckets": buckets, "mask": {"size": size} if size else None}}


def _retention(dim, vdim, decay, dims, mlp, base=10000.0):
    return {"type": "retention", "mlp": mlp, "mixer": {"heads": len(decay), "dim": dim, "vdim": vdim, "decay": decay,
                                                       "rot": {"base": base, "dims": dims} if dims else None}}


def _mamba(heads, vdim, state, groups, conv, norm_groups, mlp):
    return {"type": "mamba2", "mlp": mlp, "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv,
                                                    "norm_groups": norm_groups}}


def _dense(ff):
    return {"kind": "dense", "ff": ff}


def _moe(experts, top, ff, groups=None, shared=None):
    return {"kind": "moe", "router": {"experts": experts, "top": top, "groups": {"count": groups[0], "keep": groups[1]} if groups else None},
            "expert": {"ff": ff}, "shared": {"ff": shared} if shared else None}


ATTENTION_ONLY = {
    "architecture": "Dozotar", "vocab": 160, "width": 48, "norm": {"eps": 1e-5},
    "layers": [
        _attention(3, 3, 16, 24, 2, 0.25, 20, 8, 7, None),
        _attention(6, 2, 8, 8, 5, 0.4, 64, 32, 50, _dense(40)),
        _attention(2, 1, 24, 40, 1, 0.2, 9, 4, 1, _moe(6, 2, 24)),
        _attention(4, 4, 12, 10, 4, 0.3, 500, 16, 400, _moe(9, 3, 16, (3, 2), 20)),
        _attention(2, 2, 16, 16, 3, 0.25, 40, 12, None, None),
    ],
}

RETENTION_ONLY = {
    "architecture": "Dozotar", "vocab": 150, "width": 40, "norm": {"eps": 1e-6},
    "layers": [
        _retention(24, 33, [0.999, 0.93], 8, None),
        _retention(8, 16, [1.0, 0.98, 0.9, 0.8, 0.96], 8, _dense(72), base=50.0),
        _retention(72, 20, [0.995], 2, _moe(8, 4, 24, (2, 1), 16)),
        _retention(40, 7, [0.97, 0.99, 0.85], None, None),
    ],
}

MAMBA_ONLY = {
    "architecture": "Dozotar", "vocab": 170, "width": 56, "norm": {"eps": 1e-5},
    "layers": [
        _mamba(3, 10, 20, 1, 2, 5, None),
        _mamba(6, 8, 12, 3, 4, 4, _dense(64)),
        _mamba(2, 33, 70, 2, 1, 1, _moe(16, 5, 16, (4, 4), 24)),
        _mamba(4, 16, 40, 2, 6, 2, None),
    ],
}

ALL_KINDS = {
    "architecture": "Dozotar", "vocab": 300, "width": 96, "norm": {"eps": 1e-6},
    "layers": [
        _retention(16, 24, [0.999, 0.96, 0.8], 10, _dense(128), base=1e5),
        _attention(4, 2, 16, 16, 3, 0.25, 60, 16, 45, _moe(10, 3, 32, (5, 2), 40)),
        _mamba(6, 16, 24, 2, 3, 3, _moe(10, 3, 32, (5, 3), 56)),
        _attention(2, 1, 32, 48, 4, 0.18, 30, 10, 20, _dense(96)),
        _mamba(3, 32, 16, 1, 4, 1, _moe(8, 2, 40, (4, 2), 40)),
        _retention(32, 16, [0.99, 0.9, 0.97, 0.7], 32, None),
    ],
}

# sizes at which the bfloat16 path takes its tensor-core kernels (heads of 64 and 128, widths and experts in 64s)
TENSOR_CORE_SIZES = {
    "architecture": "Dozotar", "vocab": 384, "width": 192, "norm": {"eps": 1e-6},
    "layers": [
        _attention(4, 2, 128, 128, 4, 0.09, 90, 32, 100, _moe(12, 3, 64, (3, 2), 128)),
        _mamba(4, 64, 64, 1, 4, 2, _dense(256)),
        _attention(4, 1, 64, 64, 3, 0.125, 40, 16, 70, _moe(8, 2, 128, (4, 3), 64)),
        _retention(64, 128, [0.998, 0.9], 64, _dense(192)),
        _attention(6, 2, 128, 64, 2, 0.09, 128, 24, 64, _moe(12, 4, 64, (6, 3), 64)),
        _mamba(6, 64, 128, 2, 3, 3, _moe(8, 2, 64, (2, 2), 192)),
    ],
}

# name -> (config.json contents, seed of the random weights)
DOZOTAR = {"attention_only": (ATTENTION_ONLY, 3), "retention_only": (RETENTION_ONLY, 4), "mamba_only": (MAMBA_ONLY, 5),
           "all_kinds": (ALL_KINDS, 6), "tensor_core_sizes": (TENSOR_CORE_SIZES, 7)}
