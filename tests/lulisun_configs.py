"""Tiny Lulisun configurations for the tests: they differ in every size, option and layer order.

LUL_A: two layers with tensors of their own and three that borrow them (two directly, one through a borrower's entry);
values wider than keys; chunks of 10; six experts in three groups of which two are kept; a shared expert of another
width than the experts.
LUL_B: what a configuration may leave out: no rotation, no chunks, no groups, no shared expert, a layer without
feed-forward; one head; the left scale 0 in one layer; the best one of three experts; odd sizes.
LUL_C: sizes of the tensor-core kernels (keys and values of 64, and of 128 with values of 256, chunks longer than a tile
of keys; experts on tensor-core tiles, a shared expert twice as wide as an expert).
LUL_D: sizes that are multiples of little (width 36, heads of 6 with 2 dimensions turning, values of 10, a memory of 5 x
7), a chunk of one token, every expert chosen, eight experts in four groups with one kept.
LUL_E: heads that are rounded up to the tensor cores' sizes (keys of 40 with values of 136, keys of 80 with values of 112),
chunks of some dozens, prompts of a few hundred tokens, a memory of 72 x 40.
"""

import random


def _layer(left, right, mlp, scales=(1.1, 0.7), **more):
    return {"type": "parallel", "mixer": {"left": left, "right": right, "left_scale": scales[0], "right_scale": scales[1]},
            "mlp": mlp, **more}


def _moe(ff, experts, top, groups=None, shared=None):
    router = {"experts": experts, "top": top}
    if groups:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    out = {"kind": "moe", "expert": {"ff": ff}, "router": router}
    if shared:
        out["shared"] = {"ff": shared}
    return out


def _left(heads, kv_heads, dim, vdim, scale, chunk=None, rot=None):
    out = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if chunk:
        out["mask"] = {"size": chunk}
    if rot:
        out["rot"] = {"dims": rot[0], "base": rot[1]}
    return out


def _right(heads, dim, vdim):
    return {"heads": heads, "dim": dim, "vdim": vdim}


_A0 = (_left(4, 2, 16, 24, 0.3, 10, (8, 500.0)), _right(3, 12, 20), _moe(20, 6, 2, (3, 2), 28), (0.9, 1.3))
_A1 = (_left(2, 1, 12, 8, 0.25, 17, (12, 10000.0)), _right(2, 20, 12), _moe(12, 4, 3, (2, 2), 12), (-0.6, 0.8))

LUL_A = {
    "architecture": "Lulisun", "vocab": 211, "width": 64, "norm": {"eps": 1e-5},
    "layers": [_layer(*_A0), _layer(*_A1), _layer(*_A0, weights_of=0), _layer(*_A1, weights_of=1), _layer(*_A0, weights_of=2)],
}

LUL_B = {
    "architecture": "Lulisun", "vocab": 129, "width": 48, "norm": {"eps": 1e-6},
    "layers": [
        _layer(_left(1, 1, 20, 28, 0.5), _right(1, 9, 11), _moe(16, 3, 1)),
        _layer(_left(3, 3, 8, 8, 0.35, 6, (4, 100.0)), _right(2, 16, 16), None, (0.0, 1.0)),
        _layer(_left(2, 2, 10, 7, 0.4, None, (10, 50.0)), _right(3, 7, 5), _moe(24, 5, 2, None, 17), (1.0, 0.0)),
    ],
}

LUL_C = {
    "architecture": "Lulisun", "vocab": 200, "width": 128, "norm": {"eps": 1e-5},
    "layers": [
        _layer(_left(4, 2, 64, 64, 0.15, 70, (32, 5000.0)), _right(2, 64, 48), _moe(64, 8, 2, (4, 3), 128), (0.8, 0.9)),
        _layer(_left(2, 1, 128, 256, 0.1, 130, (128, 20000.0)), _right(1, 128, 64), _moe(32, 4, 4, None, 32), (1.4, 0.5)),
        _layer(_left(4, 4, 64, 128, 0.12, 33), _right(4, 32, 32), None),
    ],
}

LUL_D = {
    "architecture": "Lulisun", "vocab": 97, "width": 36, "norm": {"eps": 1e-4},
    "layers": [
        _layer(_left(3, 3, 6, 10, 0.5, 1, (2, 37.0)), _right(5, 5, 7), _moe(10, 8, 2, (4, 1), 6), (2.0, 0.4)),
        _layer(_left(4, 2, 12, 4, 0.2, 21, (8, 900.0)), _right(1, 33, 3), _moe(7, 4, 4, (1, 1), 14), (0.3, 1.7)),
        _layer(_left(5, 1, 7, 3, 0.6, 4), _right(2, 1, 6), _moe(5, 6, 2, (6, 3), 5)),
    ],
}

LUL_E = {
    "architecture": "Lulisun", "vocab": 500, "width": 192, "norm": {"eps": 1e-5},
    "layers": [
        _layer(_left(6, 2, 40, 136, 0.16, 48, (24, 3000.0)), _right(4, 72, 40), _moe(96, 6, 3, (2, 1), 48), (0.7, 1.1)),
        _layer(_left(4, 4, 80, 112, 0.11, 150, (80, 10000.0)), _right(2, 40, 136), _moe(56, 4, 2, None, 112), (1.2, 0.6)),
    ],
}

# name -> (config, seed, page size)
ALL = {"lul_a": (LUL_A, 51, 16), "lul_b": (LUL_B, 52, 4), "lul_c": (LUL_C, 53, 16), "lul_d": (LUL_D, 54, 8),
       "lul_e": (LUL_E, 55, 16)}


def random_config(seed: int) -> dict:
    """A configuration drawn at random: two to five layers, some of which borrow another one's tensors, sizes of the SIMT
    kernels and of the tensor-core ones, chunks, rotations, groups, shared experts and feed-forwards or none."""
    rng = random.Random(seed)
    layers = []
    for i in range(rng.randint(2, 5)):
        owners = [j for j, layer in enumerate(layers) if "weights_of" not in layer]
        if owners and rng.random() < 0.4:
            j = rng.choice(owners)
            layers.append({**layers[j], "weights_of": j})
            continue
        heads, dim = rng.choice([2, 4, 6, 8]), rng.choice([24, 32, 56, 64, 88, 128])
        left = _left(heads, rng.choice([k for k in (1, 2, 3, 4, 8) if heads % k == 0]), dim,
                     rng.choice([dim, dim, 2 * dim, 32, 64, 176]), dim ** -0.5, rng.choice([None, 16, 37, 64, 100, 128]),
                     rng.choice([None, (dim // 4 * 2, 10000.0), (dim, 500.0)]))
        right = _right(rng.choice([1, 2, 3, 4]), rng.choice([16, 30, 64, 100, 128]), rng.choice([16, 24, 50, 64, 128]))
        mlp = None
        if rng.random() < 0.85:
            groups, per, ff = rng.choice([1, 2, 4]), rng.choice([2, 3, 4]), rng.choice([24, 64, 96])
            keep = rng.randint(1, groups)
            mlp = _moe(ff, groups * per, rng.randint(1, min(keep * per, 4)),
                       (groups, keep) if groups > 1 or rng.random() < 0.5 else None,
                       rng.choice([None, ff, 2 * ff, 40, 100]))
        layers.append(_layer(left, right, mlp, (rng.choice([0.5, 1.0, 1.5]), rng.choice([0.4, 1.0, -0.8]))))
    return {"architecture": "Lulisun", "vocab": rng.choice([300, 777, 1000]), "width": rng.choice([96, 128, 160, 320]),
            "norm": {"eps": 1e-5}, "layers": layers}


def prompt(vocab: int, length: int, seed: int) -> list[int]:
    rng = random.Random(seed)
    return [rng.randrange(vocab) for _ in range(length)]


# Largest absolute difference of float32 logits from the float64 plain implementation that rounding alone explains.
FLOAT32_TOLERANCE = {"lul_a": 5e-5, "lul_b": 5e-5, "lul_c": 1e-4, "lul_d": 5e-5, "lul_e": 1e-4}
