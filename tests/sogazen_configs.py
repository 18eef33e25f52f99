"""Tiny Sogazen configurations for the tests: they differ in every size, option and layer order.

SOG_A: both mixers, a dense feed-forward and two mixtures; six query heads on two key heads, a part of the head turning;
heads in groups, the row normalised in other parts than heads; two identity experts among five outputs' choices.
SOG_B: what a configuration may leave out: no rotation, no caps, no identity experts, a layer without feed-forward; one head;
one tap (no convolution tail); the best one of three experts; time mixing first.
SOG_C: sizes of the tensor-core kernels (heads of 64 and of 128, experts on tensor-core tiles), a state of 128, time mixers of
64 and 128 numbers a head, a dense feed-forward of many rows.
SOG_D: sizes that are multiples of little (width 36, heads of 6 with 2 dimensions turning, a state of 5, time-mixing heads of
7, an odd inner width of the decay), every output of the router chosen.
SOG_E: heads that are rounded up to the tensor cores' sizes (40 and 80), long prompts, six taps, one expert beside
three identity experts.
"""

import json
import random
from pathlib import Path

import torch


def _pair(left, right, mlp):
    return {"type": "parallel", "mixer": {"left": left, "right": right}, "mlp": mlp}


def _time(heads, dim, mlp, rank=None):
    mixer = {"heads": heads, "dim": dim}
    if rank:
        mixer["decay_rank"] = rank
    return {"type": "wkv", "mixer": mixer, "mlp": mlp}


def _left(heads, kv_heads, dim, scale, softcap=None, rot=None):
    out = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale}
    if softcap:
        out["softcap"] = softcap
    if rot:
        out["rot"] = {"dims": rot[0], "base": rot[1]}
    return out


def _right(heads, vdim, state, groups, conv, norm_groups):
    return {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv, "norm_groups": norm_groups}


def _dense(ff, limit):
    return {"kind": "dense", "ff": ff, "limit": limit}


def _moe(ff, experts, top, identity=None):
    router = {"experts": experts, "top": top}
    if identity:
        router["identity"] = identity
    return {"kind": "moe", "expert": {"ff": ff}, "router": router}


SOG_A = {
    "architecture": "Sogazen", "vocab": 211, "width": 64, "norm": {"eps": 1e-5}, "logit_softcap": 9.0,
    "layers": [
        _pair(_left(6, 2, 16, 0.3, 20.0, (8, 500.0)), _right(4, 12, 20, 2, 3, 3), _dense(40, 0.9)),
        _time(3, 20, _moe(24, 3, 2, 2), 12),
        _pair(_left(4, 4, 12, 0.4, 6.0, (12, 10000.0)), _right(6, 8, 16, 3, 4, 1), _moe(20, 6, 3, 1)),
    ],
}

SOG_B = {
    "architecture": "Sogazen", "vocab": 129, "width": 48, "norm": {"eps": 1e-6},
    "layers": [
        _time(1, 20, _moe(16, 3, 1), 5),
        _pair(_left(1, 1, 20, 0.5), _right(1, 9, 11, 1, 1, 1), None),
        _pair(_left(3, 3, 8, 0.35, None, (4, 100.0)), _right(2, 16, 24, 1, 2, 4), _dense(24, 2.5)),
        _time(2, 16, None),
    ],
}

SOG_C = {
    "architecture": "Sogazen", "vocab": 200, "width": 128, "norm": {"eps": 1e-5}, "logit_softcap": 12.0,
    "layers": [
        _pair(_left(4, 2, 64, 0.15, 15.0, (32, 5000.0)), _right(4, 64, 128, 2, 4, 2), _moe(64, 6, 3, 2)),
        _time(2, 64, _dense(256, 1.2)),
        _pair(_left(3, 1, 128, 0.1, 30.0, (128, 20000.0)), _right(2, 48, 64, 1, 4, 1), _moe(32, 4, 4, 4)),
        _time(1, 128, _moe(96, 4, 2)),
    ],
}

SOG_D = {
    "architecture": "Sogazen", "vocab": 97, "width": 36, "norm": {"eps": 1e-4}, "logit_softcap": 5.0,
    "layers": [
        _pair(_left(3, 3, 6, 0.5, 3.0, (2, 37.0)), _right(3, 7, 5, 3, 5, 7), _moe(10, 3, 5, 2)),
        _time(5, 7, _dense(11, 0.5), 3),
        _pair(_left(5, 1, 7, 0.6), _right(10, 1, 3, 5, 2, 2), _moe(7, 2, 3, 5)),
    ],
}

SOG_E = {
    "architecture": "Sogazen", "vocab": 500, "width": 160, "norm": {"eps": 1e-5}, "logit_softcap": 20.0,
    "layers": [
        _pair(_left(6, 2, 40, 0.16, 25.0, (24, 3000.0)), _right(4, 40, 48, 4, 6, 2), _dense(224, 1.0)),
        _pair(_left(4, 4, 80, 0.11, 40.0, (80, 10000.0)), _right(8, 24, 136, 2, 4, 8), _moe(56, 5, 2, 3)),
        _time(4, 48, _moe(40, 1, 1, 3), 24),
    ],
}

# name -> (config, seed, page size)
ALL = {"sog_a": (SOG_A, 61, 16), "sog_b": (SOG_B, 62, 4), "sog_c": (SOG_C, 63, 16), "sog_d": (SOG_D, 64, 8),
       "sog_e": (SOG_E, 65, 16)}


def write_model(config: dict, out_dir, seed: int) -> Path:
    """A random model whose vectors (biases, corrections, weights of norms) are far from their neutral values and whose
    matrices give every mechanism something to do."""
    from safetensors.torch import load_file, save_file

    from liteinfer_b200.weights.random_init import write_random_model

    path = write_random_model(config, out_dir, seed)
    tensors = load_file(str(path / "model.safetensors"))
    g = torch.Generator().manual_seed(seed + 1000)
    for name in sorted(tensors):
        t = tensors[name]
        noise = torch.randn(t.shape, generator=g)
        if name.endswith((".q.b", ".k.b", ".conv.b")):
            t = 0.3 * noise
        elif name.endswith((".norm", ".norm1", ".norm2", ".out", ".D")):
            t = 1.0 + 0.3 * noise
        elif name.endswith(".correction"):
            t = 0.2 * noise
        elif name.endswith((".dt_bias", ".A_log", ".w0", ".u", ".conv")) or ".mu." in name:
            continue
        elif t.dim() == 2:
            t = noise * t.shape[1] ** -0.5
        tensors[name] = t.to(torch.bfloat16)
    save_file({n: t.to(torch.bfloat16).contiguous() for n, t in tensors.items()}, str(path / "model.safetensors"))
    return path


def random_config(seed: int) -> dict:
    """A configuration drawn at random: two to five layers of both kinds, sizes of the SIMT kernels and of the tensor-core
    ones, rotations, caps, groups, identity experts and feed-forwards or none."""
    rng = random.Random(seed)
    layers = []
    for _ in range(rng.randint(2, 5)):
        mlp, kind = None, rng.random()
        if kind < 0.35:
            mlp = _dense(rng.choice([24, 64, 200, 96]), rng.choice([0.7, 1.5, 4.0]))
        elif kind < 0.9:
            experts, identity = rng.choice([1, 2, 4, 7]), rng.choice([None, 1, 3, 6])
            mlp = _moe(rng.choice([24, 64, 96, 33]), experts, rng.randint(1, min(experts + (identity or 0), 5)), identity)
        if rng.random() < 0.4:
            layers.append(_time(rng.choice([1, 2, 4, 5]), rng.choice([16, 30, 64, 72, 128]), mlp, rng.choice([None, 4, 20, 33])))
            continue
        heads, dim = rng.choice([2, 4, 6, 8]), rng.choice([24, 32, 56, 64, 88, 128])
        left = _left(heads, rng.choice([k for k in (1, 2, 3, 4, 8) if heads % k == 0]), dim, dim ** -0.5,
                     rng.choice([None, 5.0, 30.0]), rng.choice([None, (dim // 4 * 2, 10000.0), (dim, 500.0)]))
        groups = rng.choice([1, 2, 3])
        heads, vdim = groups * rng.choice([1, 2, 4]), rng.choice([8, 24, 32, 64])
        right = _right(heads, vdim, rng.choice([16, 24, 64, 100, 128]), groups, rng.choice([1, 2, 3, 4, 7]),
                       rng.choice([1, 2, 4, heads]))
        layers.append(_pair(left, right, mlp))
    config = {"architecture": "Sogazen", "vocab": rng.choice([300, 777, 1000]), "width": rng.choice([96, 128, 160, 320]),
              "norm": {"eps": rng.choice([1e-5, 1e-6])}, "layers": layers}
    if rng.random() < 0.7:
        config["logit_softcap"] = rng.choice([10.0, 25.0])
    return config


def prompt(vocab: int, length: int, seed: int) -> list[int]:
    rng = random.Random(seed)
    return [rng.randrange(vocab) for _ in range(length)]


def changed(config: dict, path, value) -> dict:
    """A copy of `config` with the entry at `path` replaced."""
    out = json.loads(json.dumps(config))
    at = out
    for key in path[:-1]:
        at = at[key]
    at[path[-1]] = value
    return out


# Largest absolute difference of float32 logits from the float64 plain implementation that rounding alone explains.
FLOAT32_TOLERANCE = {"sog_a": 1e-4, "sog_b": 1e-4, "sog_c": 2e-4, "sog_d": 1e-4, "sog_e": 2e-4}
