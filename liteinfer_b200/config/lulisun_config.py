"""Typed configuration of the Lulisun decoder, read from its config.json.

A Lulisun config.json names everything per layer:

    {"architecture": "Lulisun", "vocab": V, "width": D, "norm": {"eps": e},
     "layers": [{"type": "parallel",
                 "mixer": {"left": {"heads", "kv_heads", "dim", "vdim", "scale", "rot": {dims, base} | null,
                                    "mask": {size} | null},
                           "right": {"heads", "dim", "vdim"}, "left_scale": a, "right_scale": b},
                 "mlp": {"kind": "moe", "expert": {"ff": F}, "shared": {"ff": F'} | null,
                         "router": {"experts": E, "top": k, "groups": {"count": n, "keep": g} | null}} | null,
                 "weights_of": j | null}, ...]}

Sizes and constants have no defaults: a missing one is a `ConfigError`.  An option that is absent or null is off (no
rotation, every earlier key visible, no expert groups, no shared expert, no feed-forward, weights of its own).  A layer
with `weights_of` is another run of layer j, with a cache and state of its own.
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Any

from liteinfer_b200.config.kegizen_config import _need
from liteinfer_b200.config.model_config import ConfigError

MIXER_TYPES = ("parallel",)


def _at_least_one(where: str, **sizes: int) -> None:
    for name, value in sizes.items():
        if value < 1:
            raise ConfigError(f"config.json {where}.{name} must be >= 1, got {value}")


@dataclass(frozen=True)
class LulisunAttention:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    chunk: int | None = None         # a position reads the positions of its own chunk of this many, up to itself
    rot_dims: int = 0                # the first dimensions of a head that turn (0: none)
    rot_base: float = 0.0

    @classmethod
    def from_dict(cls, raw: dict[str, Any], where: str) -> "LulisunAttention":
        heads, kv_heads, dim, vdim = (_need(raw, n, int, where) for n in ("heads", "kv_heads", "dim", "vdim"))
        _at_least_one(where, heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim)
        if heads % kv_heads:
            raise ConfigError(f"config.json {where}: heads={heads} is not a multiple of kv_heads={kv_heads}")
        mask, rot = raw.get("mask"), raw.get("rot")
        chunk = None
        if mask:
            chunk = _need(mask, "size", int, where + ".mask")
            _at_least_one(where + ".mask", size=chunk)
        dims, base = 0, 0.0
        if rot and rot.get("dims") != 0:
            dims, base = _need(rot, "dims", int, where + ".rot"), _need(rot, "base", float, where + ".rot")
            if dims < 2 or dims % 2 or dims > dim or not base > 0:
                raise ConfigError(f"config.json {where}.rot: dims={dims} must be even and within the head's {dim} "
                                  "dimensions, base > 0")
        return cls(heads, kv_heads, dim, vdim, _need(raw, "scale", float, where), chunk, dims, base)

    def to_dict(self) -> dict[str, Any]:
        out: dict[str, Any] = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim,
                               "scale": self.scale}
        if self.chunk is not None:
            out["mask"] = {"size": self.chunk}
        if self.rot_dims:
            out["rot"] = {"dims": self.rot_dims, "base": self.rot_base}
        return out


@dataclass(frozen=True)
class LulisunMemory:
    heads: int
    dim: int
    vdim: int

    @classmethod
    def from_dict(cls, raw: dict[str, Any], where: str) -> "LulisunMemory":
        sizes = {n: _need(raw, n, int, where) for n in ("heads", "dim", "vdim")}
        _at_least_one(where, **sizes)
        return cls(**sizes)

    def to_dict(self) -> dict[str, Any]:
        return {"heads": self.heads, "dim": self.dim, "vdim": self.vdim}


@dataclass(frozen=True)
class LulisunMoE:
    ff: int                          # the width of one expert
    experts: int
    top: int
    groups: int = 1                  # experts form this many equal groups of neighbours ...
    groups_keep: int = 1             # ... of which only the best this many can be chosen from
    shared_ff: int = 0               # the width of the expert that every token runs (0: there is none)

    @classmethod
    def from_dict(cls, raw: dict[str, Any], where: str) -> "LulisunMoE":
        if raw.get("kind", "moe") != "moe":
            raise ConfigError(f"config.json {where} has kind {raw.get('kind')!r}; known: ['moe']")
        router, groups, shared = raw.get("router"), (raw.get("router") or {}).get("groups"), raw.get("shared")
        moe = cls(_need(raw.get("expert"), "ff", int, where + ".expert"),
                  _need(router, "experts", int, where + ".router"), _need(router, "top", int, where + ".router"),
                  _need(groups, "count", int, where + ".router.groups") if groups else 1,
                  _need(groups, "keep", int, where + ".router.groups") if groups else 1,
                  _need(shared, "ff", int, where + ".shared") if shared else 0)
        _at_least_one(where, ff=moe.ff, experts=moe.experts, top=moe.top, groups=moe.groups, keep=moe.groups_keep)
        if shared:
            _at_least_one(where + ".shared", ff=moe.shared_ff)
        if moe.experts % moe.groups or moe.groups_keep > moe.groups:
            raise ConfigError(f"config.json {where}.router.groups: count={moe.groups} must divide experts={moe.experts}, "
                              f"and keep={moe.groups_keep} must not exceed it")
        if moe.top > moe.groups_keep * (moe.experts // moe.groups):
            raise ConfigError(f"config.json {where}.router: the kept groups hold fewer experts than top={moe.top}")
        return moe

    def to_dict(self) -> dict[str, Any]:
        router: dict[str, Any] = {"experts": self.experts, "top": self.top}
        if self.groups > 1:
            router["groups"] = {"count": self.groups, "keep": self.groups_keep}
        out: dict[str, Any] = {"kind": "moe", "expert": {"ff": self.ff}, "router": router}
        if self.shared_ff:
            out["shared"] = {"ff": self.shared_ff}
        return out


@dataclass(frozen=True)
class LulisunLayer:
    left: LulisunAttention
    right: LulisunMemory
    left_scale: float
    right_scale: float
    mlp: LulisunMoE | None
    weights_of: int | None = None    # the layer whose tensors this one uses (never one that borrows them itself)

    @classmethod
    def from_dict(cls, raw: dict[str, Any], where: str) -> "LulisunLayer":
        if raw.get("type") not in MIXER_TYPES:
            raise ConfigError(f"config.json {where} has type {raw.get('type')!r}; known: {list(MIXER_TYPES)}")
        mixer, at, mlp = raw.get("mixer"), where + ".mixer", raw.get("mlp")
        if not isinstance(mixer, dict):
            raise ConfigError(f"config.json {where} has no 'mixer'")
        return cls(LulisunAttention.from_dict(mixer.get("left"), at + ".left"),
                   LulisunMemory.from_dict(mixer.get("right"), at + ".right"),
                   _need(mixer, "left_scale", float, at), _need(mixer, "right_scale", float, at),
                   None if mlp is None else LulisunMoE.from_dict(mlp, where + ".mlp"))

    def to_dict(self) -> dict[str, Any]:
        out: dict[str, Any] = {"type": "parallel",
                               "mixer": {"left": self.left.to_dict(), "right": self.right.to_dict(),
                                         "left_scale": self.left_scale, "right_scale": self.right_scale},
                               "mlp": None if self.mlp is None else self.mlp.to_dict()}
        if self.weights_of is not None:
            out["weights_of"] = self.weights_of
        return out


@dataclass(frozen=True)
class LulisunConfig:
    vocab_size: int
    hidden_size: int
    norm_eps: float
    layers: tuple[LulisunLayer, ...]
    eos_token_id: tuple[int, ...] = ()
    architecture: str = "Lulisun"

    @classmethod
    def from_dict(cls, raw: dict[str, Any]) -> "LulisunConfig":
        entries = raw.get("layers")
        if not isinstance(entries, list) or not entries:
            raise ConfigError("config.json has no 'layers' list")
        layers = []
        for i, entry in enumerate(entries):
            source, seen = i, {i}
            while entries[source].get("weights_of") is not None:
                source = _need(entries[source], "weights_of", int, f"layers[{source}]")
                if not 0 <= source < len(entries) or source in seen:
                    raise ConfigError(f"config.json layers[{i}].weights_of leads to no layer with tensors of its own")
                seen.add(source)
            layer = LulisunLayer.from_dict(entries[source], f"layers[{source}]")
            layers.append(layer if source == i else LulisunLayer(layer.left, layer.right, layer.left_scale,
                                                                 layer.right_scale, layer.mlp, source))
        eos = raw.get("eos_token_id")
        eos_ids = () if eos is None else tuple(int(e) for e in (eos if isinstance(eos, (list, tuple)) else [eos]))
        config = cls(_need(raw, "vocab", int, ""), _need(raw, "width", int, ""),
                     _need(raw.get("norm"), "eps", float, "norm"), tuple(layers), eos_ids,
                     str(raw.get("architecture", "Lulisun")))
        _at_least_one("", vocab=config.vocab_size, width=config.hidden_size)
        if not config.norm_eps > 0:
            raise ConfigError("norm.eps must be > 0")
        return config

    def to_dict(self) -> dict[str, Any]:
        """config.json contents that `from_dict` reads back to an equal config."""
        out: dict[str, Any] = {"architecture": self.architecture, "vocab": self.vocab_size, "width": self.hidden_size,
                               "norm": {"eps": self.norm_eps}, "layers": [layer.to_dict() for layer in self.layers]}
        if self.eos_token_id:
            out["eos_token_id"] = list(self.eos_token_id)
        return out
