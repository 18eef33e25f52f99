"""Typed configuration of the Sogazen decoder, read from its config.json.

A Sogazen config.json names everything per layer:

    {"architecture": "Sogazen", "vocab": V, "width": D, "norm": {"eps": e}, "logit_softcap": c | null,
     "layers": [{"type": "parallel",
                 "mixer": {"left": {"heads", "kv_heads", "dim", "vdim", "scale", "softcap": c | null,
                                    "rot": {"dims", "base"} | null},
                           "right": {"heads", "vdim", "state", "groups", "conv", "norm_groups"}},
                 "mlp": ...},
                {"type": "wkv", "mixer": {"heads", "dim"}, "mlp": ...}, ...]}

with "mlp" one of null, {"kind": "dense", "ff": F, "limit": L} and {"kind": "moe", "expert": {"ff": F}, "router":
{"experts": E, "top": k, "identity": n | null}}.  Sizes and constants have no defaults: a missing one is a `ConfigError`.  An
option that is absent or null is off (no cap, no rotation, no identity experts, no feed-forward).  A `wkv` mixer may name the
width of its decay's inner product, `decay_rank`; otherwise the checkpoint's tensors say it.
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Any

from liteinfer_b200.config.kegizen_config import _need
from liteinfer_b200.config.lulisun_config import _at_least_one
from liteinfer_b200.config.model_config import ConfigError

LAYER_TYPES = ("parallel", "wkv")


def _cap(raw: dict[str, Any], key: str, where: str) -> float:
    """A cap on scores or logits; 0: none."""
    if raw.get(key) is None:
        return 0.0
    value = _need(raw, key, float, where)
    if value < 0:
        raise ConfigError(f"config.json {where} {key!r} must be >= 0, got {value}")
    return value


@dataclass(frozen=True)
class SogazenAttention:
    heads: int
    kv_heads: int
    dim: int                         # of keys, and of the values, which are the keys as projected
    scale: float
    softcap: float = 0.0             # a scaled score passes c * tanh(. / c) (0: as it is)
    rot_dims: int = 0                # the first dimensions of a head that turn (0: none)
    rot_base: float = 0.0

    @classmethod
    def from_dict(cls, raw: dict[str, Any], where: str) -> "SogazenAttention":
        heads, kv_heads, dim, vdim = (_need(raw, n, int, where) for n in ("heads", "kv_heads", "dim", "vdim"))
        _at_least_one(where, heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim)
        if heads % kv_heads:
            raise ConfigError(f"config.json {where}: heads={heads} is not a multiple of kv_heads={kv_heads}")
        if vdim != dim:
            raise ConfigError(f"config.json {where}: the values are the keys, so vdim={vdim} must be dim={dim}")
        rot, dims, base = raw.get("rot"), 0, 0.0
        if rot and rot.get("dims") != 0:
            dims, base = _need(rot, "dims", int, where + ".rot"), _need(rot, "base", float, where + ".rot")
            if dims < 2 or dims % 2 or dims > dim or not base > 0:
                raise ConfigError(f"config.json {where}.rot: dims={dims} must be even and within the head's {dim} "
                                  "dimensions, base > 0")
        return cls(heads, kv_heads, dim, _need(raw, "scale", float, where), _cap(raw, "softcap", where), dims, base)

    def to_dict(self) -> dict[str, Any]:
        out: dict[str, Any] = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.dim,
                               "scale": self.scale}
        if self.softcap:
            out["softcap"] = self.softcap
        if self.rot_dims:
            out["rot"] = {"dims": self.rot_dims, "base": self.rot_base}
        return out


@dataclass(frozen=True)
class SogazenStateSpace:
    heads: int
    vdim: int
    state: int
    groups: int                      # heads share B and C within a group
    conv: int                        # taps
    norm_groups: int                 # parts of the row that are normalised each by itself

    @classmethod
    def from_dict(cls, raw: dict[str, Any], where: str) -> "SogazenStateSpace":
        sizes = {n: _need(raw, n, int, where) for n in ("heads", "vdim", "state", "groups", "conv", "norm_groups")}
        _at_least_one(where, **sizes)
        if sizes["heads"] % sizes["groups"] or sizes["heads"] * sizes["vdim"] % sizes["norm_groups"]:
            raise ConfigError(f"config.json {where}: groups must divide the heads, norm_groups their numbers")
        return cls(**sizes)

    def to_dict(self) -> dict[str, Any]:
        return {n: getattr(self, n) for n in ("heads", "vdim", "state", "groups", "conv", "norm_groups")}


@dataclass(frozen=True)
class SogazenTimeMixer:
    heads: int
    dim: int
    decay_rank: int | None = None    # the width of the decay's inner product (None: the checkpoint's)

    @classmethod
    def from_dict(cls, raw: dict[str, Any], where: str) -> "SogazenTimeMixer":
        sizes = {n: _need(raw, n, int, where) for n in ("heads", "dim")}
        if isinstance(raw, dict) and raw.get("decay_rank") is not None:
            sizes["decay_rank"] = _need(raw, "decay_rank", int, where)
        _at_least_one(where, **sizes)
        return cls(**sizes)

    def to_dict(self) -> dict[str, Any]:
        out = {"heads": self.heads, "dim": self.dim}
        if self.decay_rank is not None:
            out["decay_rank"] = self.decay_rank
        return out


@dataclass(frozen=True)
class SogazenMLP:
    kind: str
    ff: int                          # the width of the feed-forward, or of one expert
    limit: float = 0.0               # dense: the caps of gate and up
    experts: int = 0
    top: int = 0
    identity: int = 0                # experts without tensors, which give back what they read

    @classmethod
    def from_dict(cls, raw: dict[str, Any], where: str) -> "SogazenMLP":
        kind = raw.get("kind", "dense")
        if kind == "dense":
            mlp = cls(kind, _need(raw, "ff", int, where), _need(raw, "limit", float, where))
            _at_least_one(where, ff=mlp.ff)
            if not mlp.limit > 0:
                raise ConfigError(f"config.json {where}.limit must be > 0, got {mlp.limit}")
            return mlp
        if kind != "moe":
            raise ConfigError(f"config.json {where} has kind {kind!r}; known: ['dense', 'moe']")
        router = raw.get("router")
        mlp = cls(kind, _need(raw.get("expert"), "ff", int, where + ".expert"),
                  experts=_need(router, "experts", int, where + ".router"), top=_need(router, "top", int, where + ".router"),
                  identity=_need(router, "identity", int, where + ".router") if router.get("identity") is not None else 0)
        _at_least_one(where, ff=mlp.ff, experts=mlp.experts, top=mlp.top)
        if mlp.identity < 0 or mlp.top > mlp.experts + mlp.identity:
            raise ConfigError(f"config.json {where}.router: identity must be >= 0, and top={mlp.top} at most experts + identity")
        return mlp

    def to_dict(self) -> dict[str, Any]:
        if self.kind == "dense":
            return {"kind": "dense", "ff": self.ff, "limit": self.limit}
        router: dict[str, Any] = {"experts": self.experts, "top": self.top}
        if self.identity:
            router["identity"] = self.identity
        return {"kind": "moe", "expert": {"ff": self.ff}, "router": router}


@dataclass(frozen=True)
class SogazenLayer:
    mixer: SogazenTimeMixer | None               # of a "wkv" layer ...
    left: SogazenAttention | None                # ... or both of a "parallel" one
    right: SogazenStateSpace | None
    mlp: SogazenMLP | None

    @classmethod
    def from_dict(cls, raw: dict[str, Any], where: str) -> "SogazenLayer":
        kind, mixer, at, mlp = raw.get("type"), raw.get("mixer"), where + ".mixer", raw.get("mlp")
        if kind not in LAYER_TYPES:
            raise ConfigError(f"config.json {where} has type {kind!r}; known: {list(LAYER_TYPES)}")
        if not isinstance(mixer, dict):
            raise ConfigError(f"config.json {where} has no 'mixer'")
        feed_forward = None if mlp is None else SogazenMLP.from_dict(mlp, where + ".mlp")
        if kind == "wkv":
            return cls(SogazenTimeMixer.from_dict(mixer, at), None, None, feed_forward)
        return cls(None, SogazenAttention.from_dict(mixer.get("left"), at + ".left"),
                   SogazenStateSpace.from_dict(mixer.get("right"), at + ".right"), feed_forward)

    def to_dict(self) -> dict[str, Any]:
        mixer = (self.mixer.to_dict() if self.mixer is not None
                 else {"left": self.left.to_dict(), "right": self.right.to_dict()})
        return {"type": "parallel" if self.mixer is None else "wkv", "mixer": mixer,
                "mlp": None if self.mlp is None else self.mlp.to_dict()}


@dataclass(frozen=True)
class SogazenConfig:
    vocab_size: int
    hidden_size: int
    norm_eps: float
    layers: tuple[SogazenLayer, ...]
    logit_softcap: float = 0.0
    eos_token_id: tuple[int, ...] = ()
    architecture: str = "Sogazen"

    @classmethod
    def from_dict(cls, raw: dict[str, Any]) -> "SogazenConfig":
        entries = raw.get("layers")
        if not isinstance(entries, list) or not entries:
            raise ConfigError("config.json has no 'layers' list")
        eos = raw.get("eos_token_id")
        eos_ids = () if eos is None else tuple(int(e) for e in (eos if isinstance(eos, (list, tuple)) else [eos]))
        config = cls(_need(raw, "vocab", int, ""), _need(raw, "width", int, ""), _need(raw.get("norm"), "eps", float, "norm"),
                     tuple(SogazenLayer.from_dict(entry, f"layers[{i}]") for i, entry in enumerate(entries)),
                     _cap(raw, "logit_softcap", ""), eos_ids, str(raw.get("architecture", "Sogazen")))
        _at_least_one("", vocab=config.vocab_size, width=config.hidden_size)
        if not config.norm_eps > 0:
            raise ConfigError("norm.eps must be > 0")
        return config

    def to_dict(self) -> dict[str, Any]:
        """config.json contents that `from_dict` reads back to an equal config."""
        out: dict[str, Any] = {"architecture": self.architecture, "vocab": self.vocab_size, "width": self.hidden_size,
                               "norm": {"eps": self.norm_eps}, "layers": [layer.to_dict() for layer in self.layers]}
        if self.logit_softcap:
            out["logit_softcap"] = self.logit_softcap
        if self.eos_token_id:
            out["eos_token_id"] = list(self.eos_token_id)
        return out
