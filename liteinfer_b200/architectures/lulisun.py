"""The Lulisun decoder as a `ModelSpec`.

Every layer runs two sublayers on the same stream, each behind a norm of its own (weights stored around zero), and adds
both: x <- x + (mixer(norm1(x)) + ff(norm2(x))), summed in 32-bit.  The mixer is itself two mixers side by side with a
scale each: a grouped-query softmax attention within chunks of positions, with a half-split rotation of the first
`rot.dims` dimensions and values of another size than keys; and an HGRN2 memory.  The feed-forward is a mixture of
experts: sigmoid scores, a correction per expert that only the choice goes by, groups of neighbours ranked by their two
best, weights that add up to 1, and a shared expert weighted by a sigmoid of its own.  A layer may use the tensors of
another one: it is then another stop of the schedule, with pages and states of its own.  The head is a table of its own.
Tensor names: `embed`, `l<i>.norm1|norm2`, `l<i>.mix.left.*`, `l<i>.mix.right.*`, `l<i>.mlp.router|correction`,
`l<i>.mlp.e<j>.gate|up|down`, `l<i>.mlp.shared.gate|up|down|sg`, `final.norm`, `head`.
"""

from __future__ import annotations

from liteinfer_b200.config.lulisun_config import LulisunAttention, LulisunConfig, LulisunLayer, LulisunMoE
from liteinfer_b200.config.registry import register_architecture
from liteinfer_b200.parts.spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry

_BARE = {"weight": ""}      # a tensor stored under the part's prefix itself
_PROJECTIONS = {"gate_proj.weight": "gate", "up_proj.weight": "up", "down_proj.weight": "down"}
_MIXER_NAMES = {**{f"left.{n}_proj.weight": f"left.{n}" for n in "qkvo"},
                **{f"right.{n}_proj.weight": f"right.{n}" for n in "qfvo"},
                "right.f_proj.bias": "right.f.b", "right.lower": "right.lower", "right.norm.weight": "right.norm"}

WEIGHT_SUM_FLOOR = 1e-20    # added to the sum that the chosen experts' scores are divided by


def _attention(config: LulisunConfig, left: LulisunAttention) -> PartSpec:
    position = (PartSpec("rotary", {"head_dim": left.dim, "rotary_dim": left.rot_dims, "theta": left.rot_base, "exact": True})
                if left.rot_dims else PartSpec("none", {}))
    return PartSpec("attention", {
        "hidden_size": config.hidden_size, "heads": left.heads, "kv_heads": left.kv_heads, "head_dim": left.dim,
        "v_head_dim": left.vdim, "position": position, "scale": left.scale, "chunk": left.chunk, "pad_heads": True})


def _mixer(config: LulisunConfig, layer: LulisunLayer) -> PartSpec:
    right = PartSpec("hgrn2", {"hidden_size": config.hidden_size, "heads": layer.right.heads, "dim": layer.right.dim,
                               "vdim": layer.right.vdim, "norm_eps": config.norm_eps})
    return PartSpec("side_by_side", {"hidden_size": config.hidden_size, "members": (_attention(config, layer.left), right),
                                     "scales": (layer.left_scale, layer.right_scale), "prefixes": ("left.", "right.")})


def _feed_forward(config: LulisunConfig, mlp: LulisunMoE) -> tuple[PartSpec, dict[str, str]]:
    names = {"router.weight": "router", "correction": "correction", "shared.sg.weight": "shared.sg"}
    names.update({f"shared.{ours}": f"shared.{theirs}" for ours, theirs in _PROJECTIONS.items()})
    for e in range(mlp.experts):
        names.update({f"experts.{e}.{ours}": f"e{e}.{theirs}" for ours, theirs in _PROJECTIONS.items()})
    return PartSpec("routed_experts", {
        "hidden_size": config.hidden_size, "intermediate_size": mlp.ff, "experts": mlp.experts, "top": mlp.top,
        "groups": mlp.groups, "groups_keep": mlp.groups_keep, "scores": "sigmoid", "correction": True, "group_rank": 2,
        "renormalise": True, "floor": WEIGHT_SUM_FLOOR, "shared_size": mlp.shared_ff, "gives_sum": True}), names


def lulisun_spec(config: LulisunConfig) -> ModelSpec:
    norm = PartSpec("rmsnorm_unit_offset", {"size": config.hidden_size, "eps": config.norm_eps})
    layers, ignored, index_of = [], [], {}
    for i, layer in enumerate(config.layers):
        if layer.weights_of is not None:
            continue
        index_of[i] = len(layers)
        parts = {"mixer_norm": norm, "mixer": _mixer(config, layer)}
        prefixes = {"mixer_norm": f"l{i}.norm1", "mixer": f"l{i}.mix."}
        renames = {"mixer_norm": _BARE, "mixer": _MIXER_NAMES}
        if layer.mlp is not None:
            feed_forward, names = _feed_forward(config, layer.mlp)
            parts.update({"feed_forward_norm": norm, "feed_forward": feed_forward})
            prefixes.update({"feed_forward_norm": f"l{i}.norm2", "feed_forward": f"l{i}.mlp."})
            renames.update({"feed_forward_norm": _BARE, "feed_forward": names})
        else:
            ignored.append(f"l{i}.norm2")
        layers.append(LayerSpec("parallel_norms" if layer.mlp is not None else "parallel_norms_mixer_only", parts,
                                prefixes, renames))
    schedule = tuple(ScheduleEntry(index_of[i if layer.weights_of is None else layer.weights_of])
                     for i, layer in enumerate(config.layers))
    sizes = {"vocab_size": config.vocab_size, "hidden_size": config.hidden_size}
    return ModelSpec(
        vocab_size=config.vocab_size, hidden_size=config.hidden_size,
        embedding=PartSpec("token_embedding", sizes), embedding_prefix="embed", layers=tuple(layers), schedule=schedule,
        final_norm=norm, final_norm_prefix="final.norm", head=PartSpec("linear", sizes), head_prefix="head",
        stream_dtype="float32", widened_embedding=True,
        renames={"embedding": _BARE, "final_norm": _BARE, "head": _BARE}, ignored=tuple(ignored),
    )


register_architecture("Lulisun", LulisunConfig, lulisun_spec, replace=True)
