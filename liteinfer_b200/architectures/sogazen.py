"""The Sogazen decoder as a `ModelSpec`.

Every layer has one of two mixers and an optional feed-forward.  The mixers: a grouped-query softmax attention and a Mamba-2
state space side by side, each normalised over the width, the mean of both; and an RWKV-style time mixer.  The attention's
values are its keys as projected; q and k have biases, a norm over the whole projection and a half-split rotation of the first
`rot.dims` dimensions; scores are capped, and the softmax's denominator is one more than the sum of the exponentials.  The
feed-forward is a gated one with capped products, or a mixture of experts: softmax scores, a correction per expert that only
the choice goes by, weights not renormalised, experts of one projection through the square of relu, and identity experts,
which give back what they read.  The sublayers read the residual stream as it is; only what they give back is normalised:
x <- x + norm(sublayer(x)), summed in 32-bit.  The head is a table of its own and the logits pass c * tanh(. / c).
Tensor names: `embed`, `l<i>.norm1|norm2`, `l<i>.mix.left.*`, `l<i>.mix.right.*` or `l<i>.mix.*`, `l<i>.mlp.gate|up|down` or
`l<i>.mlp.router|correction`, `l<i>.mlp.e<j>.up|down`, `final.norm`, `head`.
"""

from __future__ import annotations

from liteinfer_b200.config.registry import register_architecture
from liteinfer_b200.config.sogazen_config import SogazenConfig, SogazenLayer, SogazenMLP
from liteinfer_b200.parts.spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry

_BARE = {"weight": ""}      # a tensor stored under the part's prefix itself
_PAIR_NAMES = {**{f"left.{n}_proj.weight": f"left.{n}" for n in "qko"},
               **{f"left.{n}_proj.bias": f"left.{n}.b" for n in "qk"},
               **{f"left.{n}_norm.weight": f"left.{n}.norm" for n in "qk"},
               "left.out.weight": "left.out", "right.out.weight": "right.out", "right.in_proj.weight": "right.in",
               "right.conv.weight": "right.conv", "right.conv.bias": "right.conv.b", "right.norm.weight": "right.norm",
               "right.o_proj.weight": "right.o"}
_TIME_NAMES = {**{f"{n}_proj.weight": n for n in "rkvgo"}, "w1.weight": "w1", "w2.weight": "w2", "norm.weight": "norm"}
_MLP_NAMES = {"gate_proj.weight": "gate", "up_proj.weight": "up", "down_proj.weight": "down"}

GATE_SLOPE = 1.702          # a dense feed-forward's gate passes g * sigmoid(1.702 g)
PAIR_SCALES = (0.5, 0.5)    # the mixers side by side: their mean
SINK = 0.0                  # the score of the attention's sink


def _mixer(config: SogazenConfig, layer: SogazenLayer) -> tuple[PartSpec, dict[str, str]]:
    common = {"hidden_size": config.hidden_size, "norm_eps": config.norm_eps}
    if layer.mixer is not None:
        return PartSpec("wkv", {**common, "heads": layer.mixer.heads, "dim": layer.mixer.dim,
                                "decay_rank": layer.mixer.decay_rank}), _TIME_NAMES
    left, right = layer.left, layer.right
    position = (PartSpec("rotary", {"head_dim": left.dim, "rotary_dim": left.rot_dims, "theta": left.rot_base, "exact": True})
                if left.rot_dims else PartSpec("none", {}))
    attention = PartSpec("attention", {
        "hidden_size": config.hidden_size, "heads": left.heads, "kv_heads": left.kv_heads, "head_dim": left.dim,
        "position": position, "scale": left.scale, "softcap": left.softcap, "bias": True, "out_bias": False,
        "qk_norm": "projection", "qk_norm_eps": config.norm_eps, "values_are_keys": True, "fixed_sink": SINK,
        "pad_heads": True})
    space = PartSpec("mamba2", {**common, "heads": right.heads, "vdim": right.vdim, "state": right.state,
                                "groups": right.groups, "conv": right.conv, "norm_groups": right.norm_groups})
    return PartSpec("side_by_side", {**common, "members": (attention, space), "scales": PAIR_SCALES,
                                     "prefixes": ("left.", "right.")}), _PAIR_NAMES


def _feed_forward(config: SogazenConfig, mlp: SogazenMLP) -> tuple[PartSpec, dict[str, str]]:
    sizes = {"hidden_size": config.hidden_size, "intermediate_size": mlp.ff}
    if mlp.kind == "dense":
        return PartSpec("gated_mlp", {**sizes, "activation": "capped_swiglu", "limit": mlp.limit,
                                      "alpha": GATE_SLOPE}), _MLP_NAMES
    names = {"router.weight": "router", "correction": "correction"}
    for e in range(mlp.experts):
        names.update({f"experts.{e}.{ours}": f"e{e}.{theirs}" for ours, theirs in _MLP_NAMES.items() if theirs != "gate"})
    return PartSpec("routed_experts", {
        **sizes, "experts": mlp.experts, "identity": mlp.identity, "top": mlp.top, "activation": "relu_squared",
        "correction": True, "renormalise": False, "gives_sum": True}), names


def sogazen_spec(config: SogazenConfig) -> ModelSpec:
    norm = PartSpec("rmsnorm_affine", {"size": config.hidden_size, "eps": config.norm_eps})
    layers, ignored = [], []
    for i, layer in enumerate(config.layers):
        mixer, mixer_names = _mixer(config, layer)
        parts = {"mixer": mixer, "mixer_out_norm": norm}
        prefixes = {"mixer": f"l{i}.mix.", "mixer_out_norm": f"l{i}.norm1"}
        renames = {"mixer": mixer_names, "mixer_out_norm": _BARE}
        if layer.mlp is not None:
            feed_forward, names = _feed_forward(config, layer.mlp)
            parts.update({"feed_forward_out_norm": norm, "feed_forward": feed_forward})
            prefixes.update({"feed_forward": f"l{i}.mlp.", "feed_forward_out_norm": f"l{i}.norm2"})
            renames.update({"feed_forward": names, "feed_forward_out_norm": _BARE})
        else:
            ignored.append(f"l{i}.norm2")
        layers.append(LayerSpec("output_norm" if layer.mlp is not None else "output_norm_mixer_only", parts, prefixes,
                                renames))
    sizes = {"vocab_size": config.vocab_size, "hidden_size": config.hidden_size}
    return ModelSpec(
        vocab_size=config.vocab_size, hidden_size=config.hidden_size,
        embedding=PartSpec("token_embedding", sizes), embedding_prefix="embed",
        layers=tuple(layers), schedule=tuple(ScheduleEntry(i) for i in range(len(layers))),
        final_norm=norm, final_norm_prefix="final.norm",
        head=PartSpec("linear", {**sizes, "softcap": config.logit_softcap}), head_prefix="head",
        stream_dtype="float32", widened_embedding=True,
        renames={"embedding": _BARE, "final_norm": _BARE, "head": _BARE}, ignored=tuple(ignored),
    )


register_architecture("Sogazen", SogazenConfig, sogazen_spec, replace=True)
