"""Feed-forward parts.  Interface of a feed-forward:

    tensor_specs() / bind(tensors)
    forward(x, ctx) -> Tensor [tokens, hidden]
"""

from __future__ import annotations

import torch

from liteinfer_b200 import ops
from liteinfer_b200.parts.context import StepContext
from liteinfer_b200.parts.registry import register_feed_forward
from liteinfer_b200.parts.spec import TensorSpec


class GatedMLP:
    """down(act(gate(x)) * up(x)) — liteinfer/models/llama.py:105-114.

    gate and up are one product against the concatenated weights; the activation
    and the multiply are one kernel.  `activation` "capped_swiglu" joins them with caps instead: with g' = min(g, limit),
    g' * sigmoid(alpha g') * (clamp(u, -limit, limit) + 1).
    """

    def __init__(self, hidden_size: int, intermediate_size: int, activation: str, dtype: torch.dtype,
                 device: torch.device, bias: bool = False, limit: float = 0.0, alpha: float = 1.0) -> None:
        if activation not in ops.GATED_ACTIVATIONS:
            raise ValueError(f"activation {activation!r} has no kernel; known: {sorted(ops.GATED_ACTIVATIONS)}")
        if activation == "capped_swiglu" and not limit > 0:
            raise ValueError("the caps of 'capped_swiglu' must be > 0")
        self.caps = dict(limit=float(limit), alpha=float(alpha)) if activation == "capped_swiglu" else {}
        self.hidden_size, self.intermediate_size, self.activation, self.bias = (
            hidden_size, intermediate_size, activation, bias)
        self.gate_up_weight = self.gate_up_bias = self.down_weight = self.down_bias = None
        self.interleaved = False

    def tensor_specs(self) -> dict[str, TensorSpec]:
        i, h = self.intermediate_size, self.hidden_size
        specs = {"gate_proj.weight": TensorSpec((i, h)), "up_proj.weight": TensorSpec((i, h)),
                 "down_proj.weight": TensorSpec((h, i))}
        if self.bias:
            specs.update({"gate_proj.bias": TensorSpec((i,), init="zeros"), "up_proj.bias": TensorSpec((i,), init="zeros"),
                          "down_proj.bias": TensorSpec((h,), init="zeros")})
        return specs

    def bind(self, tensors: dict[str, torch.Tensor]) -> None:
        gate, up = tensors["gate_proj.weight"], tensors["up_proj.weight"]
        # bfloat16: gate and up rows interleaved in eights, the layout whose product, activation and
        # multiply one decode kernel can do together; otherwise gate rows first, then up rows.
        self.interleaved = gate.dtype == torch.bfloat16 and self.intermediate_size % 8 == 0
        self.gate_up_weight = self._pair(gate, up)
        self.down_weight = tensors["down_proj.weight"]
        if self.bias:
            self.gate_up_bias = self._pair(tensors["gate_proj.bias"], tensors["up_proj.bias"])
            self.down_bias = tensors["down_proj.bias"]

    def _pair(self, gate: torch.Tensor, up: torch.Tensor) -> torch.Tensor:
        if not self.interleaved:
            return torch.cat([gate, up])
        rest = gate.shape[1:]
        stacked = torch.stack([gate.reshape(-1, 8, *rest), up.reshape(-1, 8, *rest)], dim=1)
        return stacked.reshape(2 * gate.shape[0], *rest).contiguous()

    takes_pending_norm = True       # x may be an ops.PendingNorm: the gate_up product folds the norm in
    adds_to_residual = True         # the down projection adds into the residual stream where its kernel can

    def forward(self, x, ctx: StepContext, residual: torch.Tensor | None = None):
        tokens = x.shape[0]
        hidden = torch.empty((tokens, self.intermediate_size), dtype=x.dtype, device=x.device)
        if self.interleaved and ops.gated_linear_supported(x, self.gate_up_weight):
            ops.gated_linear(x, self.gate_up_weight, hidden, self.activation, self.gate_up_bias, **self.caps)
        else:
            gate_up = torch.empty((tokens, 2 * self.intermediate_size), dtype=x.dtype, device=x.device)
            ops.linear(x, self.gate_up_weight, gate_up, self.gate_up_bias)
            if self.interleaved:
                ops.act_mul_interleaved(gate_up, hidden, self.activation, **self.caps)
            else:
                ops.act_mul(gate_up, hidden, self.activation, **self.caps)
        return ops.linear(hidden, self.down_weight, None, self.down_bias, residual=residual)


class DenseMLP:
    """down(act(up(x))): a feed-forward without a gate; `activation` from `ops.UNARY_ACTIVATIONS`
    ("relu_squared": the square of relu)."""

    def __init__(self, hidden_size: int, intermediate_size: int, activation: str, dtype: torch.dtype,
                 device: torch.device) -> None:
        if activation not in ops.UNARY_ACTIVATIONS:
            raise ValueError(f"activation {activation!r} has no kernel; known: {sorted(ops.UNARY_ACTIVATIONS)}")
        self.hidden_size, self.intermediate_size, self.activation = hidden_size, intermediate_size, activation
        self.up_weight = self.down_weight = None

    def tensor_specs(self) -> dict[str, TensorSpec]:
        i, h = self.intermediate_size, self.hidden_size
        return {"up_proj.weight": TensorSpec((i, h)), "down_proj.weight": TensorSpec((h, i))}

    def bind(self, tensors: dict[str, torch.Tensor]) -> None:
        self.up_weight, self.down_weight = tensors["up_proj.weight"], tensors["down_proj.weight"]

    def forward(self, x, ctx: StepContext):
        hidden = ops.linear(x, self.up_weight, None, activation=self.activation)      # one kernel for a few rows of x
        return ops.linear(hidden, self.down_weight, None)


class RoutedExperts:
    """A mixture of experts: every token runs `top` of `experts` small gated feed-forwards and adds up their
    outputs, weighted by the router's scores.

    Router: logits = `router.weight` x in 32-bit; scores = softmax over all experts, or (`scores` "sigmoid") the sigmoid
    of each logit.  The choice goes by the scores, plus (`correction`) a stored number per expert, `correction`.  With
    `groups` > 1 the experts form that many equal groups of neighbours; a group's score is its largest choice score, or
    (`group_rank` 2) the sum of its two largest, and only experts of the best `groups_keep` groups can be chosen.  The
    `top` largest choice scores among those are chosen; the weights are the chosen experts' scores (`renormalise`:
    divided by their sum + `floor`).  Expert e: down_e(act(gate_e x, up_e x)), without biases, `activation` of
    `ops.EXPERT_ACTIVATIONS` ("swiglu": silu(g) * u; "capped_swiglu": g' = min(g, limit), u' = clamp(u, -limit, limit),
    g' * sigmoid(alpha * g') * (u' + 1)).  The step's (token, slot) pairs are ordered by expert on the device, and both
    products run tile by tile over each expert's rows, so an expert's weights are read once per tile of its tokens and
    nothing is read on the host.

    `shared_size` > 0: a shared expert of that width (`shared.gate_proj.weight` ...) runs for every token and is added,
    times sigmoid(`shared.sg.weight` x), one number per token (the router's product makes that logit too).  Where its
    width is a multiple of an expert's, it is cut into experts of that width which every token runs, with that number as
    their weight: a down projection adds up over its columns, so the sum is the same and the grouped products do it all.
    Otherwise it runs as a gated feed-forward of its own.

    `activation` of `ops.UNGATED_EXPERT_ACTIVATIONS`: the experts have no gate, down_e(act(up_e x)).

    `identity` > 0: the router has that many more outputs, the last ones, which stand for experts without tensors that give
    back what they read; they are scored and chosen like the others.

    `gives_sum`: `forward` returns the rows and terms not yet added up (`ops.SumDelta`).
    """

    def __init__(self, hidden_size: int, intermediate_size: int, experts: int, top: int, dtype: torch.dtype,
                 device: torch.device, groups: int = 1, groups_keep: int = 1, activation: str = "swiglu",
                 limit: float = 0.0, alpha: float = 1.0, renormalise: bool = False, scores: str = "softmax",
                 correction: bool = False, group_rank: int = 1, floor: float = 0.0, shared_size: int = 0,
                 gives_sum: bool = False, identity: int = 0) -> None:
        known = sorted((*ops.EXPERT_ACTIVATIONS, *ops.UNGATED_EXPERT_ACTIVATIONS))
        if activation not in known:
            raise ValueError(f"activation {activation!r} has no kernel; known: {known}")
        if identity < 0 or (identity and (not gives_sum or groups != 1 or shared_size)):
            raise ValueError("identity experts go with an output left to the stream's sum (gives_sum), without groups and "
                             "without a shared expert")
        if scores not in ops.ROUTER_SCORES:
            raise ValueError(f"scores {scores!r} are not supported; known: {sorted(ops.ROUTER_SCORES)}")
        if group_rank not in (1, 2):
            raise ValueError("a group ranks by its largest choice score (1) or by the sum of its two largest (2)")
        if not 1 <= top <= experts + identity or groups < 1 or experts % groups or not 1 <= groups_keep <= groups:
            raise ValueError("a mixture of experts needs 1 <= top <= experts, groups that divide experts, and "
                             "1 <= groups_keep <= groups")
        if groups_keep * (experts // groups) + identity < top:
            raise ValueError("the kept groups hold fewer experts than `top`")
        if shared_size and (not gives_sum or activation != "swiglu"):
            raise ValueError("a shared expert is a plain gated silu one, and its output is left to the stream's sum "
                             "(gives_sum)")
        self.hidden_size, self.intermediate_size, self.experts, self.top = hidden_size, intermediate_size, experts, top
        self.groups, self.groups_keep, self.activation = groups, groups_keep, activation
        self.limit, self.alpha, self.renormalise = float(limit), float(alpha), bool(renormalise)
        self.scores, self.has_correction, self.group_rank, self.floor = scores, bool(correction), group_rank, float(floor)
        self.shared_size, self.gives_sum = int(shared_size), bool(gives_sum)
        self.identity, self.gated = int(identity), activation in ops.EXPERT_ACTIVATIONS
        # The shared expert as so many experts that every token runs (0: it has a feed-forward of its own).
        self.shared_slots = shared_size // intermediate_size if shared_size % intermediate_size == 0 else 0
        self.shared = (GatedMLP(hidden_size, shared_size, "silu", dtype, device)
                       if shared_size and not self.shared_slots else None)
        self.dtype, self.device = dtype, device
        self.router = self.correction = self.gate_up = self.down = None
        self.eights = False

    def tensor_specs(self) -> dict[str, TensorSpec]:
        f, h = self.intermediate_size, self.hidden_size
        outputs = self.experts + self.identity
        specs = {"router.weight": TensorSpec((outputs, h), kind="f32")}
        if self.has_correction:
            specs["correction"] = TensorSpec((outputs,), kind="f32", init=_correction_init)
        for e in range(self.experts):
            specs.update(_expert_specs(f"experts.{e}.", h, f, self.gated))
        if self.shared_size:
            specs.update(_expert_specs("shared.", h, self.shared_size))
            specs["shared.sg.weight"] = TensorSpec((1, h), kind="f32")
        return specs

    def bind(self, tensors: dict[str, torch.Tensor]) -> None:
        router = tensors["router.weight"].to(torch.float32)
        if self.shared_size:
            router = torch.cat([router, tensors["shared.sg.weight"].to(torch.float32)])
        self.router = router.contiguous()
        self.correction = tensors["correction"].to(torch.float32).contiguous() if self.has_correction else None
        if not self.gated:
            stack = lambda n: torch.stack([tensors[f"experts.{e}.{n}_proj.weight"] for e in range(self.experts)]).contiguous()
            self.gate_up, self.down = stack("up"), stack("down")        # [experts, ff, hidden]: the up rows alone
            return
        # [experts, 2 * ff, hidden]: an expert's gate rows, then its up rows; in bfloat16 with a width in eights both
        # interleaved in eights (eight gate rows, then their eight up rows), the layout whose product and activation
        # the tensor-core kernels do together.  [experts, hidden, ff].
        gates, ups, downs = ([tensors[f"experts.{e}.{n}_proj.weight"] for e in range(self.experts)]
                             for n in ("gate", "up", "down"))
        for k in range(self.shared_slots):
            part = slice(k * self.intermediate_size, (k + 1) * self.intermediate_size)
            gates.append(tensors["shared.gate_proj.weight"][part])
            ups.append(tensors["shared.up_proj.weight"][part])
            downs.append(tensors["shared.down_proj.weight"][:, part])
        if self.shared is not None:
            self.shared.bind({n: tensors["shared." + n] for n in self.shared.tensor_specs()})
        self.eights = gates[0].dtype == torch.bfloat16 and self.intermediate_size % 8 == 0
        if self.eights:
            pair = lambda g, u: torch.stack([g.unflatten(0, (-1, 8)), u.unflatten(0, (-1, 8))], dim=1).flatten(0, 2)
        else:
            pair = lambda g, u: torch.cat([g, u])
        self.gate_up = torch.stack([pair(g, u) for g, u in zip(gates, ups)]).contiguous()
        self.down = torch.stack(downs).contiguous()

    def route(self, x: torch.Tensor, gate: torch.Tensor | None = None,
              identity: torch.Tensor | None = None) -> tuple[torch.Tensor, torch.Tensor]:
        """(chosen experts [tokens, top + shared slots] int32, their weights, float32); `gate` [tokens] float32 receives
        the shared expert's weight, `identity` [tokens] float32 the sum of the identity experts' weights."""
        tokens, slots = x.shape[0], self.top + self.shared_slots
        ids = torch.empty((tokens, slots), dtype=torch.int32, device=x.device)
        weights = torch.empty((tokens, slots), dtype=torch.float32, device=x.device)
        options = {}
        if self.scores != "softmax" or self.has_correction or self.group_rank != 1 or self.floor or self.shared_size:
            options = dict(scores=self.scores, correction=self.correction, rank_by=self.group_rank, floor=self.floor,
                           gated=bool(self.shared_size), gate=gate)
        if self.identity:
            options.update(identity=identity, identity_experts=self.identity)
        ops.moe_router(x, self.router, self.top, self.groups, self.groups_keep, self.renormalise, ids, weights, **options)
        return ids, weights

    def forward(self, x, ctx: StepContext):
        if not self.gives_sum:
            ids, weights = self.route(x)
            out = torch.empty((x.shape[0], self.hidden_size), dtype=x.dtype, device=x.device)
            return ops.moe_experts(x, self.gate_up, self.down, ids, weights, self.activation, self.limit, self.alpha,
                                   self.eights, out)
        gate = torch.empty((x.shape[0],), dtype=torch.float32, device=x.device) if self.shared is not None else None
        if self.identity:
            same = torch.empty((x.shape[0],), dtype=torch.float32, device=x.device)
            ids, weights = self.route(x, None, same)
            rows = ops.moe_expert_rows(x, self.gate_up, self.down, ids, weights, self.activation, self.limit, self.alpha,
                                       self.eights, partial=True)
            return ops.SumDelta((ops.SumTerm(x, 1.0, same),), rows)
        ids, weights = self.route(x, gate)
        rows = ops.moe_expert_rows(x, self.gate_up, self.down, ids, weights, self.activation, self.limit, self.alpha,
                                   self.eights)
        terms = () if self.shared is None else (ops.SumTerm(self.shared.forward(x, ctx), 1.0, gate),)
        return ops.SumDelta(terms, rows)


def _expert_specs(prefix: str, hidden: int, width: int, gated: bool = True) -> dict[str, TensorSpec]:
    if not gated:
        return {prefix + "up_proj.weight": TensorSpec((width, hidden)), prefix + "down_proj.weight": TensorSpec((hidden, width))}
    return {prefix + "gate_proj.weight": TensorSpec((width, hidden)), prefix + "up_proj.weight": TensorSpec((width, hidden)),
            prefix + "down_proj.weight": TensorSpec((hidden, width))}


def _correction_init(shape, generator):
    return 0.1 * torch.randn(shape, generator=generator)


register_feed_forward("gated_mlp", GatedMLP)
register_feed_forward("routed_experts", RoutedExperts)
register_feed_forward("dense_mlp", DenseMLP)
