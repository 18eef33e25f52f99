"""The Mamba-2 mixer (state-space duality): a linear recurrence with one decay per head and token.

Per token, with h the mixer's input, `heads` heads of `vdim` and `groups` groups of `state` numbers:

    [z | x | B | C | dt] = W_in h
    x, B, C = silu(conv([x | B | C]))                # causal, per channel, a few taps, with a bias
    d = softplus(dt + dt_bias)                       # per head
    S <- exp(-exp(A_log) d) S + d B x^T;  y = S^T C + D x     # S [state, vdim] per head; head h reads group h // (heads / groups)
    out = W_o (norm_weight * rms_by_part(y * silu(z)))        # the gate in front of the norm; the heads' row in equal parts

What a request keeps between steps is S, 32-bit and zero at its start, and the last taps - 1 inputs of the convolution,
so a sequence may arrive whole, in portions or one token at a time.  Everything besides the projections and the
convolution is computed in 32-bit.
"""

from __future__ import annotations

import torch

from liteinfer_b200 import ops
from liteinfer_b200.parts.context import LayerCache, StateNeed, StepContext
from liteinfer_b200.parts.registry import register_mixer
from liteinfer_b200.parts.spec import TensorSpec


def _decay_init(shape, generator):
    """A_log such that exp(A_log) lies in [1, 8]."""
    return torch.log(1.0 + 7.0 * torch.rand(shape, generator=generator))


def _step_init(shape, generator):
    """Biases whose softplus lies around 0.01 to 0.1."""
    return -4.6 + 2.3 * torch.rand(shape, generator=generator)


def _conv_init(shape, generator):
    return 0.4 * torch.randn(shape, generator=generator)


class Mamba2:
    """Runs alone or as one of several mixers side by side (parts/side_by_side.py)."""

    has_biases = False

    def __init__(self, hidden_size: int, heads: int, vdim: int, state: int, groups: int, conv: int, norm_groups: int,
                 norm_eps: float, dtype: torch.dtype, device: torch.device, state_name: str = "mamba2",
                 tail_name: str = "mamba2_conv") -> None:
        if min(heads, vdim, state, groups, conv, norm_groups) < 1:
            raise ValueError("a Mamba-2 mixer's sizes are at least 1")
        if heads % groups or (heads * vdim) % norm_groups:
            raise ValueError(f"heads={heads} must be a multiple of groups={groups}, and {heads * vdim} numbers must fall into "
                             f"norm_groups={norm_groups} equal parts")
        self.hidden_size, self.heads, self.vdim, self.state, self.groups = hidden_size, heads, vdim, state, groups
        self.taps, self.norm_groups, self.norm_eps = conv, norm_groups, float(norm_eps)
        self.state_name, self.tail_name = state_name, tail_name
        self.mixed_width = heads * vdim
        self.channels = self.mixed_width + 2 * groups * state       # what the convolution runs over: x, B, C
        self.dt_at = self.mixed_width + self.channels               # columns of the projection: [z | x | B | C | dt]
        self.in_weight = self.conv_weight = self.conv_bias = self.dt_bias = self.a_log = self.skip = None
        self.norm_weight = self.out_weight = None

    def tensor_specs(self) -> dict[str, TensorSpec]:
        d, h = self.hidden_size, self.heads
        return {
            "in_proj.weight": TensorSpec((self.dt_at + h, d)),
            "conv.weight": TensorSpec((self.channels, self.taps), init=_conv_init),
            "conv.bias": TensorSpec((self.channels,), kind="f32"),
            "dt_bias": TensorSpec((h,), kind="f32", init=_step_init), "A_log": TensorSpec((h,), kind="f32", init=_decay_init),
            "D": TensorSpec((h,), kind="f32", init="ones_normal"),
            "norm.weight": TensorSpec((self.mixed_width,), kind="f32", init="ones_normal"),
            "o_proj.weight": TensorSpec((d, self.mixed_width)),
        }

    def bind(self, tensors: dict[str, torch.Tensor]) -> None:
        weight = tensors["in_proj.weight"]
        pad = -weight.shape[0] % 16
        self.in_weight = torch.cat([weight, weight.new_zeros((pad, self.hidden_size))]).contiguous() if pad else weight
        self.conv_weight = tensors["conv.weight"].t().contiguous()      # tap by tap: [taps, channels]
        self.conv_bias, self.dt_bias = tensors["conv.bias"].contiguous(), tensors["dt_bias"].contiguous()
        self.a_log, self.skip = tensors["A_log"].contiguous(), tensors["D"].contiguous()
        self.norm_weight, self.out_weight = tensors["norm.weight"].contiguous(), tensors["o_proj.weight"]

    def cache_needs(self) -> tuple:
        return (StateNeed((self.heads, self.vdim, self.state), "f32", name=self.state_name),      # S^T: column by column
                StateNeed((self.taps - 1, self.channels), "weight", name=self.tail_name))

    def mix(self, proj: torch.Tensor, ctx: StepContext, cache: LayerCache, out: torch.Tensor) -> None:
        """From the projection's rows to the gated and normed read-outs, out [tokens, mixed_width] (column slices are fine)."""
        if cache.read_only:
            raise ValueError("a Mamba-2 mixer cannot read another stop's state: its state moves with every token")
        tokens, inner = proj.shape[0], self.mixed_width
        conved = torch.empty((tokens, self.channels), dtype=proj.dtype, device=proj.device)
        ops.short_conv_step(proj[:, inner:self.dt_at], self.conv_weight, cache.states[self.tail_name], ctx.seq_of_token,
                            ctx.query_start_loc, ctx.state_slots, ctx.num_seqs, conved, "silu",
                            single_tokens=ctx.max_query_len == 1, bias=self.conv_bias)
        read = torch.empty((tokens, inner), dtype=torch.float32, device=proj.device)
        ops.state_space(conved, proj[:, self.dt_at:self.dt_at + self.heads], self.dt_bias, self.a_log,
                        cache.states[self.state_name], ctx.query_start_loc, ctx.state_slots, ctx.num_seqs, self.heads,
                        self.groups, self.state, self.vdim, read, ctx.max_query_len)
        ops.gated_group_norm(read, proj[:, :inner], self.norm_weight, self.norm_eps, out, self.norm_groups,
                             add=conved[:, :inner], skip=self.skip)

    def forward(self, x: torch.Tensor, ctx: StepContext, cache: LayerCache) -> torch.Tensor:
        out = torch.empty((x.shape[0], self.mixed_width), dtype=x.dtype, device=x.device)
        self.mix(ops.linear(x, self.in_weight, None), ctx, cache, out)
        return ops.linear(out, self.out_weight, None)


register_mixer("mamba2", Mamba2)
