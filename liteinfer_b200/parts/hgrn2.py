"""The HGRN2 mixer: linear attention in which the forget gate also decides what is written.

Per token, with h the mixer's input and per head (dim, vdim the sizes of queries and values):

    q = silu(W_q h);  v = W_v h
    f = lower + (1 - lower) * sigmoid(W_f h + b_f)          # per head and channel; `lower` a bound of the same size
    S <- diag(f) S + (1 - f) v^T;  o = S^T q                # S [dim, vdim] per head, from zero
    y = W_o [norm_weight * o / rms(o)]                      # rms per head over vdim, one weight for all heads

What a request keeps between steps is S, 32-bit and zero at its start, so a sequence may arrive whole, in portions or
one token at a time.  Everything besides the projections is computed in 32-bit.
"""

from __future__ import annotations

import torch

from liteinfer_b200 import ops
from liteinfer_b200.parts.context import LayerCache, StateNeed, StepContext
from liteinfer_b200.parts.registry import register_mixer
from liteinfer_b200.parts.spec import TensorSpec


def _lower_init(shape, generator):
    """Lower bounds between 0.2 and 0.9."""
    return 0.2 + 0.7 * torch.rand(shape, generator=generator)


def _forget_init(shape, generator):
    return 0.3 * torch.randn(shape, generator=generator)


class HGRN2:
    """Runs alone or as one of several mixers side by side (parts/side_by_side.py), which uses `in_weight`,
    `out_weight`, `mix` and `scale_output`."""

    has_biases = False

    def __init__(self, hidden_size: int, heads: int, dim: int, vdim: int, norm_eps: float, dtype: torch.dtype,
                 device: torch.device, state_name: str = "hgrn2") -> None:
        if min(heads, dim, vdim) < 1:
            raise ValueError("an HGRN2 mixer needs heads, dim and vdim of at least 1")
        self.hidden_size, self.heads, self.dim, self.vdim = hidden_size, heads, dim, vdim
        self.norm_eps, self.state_name = float(norm_eps), state_name
        self.q_width, self.mixed_width = heads * dim, heads * vdim
        self.f_at, self.v_at = self.q_width, 2 * self.q_width        # columns of the fused projection: [q | f | v]
        self.in_weight = self.f_bias = self.lower = self.norm_weight = self.out_weight = None

    def tensor_specs(self) -> dict[str, TensorSpec]:
        d = self.hidden_size
        return {
            "q_proj.weight": TensorSpec((self.q_width, d)), "f_proj.weight": TensorSpec((self.q_width, d), init=_forget_init),
            "f_proj.bias": TensorSpec((self.q_width,), kind="f32"),
            "lower": TensorSpec((self.q_width,), kind="f32", init=_lower_init),
            "v_proj.weight": TensorSpec((self.mixed_width, d)),
            "norm.weight": TensorSpec((self.vdim,), kind="f32", init="ones_normal"),
            "o_proj.weight": TensorSpec((d, self.mixed_width)),
        }

    def bind(self, tensors: dict[str, torch.Tensor]) -> None:
        # One product for everything that reads h, filled up to a multiple of 16 rows.
        parts = [tensors[n + "_proj.weight"] for n in ("q", "f", "v")]
        pad = -sum(p.shape[0] for p in parts) % 16
        if pad:
            parts.append(parts[0].new_zeros((pad, self.hidden_size)))
        self.in_weight = torch.cat(parts).contiguous()
        self.f_bias, self.lower = tensors["f_proj.bias"].contiguous(), tensors["lower"].contiguous()
        self.norm_weight, self.out_weight = tensors["norm.weight"].contiguous(), tensors["o_proj.weight"]

    def scale_output(self, factor: float) -> bool:
        """Makes the mixer's output `factor` times what it is (in the norm's 32-bit weight), once, when bound."""
        self.norm_weight = self.norm_weight * factor
        return True

    def cache_needs(self) -> tuple:
        return (StateNeed((self.heads, self.vdim, self.dim), "f32", name=self.state_name),)     # S^T: column by column

    def mix(self, proj: torch.Tensor, ctx: StepContext, cache: LayerCache, out: torch.Tensor) -> None:
        """From the projection's rows to the normed read-outs, out [tokens, mixed_width] (column slices are fine)."""
        if cache.read_only:
            raise ValueError("an HGRN2 mixer cannot read another stop's state: its state moves with every token")
        ops.hgrn2(proj, (0, self.f_at, self.v_at), self.f_bias, self.lower, cache.states[self.state_name],
                  ctx.query_start_loc, ctx.state_slots, ctx.num_seqs, self.heads, self.dim, self.vdim, self.norm_weight,
                  self.norm_eps, out, ctx.max_query_len)

    def forward(self, x: torch.Tensor, ctx: StepContext, cache: LayerCache) -> torch.Tensor:
        out = torch.empty((x.shape[0], self.mixed_width), dtype=x.dtype, device=x.device)
        self.mix(ops.linear(x, self.in_weight, None), ctx, cache, out)
        return ops.linear(out, self.out_weight, None)


register_mixer("hgrn2", HGRN2)
