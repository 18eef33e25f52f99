"""Several mixers side by side: y = sum_i scale_i * mixer_i(h), all reading the same h.

Everything that reads h is one product against the members' projections, and the members' outputs, next to each other in
one row, pass one product against their output projections, so the members' results are added up inside it.  The scales:
one is left to whoever adds y into the residual stream (a constant factor of that sum), the others, divided by it, go
where a member can take a constant without a rounding (`scale_output`) or, failing that, into its rows of the output
projection.

With `norm_eps` every member's result is divided by its root mean square over the width and multiplied by a weight of its
own (`out.weight` behind its prefix) before it is scaled and added up: the output projections are then products of their
own, and norms, scales and the sum are left to whoever normalises y on its way into the stream (`ops.output_norm`).  In steps
of few tokens, where each kernel alone leaves most of the device idle, the second member runs on a second stream beside the
first.

A member is a mixer with `in_weight`, `out_weight`, `mixed_width` and `mix(projection rows, ctx, cache, out)`; each
finds its pages or state under the name its own need declares, so members that keep the same kind of thing are given
different names (`cache_name`, `state_name`).  Their tensors lie behind the members' prefixes.
"""

from __future__ import annotations

from typing import Mapping, Sequence

import torch

from liteinfer_b200 import ops
from liteinfer_b200.parts.block import PARALLEL_SUBLAYERS
from liteinfer_b200.parts.context import LayerCache, StepContext
from liteinfer_b200.parts.registry import build_part, register_mixer
from liteinfer_b200.parts.spec import PartSpec, TensorSpec


class SideBySide:
    """`members`: the mixers' specs; `scales`: their factors; `prefixes`: what stands in front of each member's tensor
    names (default "0.", "1.", ...); `norm_eps`: every member's result is normalised first."""

    gives_sum = True        # `forward` returns an ops.SumDelta

    def __init__(self, hidden_size: int, members: Sequence[PartSpec], scales: Sequence[float], dtype: torch.dtype,
                 device: torch.device, prefixes: Sequence[str] | None = None, norm_eps: float | None = None) -> None:
        if not members or len(members) != len(scales):
            raise ValueError("mixers side by side need at least one member and a scale for each")
        if norm_eps is not None and len(members) > 2:
            raise ValueError("at most two mixers side by side can be normalised on their way out")
        self.norm_eps = None if norm_eps is None else float(norm_eps)
        self.out_norms: list[torch.Tensor] = []
        self.hidden_size = hidden_size
        self.members = [build_part("mixer", spec, dtype=dtype, device=device) for spec in members]
        self.scales = [float(s) for s in scales]
        self.prefixes = [f"{i}." for i in range(len(members))] if prefixes is None else list(prefixes)
        for member in self.members:
            if not hasattr(member, "mix") or member.has_biases:
                raise ValueError(f"a {type(member).__name__} with these options cannot run side by side with another mixer")
        self.factor = 1.0       # what the sum into the stream still has to multiply by
        self.in_weight = self.out_weight = None
        # Where each member's columns lie in the joined projection and in the joined outputs: both start on a multiple of
        # 16 columns, so that every member's rows are aligned for 16-byte accesses whatever its neighbours' sizes.
        self.in_at: list[tuple[int, int]] = []
        self.out_at: list[tuple[int, int]] = []

    def tensor_specs(self) -> dict[str, TensorSpec]:
        specs = {prefix + name: spec for prefix, member in zip(self.prefixes, self.members)
                 for name, spec in member.tensor_specs().items()}
        if self.norm_eps is not None:
            specs.update({prefix + "out.weight": TensorSpec((self.hidden_size,), kind="f32", init="ones_normal")
                          for prefix in self.prefixes})
        return specs

    def bind(self, tensors: Mapping[str, torch.Tensor]) -> None:
        for prefix, member in zip(self.prefixes, self.members):
            member.bind({name: tensors[prefix + name] for name in member.tensor_specs()})
        # The factor left to the sum: that of the first member which cannot scale itself, if it is not 0.
        rigid = [s for s, m in zip(self.scales, self.members) if not hasattr(m, "scale_output") and s != 0.0]
        self.factor = rigid[0] if rigid else 1.0
        ins, outs = [], []
        self.in_at, self.out_at = [], []
        at = out_end = 0
        for scale, member in zip(self.scales, self.members):
            rows = member.in_weight
            pad = -rows.shape[0] % 16
            ins += [rows, rows.new_zeros((pad, rows.shape[1]))]
            self.in_at.append((at, at + rows.shape[0]))
            at += rows.shape[0] + pad
            if self.norm_eps is not None:
                continue
            out, own = member.out_weight, scale / self.factor
            if own != 1.0 and not (hasattr(member, "scale_output") and member.scale_output(own)):
                out = (out.to(torch.float32) * own).to(out.dtype)
            pad = -out.shape[1] % 16
            outs += [out, out.new_zeros((out.shape[0], pad))]
            self.out_at.append((out_end, out_end + out.shape[1]))
            out_end += out.shape[1] + pad
        self.in_weight = torch.cat(ins).contiguous()
        if self.norm_eps is not None:
            self.out_norms = [tensors[prefix + "out.weight"].to(torch.float32).contiguous() for prefix in self.prefixes]
            for member in self.members:          # (their projections are kept in the joined copy only)
                for name in ("qkv_weight", "in_weight"):
                    if name in vars(member):
                        setattr(member, name, None)
            return
        self.out_weight = torch.cat(outs, dim=1).contiguous()
        for member in self.members:             # only the joined copies are kept
            for name in ("qkv_weight", "o_weight", "in_weight", "out_weight"):
                if name in vars(member):
                    setattr(member, name, None)

    def cache_needs(self) -> tuple:
        return tuple(need for member in self.members for need in member.cache_needs())

    def forward(self, x: torch.Tensor, ctx: StepContext, cache: LayerCache) -> "ops.SumDelta":
        proj = ops.linear(x, self.in_weight, None)
        if self.norm_eps is not None:
            return self._normed(proj, ctx, cache)
        # (The columns between the members' meet zeros in the product, so they must hold numbers.)
        gaps = sum(end - start for start, end in self.out_at) != self.out_weight.shape[1]
        mixed = (torch.zeros if gaps else torch.empty)((x.shape[0], self.out_weight.shape[1]), dtype=x.dtype, device=x.device)
        for (in_start, in_end), (out_start, out_end), member in zip(self.in_at, self.out_at, self.members):
            member.mix(proj[:, in_start:in_end], ctx, cache, mixed[:, out_start:out_end])
        return ops.SumDelta((ops.SumTerm(ops.linear(mixed, self.out_weight, None), self.factor),))


    def _normed(self, proj: torch.Tensor, ctx: StepContext, cache: LayerCache) -> "ops.SumDelta":
        def term(i: int) -> "ops.SumTerm":
            member, (start, end) = self.members[i], self.in_at[i]
            mixed = torch.empty((proj.shape[0], member.mixed_width), dtype=proj.dtype, device=proj.device)
            member.mix(proj[:, start:end], ctx, cache, mixed)
            return ops.SumTerm(ops.linear(mixed, member.out_weight, None), self.scales[i], None, self.out_norms[i], self.norm_eps)

        if len(self.members) == 2 and proj.is_cuda and proj.shape[0] <= PARALLEL_SUBLAYERS:
            lane = ops.beside(proj.device)
            with lane:
                second = term(1)
            first = term(0)
            lane.join()
            return ops.SumDelta((first, second))
        return ops.SumDelta(tuple(term(i) for i in range(len(self.members))))


register_mixer("side_by_side", SideBySide)
