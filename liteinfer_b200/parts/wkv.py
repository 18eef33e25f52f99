"""The RWKV-style time mixer: a matrix memory per head with a decay per key channel that the token chooses.

Per token, with h the mixer's input and h' the one of the token before (zeros before the first), per head (`dim` the size of
keys and values):

    m_s = h + (h' - h) * mu_s  for s in r, k, v, g, w
    r, k, v = W_r m_r, W_k m_k, W_v m_v;  gate = silu(W_g m_g)
    w = exp(-exp(W_w2 tanh(W_w1 m_w) + w0))                  # in (0, 1), per head and key channel
    o = (S + diag(u) k v^T)^T r;  S <- diag(w) S + k v^T      # the bonus u is for the token's own key and value only
    y = W_o (norm_weight * [o / rms(o) per head] * gate)      # norm_weight: all heads' size

What a request keeps between steps is S, 32-bit and zero at its start, and its last h, so a sequence may arrive whole, in
portions or one token at a time.  Everything besides the projections is computed in 32-bit.  The width of the decay's inner
product is the checkpoint's.
"""

from __future__ import annotations

import torch

from liteinfer_b200 import ops
from liteinfer_b200.parts.context import LayerCache, StateNeed, StepContext
from liteinfer_b200.parts.registry import register_mixer
from liteinfer_b200.parts.spec import TensorSpec

MIXES = ("r", "k", "v", "g", "w")


def _mu_init(shape, generator):
    return torch.rand(shape, generator=generator)


def _decay_init(shape, generator):
    """Decays between exp(-exp(-6)) and exp(-exp(-1))."""
    return -6.0 + 5.0 * torch.rand(shape, generator=generator)


def _bonus_init(shape, generator):
    return 0.5 * torch.randn(shape, generator=generator)


class WKV:
    def __init__(self, hidden_size: int, heads: int, dim: int, norm_eps: float, dtype: torch.dtype, device: torch.device,
                 decay_rank: int | None = None, state_name: str = "wkv", last_name: str = "wkv_last") -> None:
        if min(heads, dim) < 1:
            raise ValueError("a time mixer needs heads and dim of at least 1")
        self.hidden_size, self.heads, self.dim, self.norm_eps = hidden_size, heads, dim, float(norm_eps)
        self.decay_rank, self.state_name, self.last_name = decay_rank, state_name, last_name
        self.width = heads * dim
        self.mu = self.weights = self.w1 = self.w2 = self.w2t = self.w0 = self.bonus = None
        self.norm_weight = self.o_weight = None

    def tensor_specs(self) -> dict[str, TensorSpec]:
        d, n, rank = self.hidden_size, self.width, self.decay_rank
        free = max(16, d // 32)
        specs = {f"mu.{s}": TensorSpec((d,), kind="f32", init=_mu_init) for s in MIXES}
        specs.update({f"{s}_proj.weight": TensorSpec((n, d)) for s in "rkvg"})
        specs.update({
            "w1.weight": TensorSpec((rank, d), free=free), "w2.weight": TensorSpec((n, rank), free=free),
            "w0": TensorSpec((n,), kind="f32", init=_decay_init),
            "u": TensorSpec((self.heads, self.dim), kind="f32", init=_bonus_init),
            "norm.weight": TensorSpec((n,), kind="f32", init="ones_normal"), "o_proj.weight": TensorSpec((d, n)),
        })
        return specs

    def bind(self, tensors: dict[str, torch.Tensor]) -> None:
        self.mu = torch.stack([tensors[f"mu.{s}"] for s in MIXES]).contiguous()
        self.weights = torch.stack([tensors[f"{s}_proj.weight"] for s in "rkvg"]).contiguous()      # [4, width, hidden]
        self.w1, self.w2 = tensors["w1.weight"].contiguous(), tensors["w2.weight"].contiguous()
        if self.w1.shape[0] != self.w2.shape[1]:
            raise ValueError(f"the decay's two products do not fit: {tuple(self.w1.shape)} and {tuple(self.w2.shape)}")
        self.w2t = self.w2.t().contiguous()
        self.w0, self.bonus = tensors["w0"].contiguous(), tensors["u"].reshape(-1).contiguous()
        self.norm_weight, self.o_weight = tensors["norm.weight"].contiguous(), tensors["o_proj.weight"]

    def cache_needs(self) -> tuple:
        return (StateNeed((self.heads, self.dim, self.dim), "f32", name=self.state_name),         # S^T: column by column
                StateNeed((1, self.hidden_size), "weight", name=self.last_name))

    def forward(self, x: torch.Tensor, ctx: StepContext, cache: LayerCache) -> torch.Tensor:
        if cache.read_only:
            raise ValueError("a time mixer cannot read another stop's state: its state moves with every token")
        tokens = x.shape[0]
        mixed = torch.empty((len(MIXES), tokens, self.hidden_size), dtype=x.dtype, device=x.device)
        ops.token_shift_step(x, self.mu, cache.states[self.last_name], ctx.seq_of_token, ctx.query_start_loc, ctx.state_slots,
                             ctx.num_seqs, mixed, single_tokens=ctx.max_query_len == 1)
        r, k, v, gate = ops.batched_linear(mixed[:4], self.weights,
                                           torch.empty((4, tokens, self.width), dtype=x.dtype, device=x.device))
        low = ops.linear(mixed[4], self.w1, None)
        out = torch.empty((tokens, self.width), dtype=x.dtype, device=x.device)
        ops.wkv_memory(r, k, v, gate, low, self.w2, self.w2t, self.w0, self.bonus, cache.states[self.state_name],
                       ctx.query_start_loc, ctx.state_slots, ctx.num_seqs, self.heads, self.dim, self.norm_weight,
                       self.norm_eps, out, ctx.max_query_len)
        return ops.linear(out, self.o_weight, None)


register_mixer("wkv", WKV)
