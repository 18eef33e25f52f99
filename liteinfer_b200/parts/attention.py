"""The attention mixer.  Interface of a mixer:

    tensor_specs() / bind(tensors)
    cache_needs() -> tuple of KVNeed / StateNeed     # what the cache manager must keep for this layer
    forward(x, ctx, cache) -> Tensor [tokens, hidden]

`x` holds the step's tokens of every sequence end to end; `ctx` (StepContext)
says which token belongs to which sequence and position; `cache` (LayerCache) is
this layer's pages or state.  A mixer writes what it must remember into `cache`
and reads earlier tokens from there only, so a sequence may arrive whole, in
portions, or one token at a time.
"""

from __future__ import annotations

import torch

from liteinfer_b200 import ops
from liteinfer_b200.parts.context import KVNeed, LayerCache, StepContext
from liteinfer_b200.parts.registry import build_part, register_mixer
from liteinfer_b200.parts.spec import PartSpec, TensorSpec


class Attention:
    """Causal grouped-query attention over a paged cache.

    liteinfer/models/llama.py:117-163: q/k/v projections, the position encoding
    on q and k, keys and values stored, attention of the new queries over
    everything stored, output projection.  Query head h reads KV head
    h // (heads // kv_heads); scores are scaled by `scale` (head_dim^-0.5 unless
    given).  `window` keeps only the newest `window` keys visible, and beside
    them the first `keep_first` of the sequence.  `v_head_dim`: values of another
    size than keys.  `softcap` > 0: a scaled score s becomes softcap * tanh(s / softcap).
    `qk_norm` "projection": q and k are each divided by their root mean square over the
    whole projection (all heads at once; eps `qk_norm_eps`) and multiplied by the weights
    `q_norm.weight` / `k_norm.weight`, before the position encoding; "head": each head of q and of k is divided
    by its own root mean square and multiplied by a weight of `head_dim` entries that the heads share
    (`qk_norm_weight` False: by no weight; `qk_norm_after_rotation`: the norm comes behind the position encoding).
    `sink`: a learned number per head (`sink`, 32-bit) whose exponential joins the denominator of that head's
    softmax; it has no key and no value and is not scaled.  `output_gate`: the concatenated heads are multiplied
    element by element by sigmoid(`gate_proj.weight` x) before the output projection.
    `head_gate`: head h of the attention's output is multiplied by sigmoid(g_h), g = `g_proj.weight` x, one number
    per head, before the output projection.  `value_mix`: "source" leaves this layer's values of the step's tokens
    in `ctx.extras[value_mix_key]` for later layers; "mixed" stores (1 - l) v + l v_source instead of v, l the
    scalar tensor `value_mix` and v_source what the source layer left for the same tokens.  `chunk` (instead of a
    window): positions form chunks of that many from the sequence's start, and a query reads the keys of its own chunk
    only.  `values_are_keys`: there is no value projection; what is stored as a token's value is its key as projected (with
    its bias, before norm and rotation).  `fixed_sink`: a sink as above whose number is a constant for all heads (0: the
    softmax's denominator is 1 larger than the sum of the exponentials).  Everything that reads x is one product against the
    concatenated weights; where q and k are normalised over the projection and there are biases or no values of their own,
    biases, norm, rotation and the cache write are one kernel behind it (`joint_norm`).

    `pad_heads`: in bfloat16 on a GPU, keys and values whose sizes no tensor-core kernel takes are rounded up to sizes
    that one does (`tensor_core_sizes`): the added rows of the projections and columns of `o_proj.weight` are zeros, so
    every score and every output is the same sum.  (Not with mixed values or an output gate; with q/k norms or biases only
    where they are those of `joint_norm`.)

    A mixer that runs several side by side (parts/side_by_side.py) makes one product of their projections and one of
    their output projections; it uses `in_weight`, `out_weight` and `mix`.
    """

    def __init__(self, hidden_size: int, heads: int, kv_heads: int, head_dim: int, position: PartSpec,
                 dtype: torch.dtype, device: torch.device, bias: bool = False, out_bias: bool | None = None,
                 window: int | None = None, scale: float | None = None, cache_name: str = "kv",
                 v_head_dim: int | None = None, keep_first: int = 0, softcap: float = 0.0,
                 qk_norm: str | None = None, qk_norm_eps: float = 1e-6, head_gate: bool = False,
                 value_mix: str | None = None, value_mix_key: str = "value_mix", qk_norm_weight: bool = True,
                 qk_norm_after_rotation: bool = False, sink: bool = False, output_gate: bool = False,
                 chunk: int | None = None, pad_heads: bool = False, values_are_keys: bool = False,
                 fixed_sink: float | None = None) -> None:
        if values_are_keys and (qk_norm != "projection" or v_head_dim not in (None, head_dim) or value_mix or head_gate
                                or output_gate):
            raise ValueError("values that are the keys as projected go with qk_norm='projection', heads of one size, and "
                             "neither gates nor mixed values")
        if sink and fixed_sink is not None:
            raise ValueError("an attention has learned sinks or a fixed one")
        if window is not None and chunk is not None:
            raise ValueError("an attention has a window or chunks, not both")
        if heads % kv_heads:
            raise ValueError(f"heads={heads} is not a multiple of kv_heads={kv_heads}")
        if qk_norm not in (None, "projection", "head"):
            raise ValueError(f"qk_norm {qk_norm!r} is not supported; known: None, 'projection', 'head'")
        if value_mix not in (None, "source", "mixed"):
            raise ValueError(f"value_mix {value_mix!r} is not supported; known: None, 'source', 'mixed'")
        if (not qk_norm_weight or qk_norm_after_rotation) and qk_norm != "head":
            raise ValueError("a norm without a weight, or behind the rotation, is an option of qk_norm='head'")
        if head_gate and output_gate:
            raise ValueError("an attention has one gate: per head (head_gate) or per element (output_gate)")
        self.qk_norm_weight, self.qk_norm_after_rotation = bool(qk_norm_weight), bool(qk_norm_after_rotation)
        self.has_sink, self.output_gate = bool(sink), bool(output_gate)
        self.sink: torch.Tensor | None = None
        self.values_are_keys = bool(values_are_keys)
        self.fixed_sink = None if fixed_sink is None else float(fixed_sink)
        self.head_gate, self.value_mix, self.value_mix_key = bool(head_gate), value_mix, value_mix_key
        self.blend: torch.Tensor | None = None
        self.hidden_size, self.heads, self.kv_heads, self.head_dim = hidden_size, heads, kv_heads, head_dim
        self.v_head_dim = head_dim if v_head_dim is None else v_head_dim
        self.keep_first = int(keep_first) if window is not None else 0
        self.softcap = float(softcap or 0.0)
        self.qk_norm, self.qk_norm_eps = qk_norm, float(qk_norm_eps)
        self.q_norm_weight = self.k_norm_weight = None
        self.bias = bias
        self.out_bias = bias if out_bias is None else out_bias
        self.window, self.chunk = window, chunk
        self.cache_name = cache_name    # under which name this mixer's pages lie in its layer's cache
        self.scale = float(scale) if scale is not None else head_dim ** -0.5
        self.dtype, self.device = dtype, device
        self.position = build_part("position", position, dtype=dtype, device=device)
        # The sizes of the checkpoint's heads; head_dim and v_head_dim are those of the rows that are computed and kept.
        self.key_size, self.value_size = self.head_dim, self.v_head_dim
        self.joint_norm = (qk_norm == "projection" and (values_are_keys or self.bias or pad_heads)
                           and not (self.head_gate or self.output_gate or value_mix))
        self.prep_bias: torch.Tensor | None = None      # float32, of the kernel behind the projection (joint_norm)
        if (pad_heads and dtype == torch.bfloat16 and torch.device(device).type == "cuda"
                and (self.joint_norm or not (qk_norm or bias)) and not (value_mix or output_gate)):
            sizes = ops.tensor_core_sizes(self.head_dim, self.v_head_dim, heads, kv_heads)
            if sizes is not None:
                self.head_dim, self.v_head_dim = sizes
        self.qkv_weight: torch.Tensor | None = None
        self.qkv_bias: torch.Tensor | None = None
        self.o_weight: torch.Tensor | None = None
        self.o_bias: torch.Tensor | None = None

    def tensor_specs(self) -> dict[str, TensorSpec]:
        q, kv, v = self.heads * self.key_size, self.kv_heads * self.key_size, self.kv_heads * self.value_size
        specs = {
            "q_proj.weight": TensorSpec((q, self.hidden_size)),
            "k_proj.weight": TensorSpec((kv, self.hidden_size)),
            "v_proj.weight": TensorSpec((v, self.hidden_size)),
            "o_proj.weight": TensorSpec((self.hidden_size, self.heads * self.value_size)),
        }
        if self.values_are_keys:
            del specs["v_proj.weight"]
        if self.qk_norm == "head":
            if self.qk_norm_weight:
                specs.update({"q_norm.weight": TensorSpec((self.head_dim,), init="ones_normal"),
                              "k_norm.weight": TensorSpec((self.head_dim,), init="ones_normal")})
        elif self.qk_norm:
            kind = "f32" if self.joint_norm else "weight"
            specs.update({"q_norm.weight": TensorSpec((q,), kind, init="ones_normal"),
                          "k_norm.weight": TensorSpec((kv,), kind, init="ones_normal")})
        if self.head_gate:
            specs["g_proj.weight"] = TensorSpec((self.heads, self.hidden_size))
        if self.output_gate:
            specs["gate_proj.weight"] = TensorSpec((self.heads * self.value_size, self.hidden_size))
        if self.has_sink:
            specs["sink"] = TensorSpec((self.heads,), kind="f32", init=_sink_init)
        if self.value_mix == "mixed":
            specs["value_mix"] = TensorSpec((), kind="f32", init=_blend_init)
        if self.bias:
            specs.update({"q_proj.bias": TensorSpec((q,), init="zeros"), "k_proj.bias": TensorSpec((kv,), init="zeros"),
                          "v_proj.bias": TensorSpec((v,), init="zeros")})
            if self.values_are_keys:
                del specs["v_proj.bias"]
        if self.out_bias:
            specs["o_proj.bias"] = TensorSpec((self.hidden_size,), init="zeros")
        for name, spec in self.position.tensor_specs().items():
            specs["position." + name] = spec
        return specs

    def bind(self, tensors: dict[str, torch.Tensor]) -> None:
        names = ("q_proj", "k_proj") if self.values_are_keys else ("q_proj", "k_proj", "v_proj")
        weights = [tensors[n + ".weight"] for n in names]
        biases = [tensors[n + ".bias"] for n in names] if self.bias else []
        order = self.position.pair_order() if hasattr(self.position, "pair_order") else None
        if order is not None:
            # The checkpoint pairs neighbouring dimensions: every head's rows of q and k (and what belongs to those
            # dimensions) are brought into the order whose pairs are half a rotary width apart.
            at = torch.tensor(order, device=weights[0].device)
            per_head = lambda t: t.unflatten(0, (-1, self.key_size))[:, at].flatten(0, 1)
            weights[0], weights[1] = per_head(weights[0]), per_head(weights[1])
            if self.bias:
                biases[0], biases[1] = per_head(biases[0]), per_head(biases[1])
        o_weight = tensors["o_proj.weight"]
        if (self.head_dim, self.v_head_dim) != (self.key_size, self.value_size):
            sizes = ((self.key_size, self.head_dim), (self.key_size, self.head_dim), (self.value_size, self.v_head_dim))
            weights = [_padded_heads(w, *size) for w, size in zip(weights, sizes)]
            biases = [_padded_heads(b[:, None], *size)[:, 0] for b, size in zip(biases, sizes)]
            o_weight = _padded_heads(o_weight.t(), self.value_size, self.v_head_dim).t().contiguous()
        if self.head_gate or self.output_gate:
            # The gate's rows ride behind v, filled up to a multiple of 16 rows (what the products' tiles like).
            gate = tensors["g_proj.weight" if self.head_gate else "gate_proj.weight"]
            pad = -(sum(w.shape[0] for w in weights) + gate.shape[0]) % 16
            weights += [gate, gate.new_zeros((pad, self.hidden_size))]
            if self.bias:
                biases.append(biases[0].new_zeros(gate.shape[0] + pad))
        self.qkv_weight = torch.cat(weights).contiguous()
        if self.bias and self.joint_norm:
            self.prep_bias = torch.cat(biases).to(torch.float32).contiguous()
        elif self.bias:
            self.qkv_bias = torch.cat(biases).contiguous()
        if self.value_mix == "mixed":
            self.blend = tensors["value_mix"].to(torch.float32).reshape(1).contiguous()
        self.o_weight = o_weight
        if self.qk_norm and self.qk_norm_weight:
            self.q_norm_weight, self.k_norm_weight = tensors["q_norm.weight"], tensors["k_norm.weight"]
            if order is not None and self.qk_norm == "head":
                self.q_norm_weight, self.k_norm_weight = self.q_norm_weight[at].contiguous(), self.k_norm_weight[at].contiguous()
            elif order is not None:
                self.q_norm_weight, self.k_norm_weight = per_head(self.q_norm_weight), per_head(self.k_norm_weight)
        if self.joint_norm and self.head_dim != self.key_size:
            self.q_norm_weight, self.k_norm_weight = (_padded_heads(w[:, None], self.key_size, self.head_dim)[:, 0].contiguous()
                                                      for w in (self.q_norm_weight, self.k_norm_weight))
        if self.has_sink:
            self.sink = tensors["sink"].to(torch.float32).contiguous()
        elif self.fixed_sink is not None:
            self.sink = torch.full((self.heads,), self.fixed_sink, dtype=torch.float32, device=self.qkv_weight.device)
        self.o_bias = tensors.get("o_proj.bias") if self.out_bias else None
        self.position.bind({n[len("position."):]: t for n, t in tensors.items() if n.startswith("position.")})

    def cache_needs(self) -> tuple:
        return (KVNeed(self.kv_heads, self.head_dim, self.window, name=self.cache_name,
                       v_head_dim=None if self.v_head_dim == self.head_dim else self.v_head_dim,
                       keep_first=self.keep_first, chunk=self.chunk),)

    # ------------------------------------------------- what a mixer made of several uses
    @property
    def in_weight(self) -> torch.Tensor:
        return self.qkv_weight

    @property
    def out_weight(self) -> torch.Tensor:
        return self.o_weight

    @property
    def mixed_width(self) -> int:
        return self.heads * self.v_head_dim

    @property
    def has_biases(self) -> bool:
        return (self.bias and not self.joint_norm) or self.out_bias

    takes_pending_norm = True       # x may be an ops.PendingNorm: the qkv product folds the norm in
    adds_to_residual = True         # the output projection adds into the residual stream where its kernel can

    def forward(self, x, ctx: StepContext, cache: LayerCache, residual: torch.Tensor | None = None):
        qkv = torch.empty((x.shape[0], self.qkv_weight.shape[0]), dtype=x.dtype, device=x.device)
        ops.linear(x, self.qkv_weight, qkv, self.qkv_bias)
        attended = torch.empty((x.shape[0], self.mixed_width), dtype=x.dtype, device=x.device)
        self.mix(qkv, ctx, cache, attended)
        return ops.linear(attended, self.o_weight, None, self.o_bias, residual=residual)

    def mix(self, qkv: torch.Tensor, ctx: StepContext, cache: LayerCache, attended: torch.Tensor) -> None:
        """From the projection's rows to the heads' outputs, `attended` [tokens, mixed_width] (both may be column slices
        of wider tensors; q is rotated in place)."""
        kv = cache.kvs[self.cache_name]
        q_width, kv_width = self.heads * self.head_dim, self.kv_heads * self.head_dim
        table = ctx.block_tables[kv.group]
        rotary = self.position.rotary()
        masked = dict(keep_first=self.keep_first, softcap=self.softcap) if (self.keep_first or self.softcap) else {}
        if self.sink is not None:
            masked["sink"] = self.sink
        prepared = self.qk_norm == "head" or self.head_gate or self.output_gate or self.value_mix
        if self.qk_norm and not prepared and not self.joint_norm:
            ops.qk_projection_rmsnorm_(qkv[:, :q_width], self.q_norm_weight, qkv[:, q_width:q_width + kv_width],
                                       self.k_norm_weight, self.qk_norm_eps)
        plain = (not masked and not prepared and not self.joint_norm and self.v_head_dim % self.head_dim == 0
                 and (rotary is None or rotary.attention_scaling == 1.0))
        newest = {}
        if plain and rotary is not None and ops.fused_decode_supports(qkv.dtype, self.heads, self.kv_heads, self.head_dim,
                                                                      rotary.rotary_dim, ctx.plan):
            # Every sequence brings one token: one launch rotates q and k, stores k and v and attends.
            newest["newest"] = ops.NewestToken(rotary.inv_freq, qkv[:, q_width:], qkv[:, q_width + kv_width:],
                                               store=not cache.read_only)
        else:
            self._store(qkv, ctx, cache, kv, table, rotary, prepared)
        if self.chunk is not None:
            masked["chunk"] = self.chunk
        ops.paged_attention(qkv, qkv.stride(0), attended, kv.k_pool, kv.v_pool, table, ctx.query_start_loc,
                            ctx.context_lens, ctx.num_seqs, ctx.max_query_len, self.heads, self.kv_heads,
                            self.head_dim, self.scale, self.window or 0, plan=ctx.plan,
                            decode_splits=ctx.decode_splits, **masked, **newest)
        gate_at = q_width + kv_width + self.kv_heads * self.v_head_dim
        if self.head_gate:
            ops.sigmoid_gate_heads_(attended, qkv[:, gate_at:gate_at + self.heads], self.heads)
        elif self.output_gate:
            ops.sigmoid_gate_(attended, qkv[:, gate_at:gate_at + self.heads * self.v_head_dim])

    def _store(self, qkv: torch.Tensor, ctx: StepContext, cache: LayerCache, kv, table, rotary, prepared) -> None:
        """q rotated in place, k rotated and stored, v stored; for an attention with per-head q/k norms or mixed values,
        or whose rows lie in a wider tensor, one kernel that also normalises q and k and blends v."""
        q_width, kv_width = self.heads * self.head_dim, self.kv_heads * self.head_dim
        v_width = self.kv_heads * self.v_head_dim
        if rotary is None:
            self.position.apply(qkv[:, :q_width].unflatten(1, (self.heads, self.head_dim)),
                                qkv[:, q_width:q_width + kv_width].unflatten(1, (self.kv_heads, self.head_dim)), ctx)
        if self.joint_norm:
            ops.projection_norm_rope_kv_write(
                qkv, ctx.positions, ctx.seq_of_token, table, kv.k_pool, kv.v_pool, rotary.inv_freq if rotary else None,
                self.heads, self.kv_heads, self.head_dim, rotary.rotary_dim if rotary else 0, self.q_norm_weight,
                self.k_norm_weight, self.heads * self.key_size, self.kv_heads * self.key_size, self.qk_norm_eps,
                bias=self.prep_bias, values_are_keys=self.values_are_keys, store=not cache.read_only,
                cos_sin_scale=rotary.attention_scaling if rotary else 1.0)
            return
        if not prepared and qkv.is_contiguous() and qkv.shape[1] == q_width + kv_width + v_width:
            plain = self.v_head_dim == self.head_dim and (rotary is None or rotary.attention_scaling == 1.0)
            wide = {} if plain else dict(v_head_dim=self.v_head_dim,
                                         cos_sin_scale=rotary.attention_scaling if rotary else 1.0)
            ops.rope_kv_write(qkv, ctx.positions, ctx.seq_of_token, table, kv.k_pool, kv.v_pool,
                              rotary.inv_freq if rotary else None, self.heads, self.kv_heads, self.head_dim,
                              rotary.rotary_dim if rotary else 0, store=not cache.read_only, **wide)
            return
        values = qkv[:, q_width + kv_width:q_width + kv_width + v_width]
        other = None
        if self.value_mix == "source":
            ctx.extras[self.value_mix_key] = values
        elif self.value_mix == "mixed":
            other = ctx.extras.get(self.value_mix_key)
            if other is None or other.shape != values.shape:
                raise ValueError("a layer that mixes values runs behind the layer whose values it mixes in, "
                                 "with values of the same shape")
        per_head = self.qk_norm == "head"
        options = {}
        if per_head and (not self.qk_norm_weight or self.qk_norm_after_rotation):
            options = dict(unit_norm=not self.qk_norm_weight, norm_after_rotation=self.qk_norm_after_rotation)
        if rotary is not None and rotary.attention_scaling != 1.0:
            options["cos_sin_scale"] = rotary.attention_scaling
        ops.head_norm_rope_kv_write(qkv, ctx.positions, ctx.seq_of_token, table, kv.k_pool, kv.v_pool,
                                    rotary.inv_freq if rotary else None, self.heads, self.kv_heads, self.head_dim,
                                    rotary.rotary_dim if rotary else 0,
                                    self.q_norm_weight if per_head else None, self.k_norm_weight if per_head else None,
                                    self.qk_norm_eps, store=not cache.read_only, v_other=other,
                                    blend=self.blend if other is not None else None, **options)


def _padded_heads(weight: torch.Tensor, old: int, new: int) -> torch.Tensor:
    """[heads * old, n] with zero rows behind every head's, [heads * new, n]."""
    heads = weight.unflatten(0, (-1, old))
    return torch.cat([heads, heads.new_zeros((heads.shape[0], new - old, heads.shape[2]))], dim=1).flatten(0, 1)


def _sink_init(shape, generator):
    return torch.randn(shape, generator=generator)


def _blend_init(shape, generator):
    """A blending weight in [0.2, 0.8]."""
    return 0.2 + 0.6 * torch.rand(shape, generator=generator)


register_mixer("attention", Attention)
