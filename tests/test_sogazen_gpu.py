"""Sogazen's kernels each against the plain torch function of the same name (`torch_kernels.py`), the plain mechanisms of
`plain_sogazen.py` or a closed form, and the whole model through `bin/trace_run` in float32 and bfloat16 against
`plain_sogazen.py`."""

from __future__ import annotations

import pytest
import torch

import plain_sogazen
import replay_harness as rh
import sogazen_configs as sc
import torch_kernels as ref
from test_gifudra_gpu import _batch
from test_kernels_gpu import _plan_for
from test_lulisun_gpu import _case, _filled, _ints, _randn, _tol, _typical_error

pytestmark = pytest.mark.gpu

DEV = "cuda:0"
DTYPES = [torch.float32, torch.bfloat16]


# ------------------------------------------------------------------ norms, rotation and cache write in one
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,kv_heads,dim,real,rot,page,lead", [
    (6, 2, 16, 16, 8, 16, 8), (4, 1, 128, 96, 64, 16, 16), (3, 3, 6, 6, 2, 8, 3), (5, 1, 7, 7, 0, 4, 1), (8, 2, 64, 64, 64, 16, 0),
    (2, 2, 64, 40, 24, 16, 8), (32, 8, 128, 128, 128, 32, 0)])
@pytest.mark.parametrize("tied,biased", [(True, True), (True, False), (False, True), (False, False)])
def test_norm_over_the_projection_rotation_and_cache_write(dtype, heads, kv_heads, dim, real, rot, page, lead, tied, biased):
    """Heads rounded up with zeros, rows in wider tensors, values of their own or the keys as projected, with and without
    biases and rotation, portions and single tokens, rows of padding."""
    from liteinfer_b200 import ops

    q_lens, ctx_lens = [3, 1, 20], [11, 40, 20]
    T, pad = sum(q_lens), 2
    pages = sum(-(-c // page) for c in ctx_lens) + 2
    table, positions, seq_of, _, _ = _batch(q_lens, ctx_lens, page, pages, 3)
    positions, seq_of = torch.cat([positions, _ints([0] * pad)]), torch.cat([seq_of, _ints([-1] * pad)])
    qk = (heads + kv_heads) * dim
    columns = qk + (0 if tied else kv_heads * dim)
    live = (torch.arange(dim, device=DEV) < real).float().repeat(columns // dim)
    rows = (_randn(T + pad, columns, seed=1, scale=2.0) * live).to(dtype)
    bias = _randn(columns, seed=2) * live if biased else None
    q_norm, k_norm = ((1 + 0.3 * _randn(n * dim, seed=3 + n)) * live[:n * dim] for n in (heads, kv_heads))
    inv_freq = (1000.0 ** (-torch.arange(rot // 2, dtype=torch.float64) * 2 / max(rot, 1))).float().to(DEV) if rot else None
    results = []
    for impl in (ops, ref):
        wide = torch.zeros(T + pad, lead + columns + 8, dtype=dtype, device=DEV)
        row = wide[:, lead:lead + columns + 8]
        row[:, :columns] = rows
        pools = [torch.zeros(pages, kv_heads, page, dim, dtype=dtype, device=DEV) for _ in range(2)]
        impl.projection_norm_rope_kv_write(row, positions, seq_of, table, *pools, inv_freq, heads, kv_heads, dim, rot, q_norm,
                                           k_norm, heads * real, kv_heads * real, 1e-4, bias=bias, values_are_keys=tied)
        results.append((row[:T, :heads * dim], *pools, row[:, qk:columns], wide[:, lead + columns:]))
    for got, want in zip(*results):
        torch.testing.assert_close(got.float(), want.float(), **_tol(dtype))
    # One head of the plain mechanism: the mean runs over the real numbers of the projection alone.
    q = rows[:T].double().cpu()[:, :heads * dim] + (bias.double().cpu()[:heads * dim] if biased else 0.0)
    q = q.view(T, heads, dim)[:, :, :real].reshape(T, heads * real)
    want = plain_sogazen.unit_rms(q, 1e-4) * q_norm.double().cpu().view(heads, dim)[:, :real].reshape(-1)
    if not rot:
        torch.testing.assert_close(results[0][0].double().cpu(), want, **_tol(dtype))


# ------------------------------------------------------------------ a fixed sink and capped scores on every attention kernel
@pytest.mark.parametrize("heads,kv_heads,d,page", [(4, 2, 64, 16), (8, 1, 128, 16), (6, 3, 128, 32), (3, 1, 64, 64), (4, 2, 20, 8)])
@pytest.mark.parametrize("softcap", [0.0, 4.0, 30.0])
@pytest.mark.parametrize("splits", [None, 1, 3])
@pytest.mark.parametrize("dtype", DTYPES)
def test_sink_of_zero_and_capped_scores(dtype, heads, kv_heads, d, page, softcap, splits):
    """Prompts and portions on tcgen05, single tokens on the split kernels (bfloat16), everything on the plain one (32-bit,
    other sizes): scores scaled so that the cap bends them and the sink's weight is far from none."""
    from liteinfer_b200 import ops

    q_lens, ctx_lens = [1, 130, 1, 7, 1, 257], [500, 190, 1, 7, 129, 300]
    q, rest = _case(dtype, heads, kv_heads, d, d, page, q_lens, ctx_lens, 0, lead=8)
    sink = torch.zeros(heads, device=DEV)
    for scale in (3.0 * d ** -0.5, 1e-4):       # scores of several units, and scores of nothing: n keys weigh 1 / (n + 1)
        tail = (len(q_lens), max(q_lens), heads, kv_heads, d, scale)
        out = lambda: torch.full((sum(q_lens), heads * d), float("nan"), dtype=dtype, device=DEV)
        options = dict(softcap=softcap, sink=sink)
        want = ref.paged_attention(q, q.stride(0), out(), *_filled(rest), *tail, **options)
        got = ops.paged_attention(q, q.stride(0), out(), *rest, *tail, plan=_plan_for(q_lens, ctx_lens), decode_splits=splits,
                                  **options)
        torch.testing.assert_close(got.float(), want.float(), **_tol(dtype))
    assert ops.gemm_error_flag(DEV) == 0


@pytest.mark.parametrize("d,page,dtype", [(64, 16, torch.bfloat16), (128, 16, torch.bfloat16), (48, 8, torch.bfloat16),
                                          (64, 16, torch.float32)])
@pytest.mark.parametrize("decode", [False, True])
def test_one_key_stands_out_under_the_cap_and_all_keys_vanish_behind_the_sink(d, page, dtype, decode):
    """A far key whose score is lifted high above all others is found by the last query through the cap; with every score
    far below the sink's 0 the output is nothing."""
    from liteinfer_b200 import ops

    heads, kv_heads, ctx, cap = 4, 2, 700, 25.0
    n = 1 if decode else 9
    sink = torch.zeros(heads, device=DEV)
    for target in (0, 15, 16, 63, 64, 350, 698, 699):
        q, rest = _case(dtype, heads, kv_heads, d, d, page, [n], [ctx], 0)
        k_pool, v_pool, table = rest[:3]
        k_pool.nan_to_num_(0.0).mul_(0.01)
        v_pool.nan_to_num_(0.0)
        lifted = _randn(d, seed=3)
        k_pool[int(table[0, target // page]), :, target % page] = lifted.to(dtype)
        q[-1] = (lifted * 3.0).to(dtype).repeat(heads)
        found = v_pool[int(table[0, target // page]), :, target % page].float().repeat_interleave(heads // kv_heads, 0)
        run = lambda scale: ops.paged_attention(q, q.stride(0), torch.empty(n, heads * d, dtype=dtype, device=DEV), *rest, 1, n, heads,
                                                kv_heads, d, scale, plan=_plan_for([n], [ctx]), softcap=cap,
                                                sink=sink)[-1].float().view(heads, d)
        torch.testing.assert_close(run(1.0), found, rtol=3e-2, atol=3e-2)
        k_pool.zero_()
        k_pool[:] = -lifted.to(dtype)
        assert float(run(1.0).abs().max()) < 1e-4


# ------------------------------------------------------------------ the state space
def _space_case(dtype, heads, groups, dim, vdim, tokens, seed=1, lead=0):
    conved = _randn(tokens, heads * vdim + 2 * groups * dim, seed=seed, dtype=dtype)
    dt = _randn(tokens, lead + heads + 3, seed=seed + 1, dtype=dtype)[:, lead:lead + heads]
    return conved, dt, _randn(heads, seed=seed + 2), _randn(heads, seed=seed + 3, scale=0.5)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,groups,dim,vdim", [(4, 2, 20, 12), (6, 3, 64, 64), (2, 1, 128, 48), (3, 3, 5, 7), (4, 1, 1, 6),
                                                   (2, 2, 200, 33), (1, 1, 300, 130), (32, 4, 128, 64), (10, 5, 3, 1)])
def test_state_space_against_the_plain_recurrence(dtype, heads, groups, dim, vdim):
    """Whole prompts, portions and single tokens in one launch, states in shuffled slots, sequences that bring nothing;
    then a step of single tokens only."""
    from liteinfer_b200 import ops

    slots = [3, 0, 6, 5, 1, 7]
    for counts in ([17, 1, 0, 2, 40, 8], [1, 1, 0, 1, 1, 1]):
        qsl = [0]
        for n in counts:
            qsl.append(qsl[-1] + n)
        conved, dt, bias, a_log = _space_case(dtype, heads, groups, dim, vdim, qsl[-1], lead=5)
        states = [_randn(8, heads, vdim, dim, seed=7) for _ in range(2)]
        outs = [torch.zeros(qsl[-1], heads * vdim, device=DEV) for _ in range(2)]
        for impl, state, out in zip((ops, ref), states, outs):
            impl.state_space(conved, dt, bias, a_log, state, _ints(qsl), _ints(slots), len(counts), heads, groups, dim, vdim,
                             out, max(counts))
        torch.testing.assert_close(outs[0], outs[1], rtol=1e-4, atol=1e-4)
        torch.testing.assert_close(states[0], states[1], rtol=1e-4, atol=1e-4)
        assert torch.equal(states[0][6], _randn(8, heads, vdim, dim, seed=7)[6])      # its sequence brings nothing


def test_state_space_of_the_plain_implementation():
    from liteinfer_b200 import ops

    heads, groups, dim, vdim, T = 6, 2, 24, 40, 70
    conved, dt, bias, a_log = _space_case(torch.float32, heads, groups, dim, vdim, T)
    skip = _randn(heads, seed=9)
    out = torch.empty(T, heads * vdim, device=DEV)
    ops.state_space(conved, dt, bias, a_log, torch.zeros(1, heads, vdim, dim, device=DEV), _ints([0, T]), _ints([0]), 1, heads,
                    groups, dim, vdim, out, T)
    z, weight = _randn(T, heads * vdim, seed=10), 1 + 0.2 * _randn(heads * vdim, seed=11)
    got = torch.empty(T, heads * vdim, device=DEV)
    ops.gated_group_norm(out, z, weight, 1e-4, got, 5, add=conved[:, :heads * vdim], skip=skip)
    c = conved.double().cpu()
    x, b, cc = torch.split(c, [heads * vdim, groups * dim, groups * dim], dim=1)
    y = plain_sogazen.state_space(x.view(T, heads, vdim), b.reshape(T, groups, dim), cc.reshape(T, groups, dim),
                                  plain_sogazen.softplus(dt.double().cpu() + bias.double().cpu()), a_log.double().cpu(), skip.double().cpu())
    want = plain_sogazen.gated_group_norm(y.reshape(T, -1), z.double().cpu(), weight.double().cpu(), 5, 1e-4)
    torch.testing.assert_close(got.double().cpu(), want, rtol=2e-5, atol=2e-5)


@pytest.mark.parametrize("single", [False, True])
def test_state_space_holds_a_token_across_a_thousand_others(single):
    """Steps of exactly 0 keep what is held and write nothing; one token with a step of its own is read ever after."""
    from liteinfer_b200 import ops

    heads, dim, vdim, T, written = 2, 64, 32, 1001, 300
    conved = _randn(T, heads * vdim + 2 * dim, seed=4)
    dt = torch.full((T, heads), -200.0, device=DEV)          # softplus: 0 in 32-bit
    dt[written] = 3.0
    zero = torch.zeros(heads, device=DEV)
    state, out = torch.zeros(1, heads, vdim, dim, device=DEV), torch.empty(T, heads * vdim, device=DEV)
    for a, b in ([(0, T)] if not single else [(0, 990)] + [(i, i + 1) for i in range(990, T)]):
        ops.state_space(conved[a:b], dt[a:b], zero, zero, state, _ints([0, b - a]), _ints([0]), 1, heads, 1, dim, vdim, out[a:b], b - a)
    step = float(torch.nn.functional.softplus(torch.tensor(3.0)))
    x, b, c = torch.split(conved, [heads * vdim, dim, dim], dim=1)
    want = step * (c[written:] @ b[written])[:, None] * x[written]
    assert float(out[:written].abs().max()) == 0.0
    torch.testing.assert_close(out[written:], want, rtol=1e-4, atol=1e-4)


# ------------------------------------------------------------------ the time mixer
def _wkv_case(dtype, heads, dim, rank, tokens, seed=1):
    width = heads * dim
    r, k, v, g = _randn(4, tokens, width, seed=seed, dtype=dtype)
    low = _randn(tokens, rank + 3, seed=seed + 1, dtype=dtype)[:, :rank]
    w2 = _randn(width, rank, seed=seed + 2, scale=rank ** -0.5, dtype=dtype)
    w0, u, weight = _randn(width, seed=seed + 3) - 2.0, _randn(width, seed=seed + 4, scale=0.5), 1 + 0.2 * _randn(width, seed=seed + 5)
    return (r, k, v, g, low, w2, w2.t().contiguous(), w0, u), weight


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,dim,rank", [(3, 20, 12), (4, 64, 64), (2, 128, 16), (5, 7, 3), (4, 1, 1), (1, 200, 100), (16, 64, 33),
                                            (1, 300, 5)])
def test_time_mixing_against_the_plain_recurrence(dtype, heads, dim, rank):
    from liteinfer_b200 import ops

    slots = [3, 0, 6, 5, 1, 7]
    for counts in ([17, 1, 0, 2, 40, 8], [1, 1, 0, 1, 1, 1]):
        qsl = [0]
        for n in counts:
            qsl.append(qsl[-1] + n)
        inputs, weight = _wkv_case(dtype, heads, dim, rank, qsl[-1])
        states = [_randn(8, heads, dim, dim, seed=7) for _ in range(2)]
        outs = [torch.zeros(qsl[-1], heads * dim, dtype=dtype, device=DEV) for _ in range(2)]
        for impl, state, out in zip((ops, ref), states, outs):
            impl.wkv_memory(*inputs, state, _ints(qsl), _ints(slots), len(counts), heads, dim, weight, 1e-5, out, max(counts))
        # (where a head is one number, the norm leaves its sign alone: a read-out near zero may fall either way)
        if dim > 1:
            torch.testing.assert_close(outs[0].float(), outs[1].float(), **_tol(dtype))
        torch.testing.assert_close(states[0], states[1], rtol=1e-4, atol=1e-4)
        assert torch.equal(states[0][6], _randn(8, heads, dim, dim, seed=7)[6])


def test_time_mixing_of_the_plain_implementation():
    from liteinfer_b200 import ops

    heads, dim, rank, T = 2, 24, 6, 70
    (r, k, v, g, low, w2, w2t, w0, u), weight = _wkv_case(torch.float32, heads, dim, rank, T)
    out = torch.empty(T, heads * dim, device=DEV)
    ops.wkv_memory(r, k, v, g, low, w2, w2t, w0, u, torch.zeros(1, heads, dim, dim, device=DEV), _ints([0, T]), _ints([0]), 1, heads,
                   dim, weight, 1e-4, out, T)
    f = lambda x: x.double().cpu()
    decay = torch.exp(-torch.exp(torch.tanh(f(low)) @ f(w2).T + f(w0)))
    o = plain_sogazen.bonus_memory(*(f(x).view(T, heads, dim) for x in (r, k, v)), decay.view(T, heads, dim), f(u).view(heads, dim))
    want = plain_sogazen.unit_rms(o, 1e-4).reshape(T, -1) * f(weight) * plain_sogazen.silu(f(g))
    torch.testing.assert_close(f(out), want, rtol=5e-5, atol=5e-5)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("dim", [32, 64, 128])
def test_memories_do_not_depend_on_the_cut(dtype, dim):
    """A sequence whole, in portions of every kind (two tokens, a chunk of the kernel's less one, ...) and token by token."""
    from liteinfer_b200 import ops

    heads, groups, vdim, rank, T = 4, 2, 24, 8, 83
    conved, dt, bias, a_log = _space_case(dtype, heads, groups, dim, vdim, T)
    inputs, weight = _wkv_case(dtype, heads, dim, rank, T)

    def run(cuts):
        space, read = torch.zeros(2, heads, vdim, dim, device=DEV), torch.empty(T, heads * vdim, device=DEV)
        memory, out = torch.zeros(2, heads, dim, dim, device=DEV), torch.empty(T, heads * dim, dtype=dtype, device=DEV)
        for a, b in zip(cuts, cuts[1:]):
            at = (_ints([0, b - a]), _ints([1]), 1)
            ops.state_space(conved[a:b], dt[a:b], bias, a_log, space, *at, heads, groups, dim, vdim, read[a:b], b - a)
            ops.wkv_memory(*(x[a:b] for x in inputs[:5]), *inputs[5:], memory, *at, heads, dim, weight, 1e-5, out[a:b], b - a)
        return read, space[1], out, memory[1]

    whole = run([0, T])
    for cuts in ([0, 2, 4, 11, 26, 27, 43, 59, 60, T], [0, 7, 15, 16, 64, 82, T], list(range(T + 1))):
        for i, (got, want) in enumerate(zip(run(cuts), whole)):
            tol = _tol(dtype) if i == 2 else dict(rtol=5e-5, atol=5e-5)
            torch.testing.assert_close(got.float(), want.float(), **tol)


@pytest.mark.parametrize("single", [False, True])
def test_time_mixing_holds_a_token_across_a_thousand_others(single):
    """Decays of exactly 1 and keys of 0: the read-out of the last token is the value of the one that was written, and a
    channel whose decay is 0 has forgotten it by the second next token."""
    from liteinfer_b200 import ops

    dim, T, written = 64, 1001, 300
    r = torch.ones(T, dim, device=DEV)
    k = torch.zeros(T, dim, device=DEV)
    k[written] = 1.0
    v, g = _randn(T, dim, seed=4), torch.full((T, dim), 30.0, device=DEV)
    low, w2 = torch.zeros(T, 2, device=DEV), torch.zeros(dim, 2, device=DEV)
    ones, none = torch.ones(dim, device=DEV), torch.zeros(dim, device=DEV)
    for w0, keeps in ((-200.0, True), (200.0, False)):
        state, out = torch.zeros(1, 1, dim, dim, device=DEV), torch.empty(T, dim, device=DEV)
        for a, b in ([(0, T)] if not single else [(0, 290)] + [(i, i + 1) for i in range(290, T)]):
            ops.wkv_memory(r[a:b], k[a:b], v[a:b], g[a:b], low[a:b], w2, w2.t().contiguous(), none + w0, none, state,
                           _ints([0, b - a]), _ints([0]), 1, 1, dim, ones, 1e-6, out[a:b], b - a)
        want = v[written] / torch.sqrt(v[written].pow(2).mean()) * 30.0
        assert float(out[:written + 1].abs().max()) == 0.0
        torch.testing.assert_close(out[written + 1], want, rtol=1e-4, atol=1e-4)
        if keeps:
            torch.testing.assert_close(out[written + 1:], want.expand(T - written - 1, dim), rtol=1e-4, atol=1e-4)
        else:
            assert float(out[written + 2:].abs().max()) == 0.0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [64, 37, 2048, 4104])
def test_token_shift(dtype, width):
    """Portions and single tokens whose `before` lies in shuffled slots, rows of padding; the step of single tokens that moves
    it on in the same launch."""
    from liteinfer_b200 import ops

    slots, mu = [3, 0, 5, 1], torch.rand(5, width, device=DEV)
    for counts in ([7, 1, 0, 30], [1, 1, 0, 1], [1, 1, 1, 1]):
        qsl = [0]
        for n in counts:
            qsl.append(qsl[-1] + n)
        T = qsl[-1]
        seq_of = _ints([s for s, n in enumerate(counts) for _ in range(n)] + [-1])
        x = _randn(T + 1, width, seed=1, dtype=dtype)
        results = []
        for impl in (ops, ref):
            before, out = _randn(7, 1, width, seed=2, dtype=dtype), torch.empty(5, T + 1, width, dtype=dtype, device=DEV)
            impl.token_shift_step(x, mu, before, seq_of, _ints(qsl), _ints(slots), 4, out, single_tokens=counts == [1] * 4)
            results.append((out, before))
        torch.testing.assert_close(results[0][0].float(), results[1][0].float(), **_tol(dtype))
        assert torch.equal(results[0][1], results[1][1])
        assert torch.equal(results[0][1][6], _randn(7, 1, width, seed=2, dtype=dtype)[6])
    whole = torch.empty(5, T + 1, width, dtype=dtype, device=DEV)
    ops.token_shift_step(x, mu, torch.zeros(1, 1, width, dtype=dtype, device=DEV), torch.zeros(T + 1, dtype=torch.int32, device=DEV),
                         _ints([0, T + 1]), _ints([0]), 1, whole)
    want = plain_sogazen.token_shift(x.double().cpu(), mu[2].double().cpu())
    torch.testing.assert_close(whole[2].double().cpu(), want, **_tol(dtype))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("channels,taps", [(64, 4), (37, 3), (128, 1), (40, 7)])
def test_short_convolution_with_a_bias(dtype, channels, taps):
    from liteinfer_b200 import ops

    bias, weight = _randn(channels, seed=1), _randn(taps, channels, seed=2, scale=0.5, dtype=dtype)
    for counts in ([9, 1, 0, 2], [1, 1, 1, 1]):
        qsl = [0]
        for n in counts:
            qsl.append(qsl[-1] + n)
        x = _randn(qsl[-1], 8 + channels + 8, seed=3, dtype=dtype)[:, 8:8 + channels]
        seq_of = _ints([s for s, n in enumerate(counts) for _ in range(n)])
        results = []
        for impl in (ops, ref):
            tail, out = _randn(6, taps - 1, channels, seed=4, dtype=dtype), torch.empty(qsl[-1], channels, dtype=dtype, device=DEV)
            impl.short_conv_step(x, weight, tail, seq_of, _ints(qsl), _ints([4, 2, 0, 1]), 4, out,
                                 single_tokens=counts == [1] * 4, bias=bias)
            results.append((out, tail))
        torch.testing.assert_close(results[0][0].float(), results[1][0].float(), **_tol(dtype))
        assert torch.equal(results[0][1], results[1][1])
    out = torch.empty(9, channels, dtype=dtype, device=DEV)
    ops.short_conv_step(x.new_zeros(9, channels) + x[:1], weight, torch.zeros(1, taps - 1, channels, dtype=dtype, device=DEV),
                        torch.zeros(9, dtype=torch.int32, device=DEV), _ints([0, 9]), _ints([0]), 1, out, bias=bias)
    want = plain_sogazen.silu(plain_sogazen.causal_conv(x[:1].double().cpu().expand(9, channels), weight.double().cpu().T, bias.double().cpu()))
    torch.testing.assert_close(out.double().cpu(), want, **_tol(dtype))


# ------------------------------------------------------------------ norms
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,size,groups", [(4, 64, 2), (3, 7, 7), (8, 128, 1), (2, 48, 3), (1, 5, 5), (64, 64, 1), (64, 128, 4), (5, 12, 60)])
def test_gate_in_front_of_a_norm_of_parts(dtype, heads, size, groups):
    from liteinfer_b200 import ops

    T, width = 11, heads * size
    x, weight, skip = _randn(T, width, seed=1), 1 + 0.3 * _randn(width, seed=2), _randn(heads, seed=3)
    wide = _randn(T, 2 * width + 16, seed=4, dtype=dtype)
    gate, add = wide[:, 8:8 + width], wide[:, 8 + width:8 + 2 * width]
    for options in ({}, dict(add=add, skip=skip)):
        outs = [torch.empty(T, width + 8, dtype=dtype, device=DEV)[:, :width] for _ in range(2)]
        for impl, out in zip((ops, ref), outs):
            impl.gated_group_norm(x, gate, weight, 1e-5, out, groups, **options)
        torch.testing.assert_close(outs[0].float(), outs[1].float(), **_tol(dtype))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,size", [(4, 64), (3, 7), (2, 200), (16, 128)])
def test_gated_norm_per_head_with_an_addend(dtype, heads, size):
    from liteinfer_b200 import ops

    T, width = 9, heads * size
    x, weight, share = _randn(T, width, seed=1), 1 + 0.3 * _randn(width, seed=2), _randn(T, heads, seed=3)
    gate, add = (_randn(T, width + 8, seed=4 + i, dtype=dtype)[:, :width] for i in range(2))
    outs = [torch.empty(T, width, dtype=dtype, device=DEV) for _ in range(2)]
    for impl, out in zip((ops, ref), outs):
        impl.gated_rmsnorm(x, gate, weight, 1e-5, out, heads, add=add, add_scale=share)
    torch.testing.assert_close(outs[0].float(), outs[1].float(), **_tol(dtype))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [48, 37, 2048, 5120, 12288])
def test_output_norm(dtype, width):
    """Two normed terms, a dense one with a factor a row beside experts' rows of which some are missing, one term: the sum
    normed, added into the stream; the stream rounded, normed (all rows or some), or only moved on."""
    from liteinfer_b200 import ops

    T, top = 9, 3
    x0 = _randn(T, width, seed=1, scale=5.0)
    weights = [1 + 0.3 * _randn(width, seed=6 + i) for i in range(4)]
    dense = [_randn(T, width, seed=2 + i, scale=3.0, dtype=dtype) for i in range(2)]
    rows = _randn(T * top, width, seed=4, dtype=dtype)
    place = torch.randperm(T * top, generator=torch.Generator().manual_seed(5)).to(torch.int32)
    place[::4] = -1
    routed = ops.RoutedRows(rows, top, place.to(DEV))
    share = torch.rand(T, device=DEV)
    pick = _ints([7, 0, 7])
    for total in (ops.SumDelta((ops.SumTerm(dense[0], 0.5, None, weights[0], 1e-3), ops.SumTerm(dense[1], 0.7, None, weights[1], 1e-5))),
                  ops.SumDelta((ops.SumTerm(dense[0], 1.0, share),), routed), ops.SumDelta((ops.SumTerm(dense[1], 1.3),)),
                  ops.SumDelta((), ops.RoutedRows(rows, top)),
                  ops.SumDelta((ops.SumTerm(dense[0], 1.0), ops.SumTerm(dense[1], 0.7, share, weights[1], 1e-5)), routed)):
        delta = ops.NormedDelta(total, weights[2], 1e-4, centred=False)
        for out_rows, final, write in ((T, None, True), (T, weights[3], True), (3, weights[3], False), (0, None, True)):
            results = []
            for impl in (ops, ref):
                x = x0.clone()
                out = torch.empty(out_rows, width, dtype=dtype, device=DEV) if out_rows else None
                impl.output_norm(x, delta, out, final, 1e-5, rows=pick if out_rows == 3 else None, write_stream=write)
                results.append((x, out))
            torch.testing.assert_close(results[0][0], results[1][0], rtol=1e-5, atol=1e-4)
            if out_rows:
                torch.testing.assert_close(results[0][1].float(), results[1][1].float(), **_tol(dtype))
            assert write or torch.equal(results[0][0], x0)


# ------------------------------------------------------------------ feed-forwards
@pytest.mark.parametrize("experts,identity,top", [(4, 2, 2), (3, 5, 4), (1, 1, 1), (8, 8, 8), (60, 30, 6), (128, 64, 8), (2, 3, 5)])
def test_router_with_identity_experts_against_the_plain_mechanism(experts, identity, top):
    from liteinfer_b200 import ops

    outputs = experts + identity
    correction, w = 0.3 * _randn(outputs, seed=outputs), _randn(outputs, 40, seed=6, scale=0.7)
    for dtype in DTYPES:
        for count in (1, 77, 300):
            x = _randn(count, 3 + 40 + 2, seed=5, dtype=dtype)[:, 3:43]
            ids, weights = torch.empty(count, top, dtype=torch.int32, device=DEV), torch.empty(count, top, device=DEV)
            same = torch.full((count,), float("nan"), device=DEV)
            ops.moe_router(x, w, top, 1, 1, False, ids, weights, correction=correction, identity=same, identity_experts=identity)
            chosen, want = plain_sogazen.route(x.double().cpu() @ w.double().cpu().T, correction.double().cpu(), top)
            agree = (ids.cpu().long() == chosen).all(-1)
            assert float(agree.double().mean()) > 0.97       # (a close call may fall the other way)
            torch.testing.assert_close(weights.double().cpu()[agree], want[agree], rtol=1e-4, atol=1e-6)
            total = (want * (chosen >= experts)).sum(-1)
            torch.testing.assert_close(same.double().cpu()[agree], total[agree], rtol=1e-4, atol=1e-6)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width,ff,experts,identity,top", [(32, 16, 6, 2, 3), (64, 64, 4, 0, 2), (36, 10, 3, 5, 4), (128, 33, 2, 2, 4),
                                                           (64, 24, 1, 6, 2), (256, 320, 5, 3, 2)])
@pytest.mark.parametrize("tokens", [1, 5, 300])
def test_experts_without_gates_and_identity_experts(dtype, width, ff, experts, identity, top, tokens):
    """Every form of the grouped products (tcgen05, mma.sync, FFMA tiles), pairs without an expert among the others; also where
    every pair of the step goes to an identity expert."""
    from liteinfer_b200 import ops
    from liteinfer_b200.parts.feed_forward import RoutedExperts

    part = RoutedExperts(width, ff, experts, top, dtype, torch.device(DEV), activation="relu_squared", correction=True,
                         gives_sum=True, identity=identity)
    tensors = {n: _randn(*s.shape, seed=i, scale=0.3).to(torch.bfloat16).to(torch.float32 if s.kind == "f32" else dtype)
               for i, (n, s) in enumerate(part.tensor_specs().items())}
    for nothing in ((False, True) if identity >= top else (False,)):
        if nothing:
            tensors["correction"] = (torch.arange(experts + identity, device=DEV) >= experts).float() * 5.0
        part.bind(tensors)
        x = _randn(tokens, width, seed=99, dtype=torch.bfloat16).to(dtype)
        delta = part.forward(x, None)
        stream, ones = torch.zeros(tokens, width, device=DEV), torch.ones(width, device=DEV)
        # (an eps far above everything: the norm is a division by a known constant)
        ops.output_norm(stream, ops.NormedDelta(delta, ones, 1e12, centred=False))
        got = stream.double().cpu() * 1e6
        w = {n.replace("experts.", "e").replace("_proj.weight", "").replace(".weight", ""): t.double().cpu() for n, t in tensors.items()}
        want = plain_sogazen.moe_ff(x.double().cpu(), w, "", {"router": {"experts": experts, "identity": identity, "top": top}})
        off = (got - want).pow(2).mean(1).sqrt() / want.pow(2).mean().sqrt()
        assert float((off > (2e-5 if dtype == torch.float32 else 0.02)).double().mean()) <= 0.02, float(off.max())
        assert torch.isfinite(got).all()
    assert ops.gemm_error_flag(DEV) == 0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width,ff", [(64, 40), (36, 11), (256, 512), (128, 24)])
@pytest.mark.parametrize("tokens", [1, 8, 13, 100, 300])
def test_capped_feed_forward(dtype, width, ff, tokens):
    """Every kernel that joins gate and up, with inputs far beyond the caps on both sides."""
    from liteinfer_b200.parts.feed_forward import GatedMLP

    part = GatedMLP(width, ff, "capped_swiglu", dtype, torch.device(DEV), limit=0.8, alpha=1.702)
    tensors = {n: _randn(*s.shape, seed=i, scale=2.0 * s.shape[1] ** -0.5).to(torch.bfloat16).to(dtype)
               for i, (n, s) in enumerate(part.tensor_specs().items())}
    part.bind(tensors)
    x = _randn(tokens, width, seed=99, dtype=torch.bfloat16).to(dtype)
    got = part.forward(x, None)
    w = {n.replace("_proj.weight", ""): t.double().cpu() for n, t in tensors.items()}
    want = plain_sogazen.dense_ff(x.double().cpu(), w, "", {"limit": 0.8})
    off = float((got.double().cpu() - want).pow(2).mean().sqrt() / want.pow(2).mean().sqrt())
    assert off < (1e-5 if dtype == torch.float32 else 0.01)


# ------------------------------------------------------------------ the whole model
@pytest.fixture(scope="module")
def sogazen_dirs(tmp_path_factory):
    base = tmp_path_factory.mktemp("sogazen")
    return {name: sc.write_model(cfg, base / name, seed) for name, (cfg, seed, _) in sc.ALL.items()}


def _expected(model_dir, requests):
    config, tensors = plain_sogazen.read_model(model_dir)
    return {name: plain_sogazen.forward(config, tensors, tokens).float() for name, tokens in requests.items()}


@pytest.mark.parametrize("name,lengths", [("sog_a", (1, 7, 61, 90)), ("sog_b", (2, 30, 45)), ("sog_c", (5, 52, 150, 18, 270)),
                                           ("sog_d", (4, 33, 58, 21)), ("sog_e", (300, 17, 149))])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_replay_all_cuts(sogazen_dirs, tmp_path, name, lengths, dtype):
    """Whole, the tail decoded, portions down to two tokens, four live requests whose pages and slots are used again, and
    every token a step of its own from the first one on: the same logits as the plain implementation."""
    config, _, page = sc.ALL[name]
    requests = {f"r{i}": sc.prompt(config["vocab"], n, 100 + i) for i, n in enumerate(lengths)}
    expected = _expected(sogazen_dirs[name], requests)
    trace = rh.Trace()
    rh.whole(trace, requests)
    rh.tail_decoded(trace, requests, tail=40)
    rh.portions(trace, requests)
    rh.mixed(trace, requests)
    longest = max(requests, key=lambda r: len(requests[r]))
    for i, token in enumerate(requests[longest]):
        trace.add([(f"o-{longest}", [token], [0])], end=[f"o-{longest}"] if i == len(requests[longest]) - 1 else [])
    results = rh.run_program(trace, sogazen_dirs[name], dtype, tmp_path / "out", config["vocab"], page_size=page)
    wanted = rh.gather_expected(trace, expected)
    if dtype == "float32":
        worst, where = rh.worst_error(results, wanted)
        assert worst < 2 * sc.FLOAT32_TOLERANCE[name], f"worst difference {worst} at step {where}"
        return
    # bfloat16: a router's close call may choose another expert than the 64-bit run does, at a position here and there.
    rows = _typical_error(results, wanted)
    assert float(rows.median()) < 0.03, f"typical relative difference {float(rows.median())}"
    assert float((rows > 0.12).double().mean()) < 0.1, f"worst relative difference {float(rows.max())}"


@pytest.mark.parametrize("seed", [1, 2, 3, 5, 8, 13])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_configurations_drawn_at_random(tmp_path, seed, dtype):
    """Layer orders, sizes and options drawn at random, every way of cutting, against the plain implementation."""
    config = sc.random_config(seed)
    model_dir = sc.write_model(config, tmp_path / "model", seed)
    requests = {f"r{i}": sc.prompt(config["vocab"], n, 7 + i) for i, n in enumerate((1, 23, 129, 200))}
    expected = _expected(model_dir, requests)
    trace = rh.Trace()
    rh.whole(trace, requests)
    rh.tail_decoded(trace, requests, tail=40)
    rh.portions(trace, requests)
    rh.mixed(trace, requests)
    results = rh.run_program(trace, model_dir, dtype, tmp_path / "out", config["vocab"], page_size=16)
    wanted = rh.gather_expected(trace, expected)
    if dtype == "float32":
        worst, where = rh.worst_error(results, wanted)
        assert worst < 5e-4, f"worst difference {worst} at step {where}"
        return
    typical = float(_typical_error(results, wanted).median())
    assert typical < 0.03, f"typical relative difference {typical}"


def test_layers_one_by_one_against_plain(sogazen_dirs):
    """The residual stream after every layer (32-bit engine) equals the plain implementation's."""
    from liteinfer_b200.engine.loading import build_runner
    from liteinfer_b200.engine.runner import StepEntry

    for name in ("sog_a", "sog_b", "sog_c", "sog_d"):
        config, tensors = plain_sogazen.read_model(sogazen_dirs[name])
        tokens = sc.prompt(config["vocab"], 45, 3)
        want: list = []
        plain_sogazen.forward(config, tensors, tokens, want)
        runner = build_runner(sogazen_dirs[name], torch.float32, DEV, 16, 8, 2)
        runner.cache.reserve(["a"], [45])
        context = runner.build_context([StepEntry("a", tokens, [44])])
        context.layer_trace = []
        runner.model.forward(context, runner.layer_caches)
        assert len(context.layer_trace) == len(want) == len(config["layers"])
        for stop, (got, plain) in enumerate(zip(context.layer_trace, want)):
            assert float((got.cpu().double() - plain).abs().max()) < 2e-4, f"{name}: layer {stop}"


def test_bfloat16_engine_keeps_32_bit_what_must_be_and_rounds_heads_up(sogazen_dirs):
    from liteinfer_b200.engine.loading import build_runner
    from liteinfer_b200.engine.runner import StepEntry

    runner = build_runner(sogazen_dirs["sog_e"], torch.bfloat16, DEV, 16, 8, 2)
    tokens = sc.prompt(sc.SOG_E["vocab"], 20, 3)
    runner.cache.reserve(["a"], [20])
    context = runner.build_context([StepEntry("a", tokens, [19])])
    context.layer_trace = []
    runner.model.forward(context, runner.layer_caches)
    assert all(t.dtype == torch.float32 for t in context.layer_trace)
    parts, states = runner.model.layers[1].parts, runner.layer_caches[1].states
    assert parts["feed_forward"].router.dtype == parts["feed_forward"].correction.dtype == torch.float32
    assert parts["feed_forward"].gate_up.dtype == torch.bfloat16 and parts["mixer_out_norm"].weight.dtype == torch.float32
    assert states["mamba2"].dtype == torch.float32 and states["mamba2_conv"].dtype == torch.bfloat16
    assert runner.layer_caches[2].states["wkv"].dtype == torch.float32
    assert [layer.parts["mixer"].members[0].head_dim for layer in runner.model.layers[:2]] == [64, 128]
    assert runner.layer_caches[1].kv.k_pool.shape[-1] == runner.layer_caches[1].kv.v_pool.shape[-1] == 128


@pytest.mark.parametrize("graphs", [False, True])
@pytest.mark.parametrize("name", ["sog_c", "sog_e"])
def test_mixers_on_two_streams_equal_one_after_the_other(sogazen_dirs, monkeypatch, name, graphs):
    """The state space on a second stream gives what one stream gives, step for step, eager and from graphs."""
    from liteinfer_b200.engine.loading import build_runner
    from liteinfer_b200.engine.runner import StepEntry
    from liteinfer_b200.parts import side_by_side

    config = sc.ALL[name][0]
    tokens = [sc.prompt(config["vocab"], 90, 60 + i) for i in range(3)]
    results = []
    for limit in (0, 256):
        monkeypatch.setattr(side_by_side, "PARALLEL_SUBLAYERS", limit)
        runner = build_runner(sogazen_dirs[name], torch.bfloat16, DEV, 16, 32, 3)
        if graphs:
            runner.enable_decode_graphs(3, 512)
        got = [runner.step([StepEntry(str(i), t[:70 + i], [69 + i]) for i, t in enumerate(tokens)]).clone()]
        for at in range(74, 90):
            got.append(runner.step([StepEntry(str(i), t[at:at + 1], [0]) for i, t in enumerate(tokens)]).clone())
        runner.check_kernels()
        results.append(torch.cat(got))
    assert torch.isfinite(results[0].float()).all()
    torch.testing.assert_close(results[1].float(), results[0].float(), rtol=2 ** -6, atol=2 ** -6)


def test_greedy_generation_through_the_engine_on_gpu(sogazen_dirs):
    """`LLM.generate` (scheduler with portions of 16 tokens, three seats for five requests, CUDA graphs, sampler) picks the
    plain implementation's tokens over 24 decoded tokens."""
    from liteinfer_b200.engine.llm import LLM
    from liteinfer_b200.sampling.params import SamplingParams

    config, tensors = plain_sogazen.read_model(sogazen_dirs["sog_a"])
    prompts = [sc.prompt(config["vocab"], n, 40 + n) for n in (3, 26, 9, 14, 2)]
    with LLM(str(sogazen_dirs["sog_a"]), dtype="float32", block_size=4, num_gpu_blocks=96, max_num_seqs=3,
             max_model_len=80, max_num_batched_tokens=16) as llm:
        outputs = llm.generate(prompts, SamplingParams(temperature=0.0, max_tokens=24))
    for prompt, output in zip(prompts, outputs):
        tokens = list(prompt)
        for _ in range(24):
            tokens.append(int(plain_sogazen.forward(config, tensors, tokens)[-1].argmax()))
        assert list(output.token_ids) == tokens[len(prompt):]
