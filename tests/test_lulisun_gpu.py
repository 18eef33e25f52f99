"""Lulisun's kernels each against the plain torch function of the same name (`torch_kernels.py`), the plain mechanisms of
`plain_lulisun.py` or a closed form, and the whole model through `bin/trace_run` in float32 and bfloat16 against
`plain_lulisun.py`."""

from __future__ import annotations

import pytest
import torch

import lulisun_configs as lc
import plain_lulisun
import replay_harness as rh
import torch_kernels as ref
from test_gifudra_gpu import _batch
from test_kernels_gpu import _plan_for

pytestmark = pytest.mark.gpu

DEV = "cuda:0"
DTYPES = [torch.float32, torch.bfloat16]


def _tol(dtype):
    return dict(rtol=2e-5, atol=2e-5) if dtype == torch.float32 else dict(rtol=2 ** -6, atol=2 ** -6)


def _randn(*shape, seed=0, scale=1.0, dtype=torch.float32):
    g = torch.Generator(device=DEV).manual_seed(seed)
    return (torch.randn(*shape, generator=g, device=DEV) * scale).to(dtype)


def _ints(values):
    return torch.tensor(values, dtype=torch.int32, device=DEV)


# ------------------------------------------------------------------ attention within chunks, values of any width
def _case(dtype, heads, kv_heads, d, v_dim, page, q_lens, ctx_lens, chunk, lead=0, seed=0):
    """Queries (a slice of wider rows), shuffled pages; slots that no query may read hold NaN, and so do the pages before
    the chunk in which a sequence's step starts, which are given back (table entry -1)."""
    pages = sum(-(-c // page) for c in ctx_lens) + 3
    table, positions, seq_of, qsl, ctx = _batch(q_lens, ctx_lens, page, pages, seed)
    k_pool = torch.full((pages, kv_heads, page, d), float("nan"), dtype=dtype, device=DEV)
    v_pool = torch.full((pages, kv_heads, page, v_dim), float("nan"), dtype=dtype, device=DEV)
    for s, (n, c) in enumerate(zip(q_lens, ctx_lens)):
        first = (c - n) // chunk * chunk if chunk else 0
        keys, values = _randn(c, kv_heads, d, seed=seed + 10 + s, dtype=dtype), _randn(c, kv_heads, v_dim, seed=seed + 50 + s, dtype=dtype)
        at = torch.arange(first, c, device=DEV)
        rows = table[s].long()[at // page]
        k_pool[rows, :, at % page], v_pool[rows, :, at % page] = keys[first:], values[first:]
        table[s, :first // page] = -1
    wide = _randn(sum(q_lens), lead + heads * d + 8, seed=seed + 1, dtype=dtype)
    q = wide[:, lead:lead + heads * d]
    return q, (k_pool, v_pool, table, qsl, ctx)


def _filled(rest):
    """The same pools with zeros where a kernel must not read (the plain twin multiplies what it has masked by zero)."""
    return rest[0].nan_to_num(0.0), rest[1].nan_to_num(0.0), *rest[2:]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,kv_heads,d,v_dim,page,chunk", [(4, 2, 16, 24, 16, 10), (6, 3, 48, 48, 8, 33), (3, 1, 32, 20, 4, 1),
                                                               (2, 2, 300, 500, 16, 64), (5, 1, 7, 3, 8, 16), (2, 1, 64, 1000, 4, 20)])
def test_chunks_on_the_plain_kernel(dtype, heads, kv_heads, d, v_dim, page, chunk):
    from liteinfer_b200 import ops

    q_lens, ctx_lens = [1, 33, 1, 7, 2, 1], [90, 50, 1, 7, 45, 61]
    q, rest = _case(dtype, heads, kv_heads, d, v_dim, page, q_lens, ctx_lens, chunk, lead=3)
    tail = (len(q_lens), max(q_lens), heads, kv_heads, d, d ** -0.5)
    out = lambda: torch.empty(sum(q_lens), heads * v_dim + 5, dtype=dtype, device=DEV)[:, 2:2 + heads * v_dim]
    want = ref.paged_attention(q, q.stride(0), out(), *_filled(rest), *tail, chunk=chunk)
    got = ops.paged_attention(q, q.stride(0), out(), *rest, *tail, chunk=chunk)
    torch.testing.assert_close(got.float(), want.float(), **_tol(dtype))


@pytest.mark.parametrize("heads,kv_heads,d,parts,page", [(4, 2, 64, 1, 16), (8, 2, 128, 1, 16), (4, 1, 128, 2, 16), (6, 2, 64, 3, 32),
                                                         (2, 2, 128, 2, 64), (20, 1, 64, 2, 16)])
@pytest.mark.parametrize("chunk", [0, 33, 64, 200, 1000])
@pytest.mark.parametrize("splits", [None, 1, 3])
def test_chunks_and_wide_values_on_the_tensor_core_kernels(heads, kv_heads, d, parts, page, chunk, splits):
    """tcgen05 over prompts and portions, the streaming kernel (or, for wide groups, mma.sync) over single tokens with keys
    unsplit and split over blocks that merge, and the mma.sync kernel in every role: chunks shorter and longer than a tile
    of keys, steps that start in the middle of a chunk, at its first and at its last position."""
    from liteinfer_b200 import ops

    dtype, v_dim = torch.bfloat16, parts * d
    q_lens, ctx_lens = [1, 130, 1, 7, 64, 1, 257, 1], [700, 190, 1, 7, 64, 129, 300, 201]
    q, rest = _case(dtype, heads, kv_heads, d, v_dim, page, q_lens, ctx_lens, chunk, lead=8)
    tail = (len(q_lens), max(q_lens), heads, kv_heads, d, d ** -0.5)
    out = lambda: torch.full((sum(q_lens), heads * v_dim + 16), float("nan"), dtype=dtype, device=DEV)[:, 8:8 + heads * v_dim]
    want = ref.paged_attention(q, q.stride(0), out(), *_filled(rest), *tail, chunk=chunk)
    plan = _plan_for(q_lens, ctx_lens)
    got = ops.paged_attention(q, q.stride(0), out(), *rest, *tail, plan=plan, decode_splits=splits, chunk=chunk)
    torch.testing.assert_close(got.float(), want.float(), **_tol(dtype))
    alone = ops.paged_attention_mma(q, q.stride(0), out(), *rest, None, *tail, -chunk)
    torch.testing.assert_close(alone.float(), want.float(), **_tol(dtype))
    part = out()
    ops.paged_attention_mma(q, q.stride(0), part, *rest, plan.decode_seqs, plan.num_decode, 1, heads, kv_heads, d,
                            d ** -0.5, -chunk, splits or 2)
    rows = plan.decode_tokens.long()
    torch.testing.assert_close(part[rows].float(), want[rows].float(), **_tol(dtype))
    assert ops.gemm_error_flag(DEV) == 0


@pytest.mark.parametrize("d,v_dim,page", [(64, 64, 16), (128, 256, 16), (48, 72, 8)])
@pytest.mark.parametrize("decode", [False, True])
def test_one_key_stands_out_at_a_chunks_edge(d, v_dim, page, decode):
    """One key's score is lifted far above all others.  The queries of its chunk find its value, whether it is the chunk's
    first position or the query itself; the key just before the chunk is not seen, nor is one that stands as far behind
    as a window would still reach."""
    from liteinfer_b200 import ops

    dtype, heads, kv_heads, chunk = torch.bfloat16, 4, 2, 200
    for ctx in (520, 401, 600):             # the last query: in the middle of a chunk, its first position, its last
        n = 1 if decode else 9
        qpos = ctx - 1
        start = qpos // chunk * chunk
        for target in sorted({start, start - 1, start - 64, qpos, max(qpos - chunk + 1, start - 100), (start + qpos) // 2}):
            q, rest = _case(dtype, heads, kv_heads, d, v_dim, page, [n], [ctx], 0)
            k_pool, v_pool, table = rest[:3]
            k_pool.nan_to_num_(0.0).mul_(0.05)
            v_pool.nan_to_num_(0.0)
            lifted = _randn(d, seed=3)
            k_pool[int(table[0, target // page]), :, target % page] = lifted.to(dtype)
            q[-1] = (lifted * 3.0).to(dtype).repeat(heads)
            found = v_pool[int(table[0, target // page]), :, target % page].float().repeat_interleave(heads // kv_heads, 0)
            got = ops.paged_attention(q, q.stride(0), torch.empty(n, heads * v_dim, dtype=dtype, device=DEV), *rest, 1, n,
                                      heads, kv_heads, d, 1.0, plan=_plan_for([n], [ctx]), chunk=chunk)[-1].float().view(heads, v_dim)
            if target >= start:
                torch.testing.assert_close(got, found, rtol=3e-2, atol=3e-2)
            else:
                assert float((got - found).abs().max()) > 0.3, (ctx, target)


@pytest.mark.parametrize("heads,kv_heads,d,parts,chunk", [(8, 2, 64, 2, 0), (4, 4, 128, 2, 50), (6, 1, 64, 1, 33)])
@pytest.mark.parametrize("splits", [1, 4])
def test_decode_that_rotates_and_stores_wide_values_itself(heads, kv_heads, d, parts, chunk, splits):
    """The single-token launch with the rotation and the cache write fused in, on both kernels that have it, against the
    two launches, for values of several parts and rows that lie in a wider tensor."""
    from liteinfer_b200 import ops

    dtype, page, v_dim = torch.bfloat16, 16, parts * d
    ctx_lens = [300, 1, 65, 101]
    B = len(ctx_lens)
    inv_freq = (1000.0 ** (-torch.arange(d // 2, dtype=torch.float64) * 2 / d)).float().to(DEV)
    width = (heads + kv_heads) * d + kv_heads * v_dim
    k_at, v_at = heads * d, (heads + kv_heads) * d
    results = []
    for form in ("apart", "stream", "mma"):
        _, (k_pool, v_pool, table, qsl, ctx) = _case(dtype, heads, kv_heads, d, v_dim, page, [1] * B, ctx_lens, chunk)
        rows = _randn(B, width + 24, seed=9, dtype=dtype)[:, 8:8 + width]
        positions, seq_of = ctx - 1, torch.arange(B, dtype=torch.int32, device=DEV)
        for s, c in enumerate(ctx_lens):            # the newest token is not in its page yet
            k_pool[int(table[s, (c - 1) // page]), :, (c - 1) % page] = float("nan")
            v_pool[int(table[s, (c - 1) // page]), :, (c - 1) % page] = float("nan")
        newest = None
        if form == "apart":
            ops.head_norm_rope_kv_write(rows, positions, seq_of, table, k_pool, v_pool, inv_freq, heads, kv_heads, d, d,
                                        None, None, 1e-6)
        else:
            newest = ops.NewestToken(inv_freq, rows[:, k_at:], rows[:, v_at:])
        out = torch.empty(B, heads * v_dim, dtype=dtype, device=DEV)
        plan = _plan_for([1] * B, ctx_lens)
        ops.paged_attention_mma(rows, rows.stride(0), out, k_pool, v_pool, table, qsl, ctx, plan.decode_seqs, B, 1, heads,
                                kv_heads, d, d ** -0.5, -chunk, splits, newest, streaming=form == "stream")
        stored = [pool[int(table[s, (c - 1) // page]), :, (c - 1) % page] for pool in (k_pool, v_pool) for s, c in enumerate(ctx_lens)]
        results.append((out, stored))
    for out, stored in results[1:]:
        torch.testing.assert_close(out.float(), results[0][0].float(), **_tol(dtype))
        for got, want in zip(stored, results[0][1]):
            assert torch.equal(got, want)


# ------------------------------------------------------------------ the memory
def _memory_case(dtype, heads, dim, vdim, tokens, seed=1, lead=0):
    width = 2 * heads * dim + heads * vdim
    proj = _randn(tokens, lead + width + 3, seed=seed, dtype=dtype)[:, lead:]
    offsets = (0, heads * dim, 2 * heads * dim)
    return (proj, offsets, _randn(heads * dim, seed=seed + 1), torch.rand(heads * dim, device=DEV) * 0.9,
            1 + 0.2 * _randn(vdim, seed=seed + 2))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,dim,vdim,lead", [(2, 12, 20, 0), (3, 64, 64, 8), (1, 128, 48, 8), (2, 5, 7, 3), (4, 1, 6, 1),
                                                 (2, 200, 33, 0), (1, 300, 130, 4), (16, 128, 128, 0)])
def test_memory_against_the_plain_recurrence(dtype, heads, dim, vdim, lead):
    """Whole prompts, portions and single tokens in one launch, states in shuffled slots, sequences that bring nothing;
    then a step of single tokens only."""
    from liteinfer_b200 import ops

    lens, slots = [17, 1, 0, 2, 40, 8], [3, 0, 6, 5, 1, 7]
    qsl = [0]
    for n in lens:
        qsl.append(qsl[-1] + n)
    for counts in (lens, [1, 1, 0, 1, 1, 1]):
        qsl = [0]
        for n in counts:
            qsl.append(qsl[-1] + n)
        proj, offsets, bias, lower, weight = _memory_case(dtype, heads, dim, vdim, qsl[-1], lead=lead)
        states = [_randn(8, heads, vdim, dim, seed=7) for _ in range(2)]
        outs = [torch.zeros(qsl[-1], heads * vdim + 4, dtype=dtype, device=DEV)[:, :heads * vdim] for _ in range(2)]
        for impl, state, out in zip((ops, ref), states, outs):
            impl.hgrn2(proj, offsets, bias, lower, state, _ints(qsl), _ints(slots), len(counts), heads, dim, vdim, weight,
                       1e-5, out, max(counts))
        torch.testing.assert_close(outs[0].float(), outs[1].float(), **_tol(dtype))
        torch.testing.assert_close(states[0], states[1], rtol=2e-5, atol=2e-5)
        assert torch.equal(states[0][6], _randn(8, heads, vdim, dim, seed=7)[6])      # its sequence brings nothing


def test_memory_of_the_plain_implementation():
    """The kernel's read-outs from a zero state equal the oracle's gate, recurrence and norm."""
    from liteinfer_b200 import ops

    heads, dim, vdim, T = 2, 24, 40, 70
    proj, (q, f, v), bias, lower, weight = _memory_case(torch.float32, heads, dim, vdim, T)
    out = torch.empty(T, heads * vdim, device=DEV)
    ops.hgrn2(proj, (q, f, v), bias, lower, torch.zeros(1, heads, vdim, dim, device=DEV), _ints([0, T]), _ints([0]), 1, heads,
              dim, vdim, weight, 1e-4, out, T)
    p = proj.double().cpu()
    gate = plain_lulisun.forget_gate(p[:, f:v] + bias.double().cpu(), lower.double().cpu()).view(T, heads, dim)
    o = plain_lulisun.forget_memory(plain_lulisun.silu(p[:, q:f]).view(T, heads, dim), gate, p[:, v:v + heads * vdim].view(T, heads, vdim))
    want = plain_lulisun.unit_rms(o, 1e-4) * weight.double().cpu()
    torch.testing.assert_close(out.double().cpu(), want.reshape(T, -1), rtol=2e-5, atol=2e-5)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("dim,vdim", [(32, 24), (128, 128)])
def test_memory_does_not_depend_on_the_cut(dtype, dim, vdim):
    """A sequence whole, in portions of every kind (two tokens, a chunk of the kernel's less one, ...) and token by token."""
    from liteinfer_b200 import ops

    heads, T = 2, 83
    proj, offsets, bias, lower, weight = _memory_case(dtype, heads, dim, vdim, T)

    def run(cuts):
        state, out = torch.zeros(2, heads, vdim, dim, device=DEV), torch.empty(T, heads * vdim, dtype=dtype, device=DEV)
        for a, b in zip(cuts, cuts[1:]):
            ops.hgrn2(proj[a:b], offsets, bias, lower, state, _ints([0, b - a]), _ints([1]), 1, heads, dim, vdim, weight,
                      1e-5, out[a:b], b - a)
        return out, state[1]

    whole, state = run([0, T])
    for cuts in ([0, 2, 4, 11, 26, 27, 43, 59, 60, T], [0, 7, 15, 16, 64, 82, T], list(range(T + 1))):
        out, last = run(cuts)
        torch.testing.assert_close(out.float(), whole.float(), **_tol(dtype))
        torch.testing.assert_close(last, state, rtol=2e-5, atol=2e-5)


@pytest.mark.parametrize("single", [False, True])
def test_memory_holds_a_token_across_a_thousand_others(single):
    """Gates that are exactly 0 once and exactly 1 ever after: the read-out of the last token is the value of the one that
    was written, whatever the others hold, and a channel whose gate stays between forgets it."""
    from liteinfer_b200 import ops

    heads, dim, vdim, T, written = 1, 64, 32, 1001, 300
    proj = _randn(T, 2 * dim + vdim, seed=4)
    proj[:, :dim] = 30.0                         # silu(30) = 30 on every channel
    proj[:, dim:2 * dim] = 80.0                  # gates of 1: keep, write nothing
    proj[written, dim:2 * dim] = -80.0           # a gate of 0: hold this token's value alone
    bias, lower, weight = torch.zeros(dim, device=DEV), torch.zeros(dim, device=DEV), torch.ones(vdim, device=DEV)
    state, out = torch.zeros(1, heads, vdim, dim, device=DEV), torch.empty(T, vdim, device=DEV)
    steps = [(0, T)] if not single else [(0, 990)] + [(i, i + 1) for i in range(990, T)]
    for a, b in steps:
        ops.hgrn2(proj[a:b], (0, dim, 2 * dim), bias, lower, state, _ints([0, b - a]), _ints([0]), 1, heads, dim, vdim,
                  weight, 1e-6, out[a:b], b - a)
    value = proj[written, 2 * dim:]
    assert float(out[:written].abs().max()) == 0.0
    torch.testing.assert_close(state[0, 0], value[:, None].expand(vdim, dim), rtol=0, atol=0)
    want = value / torch.sqrt(value.pow(2).mean())
    torch.testing.assert_close(out[written:], want.expand(T - written, vdim), rtol=1e-5, atol=1e-5)


# ------------------------------------------------------------------ the stream's sum and the norms behind it
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [48, 37, 2048, 5120, 12288])
def test_sum_and_norms(dtype, width):
    from liteinfer_b200 import ops

    T, top = 9, 3
    x0 = _randn(T, width, seed=1, scale=5.0)
    terms = (ops.SumTerm(_randn(T, width, seed=2, dtype=dtype), 1.7),
             ops.SumTerm(_randn(T, width, seed=3, dtype=dtype), 1.0, torch.rand(T, device=DEV)))
    rows = _randn(T * top, width, seed=4, dtype=dtype)
    place = torch.randperm(T * top, generator=torch.Generator().manual_seed(5)).to(torch.int32).to(DEV)
    weights = tuple(1 + 0.3 * _randn(width, seed=6 + i) for i in range(2))
    wanted_rows = _ints([7, 0, 7])
    for delta in (ops.SumDelta(terms, ops.RoutedRows(rows, top, place)), ops.SumDelta(terms[:1], ops.RoutedRows(rows, top)),
                  ops.SumDelta(terms), ops.SumDelta(())):
        for count, pick, write in ((2, None, True), (1, None, True), (1, wanted_rows, False), (0, None, True), (2, None, False)):
            results = []
            for impl in (ops, ref):
                x = x0.clone()
                n = T if pick is None else 3
                outs = tuple(torch.empty(n, width, dtype=dtype, device=DEV) for _ in range(count))
                impl.sum_norms(x, delta, weights[:count], 1e-5, outs, rows=pick, write_stream=write)
                results.append((x, *outs))
            torch.testing.assert_close(results[0][0], results[1][0], rtol=1e-5, atol=1e-4)
            for got, want in zip(results[0][1:], results[1][1:]):
                torch.testing.assert_close(got.float(), want.float(), **_tol(dtype))
            assert write or torch.equal(results[0][0], x0)
        if delta.terms:
            sums = [torch.empty(T, width, dtype=dtype, device=DEV) for _ in range(2)]
            for impl, out in zip((ops, ref), sums):
                impl.sum_norms(None, delta, (), 0.0, (out,))
            torch.testing.assert_close(sums[0].float(), sums[1].float(), **_tol(dtype))


# ------------------------------------------------------------------ the router and the experts
@pytest.mark.parametrize("experts,top,groups,keep", [(6, 2, 3, 2), (12, 4, 4, 2), (8, 2, 4, 1), (64, 6, 8, 3), (5, 2, 1, 1),
                                                      (3, 1, 1, 1), (256, 8, 8, 4), (4, 4, 2, 2), (6, 3, 6, 4), (96, 5, 3, 1), (128, 40, 2, 1), (64, 40, 1, 1)])
def test_corrected_router_against_the_plain_mechanism(experts, top, groups, keep):
    """Scores whose corrections change the choice, negative choice scores among them, groups ranked by their two best."""
    from liteinfer_b200 import ops

    tokens = 77
    logits = _randn(tokens, experts, seed=experts, scale=2.0)
    router = {"experts": experts, "top": top, "groups": {"count": groups, "keep": keep} if groups > 1 else None}
    scores = plain_lulisun.sigmoid(logits.double().cpu())
    uncorrected, _ = plain_lulisun.route_scores(scores, torch.zeros(experts, dtype=torch.float64), router)
    for shift in (0.0, -1.5):               # behind the shift every choice score is negative
        correction = 0.6 * _randn(experts, seed=experts + 1) + shift
        ids, weights = torch.empty(tokens, top, dtype=torch.int32, device=DEV), torch.empty(tokens, top, device=DEV)
        ops.moe_route(logits, top, groups, keep, True, ids, weights, scores="sigmoid", correction=correction, rank_by=2, floor=1e-20)
        chosen, want = plain_lulisun.route_scores(scores, correction.double().cpu(), router)
        assert torch.equal(ids.cpu().long(), chosen)
        torch.testing.assert_close(weights.cpu().double(), want, rtol=1e-5, atol=1e-6)
        assert experts == top or not torch.equal(chosen, uncorrected)
    # Product and routing in one launch, in both dtypes and both widths of block, with the shared expert's row.
    for dtype in DTYPES:
        for count in (tokens, 300):
            x = _randn(count, 3 + 40 + 2, seed=5, dtype=dtype)[:, 3:43]
            w = _randn(experts + 1, 40, seed=6, scale=0.7)
            z = x.float() @ w.t()
            want_ids, want_w = torch.empty(count, top, dtype=torch.int32, device=DEV), torch.empty(count, top, device=DEV)
            ops.moe_route(z[:, :experts].contiguous(), top, groups, keep, True, want_ids, want_w, scores="sigmoid",
                          correction=correction, rank_by=2, floor=1e-20)
            got_ids, got_w = torch.empty(count, top + 2, dtype=torch.int32, device=DEV), torch.empty(count, top + 2, device=DEV)
            gate = torch.empty(count, device=DEV)
            ops.moe_router(x, w, top, groups, keep, True, got_ids, got_w, scores="sigmoid", correction=correction, rank_by=2,
                           floor=1e-20, gated=True, gate=gate)
            same = (got_ids[:, :top] == want_ids).all(-1)
            assert float(same.float().mean()) > 0.97        # (a close call may fall the other way: the sums' order differs)
            torch.testing.assert_close(got_w[same, :top], want_w[same], rtol=1e-4, atol=1e-6)
            torch.testing.assert_close(gate, torch.sigmoid(z[:, experts]), rtol=1e-4, atol=1e-6)
            assert got_ids[:, top:].tolist() == [[experts, experts + 1]] * count
            assert torch.equal(got_w[:, top:], gate[:, None].expand(count, 2))


def test_corrected_router_gives_every_row_an_expert_whatever_it_holds():
    from liteinfer_b200 import ops

    experts, top = 12, 3
    x = _randn(9, 64, seed=1, dtype=torch.bfloat16)
    x[2], x[5, 7], x[6] = float("nan"), float("inf"), float("-inf")
    ids = torch.full((9, top + 1), -7, dtype=torch.int32, device=DEV)
    ops.moe_router(x, _randn(experts + 1, 64, seed=2), top, 3, 2, True, ids, torch.empty(9, top + 1, device=DEV), scores="sigmoid",
                   correction=_randn(experts, seed=3) - 2.0, rank_by=2, floor=1e-20, gated=True)
    assert int(ids.min()) >= 0 and int(ids[:, :top].max()) < experts and bool((ids[:, top] == experts).all())
    for row in ids[:, :top].tolist():
        assert len(set(row)) == top


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("ff,shared", [(16, 16), (16, 48), (16, 24), (24, 8), (64, 128)])
@pytest.mark.parametrize("tokens", [1, 5, 300])
def test_shared_expert_among_the_others_or_on_its_own(dtype, ff, shared, tokens):
    """A shared expert as wide as an expert, several times as wide (cut into slots of the grouped products) or of a width
    of its own (a feed-forward beside them): the plain mixture of experts."""
    from liteinfer_b200 import ops
    from liteinfer_b200.parts.feed_forward import RoutedExperts

    width, experts, top = 32, 6, 2
    part = RoutedExperts(width, ff, experts, top, dtype, torch.device(DEV), groups=3, groups_keep=2, scores="sigmoid",
                         correction=True, group_rank=2, renormalise=True, floor=1e-20, shared_size=shared, gives_sum=True)
    assert part.shared_slots == (shared // ff if shared % ff == 0 else 0)
    tensors = {n: _randn(*s.shape, seed=i, scale=0.3).to(torch.bfloat16).to(torch.float32 if s.kind == "f32" else dtype)
               for i, (n, s) in enumerate(part.tensor_specs().items())}
    part.bind(tensors)
    x = _randn(tokens, width, seed=99, dtype=torch.bfloat16).to(dtype)
    delta = part.forward(x, None)
    got = torch.empty(tokens, width, dtype=dtype, device=DEV)
    ops.sum_norms(None, delta, (), 0.0, (got,))
    names = {"router.weight": "router", "shared.sg.weight": "shared.sg"}
    w = {"p." + names.get(n, n.replace("experts.", "e").replace("_proj.weight", "")): t.double().cpu() for n, t in tensors.items()}
    want = plain_lulisun.moe_ff(x.double().cpu(), w, "p.", {"router": {"experts": experts, "top": top, "groups": {"count": 3, "keep": 2}},
                                                           "shared": {"ff": shared}})
    off = (got.double().cpu() - want).pow(2).mean(1).sqrt() / want.pow(2).mean().sqrt()
    assert float((off > (1e-5 if dtype == torch.float32 else 0.02)).double().mean()) <= 0.02, float(off.max())


# ------------------------------------------------------------------ the whole model
@pytest.fixture(scope="module")
def lulisun_dirs(tmp_path_factory):
    from liteinfer_b200.weights.random_init import write_random_model

    base = tmp_path_factory.mktemp("lulisun")
    return {name: write_random_model(cfg, base / name, seed) for name, (cfg, seed, _) in lc.ALL.items()}


def _expected(model_dir, requests):
    config, tensors = plain_lulisun.read_model(model_dir)
    return {name: plain_lulisun.forward(config, tensors, tokens).float() for name, tokens in requests.items()}


def _typical_error(results, wanted):
    rows = []
    for got, want in zip(results, wanted):
        if want is not None:
            diff = got.double() - want.double()
            diff -= diff.mean(dim=1, keepdim=True)
            rows.append(diff.pow(2).mean(dim=1).sqrt() / want.double().std())
    return torch.cat(rows)


@pytest.mark.parametrize("name,lengths", [("lul_a", (1, 7, 61, 90)), ("lul_b", (2, 30, 45)), ("lul_c", (5, 52, 150, 18, 270)),
                                           ("lul_d", (4, 33, 58, 21)), ("lul_e", (300, 17, 149))])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_replay_all_cuts(lulisun_dirs, tmp_path, name, lengths, dtype):
    """Whole, the tail decoded, portions down to two tokens, four live requests whose pages and slots are used again, and
    every token a step of its own from the first one on: the same logits as the plain implementation."""
    config, _, page = lc.ALL[name]
    requests = {f"r{i}": lc.prompt(config["vocab"], n, 100 + i) for i, n in enumerate(lengths)}
    expected = _expected(lulisun_dirs[name], requests)
    trace = rh.Trace()
    rh.whole(trace, requests)
    rh.tail_decoded(trace, requests, tail=40)
    rh.portions(trace, requests)
    rh.mixed(trace, requests)
    longest = max(requests, key=lambda r: len(requests[r]))
    for i, token in enumerate(requests[longest]):
        trace.add([(f"o-{longest}", [token], [0])], end=[f"o-{longest}"] if i == len(requests[longest]) - 1 else [])
    results = rh.run_program(trace, lulisun_dirs[name], dtype, tmp_path / "out", config["vocab"], page_size=page)
    wanted = rh.gather_expected(trace, expected)
    if dtype == "float32":
        worst, where = rh.worst_error(results, wanted)
        assert worst < 2 * lc.FLOAT32_TOLERANCE[name], f"worst difference {worst} at step {where}"
        return
    # bfloat16: a router's close call may choose another expert than the 64-bit run does, at a position here and there;
    # every other position is held to the rounding's size, and so is the typical one.
    rows = _typical_error(results, wanted)
    assert float(rows.median()) < 0.02, f"typical relative difference {float(rows.median())}"
    assert float((rows > 0.08).double().mean()) < 0.05, f"worst relative difference {float(rows.max())}"


@pytest.mark.parametrize("seed", [2, 5, 8, 21])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_configurations_drawn_at_random(tmp_path, seed, dtype):
    """Layer orders, borrowed tensors, sizes and options drawn at random, every way of cutting, against the plain
    implementation."""
    from liteinfer_b200.weights.random_init import write_random_model

    config = lc.random_config(seed)
    model_dir = write_random_model(config, tmp_path / "model", seed)
    requests = {f"r{i}": lc.prompt(config["vocab"], n, 7 + i) for i, n in enumerate((1, 23, 129, 200))}
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
        assert worst < 2e-4, f"worst difference {worst} at step {where}"
        return
    typical = float(_typical_error(results, wanted).median())
    assert typical < 0.03, f"typical relative difference {typical}"


def test_layers_one_by_one_against_plain(lulisun_dirs):
    """The residual stream after every layer run (32-bit engine) equals the plain implementation's."""
    from liteinfer_b200.engine.loading import build_runner
    from liteinfer_b200.engine.runner import StepEntry

    for name in ("lul_a", "lul_b", "lul_c", "lul_d"):
        config, tensors = plain_lulisun.read_model(lulisun_dirs[name])
        tokens = lc.prompt(config["vocab"], 45, 3)
        want: list = []
        plain_lulisun.forward(config, tensors, tokens, want)
        runner = build_runner(lulisun_dirs[name], torch.float32, DEV, 16, 8, 2)
        runner.cache.reserve(["a"], [45])
        context = runner.build_context([StepEntry("a", tokens, [44])])
        context.layer_trace = []
        runner.model.forward(context, runner.layer_caches)
        assert len(context.layer_trace) == len(want) == len(config["layers"])
        for stop, (got, plain) in enumerate(zip(context.layer_trace, want)):
            assert float((got.cpu().double() - plain).abs().max()) < 2e-4, f"{name}: layer {stop}"


def test_bfloat16_engine_keeps_32_bit_what_must_be_and_rounds_heads_up(lulisun_dirs):
    from liteinfer_b200.engine.loading import build_runner
    from liteinfer_b200.engine.runner import StepEntry

    runner = build_runner(lulisun_dirs["lul_e"], torch.bfloat16, DEV, 16, 8, 2)
    tokens = lc.prompt(lc.LUL_E["vocab"], 20, 3)
    runner.cache.reserve(["a"], [20])
    context = runner.build_context([StepEntry("a", tokens, [19])])
    context.layer_trace = []
    runner.model.forward(context, runner.layer_caches)
    assert all(t.dtype == torch.float32 for t in context.layer_trace)
    parts = runner.model.layers[0].parts
    assert parts["feed_forward"].router.dtype == parts["feed_forward"].correction.dtype == torch.float32
    assert parts["feed_forward"].gate_up.dtype == torch.bfloat16 and parts["mixer_norm"].weight.dtype == torch.float32
    assert runner.layer_caches[0].states["hgrn2"].dtype == torch.float32
    sizes = [(layer.parts["mixer"].members[0].head_dim, layer.parts["mixer"].members[0].v_head_dim) for layer in runner.model.layers]
    assert sizes == [(64, 192), (128, 128)]
    assert runner.layer_caches[0].kv.k_pool.shape[-1] == 64 and runner.layer_caches[0].kv.v_pool.shape[-1] == 192


@pytest.mark.parametrize("graphs", [False, True])
@pytest.mark.parametrize("name", ["lul_c", "lul_e"])
def test_sublayers_side_by_side_equal_one_after_the_other(lulisun_dirs, monkeypatch, name, graphs):
    """The feed-forward on a second stream (its experts, and a shared expert whose products use scratch of their own)
    gives what one stream gives, step for step, eager and from graphs."""
    from liteinfer_b200.engine.loading import build_runner
    from liteinfer_b200.engine.runner import StepEntry
    from liteinfer_b200.parts import block

    config = lc.ALL[name][0]
    tokens = [lc.prompt(config["vocab"], 90, 60 + i) for i in range(3)]
    results = []
    for limit in (0, 256):
        monkeypatch.setattr(block, "PARALLEL_SUBLAYERS", limit)
        runner = build_runner(lulisun_dirs[name], torch.bfloat16, DEV, 16, 32, 3)
        if graphs:
            runner.enable_decode_graphs(3, 512)
        got = [runner.step([StepEntry(str(i), t[:70 + i], [69 + i]) for i, t in enumerate(tokens)]).clone()]
        for at in range(74, 90):
            got.append(runner.step([StepEntry(str(i), t[at:at + 1], [0]) for i, t in enumerate(tokens)]).clone())
        runner.check_kernels()
        results.append(torch.cat(got))
    assert torch.isfinite(results[0].float()).all()
    torch.testing.assert_close(results[1].float(), results[0].float(), rtol=2 ** -6, atol=2 ** -6)


def test_greedy_generation_through_the_engine_on_gpu(lulisun_dirs):
    """`LLM.generate` (scheduler with portions of 16 tokens, three seats for five requests, CUDA graphs, sampler) picks the
    plain implementation's tokens over 24 decoded tokens, chunks ending among them."""
    from liteinfer_b200.engine.llm import LLM
    from liteinfer_b200.sampling.params import SamplingParams

    config, tensors = plain_lulisun.read_model(lulisun_dirs["lul_a"])
    prompts = [lc.prompt(config["vocab"], n, 40 + n) for n in (3, 26, 9, 14, 2)]
    with LLM(str(lulisun_dirs["lul_a"]), dtype="float32", block_size=4, num_gpu_blocks=96, max_num_seqs=3,
             max_model_len=80, max_num_batched_tokens=16) as llm:
        outputs = llm.generate(prompts, SamplingParams(temperature=0.0, max_tokens=24))
    for prompt, output in zip(prompts, outputs):
        tokens = list(prompt)
        for _ in range(24):
            tokens.append(int(plain_lulisun.forward(config, tensors, tokens)[-1].argmax()))
        assert list(output.token_ids) == tokens[len(prompt):]
