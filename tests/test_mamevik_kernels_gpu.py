"""The kernels of the Mamevik mechanisms, each alone against its plain PyTorch statement (tests/plain_kernels.py) at
sizes of their own: what stands in front of the state-space scan (convolution with bias, step sizes, decays), the
scan, the gate ahead of a norm in parts, the sum that norms and packs the stream (with the experts' rows weighted in
it), the embedding of pairs, the latent rows' cache write, the router whose weights are the softmax over the chosen
logits, the experts whose branches are bounded (every way of computing them), the logits' cap."""
from __future__ import annotations

import pytest
import torch

import plain_kernels as P
from test_dutivik_kernels_gpu import _HostBatch, _states
from test_kernels_gpu import DEV, DTYPES, K, _cache_case, randn, tol
from test_pipesun_kernels_gpu import _Batch

pytestmark = pytest.mark.gpu
F32 = dict(rtol=3e-5, atol=3e-5)

#  heads, groups, state, values, taps
SSM_SIZES = [(3, 1, 6, 10, 4), (4, 2, 16, 24, 2), (2, 2, 40, 20, 1), (6, 3, 64, 32, 3), (4, 1, 128, 48, 4), (2, 1, 200, 12, 5),
             (3, 3, 9, 7, 9), (2, 1, 256, 36, 4), (1, 1, 512, 12, 7)]
LENS = [(0, 1), (5, 19), (0, 2), (11, 37)]


def _ssm_case(heads, groups, dim, vdim, taps, dtype, tokens, seed):
    channels = heads * vdim + 2 * groups * dim
    rows = randn(tokens, (channels + heads + 7) // 8 * 8 + 16, dtype=dtype, seed=seed)[:, 16:]
    return dict(rows=rows, taps=randn(channels, taps, dtype=torch.float32, seed=seed + 1),
                bias=randn(channels, dtype=torch.float32, seed=seed + 2, scale=0.5),
                a_log=randn(heads, dtype=torch.float32, seed=seed + 3), dt_bias=randn(heads, dtype=torch.float32, seed=seed + 4),
                skip=randn(heads, dtype=torch.float32, seed=seed + 5), channels=channels)


def _on_host(case):
    return {k: v.cpu() if isinstance(v, torch.Tensor) else v for k, v in case.items()}


def _prepare(module, c, state, batch, sizes, offset):
    return module.ssm_prepare(c["rows"], c["taps"], c["bias"], state, batch, c["a_log"], c["dt_bias"], state_offset=offset, **sizes)


# ---- in front of the scan ----------------------------------------------------------------------------------
@pytest.mark.parametrize("front", [3, 8])      # the state begins `front` floats into its row: off and on a 16-byte boundary
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,groups,dim,vdim,taps", SSM_SIZES)
@pytest.mark.parametrize("lens", [LENS, [(4, 1), (0, 1), (9, 1)]], ids=["portions", "single-tokens"])
def test_ssm_prepare(lens, heads, groups, dim, vdim, taps, dtype, front):
    batch = _Batch(lens, slots=[4, 0, 2, 5][:len(lens)])
    c = _ssm_case(heads, groups, dim, vdim, taps, dtype, batch.num_tokens, 1)
    state, host_state = _states(6, front + c["channels"] * (taps - 1) + (5 if front % 4 else 4), seed=9)
    sizes = dict(heads=heads, groups=groups, dim=dim, value_dim=vdim)
    got = _prepare(K(), c, state, batch, sizes, front)
    want = _prepare(P, _on_host(c), host_state, _HostBatch(batch), sizes, front)
    used = c["channels"] + 2 * heads
    torch.testing.assert_close(got.cpu()[:, :used], want[:, :used], rtol=2e-5, atol=2e-5)
    assert torch.equal(state.cpu(), host_state)                        # also the slots and floats nobody owns


def test_step_sizes_far_out():
    """softplus and the decay keep their digits where the argument is large or small, and are not clamped."""
    heads, rows = 4, torch.zeros(1, 16, dtype=torch.float32, device=DEV)
    rows[0, 6:10] = torch.tensor([60.0, -40.0, 0.0, 12.0])
    one = lambda *v: torch.tensor(v, dtype=torch.float32, device=DEV)
    zeros = torch.zeros(6, 1, dtype=torch.float32, device=DEV)
    out = K().ssm_prepare(rows, zeros, zeros[:, 0].contiguous(), torch.zeros(1, 4, dtype=torch.float32, device=DEV),
                          _Batch([(0, 1)]), one(-4.0, 2.0, 0.0, -9.0), one(0.0, 0.0, 0.0, 0.0), heads=heads, groups=1, dim=1,
                          value_dim=1, state_offset=0).cpu().double()[0]
    dt = torch.nn.functional.softplus(rows[0, 6:10].cpu().double(), threshold=1e6)
    decay = torch.exp(-torch.exp(torch.tensor([-4.0, 2.0, 0.0, -9.0], dtype=torch.float64)) * dt)
    torch.testing.assert_close(out[6:10], dt, rtol=1e-6, atol=0.0)
    torch.testing.assert_close(out[10:14], decay, rtol=1e-6, atol=0.0)


# ---- the scan -------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("columns", [None, "4"])
@pytest.mark.parametrize("front", [3, 8])
@pytest.mark.parametrize("heads,groups,dim,vdim,taps", SSM_SIZES)
def test_ssm_scan(heads, groups, dim, vdim, taps, front, columns, monkeypatch):
    monkeypatch.delenv("KVCORE_SCAN_COLS", raising=False)
    if columns:
        monkeypatch.setenv("KVCORE_SCAN_COLS", columns)
    batch = _Batch(LENS, slots=[4, 0, 2, 5])
    c = _ssm_case(heads, groups, dim, vdim, taps, torch.float32, batch.num_tokens, 11)
    state, host_state = _states(6, front + heads * dim * vdim + c["channels"] * (taps - 1) + 9, seed=13)
    sizes = dict(heads=heads, groups=groups, dim=dim, value_dim=vdim)
    behind = front + heads * dim * vdim
    prepared = _prepare(K(), c, state, batch, sizes, behind)
    host = _prepare(P, _on_host(c), host_state, _HostBatch(batch), sizes, behind)
    got = K().ssm_scan(prepared, c["skip"], state, batch, state_offset=front, **sizes)
    want = P.ssm_scan(host, c["skip"].cpu(), host_state, _HostBatch(batch), state_offset=front, **sizes)
    torch.testing.assert_close(got.cpu(), want, rtol=2e-4, atol=2e-4)
    torch.testing.assert_close(state.cpu(), host_state, rtol=2e-4, atol=2e-4)


@pytest.mark.parametrize("taps", [1, 3, 6])
def test_state_space_does_not_depend_on_the_cut(taps):
    """One portion, portions of 1, 2, 5 and 17 tokens in another slot, and token by token: the same bits out, the same
    bits in the state, convolution and recurrence together."""
    heads, groups, dim, vdim, tokens = 4, 2, 40, 24, 31
    c = _ssm_case(heads, groups, dim, vdim, taps, torch.bfloat16, tokens, 21)
    sizes = dict(heads=heads, groups=groups, dim=dim, value_dim=vdim)
    matrix = heads * dim * vdim
    floats = matrix + c["channels"] * (taps - 1)

    def run(lo, hi, state, batch):
        part = dict(c, rows=c["rows"][lo:hi])
        return K().ssm_scan(_prepare(K(), part, state, batch, sizes, matrix), c["skip"], state, batch, **sizes)
    whole_state = torch.zeros(3, floats, dtype=torch.float32, device=DEV)
    whole = run(0, tokens, whole_state, _Batch([(0, tokens)], slots=[1]))
    for cuts in ([1, 2, 5, 17, 6], [1] * tokens, [16, 15], [2] * 15 + [1]):
        state = torch.zeros(3, floats, dtype=torch.float32, device=DEV)
        outs, at = [], 0
        for n in cuts:
            outs.append(run(at, at + n, state, _Batch([(at, n)], slots=[2])))
            at += n
        assert torch.equal(torch.cat(outs), whole)
        assert torch.equal(state[2], whole_state[1])
        assert not state[:2].any()


@pytest.mark.parametrize("dim,vdim", [(40, 24), (128, 40), (128, 13), (512, 8)])
def test_ssm_scan_does_not_depend_on_the_rows_a_thread_holds(dim, vdim, monkeypatch):
    heads, groups = 2, 1
    batch = _Batch([(0, 21), (0, 1), (0, 6)], slots=[2, 0, 1])
    c = _ssm_case(heads, groups, dim, vdim, 4, torch.float32, batch.num_tokens, 31)
    sizes = dict(heads=heads, groups=groups, dim=dim, value_dim=vdim)
    held = torch.zeros(3, c["channels"] * 3, dtype=torch.float32, device=DEV)
    prepared = _prepare(K(), c, held, batch, sizes, 0)
    results = []
    for shape in ({}, {"KVCORE_SCAN_ROWS": "4"}, {"KVCORE_SCAN_ROWS": "8"}, {"KVCORE_SCAN_ROWS": "16"},
                  {"KVCORE_SCAN_COLS": "4"}, {"KVCORE_SCAN_COLS": "1"}):
        for name in ("KVCORE_SCAN_ROWS", "KVCORE_SCAN_COLS"):
            monkeypatch.delenv(name, raising=False)
        for name, value in shape.items():
            monkeypatch.setenv(name, value)
        state = torch.zeros(3, heads * dim * vdim, dtype=torch.float32, device=DEV)
        results.append((K().ssm_scan(prepared, c["skip"], state, batch, **sizes), state))
    for out, state in results[1:]:
        assert torch.equal(out, results[0][0]) and torch.equal(state, results[0][1])


# ---- behind the scan ---------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width,groups", [(21, 7), (96, 3), (256, 1), (1000, 2), (1026, 2), (2048, 1), (4100, 1), (8192, 4),
                                          (16388, 1), (33000, 2)])
def test_gate_ahead_of_a_norm_in_parts(width, groups, dtype):
    tokens = 5
    o = randn(tokens, 1, width, dtype=torch.float32, seed=41, scale=3.0)
    wide = randn(tokens, width + 16, dtype=dtype, seed=42, scale=2.0)
    gate = wide[:, 8:8 + width]
    weight = randn(width, dtype=torch.float32, seed=43) + 1.0
    got = torch.zeros(tokens, width + 8, dtype=dtype, device=DEV)
    want = torch.zeros(tokens, width, dtype=dtype)
    K().gated_group_norm(o, gate, weight, 1e-5, got[:, :width], groups)
    P.gated_group_norm(o.cpu(), gate.cpu(), weight.cpu(), 1e-5, want, groups)
    torch.testing.assert_close(got[:, :width].cpu(), want, **(F32 if dtype == torch.float32 else tol(dtype)))
    assert not got[:, width:].any()


# ---- the stream ------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("width", [42, 1000, 4096 + 24, 6001])
@pytest.mark.parametrize("dtype", DTYPES)
def test_sum_norm_and_packing_of_the_stream(width, dtype):
    tokens = 7
    x = randn(tokens, width, dtype=torch.float32, seed=51, scale=3.0)
    origin = randn(tokens, width, dtype=torch.float32, seed=52)
    a = randn(tokens, width, dtype=dtype, seed=53)
    w = randn(width, dtype=torch.float32, seed=54) + 1.0
    want = P.stream_add_rows(x.cpu().clone(), a.cpu(), weight=w.cpu(), eps=1e-5)
    stream, y, packed = K().stream_add_rows(x.clone(), a, weight=w, eps=1e-5)
    assert packed is None
    torch.testing.assert_close(stream.cpu(), want[0], **F32)
    torch.testing.assert_close(y.cpu(), want[1], **(F32 if dtype == torch.float32 else tol(dtype)))
    # the packed row, with and without something to add; the stream stays
    for addend in (a, None):
        before = x.clone()
        out = K().stream_add_rows(before, addend, out_dtype=dtype, origin=origin, keep=False)
        assert out[0] is None and out[1] is None and torch.equal(before, x)
        total = x if addend is None else x + a.float()
        assert torch.equal(out[2], torch.cat([total, origin], 1).to(dtype))
    # one row for all tokens
    row = a[2:3].contiguous()
    stream_one, y_one, _ = K().stream_add_rows(x.clone(), row, weight=w, eps=1e-5)
    stream_all, y_all, _ = K().stream_add_rows(x.clone(), row.expand(tokens, width).contiguous(), weight=w, eps=1e-5)
    assert torch.equal(stream_one, stream_all) and torch.equal(y_one, y_all)
    # some tokens only
    rows = torch.tensor([5, 0, 3], dtype=torch.int32, device=DEV)
    before = x.clone()
    _, picked, _ = K().stream_add_rows(before, a, weight=w, eps=1e-5, token_rows=rows)
    assert torch.equal(picked, y[rows.long()]) and torch.equal(before, x)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [44, 777, 5000])
def test_experts_rows_are_weighted_and_summed_into_the_stream(width, dtype):
    tokens, top, count = 9, 3, 60
    g = torch.Generator().manual_seed(5)
    x = randn(tokens, width, dtype=torch.float32, seed=61)
    rows = randn(count, width, dtype=dtype, seed=62)
    row_of_pair = torch.randperm(count, generator=g)[:tokens * top].to(torch.int32).to(DEV)
    weights = torch.rand(tokens * top, generator=g).to(DEV)
    w = randn(width, dtype=torch.float32, seed=63)
    for experts in (K().ExpertRows(rows, row_of_pair, weights, top), K().ExpertRows(rows, row_of_pair, None, top),
                    K().ExpertRows(rows[:tokens * top].contiguous(), None, None, top)):
        host = K().ExpertRows(experts.rows.cpu(), None if experts.row_of_pair is None else experts.row_of_pair.cpu(),
                              None if experts.pending_weights is None else experts.pending_weights.cpu(), top)
        want = P.stream_add_rows(x.cpu().clone(), host, weight=w.cpu(), eps=1e-6, out_dtype=dtype)
        stream, y, _ = K().stream_add_rows(x.clone(), experts, weight=w, eps=1e-6)
        torch.testing.assert_close(stream.cpu(), want[0], **F32)
        torch.testing.assert_close(y.cpu(), want[1], **(F32 if dtype == torch.float32 else tol(dtype)))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width,buckets,factors", [(40, 17, (3, 5)), (1000, 1, (1, 1)), (4096 + 24, 101, (1009, 2003)),
                                                   (36, 1000, (2 ** 31 - 1, 2 ** 31 - 3)), (45, 9, (-7, 2))])
@pytest.mark.parametrize("normed", [True, False])
def test_embedding_of_pairs(normed, width, buckets, factors, dtype):
    """First tokens, portions behind others, single tokens; the word that is left for the next portion; factors whose
    products need more than 32 bits."""
    vocab = 30
    table, pairs = randn(vocab, width, dtype=dtype, seed=71), randn(buckets + 1, width, dtype=dtype, seed=72)
    weight = randn(width, dtype=torch.float32, seed=73) + 1.0 if normed else None
    args = dict(mul_prev=factors[0], mul_cur=factors[1], eps=1e-5)
    state = torch.full((5, 1), 9, dtype=torch.int32, device=DEV)
    host_state = state.cpu().clone()
    g = torch.Generator().manual_seed(6)
    for lens in ([(0, 1), (0, 7), (0, 3)], [(1, 4), (7, 1), (3, 2)], [(5, 1), (8, 1), (5, 1)]):
        batch = _Batch(lens, slots=[3, 0, 4])
        ids = torch.randint(0, vocab, (batch.num_tokens,), dtype=torch.int32, generator=g)
        got = K().embed_pairs(table, ids.to(DEV), pairs=pairs, weight=weight, state=state, ctx=batch, **args)
        want = P.embed_pairs(table.cpu(), ids, pairs=pairs.cpu(), weight=None if weight is None else weight.cpu(),
                             state=host_state, ctx=_HostBatch(batch), **args)
        torch.testing.assert_close(got.cpu(), want, **F32)
        assert torch.equal(state.cpu(), host_state)
    assert K().read_status() == 0


def test_logits_cap():
    logits = randn(3, 1001, dtype=torch.float32, seed=81, scale=40.0)
    want = 22.0 * torch.tanh(logits.double() * 0.4 / 22.0)
    got = K().softcap(logits, 0.4, 22.0)
    assert got.data_ptr() == logits.data_ptr()
    torch.testing.assert_close(got.double(), want, rtol=1e-5, atol=1e-5)


# ---- the latent cache --------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rank,page", [(40, 16), (30, 8), (512, 16)])
def test_latent_rows_into_the_cache(rank, page, dtype):
    case = _cache_case(dtype, 2, 1, 16, page, [(0, 33), (15, 2), (64, 1)], seed=7)
    batch = _Batch([(0, 33), (15, 2), (64, 1)])
    table = case["table"]
    pages = int(table.max()) + 1
    rows = randn(batch.num_tokens, rank + 24, dtype=dtype, seed=91, scale=2.0)[:, 8:8 + rank]
    weight = randn(rank, dtype=dtype, seed=92) + 1.0
    got = randn(pages, 1, page, rank, dtype=dtype, seed=93)
    want = got.cpu().clone()
    K().latent_cache_write(rows, weight, 1e-5, batch, table, got)
    P.latent_cache_write(rows.cpu(), weight.cpu(), 1e-5, _HostBatch(batch), table.cpu(), want)
    torch.testing.assert_close(got.cpu(), want, **tol(dtype))
    assert K().read_status() == 0


# ---- the mixture ----------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("tokens,experts,top,width", [(5, 6, 2, 40), (300, 16, 4, 136), (7, 1, 1, 30), (33, 9, 9, 64)])
def test_router_with_the_softmax_over_the_chosen_logits(tokens, experts, top, width, dtype):
    x = randn(tokens, width, dtype=dtype, seed=101)
    router = randn(experts, width, dtype=torch.float32, seed=102)
    bias = randn(experts, dtype=torch.float32, seed=103, scale=3.0)
    ids, weights, _ = K().moe_route(x, router, top, score="softmax_chosen", bias=bias)
    want_ids, want_weights, _ = P.moe_route(x.cpu(), router.cpu(), top, score="softmax_chosen", bias=bias.cpu())
    same = (ids.cpu() == want_ids).all(dim=1)
    assert same.float().mean() > 0.97          # a choice may hang on the last bit of a sum taken in another order
    torch.testing.assert_close(weights.cpu()[same], want_weights[same], rtol=2e-4, atol=1e-6)
    torch.testing.assert_close(weights.sum(1), torch.ones(tokens, device=DEV), rtol=1e-5, atol=1e-5)
    if experts > 2 * top:
        free, _, _ = P.moe_route(x.cpu(), router.cpu(), top, score="softmax_chosen")
        assert (free != want_ids).any(), "the bias changes no choice in this case"


def test_router_logits_far_below_the_largest():
    """Logits a hundred apart: scores of a softmax over all experts would be zero behind the first, the choice among the
    others and their order still go by the logits."""
    router = torch.zeros(5, 8, dtype=torch.float32, device=DEV)
    bias = torch.tensor([-300.0, 0.0, -200.0, -250.0, -400.0], dtype=torch.float32, device=DEV)
    ids, weights, _ = K().moe_route(torch.zeros(2, 8, dtype=torch.float32, device=DEV), router, 3, score="softmax_chosen", bias=bias)
    assert ids.cpu().tolist() == [[1, 2, 3]] * 2
    torch.testing.assert_close(weights.cpu(), torch.tensor([[1.0, 0.0, 0.0]] * 2))


@pytest.mark.parametrize("dtype,path,tokens,experts,top,width,ff", [
    (torch.float32, "tiles", 23, 6, 2, 40, 20),
    (torch.float32, "tiles", 9, 3, 3, 21, 7),
    (torch.bfloat16, "tiles", 40, 5, 2, 48, 24),
    (torch.bfloat16, "stream", 3, 8, 2, 64, 48),            # each pair streams its expert alone
    (torch.bfloat16, "stream", 40, 4, 2, 64, 32),           # pairs grouped by expert
    (torch.bfloat16, "stream", 60, 3, 2, 72, 40),           # more than a tile of pairs an expert, ragged widths
    (torch.bfloat16, "stream", 30, 4, 1, 2120, 24),         # an input wider than a staged slab
    (torch.bfloat16, "stream", 25, 7, 2, 136, 2056),        # a hidden row wider than one, experts with few pairs
    (torch.bfloat16, "library", 300, 4, 2, 72, 40),
])
@pytest.mark.parametrize("limit", [0.7, 3.0])
def test_experts_with_bounded_branches(limit, dtype, path, tokens, experts, top, width, ff):
    x = randn(tokens, width, dtype=dtype, seed=111)
    gate_up = randn(experts, 2 * ff, width, dtype=dtype, seed=112, scale=2.0 * width ** -0.5)
    down = randn(experts, width, ff, dtype=dtype, seed=113, scale=ff ** -0.5)
    ids, weights, _ = K().moe_route(x, randn(experts, width, dtype=torch.float32, seed=114), top, score="softmax_chosen")
    join = (1.702, limit, 1.0)
    pairs = K().moe_experts(x, ids, weights, gate_up, down, weight_on_input=False, path=path, join=join)
    got = K().moe_combine(pairs, tokens, top)
    want = torch.zeros(tokens, width, dtype=torch.float64)
    for t in range(tokens):
        for e, a in zip(ids[t].tolist(), weights[t].tolist()):
            both = gate_up[e].cpu().double() @ x[t].cpu().double()
            g, u = both[:ff].clamp(max=limit), both[ff:].clamp(min=-limit, max=limit)
            want[t] += a * (down[e].cpu().double() @ (g * torch.sigmoid(1.702 * g) * (u + 1.0)))
    torch.testing.assert_close(got.cpu().double(), want, **(dict(rtol=2e-5, atol=2e-5) if dtype == torch.float32
                                                            else dict(rtol=3e-2, atol=6e-2)))
    # the sum into the stream takes the same rows
    stream = torch.zeros(tokens, width, dtype=torch.float32, device=DEV)
    K().stream_add_rows(stream, pairs)
    torch.testing.assert_close(stream.cpu().double(), want, **(dict(rtol=2e-5, atol=2e-5) if dtype == torch.float32
                                                               else dict(rtol=3e-2, atol=6e-2)))


def test_wrappers_refuse_what_does_not_fit():
    import kvcore_b200.kernels as kernels

    batch = _Batch([(0, 2)])
    x = randn(2, 16, dtype=torch.float32, seed=1)
    with pytest.raises(kernels.KernelError, match="weight"):
        K().stream_add_rows(x, x, weight=x[0, :8].contiguous())
    with pytest.raises(kernels.KernelError, match="type of the outputs"):
        K().stream_add_rows(x, None)
    with pytest.raises(kernels.KernelError, match="parts"):
        K().gated_group_norm(x, x, x[0].contiguous(), 1e-5, torch.empty_like(x), 3)
    with pytest.raises(kernels.KernelError, match="32 bits"):
        K().embed_pairs(x, torch.zeros(2, dtype=torch.int32, device=DEV), pairs=x, mul_prev=1 << 31, mul_cur=1,
                        state=torch.zeros(1, 1, dtype=torch.int32, device=DEV), ctx=batch)
    with pytest.raises(kernels.KernelError, match="limit"):
        K().moe_experts(x, torch.zeros(2, 1, dtype=torch.int32, device=DEV), torch.ones(2, 1, device=DEV),
                        randn(1, 8, 16, dtype=torch.float32), randn(1, 16, 4, dtype=torch.float32), weight_on_input=False,
                        join=(1.0, 0.0, 1.0))
