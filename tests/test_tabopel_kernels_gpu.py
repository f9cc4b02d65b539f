"""The kernels of the Tabopel mechanisms, each alone against its plain PyTorch statement (tests/plain_kernels.py) at
sizes of their own: what stands between the projections and the attention (short convolution, norm over the projection,
turn in halves, cache row), attention with capped scores, the fixed-decay scan on turned projections, the norm and gate
without a weight behind it, the kernel between two sub-layers (norm of what is added, sum, step row, norm in front of the
next), the squared positive part alone and in the streaming product, ungated experts and experts that hand their input
on in every way the products can be taken."""
from __future__ import annotations

import pytest
import torch

import plain_kernels as P
from test_dutivik_kernels_gpu import _HostBatch, _states
from test_kernels_gpu import DEV, DTYPES, K, _cache_case, randn, tol
from test_pipesun_kernels_gpu import _Batch

pytestmark = pytest.mark.gpu
F32 = dict(rtol=3e-5, atol=3e-5)


def close(dtype):
    return F32 if dtype == torch.float32 else tol(dtype)


# ---- between the projections and the attention -------------------------------------------------------------
#  q heads, k heads, dim, value entries, turned entries
PREPARE_SIZES = [(4, 2, 16, 24, 16), (3, 1, 20, 14, 6), (6, 3, 24, 36, 0), (2, 2, 10, 14, 10), (8, 4, 64, 128, 32),
                 (24, 6, 128, 96, 128), (40, 8, 128, 1024, 64), (2, 1, 40, 8, 24), (5, 5, 9, 10, 4), (16, 2, 256, 512, 256)]
PREPARE_LENS = [(0, 1), (5, 19), (0, 2), (11, 37)]


def _prepare_case(sizes, lens, dtype, seed, page=16, taps=0, norm=False):
    H, G, D, V, rot = sizes
    width = (H + G) * D + V
    batch = _Batch(lens, slots=[4, 0, 2, 5][:len(lens)])
    case = _cache_case(dtype, 1, 1, 8, page, lens, seed=seed)
    c = dict(batch=batch, host=_HostBatch(batch), table=case["table"], sizes=sizes,
             rows=randn(batch.num_tokens, (width + 7) // 8 * 8 + 16, dtype=dtype, seed=seed + 1)[:, 8:],
             cache=randn(int(case["table"].max()) + 1, 1, page, G * D + V, dtype=dtype, seed=seed + 2),
             cos_sin=None, taps=None, q_weight=None, k_weight=None, channels=width)
    if rot:
        inv = (10000.0 ** (-torch.arange(0, rot, 2, dtype=torch.float32) / rot)).to(DEV)
        c["cos_sin"] = K().rope_table(batch.positions, inv)
    if taps:
        c["taps"] = randn(taps, width, dtype=dtype, seed=seed + 3)
    if norm:
        c["q_weight"], c["k_weight"] = (randn(n * D, dtype=dtype, seed=seed + 4 + n) + 1.0 for n in (H, G))
    return c


def _run_prepare(module, c, rows, cache, state, batch, table, *, write=True, q_out=None, offset=0):
    H, G, D, V, _ = c["sizes"]
    on = (lambda t: None if t is None else t.to(rows.device))
    # convolved queries, and those of a test that keeps the rows, get rows of their own
    q_out = torch.empty(rows.shape[0], H * D, dtype=rows.dtype, device=rows.device) if q_out is None else q_out
    cos_sin = None if c["cos_sin"] is None else c["cos_sin"][c.get("lo", 0):c.get("lo", 0) + rows.shape[0]].contiguous()
    module.attention_prepare(rows, q_out, on(cos_sin), batch, table, cache, q_heads=H, k_heads=G, dim=D, value_width=V,
                             taps=on(c["taps"]), state=state, state_offset=offset, q_weight=on(c["q_weight"]),
                             k_weight=on(c["k_weight"]), eps=1e-5, write=write)
    return q_out


@pytest.mark.parametrize("lens", [PREPARE_LENS, [(4, 1), (0, 1), (9, 1)]], ids=["portions", "single-tokens"])
@pytest.mark.parametrize("norm", [False, True], ids=["", "norm"])
@pytest.mark.parametrize("taps", [0, 1, 2, 4, 6, 9, 11])
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sizes", PREPARE_SIZES)
def test_attention_prepare(sizes, dtype, taps, norm, lens):
    c = _prepare_case(sizes, lens, dtype, 3, taps=taps, norm=norm)
    floats = c["channels"] * max(0, taps - 1)
    for front in (3, 8):                              # off and on a 16-byte boundary
        state, host_state = _states(6, front + floats + (5 if front % 4 else 4), seed=9)
        got, want = c["cache"].clone(), c["cache"].cpu().clone()
        q = _run_prepare(K(), c, c["rows"], got, state, c["batch"], c["table"], offset=front)
        q_want = _run_prepare(P, c, c["rows"].cpu(), want, host_state, c["host"], c["table"].cpu(), offset=front)
        torch.testing.assert_close(q.cpu(), q_want, **close(dtype))
        torch.testing.assert_close(got.cpu(), want, **close(dtype))    # also the rows of tokens that are not there
        assert torch.equal(state.cpu(), host_state)                    # also the slots and floats nobody owns
        assert K().read_status() == 0
        if taps < 2:
            break


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("taps,norm", [(0, True), (0, False), (4, False), (3, True), (11, False)])
@pytest.mark.parametrize("sizes", [(4, 2, 16, 24, 8), (6, 3, 24, 30, 24), (8, 2, 128, 256, 64), (5, 5, 9, 10, 4)])
def test_keys_and_values_in_planes_of_their_own(sizes, taps, norm, dtype):
    H, G, D, V, _ = sizes
    c = _prepare_case(sizes, PREPARE_LENS, dtype, 23, taps=taps, norm=norm)
    pages, page = c["cache"].shape[0], c["cache"].shape[2]
    state, _ = _states(6, c["channels"] * max(0, taps - 1) + 4, seed=2)
    rows_state = state.clone()
    planes = (torch.zeros(pages, G, page, D, dtype=dtype, device=DEV), torch.zeros(pages, G, page, V // G, dtype=dtype, device=DEV))
    cache = torch.zeros_like(c["cache"])
    q = _run_prepare(K(), c, c["rows"], planes, state, c["batch"], c["table"])
    q_rows = _run_prepare(K(), c, c["rows"], cache, rows_state, c["batch"], c["table"])
    assert torch.equal(q, q_rows) and torch.equal(state, rows_state)
    assert torch.equal(planes[0], cache[:, 0, :, :G * D].reshape(pages, page, G, D).transpose(1, 2))
    assert torch.equal(planes[1], cache[:, 0, :, G * D:].reshape(pages, page, G, V // G).transpose(1, 2))
    host = (torch.zeros(planes[0].shape, dtype=dtype), torch.zeros(planes[1].shape, dtype=dtype))
    _run_prepare(P, c, c["rows"].cpu(), host, _states(6, c["channels"] * max(0, taps - 1) + 4, seed=2)[1], c["host"], c["table"].cpu())
    for got, want in zip(planes, host):
        torch.testing.assert_close(got.cpu(), want, **close(dtype))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("norm", [False, True], ids=["", "norm"])
def test_queries_in_place_and_without_a_cache_write(norm, dtype):
    c = _prepare_case((4, 2, 16, 24, 8), PREPARE_LENS, dtype, 5, norm=norm)
    q = _run_prepare(K(), c, c["rows"], c["cache"].clone(), None, c["batch"], c["table"])
    rows = torch.empty_strided(c["rows"].shape, c["rows"].stride(), dtype=dtype, device=DEV).copy_(c["rows"])
    untouched = c["cache"].clone()
    _run_prepare(K(), c, rows, untouched, None, c["batch"], c["table"], write=False, q_out=rows[:, :64])
    assert torch.equal(untouched, c["cache"])
    if norm:                                          # (the norm's sums fall to other threads without the keys)
        torch.testing.assert_close(rows[:, :64], q, **close(dtype))
    else:
        assert torch.equal(rows[:, :64], q)
    assert torch.equal(rows[:, 64:], c["rows"][:, 64:])


@pytest.mark.parametrize("norm", [False, True], ids=["", "norm"])
@pytest.mark.parametrize("taps", [2, 4, 7])
def test_convolution_does_not_depend_on_the_cut(taps, norm):
    """One portion, portions of 1, 2, 5 and 17 tokens in another slot, and token by token: the same bits in the queries,
    the cache and the state."""
    sizes, tokens, dtype = (4, 2, 16, 24, 8), 31, torch.bfloat16
    c = _prepare_case(sizes, [(0, tokens)], dtype, 7, taps=taps, norm=norm)
    floats = c["channels"] * (taps - 1)

    def run(lo, hi, cache, state, slot):
        c["lo"] = lo
        return _run_prepare(K(), c, c["rows"][lo:hi], cache, state, _Batch([(lo, hi - lo)], slots=[slot]), c["table"])
    whole_state, whole_cache = torch.zeros(3, floats, dtype=torch.float32, device=DEV), c["cache"].clone()
    whole = run(0, tokens, whole_cache, whole_state, 1)
    for cuts in ([1, 2, 5, 17, 6], [1] * tokens, [16, 15], [2] * 15 + [1]):
        state, cache = torch.zeros(3, floats, dtype=torch.float32, device=DEV), c["cache"].clone()
        outs, at = [], 0
        for n in cuts:
            outs.append(run(at, at + n, cache, state, 2))
            at += n
        assert torch.equal(torch.cat(outs), whole) and torch.equal(cache, whole_cache)
        assert torch.equal(state[2], whole_state[1]) and not state[:2].any()


def test_runs_of_many_tokens():
    """As many tokens as long runs take, in portions whose ends fall into the middle of a run."""
    lens = [(0, 700), (3, 5), (0, 333), (40, 1)]
    c = _prepare_case((4, 2, 32, 40, 16), lens, torch.float32, 11, taps=4)
    state, host_state = _states(6, c["channels"] * 3, seed=3)
    got, want = c["cache"].clone(), c["cache"].cpu().clone()
    q = _run_prepare(K(), c, c["rows"], got, state, c["batch"], c["table"])
    q_want = _run_prepare(P, c, c["rows"].cpu(), want, host_state, c["host"], c["table"].cpu())
    torch.testing.assert_close(q.cpu(), q_want, **F32)
    torch.testing.assert_close(got.cpu(), want, **F32)
    assert torch.equal(state.cpu(), host_state)


# ---- capped scores ------------------------------------------------------------------------------------------------
# dtype, heads, kv heads, key width, value width, page, requests (cached, new), cap, sink
CAP_CASES = [
    (torch.float32, 4, 2, 20, 12, 4, [(0, 40), (13, 1), (5, 9)], 2.0, True),
    (torch.float32, 3, 1, 56, 40, 16, [(70, 3), (0, 1)], 20.0, False),
    (torch.bfloat16, 4, 2, 64, 128, 16, [(100, 201), (0, 77)], 3.0, True),          # tiles of 64 rows
    (torch.bfloat16, 8, 2, 112, 40, 16, [(300, 5), (17, 3)], 1.0, False),            # the few-row form
    (torch.bfloat16, 4, 1, 128, 64, 16, [(640, 1), (1000, 1), (3, 1)], 5.0, True),   # decoded, keys in chunks
    (torch.bfloat16, 6, 3, 80, 48, 16, [(0, 300), (90, 1), (200, 1)], 50.0, True),   # portions beside single tokens
    (torch.bfloat16, 2, 2, 24, 20, 8, [(30, 4)], 2.5, True),                          # widths only the general kernel takes
]


@pytest.mark.parametrize("dtype,heads,kv_heads,dim,vdim,page,lens,cap,sink", CAP_CASES)
def test_attention_with_capped_scores(dtype, heads, kv_heads, dim, vdim, page, lens, cap, sink):
    width = kv_heads * (dim + vdim)
    case = _cache_case(dtype, 1, 1, width, page, lens, seed=31)
    plane, batch = case["k_cache"], _Batch(lens)
    q = randn(batch.num_tokens, heads, dim, dtype=dtype, seed=32, scale=3.0)      # scores far beyond the smaller caps
    sinks = randn(heads, dtype=torch.float32, seed=33) if sink else None
    args = dict(scale=dim ** -0.5, out_dtype=torch.float32, value_heads=kv_heads, group=heads // kv_heads, maps=1,
                key_width=dim, value_width=vdim, key_strides=(page * width, dim, width),
                value_strides=(page * width, vdim, width), page_size=page, num_pages=plane.shape[0])
    host = (q.cpu(), plane.cpu(), plane.cpu().view(-1)[kv_heads * dim:], case["table"].cpu(), _HostBatch(batch))
    host_sinks = None if sinks is None else sinks.cpu()
    want = P.attention_dims(*host, sink=host_sinks, softcap=cap, **args)
    free = P.attention_dims(*host, sink=host_sinks, **args)
    assert (want - free).abs().max() > (1e-2 if cap < 40 else 1e-4), "the cap moves nothing in this case"
    bound = F32 if dtype == torch.float32 else dict(rtol=2e-2, atol=2e-2)
    run = lambda **how: K().attention_dims(q, plane, plane.view(-1)[kv_heads * dim:], case["table"], batch, sink=sinks,
                                           softcap=cap, **how, **args)
    for force in (False, True):
        torch.testing.assert_close(run(force_general=force).cpu(), want, **bound)
        assert K().read_status() == 0
    if dtype == torch.bfloat16 and batch.max_query_len == 1:
        for splits in (1, 3):
            torch.testing.assert_close(run(num_splits=splits).cpu(), want, **bound)


# heads, kv heads, page, requests (cached, new, longest portion first), cap, sink, splits
PLANE_CASES = [
    (8, 2, 16, [(0, 300), (130, 140), (5, 40)], 2.0, True, None),              # prompts on tcgen05
    (8, 2, 16, [(0, 129)], None, True, None),
    (6, 2, 8, [(37, 200)], 30.0, False, None),                                  # three heads a key head: queries copied by rows
    (16, 1, 32, [(0, 40), (77, 9)], 4.0, True, None),
    (8, 2, 16, [(640, 1), (1000, 1), (3, 1), (0, 1)], 2.5, True, None),         # decoded
    (8, 2, 16, [(640, 1), (1000, 1), (3, 1)], None, True, 3),
    (8, 2, 16, [(640, 1), (1000, 1), (3, 1)], 1.0, True, 5),
    (8, 8, 64, [(300, 1)] * 40, 6.0, False, None),                              # more items than blocks fit at once
    (8, 2, 16, [(0, 300), (40, 9), (90, 1), (200, 1), (7, 1)], 3.0, True, None),  # portions beside single tokens
]


@pytest.mark.parametrize("heads,kv_heads,page,lens,cap,sink,splits", PLANE_CASES)
def test_attention_over_planes_with_sinks_and_capped_scores(heads, kv_heads, page, lens, cap, sink, splits):
    dim, dtype = 128, torch.bfloat16
    case = _cache_case(dtype, heads, kv_heads, dim, page, lens, seed=5)
    batch = _Batch(lens)
    q = randn(batch.num_tokens, heads * dim, dtype=dtype, seed=6, scale=2.0)     # scores far beyond the smaller caps
    sinks = randn(heads, dtype=torch.float32, seed=7, scale=3.0) if sink else None
    args = (heads, kv_heads, dim, dim ** -0.5, None)
    host = (q.cpu(), case["k_cache"].cpu(), case["v_cache"].cpu(), case["table"].cpu(), batch.positions.cpu(), batch.req_index.cpu(), *args)
    host_sinks = None if sinks is None else sinks.cpu()
    want = P.paged_attention_plain(*host, sink=host_sinks, softcap=cap)
    assert (want - P.paged_attention_plain(*host)).abs().max() > 0.05, "neither moves anything in this case"
    out = torch.zeros(batch.num_tokens, heads * dim + 8, dtype=dtype, device=DEV)
    got = K().paged_attention(q, case["k_cache"], case["v_cache"], case["table"], batch, *args, sink=sinks, softcap=cap,
                              num_splits=splits, out=out[:, :heads * dim])
    assert K().read_status() == 0 and not out[:, heads * dim:].any()
    torch.testing.assert_close(got.cpu(), want, rtol=2e-2, atol=2e-2)
    # the same through the kernels that address any cache by strides
    strides = (kv_heads * page * dim, page * dim, dim)
    other = K().attention_dims(q.view(-1, heads, dim), case["k_cache"], case["v_cache"], case["table"], batch, value_heads=kv_heads,
                               group=heads // kv_heads, maps=1, key_width=dim, value_width=dim, page_size=page,
                               num_pages=case["k_cache"].shape[0], key_strides=strides, value_strides=strides, scale=dim ** -0.5,
                               sink=sinks, softcap=cap)
    torch.testing.assert_close(other.reshape(-1, heads * dim).cpu(), want, rtol=2e-2, atol=2e-2)


@pytest.mark.parametrize("lens,splits", [((200, 1), None), ((200, 1), 3), ((0, 201), None), ((150, 51), None)])
@pytest.mark.parametrize("place", [0, 15, 16, 127, 128, 180])
@pytest.mark.parametrize("cap", [3.0, 25.0])
def test_a_far_key_among_planes_keeps_the_weight_that_the_cap_leaves_it(cap, place, lens, splits):
    """As below, on the TMA decode and the tcgen05 kernel: exp(cap) against the sink's exp(1.5) and one for every other key."""
    heads, kv_heads, dim, page = 4, 2, 128, 16
    case = _cache_case(torch.bfloat16, heads, kv_heads, dim, page, [lens], seed=3)
    keys, values, batch = case["k_cache"].zero_(), case["v_cache"].zero_(), _Batch([lens])
    q = torch.zeros(batch.num_tokens, heads * dim, dtype=torch.bfloat16, device=DEV)
    q.view(-1, heads, dim)[:, :, 3] = 200.0
    at = case["table"][0, place // page]
    keys[at, :, place % page, 3], values[at, :, place % page] = 100.0, 1.0
    sinks = torch.full((heads,), 1.5, dtype=torch.float32, device=DEV)
    out = K().paged_attention(q, keys, values, case["table"], batch, heads, kv_heads, dim, 1.0, None, sink=sinks, softcap=cap, num_splits=splits)
    e = torch.tensor([cap, 1.5], dtype=torch.float64).exp()
    want = e[0] / (e[0] + e[1] + sum(lens) - 1)
    torch.testing.assert_close(out[-1].cpu().double(), want.expand(heads * dim), rtol=8e-3, atol=0.0)
    assert K().read_status() == 0


def test_a_sink_that_dominates_or_vanishes_among_planes():
    """A sink far above every score leaves nothing; far below, the ordinary softmax, bit for bit within rounding."""
    heads, kv_heads, dim, page = 4, 2, 128, 16
    for lens in ([(0, 150)], [(150, 1)]):
        case = _cache_case(torch.bfloat16, heads, kv_heads, dim, page, lens, seed=9)
        batch = _Batch(lens)
        q = randn(batch.num_tokens, heads * dim, dtype=torch.bfloat16, seed=10)
        run = lambda sinks: K().paged_attention(q, case["k_cache"], case["v_cache"], case["table"], batch, heads, kv_heads, dim,
                                                dim ** -0.5, None, sink=sinks)
        free = run(None)
        assert run(torch.full((heads,), 80.0, device=DEV)).abs().max() < 1e-20
        torch.testing.assert_close(run(torch.full((heads,), -80.0, device=DEV)), free, rtol=1e-2, atol=1e-3)


@pytest.mark.parametrize("dtype,dim,lens", [(torch.float32, 16, (60, 1)), (torch.bfloat16, 64, (200, 1)), (torch.bfloat16, 64, (0, 201))])
@pytest.mark.parametrize("place", [0, 15, 16, 47])
def test_a_far_key_keeps_the_weight_that_the_cap_leaves_it(dtype, dim, lens, place):
    """One key's score lies far above the cap, the others' scores are zero: it weighs exp(cap) against one each and the
    sink's one, wherever it lies.  A tanh that overflowed or lost its digits would show in the weight."""
    heads, page, cap = 2, 16, 4.0
    width = 2 * dim
    case = _cache_case(dtype, 1, 1, width, page, [lens], seed=3)
    plane, batch = case["k_cache"].zero_(), _Batch([lens])
    q = torch.zeros(batch.num_tokens, heads, dim, dtype=dtype, device=DEV)
    q[:, :, 3] = 200.0
    at = plane[case["table"][0, place // page], 0, place % page]
    at[3], at[dim:] = 100.0, 1.0
    out = K().attention_dims(q, plane, plane.view(-1)[dim:], case["table"], batch, value_heads=1, group=heads, maps=1,
                             key_width=dim, value_width=dim, page_size=page, num_pages=plane.shape[0], scale=1.0,
                             key_strides=(page * width, 0, width), value_strides=(page * width, 0, width), softcap=cap,
                             sink=torch.zeros(heads, dtype=torch.float32, device=DEV), out_dtype=torch.float32)
    e = torch.tensor(cap, dtype=torch.float64).exp()
    want = e / (e + sum(lens) - 1 + 1)
    torch.testing.assert_close(out[-1].cpu().double(), want.expand(heads, dim), rtol=1e-4 if dtype == torch.float32 else 8e-3, atol=0.0)
    assert K().read_status() == 0


# ---- the scan on turned projections ------------------------------------------------------------------------------
#  heads, key width, value width, turned entries
RETENTION_SIZES = [(3, 6, 10, 6), (2, 16, 24, 8), (2, 24, 8, 0), (1, 40, 200, 40), (2, 64, 32, 16), (2, 128, 48, 128),
                   (1, 200, 20, 64), (1, 256, 36, 256), (1, 512, 12, 30)]


def _retention_case(heads, dim, vdim, rot, dtype, batch, seed):
    qk = heads * dim
    rows = randn(batch.num_tokens, (2 * qk + heads * vdim + 7) // 8 * 8 + 8, dtype=dtype, seed=seed)
    cos_sin = None
    if rot:
        inv = (500.0 ** (-torch.arange(0, rot, 2, dtype=torch.float32) / rot)).to(DEV)
        cos_sin = K().rope_table(batch.positions, inv)
    decay = torch.tensor([(0.7, 0.0, 1.0)[h % 3] for h in range(heads)],       # also nothing kept, and nothing lost
                          dtype=torch.float32, device=DEV)
    return rows[:, :qk], rows[:, qk:2 * qk], rows[:, 2 * qk:2 * qk + heads * vdim], cos_sin, decay


@pytest.mark.parametrize("front", [3, 8])
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,dim,vdim,rot", RETENTION_SIZES)
def test_retention_scan(heads, dim, vdim, rot, dtype, front):
    batch = _Batch([(0, 1), (5, 19), (0, 2), (11, 37)], slots=[4, 0, 2, 5])
    q, k, v, cos_sin, decay = _retention_case(heads, dim, vdim, rot, dtype, batch, 11)
    state, host_state = _states(6, front + heads * dim * vdim + (5 if front % 4 else 4), seed=13)
    sizes = dict(heads=heads, dim=dim, value_dim=vdim, k_scale=dim ** -0.5, state_offset=front)
    got = K().retention_scan(q, k, v, cos_sin, decay, state, batch, **sizes)
    want = P.retention_scan(q.cpu(), k.cpu(), v.cpu(), None if cos_sin is None else cos_sin.cpu(), decay.cpu(), host_state,
                            _HostBatch(batch), **sizes)
    torch.testing.assert_close(got.cpu(), want, rtol=2e-4, atol=2e-4)
    torch.testing.assert_close(state.cpu(), host_state, rtol=2e-4, atol=2e-4)


@pytest.mark.parametrize("dtype", DTYPES)
def test_retention_does_not_depend_on_the_cut(dtype):
    heads, dim, vdim, rot, tokens = 3, 40, 24, 16, 31
    everything = _Batch([(0, tokens)], slots=[1])
    q, k, v, cos_sin, decay = _retention_case(heads, dim, vdim, rot, dtype, everything, 17)
    floats = heads * dim * vdim

    def run(lo, hi, state, slot):
        return K().retention_scan(q[lo:hi], k[lo:hi], v[lo:hi], cos_sin[lo:hi].contiguous(), decay, state,
                                  _Batch([(lo, hi - lo)], slots=[slot]), heads=heads, dim=dim, value_dim=vdim, k_scale=0.3)
    whole_state = torch.zeros(3, floats, dtype=torch.float32, device=DEV)
    whole = run(0, tokens, whole_state, 1)
    for cuts in ([1, 2, 5, 17, 6], [1] * tokens, [2] * 15 + [1]):
        state = torch.zeros(3, floats, dtype=torch.float32, device=DEV)
        outs, at = [], 0
        for n in cuts:
            outs.append(run(at, at + n, state, 2))
            at += n
        assert torch.equal(torch.cat(outs), whole)
        assert torch.equal(state[2], whole_state[1]) and not state[:2].any()


def test_a_turned_far_token_is_read_through_the_state():
    """One token's key alone is not zero; 300 tokens on, the query reads its value with the factor that the distance gives:
    decay^300 times the turned product of query and key."""
    dim, vdim, tokens = 8, 6, 301
    inv = torch.tensor([1.0, 0.1, 0.01, 0.001], dtype=torch.float32, device=DEV)
    batch = _Batch([(0, tokens)])
    rows = torch.zeros(tokens, 2 * dim + vdim + 2, dtype=torch.float32, device=DEV)
    rows[0, dim + 3], rows[0, 2 * dim:2 * dim + vdim] = 2.0, torch.arange(1.0, vdim + 1.0, device=DEV)
    rows[-1, 3] = 5.0
    state = torch.zeros(1, dim * vdim, dtype=torch.float32, device=DEV)
    out = K().retention_scan(rows[:, :dim], rows[:, dim:2 * dim], rows[:, 2 * dim:2 * dim + vdim], K().rope_table(batch.positions, inv),
                             torch.tensor([0.995], dtype=torch.float32, device=DEV), state, batch, heads=1, dim=dim,
                             value_dim=vdim, k_scale=0.25)
    angle = torch.tensor(0.3, dtype=torch.float64)
    want = 0.995 ** 300 * 10.0 * 0.25 * torch.cos(angle) * torch.arange(1.0, vdim + 1.0, dtype=torch.float64)
    torch.testing.assert_close(out[-1, 0].cpu().double(), want, rtol=1e-4, atol=1e-6)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,vdim", [(3, 10), (2, 200), (1, 4096 + 8)])
def test_norm_without_a_weight_and_gate(heads, vdim, dtype):
    tokens = 7
    o = randn(tokens, heads, vdim, dtype=torch.float32, seed=18, scale=4.0)
    gate = randn(tokens, heads * vdim + 16, dtype=dtype, seed=19)[:, 8:8 + heads * vdim]
    got = torch.zeros(tokens, heads * vdim, dtype=dtype, device=DEV)
    want = got.cpu().clone()
    K().gated_rms_norm(o, gate, None, 1e-5, got)
    P.gated_rms_norm(o.cpu(), gate.cpu(), None, 1e-5, want)
    torch.testing.assert_close(got.cpu(), want, **close(dtype))
    ones = torch.ones(vdim, dtype=dtype, device=DEV)
    assert torch.equal(got, K().gated_rms_norm(o, gate, ones, 1e-5, torch.empty_like(got)))


@pytest.mark.parametrize("dtype", DTYPES)
def test_gate_entry_by_entry_into_a_given_tensor(dtype):
    o, gate = randn(5, 3, 24, dtype=dtype, seed=1), randn(5, 80, dtype=dtype, seed=2)[:, 8:80]
    out = torch.empty(5, 72, dtype=dtype, device=DEV)
    assert K().sigmoid_gate_mul(o, gate, out=out) is out and torch.equal(out, K().sigmoid_gate_mul(o, gate))


# ---- between two sub-layers -----------------------------------------------------------------------------------------
STREAM_WIDTHS = [42, 77, 1000, 1500, 2048, 3000, 4096, 4096 + 24, 6001, 9000]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", STREAM_WIDTHS)
def test_norm_sum_step_and_norm(width, dtype):
    tokens = 7
    x = randn(tokens, width, dtype=torch.float32, seed=51, scale=3.0)
    a = randn(tokens, width, dtype=dtype, seed=53, scale=5.0)
    behind, front = (randn(width, dtype=dtype, seed=54 + n) + 1.0 for n in range(2))
    step = randn(1, width, dtype=dtype, seed=57)
    for row in (None, step):
        want = P.stream_add_rows(x.cpu().clone(), a.cpu(), weight=front.cpu(), eps=1e-5, after=(behind.cpu(), 1e-3),
                                 step=None if row is None else row.cpu())
        stream, y, _ = K().stream_add_rows(x.clone(), a, weight=front, eps=1e-5, after=(behind, 1e-3), step=row)
        torch.testing.assert_close(stream.cpu(), want[0], **F32)
        torch.testing.assert_close(y.cpu(), want[1], **close(dtype))
        # the sum alone; a row does not depend on the rows beside it
        alone, none, _ = K().stream_add_rows(x.clone(), a, after=(behind, 1e-3), step=row)
        assert none is None and torch.equal(alone, stream)
        one, y_one, _ = K().stream_add_rows(x[3:4].clone(), a[3:4].clone(), weight=front, eps=1e-5, after=(behind, 1e-3), step=row)
        assert torch.equal(one, stream[3:4]) and torch.equal(y_one, y[3:4])
        # some tokens only; the stream stays
        rows = torch.tensor([5, 0, 3], dtype=torch.int32, device=DEV)
        before = x.clone()
        _, picked, _ = K().stream_add_rows(before, a, weight=front, eps=1e-5, token_rows=rows, after=(behind, 1e-3), step=row)
        assert torch.equal(picked, y[rows.long()]) and torch.equal(before, x)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [1000, 1028, 2048, 4096, 9000])
def test_a_row_under_a_norm_has_the_same_bits_in_a_long_batch(width, dtype):
    """Few rows take more threads each than many rows do; the sums are the same."""
    x, a = randn(900, width, dtype=torch.float32, seed=71), randn(900, width, dtype=dtype, seed=72, scale=3.0)
    behind, front = (randn(width, dtype=dtype, seed=73 + n) + 1.0 for n in range(2))
    stream, y, _ = K().stream_add_rows(x.clone(), a, weight=front, eps=1e-5, after=(behind, 1e-3))
    few, y_few, _ = K().stream_add_rows(x[400:408].clone(), a[400:408].clone(), weight=front, eps=1e-5, after=(behind, 1e-3))
    assert torch.equal(few, stream[400:408]) and torch.equal(y_few, y[400:408])
    want = P.stream_add_rows(x[400:408].cpu(), a[400:408].cpu(), weight=front.cpu(), eps=1e-5, after=(behind.cpu(), 1e-3))
    torch.testing.assert_close(few.cpu(), want[0], **F32)
    torch.testing.assert_close(y_few.cpu(), want[1], **close(dtype))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [44, 777, 2000, 5000])
def test_experts_rows_under_a_norm_with_pairs_that_have_none(width, dtype):
    """The rows of a token's experts, weighted or already weighted, some pairs with an expert that hands the token's own
    row on: summed in 32-bit, normed, added."""
    tokens, top, count, E = 9, 3, 60, 5
    g = torch.Generator().manual_seed(5)
    x, own = randn(tokens, width, dtype=torch.float32, seed=61), randn(tokens, width, dtype=dtype, seed=65)
    rows = randn(count, width, dtype=dtype, seed=62)
    ids = torch.randint(0, E + 2, (tokens, top), generator=g, dtype=torch.int32)
    ids[0], ids[1] = torch.tensor([5, 6, 5]), torch.tensor([0, 1, 2])              # all of them, none of them
    row_of_pair = torch.randperm(count, generator=g)[:tokens * top].to(torch.int32)
    row_of_pair[ids.view(-1) >= E] = -1
    weights = torch.rand(tokens, top, generator=g)
    behind, front = randn(width, dtype=dtype, seed=63), randn(width, dtype=dtype, seed=64)
    rows_nan = rows[:tokens * top].clone()
    rows_nan[(ids.view(-1) >= E).to(DEV)] = float("nan")                            # nobody has written these rows
    for host_rows, indirection, pending in ((rows, row_of_pair, weights.reshape(-1)), (rows, row_of_pair, None), (rows_nan, None, None)):
        host = K().ExpertRows(host_rows.cpu(), indirection, pending, top, (ids, weights, own.cpu(), E))
        on = lambda t: None if t is None else t.to(DEV)
        experts = K().ExpertRows(host_rows, on(indirection), on(pending), top, (ids.to(DEV), weights.to(DEV), own, E))
        want = P.stream_add_rows(x.cpu().clone(), host, weight=front.cpu(), eps=1e-6, out_dtype=dtype, after=(behind.cpu(), 1e-5))
        stream, y, _ = K().stream_add_rows(x.clone(), experts, weight=front, eps=1e-6, after=(behind, 1e-5))
        torch.testing.assert_close(stream.cpu(), want[0], **F32)
        torch.testing.assert_close(y.cpu(), want[1], **close(dtype))
        summed = K().moe_combine(experts, tokens, top)
        plain = P.stream_add_rows(torch.zeros(tokens, width), host)[0].to(dtype)
        torch.testing.assert_close(summed.cpu(), plain, **close(dtype))


# ---- the squared positive part -----------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", [(3, 7), (5, 64), (300, 1000), (1, 1)])
def test_relu_squared(shape, dtype):
    x = randn(*shape, dtype=dtype, seed=1, scale=3.0)
    want = P.relu_squared(x.clone())
    assert K().relu_squared(x) is x
    assert torch.equal(x, want)


@pytest.mark.parametrize("m,n,k", [(1, 40, 64), (7, 200, 128), (16, 1000, 448), (3, 24, 40), (17, 96, 64), (100, 56, 72)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_product_with_the_squared_positive_part(m, n, k, dtype):
    x = randn(m, k, dtype=dtype, seed=1)
    w = randn(n, k, dtype=dtype, seed=2, scale=2.0 * k ** -0.5)
    got = K().linear_relu_squared(x, w)
    want = torch.relu(x.double() @ w.double().T) ** 2
    torch.testing.assert_close(got.double(), want, **(dict(rtol=2e-5, atol=2e-5) if dtype == torch.float32 else dict(rtol=2e-2, atol=2e-2)))
    assert K().read_status() == 0


@pytest.mark.parametrize("dtype,path,tokens,experts,identity,top,width,ff", [
    (torch.float32, "tiles", 23, 6, 2, 3, 40, 20),
    (torch.float32, "tiles", 9, 3, 1, 4, 21, 7),             # every expert chosen
    (torch.float32, "tiles", 5, 4, 0, 2, 36, 12),            # none hands its input on
    (torch.bfloat16, "tiles", 40, 5, 3, 2, 48, 24),
    (torch.bfloat16, "stream", 3, 8, 2, 2, 64, 48),          # each pair streams its expert alone
    (torch.bfloat16, "stream", 40, 4, 1, 2, 64, 32),         # pairs grouped by expert
    (torch.bfloat16, "stream", 25, 7, 3, 2, 136, 2056),      # a hidden row wider than a staged slab
    (torch.bfloat16, "library", 300, 4, 1, 2, 72, 40),
    (torch.bfloat16, "library", 700, 12, 4, 1, 64, 32),
])
@pytest.mark.parametrize("skewed", [False, True], ids=["spread", "skewed"])
def test_ungated_experts_and_experts_that_hand_their_input_on(skewed, dtype, path, tokens, experts, identity, top, width, ff):
    x = randn(tokens, width, dtype=dtype, seed=111)
    up = randn(experts, ff, width, dtype=dtype, seed=112, scale=1.5 * width ** -0.5)
    down = randn(experts, width, ff, dtype=dtype, seed=113, scale=ff ** -0.5)
    router = randn(experts + identity, width, dtype=torch.float32, seed=114, scale=width ** -0.5)
    correction = randn(experts + identity, dtype=torch.float32, seed=115, scale=0.2)
    if skewed:                                               # nearly every token chooses expert 1 (and an identity expert)
        correction[1] = 3.0
        correction[-1] += 2.0
    ids, weights, _ = K().moe_route(x, router, top, score="softmax", correction=correction)
    how = dict(weight_on_input=False, activation="squared_relu", identity=identity)
    pairs = K().moe_experts(x, ids, weights, up, down, path=path, **how)
    want = torch.zeros(tokens, width, dtype=torch.float64)
    for t in range(tokens):
        for e, a in zip(ids[t].tolist(), weights[t].tolist()):
            h = x[t].cpu().double()
            want[t] += a * (h if e >= experts else down[e].cpu().double() @ torch.relu(up[e].cpu().double() @ h) ** 2)
    bound = dict(rtol=2e-5, atol=2e-5) if dtype == torch.float32 else dict(rtol=3e-2, atol=0.02 * float(want.abs().max()))
    torch.testing.assert_close(K().moe_combine(pairs, tokens, top).cpu().double(), want, **bound)
    assert K().read_status() == 0
    # the kernel between the sub-layers takes the same rows
    ones = torch.ones(width, dtype=dtype, device=DEV)
    stream = K().stream_add_rows(torch.zeros(tokens, width, dtype=torch.float32, device=DEV), pairs, after=(ones, 1e-5))[0]
    normed = want / torch.sqrt((want * want).mean(1, keepdim=True) + 1e-5)
    keep = (want * want).mean(1) > 1e-3                       # (a row near zero is all rounding once it is normed)
    assert keep.float().mean() > 0.5
    torch.testing.assert_close(stream.cpu().double()[keep], normed[keep], **(dict(rtol=1e-3, atol=1e-3) if dtype == torch.float32
                                                                            else dict(rtol=0.1, atol=0.1)))


def test_a_batch_whose_every_pair_hands_its_input_on():
    tokens, experts, identity, top, width, ff = 40, 3, 2, 2, 64, 32
    x = randn(tokens, width, dtype=torch.bfloat16, seed=1)
    up, down = randn(experts, ff, width, dtype=torch.bfloat16, seed=2), randn(experts, width, ff, dtype=torch.bfloat16, seed=3)
    ids = torch.tensor([[3, 4]] * tokens, dtype=torch.int32, device=DEV)
    weights = torch.rand(tokens, top, generator=torch.Generator().manual_seed(4)).to(DEV)
    want = (weights.sum(1, keepdim=True) * x.float()).cpu()
    for path in ("tiles", "stream", "library"):
        pairs = K().moe_experts(x, ids, weights, up, down, path=path, weight_on_input=False, activation="squared_relu", identity=identity)
        torch.testing.assert_close(K().moe_combine(pairs, tokens, top).float().cpu(), want, rtol=1e-2, atol=1e-2)
        ones = torch.ones(width, dtype=torch.bfloat16, device=DEV)
        stream = K().stream_add_rows(torch.zeros(tokens, width, dtype=torch.float32, device=DEV), pairs, after=(ones, 1e-5))[0]
        torch.testing.assert_close(stream.cpu(), P._rms(want, 1e-5), rtol=1e-3, atol=1e-3)
        assert K().read_status() == 0
    few = K().moe_experts(x[:2].contiguous(), ids[:2].contiguous(), weights[:2].contiguous(), up, down, path="stream",
                          weight_on_input=False, activation="squared_relu", identity=identity)
    torch.testing.assert_close(K().moe_combine(few, 2, top).float().cpu(), want[:2], rtol=1e-2, atol=1e-2)


def test_wrappers_refuse_what_does_not_fit():
    import kvcore_b200.kernels as kernels

    batch = _Batch([(0, 2)])
    x = randn(2, 16, dtype=torch.float32, seed=1)
    w = x[0].contiguous()
    with pytest.raises(kernels.KernelError, match="does not fit"):
        K().stream_add_rows(x, x, after=(w[:8].contiguous(), 1e-5))
    with pytest.raises(kernels.KernelError, match="step row"):
        K().stream_add_rows(x, x, step=x[:1])
    with pytest.raises(kernels.KernelError, match="step row of"):
        K().stream_add_rows(x, x, after=(w, 1e-5), step=x[:1, :8].contiguous())
    cache, table = torch.zeros(2, 1, 4, 8, dtype=torch.float32, device=DEV), torch.ones(1, 1, dtype=torch.int32, device=DEV)
    sizes = dict(q_heads=2, k_heads=1, dim=4, value_width=4)
    with pytest.raises(kernels.KernelError, match="taps"):
        K().attention_prepare(x, x[:, :8].contiguous(), None, batch, table, cache, taps=x[:, :8].contiguous(), **sizes)
    with pytest.raises(kernels.KernelError, match="state"):
        K().attention_prepare(x, x[:, :8].contiguous(), None, batch, table, cache, taps=x, **sizes)
    with pytest.raises(kernels.KernelError, match="cos_sin"):
        K().attention_prepare(x, x[:, :8], torch.zeros(2, 3, 2, device=DEV), batch, table, cache, **sizes)
    with pytest.raises(kernels.KernelError, match="decays"):
        K().retention_scan(x[:, :4], x[:, 4:8], x[:, 8:12], None, w, torch.zeros(1, 16, device=DEV), batch, heads=1, dim=4,
                           value_dim=4, k_scale=1.0)
    with pytest.raises(kernels.KernelError, match="cap"):
        K().attention_dims(x.view(2, 2, 8), cache, cache, table, batch, value_heads=1, group=2, maps=1, key_width=8, value_width=8,
                           page_size=4, num_pages=2, key_strides=(32, 0, 8), value_strides=(32, 0, 8), scale=1.0, softcap=0.0)
    q = randn(2, 64, dtype=torch.bfloat16, seed=1)
    planes = torch.zeros(2, 1, 16, 32, dtype=torch.bfloat16, device=DEV)
    with pytest.raises(kernels.KernelError, match="sinks and capped scores"):
        K().paged_attention(q, planes, planes, table, batch, 2, 1, 32, 1.0, None, softcap=5.0)
    with pytest.raises(kernels.KernelError, match="activation"):
        K().moe_experts(x, torch.zeros(2, 1, dtype=torch.int32, device=DEV), torch.ones(2, 1, device=DEV),
                        randn(1, 8, 16, dtype=torch.float32), randn(1, 16, 8, dtype=torch.float32), weight_on_input=False,
                        activation="gelu")
