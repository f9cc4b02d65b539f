"""The Mamevik decoder through the framework (configuration, loader, cache manager, step function, scheduler,
entry point) against the plain statement in tests/plain_mamevik.py, on the host with the stand-in kernels and on
the GPU with the CUDA kernels, in 32-bit and in bfloat16.

Small configurations of their own and random weights: whole prompts against token-by-token decoding, portions down
to one and two tokens, mixed batches against each request alone, pages and state slots used again (freed pages
overwritten), the first tokens of a request (no token in front, an empty convolution, a window that is not full),
long decoding across the windows and across pages, keys just inside and just outside a window and a token that only
the state carries on, loops at the start, in the middle and at the end, sizes that make mechanisms coincide (one head,
one group, groups of one head, one part and one part a head in the norm, one tap, a window of one position and one
longer than any request, every expert chosen, one expert, one pass of the loop, one bucket), and greedy generation
through the entry point."""
from __future__ import annotations

import json

import numpy as np
import pytest
import torch

import plain_kernels
import plain_mamevik as P
import replay_cases as rc
from kvcore_b200 import (CacheConfig, DeviceConfig, KVCoreConfig, ModelConfig, SamplingParams, SchedulerConfig)
from kvcore_b200.config import ConfigError
from kvcore_b200.config.registry import model_spec_from_config, model_spec_from_folder
from kvcore_b200.engine.llm_engine import GenerationRequest, LLMEngine
from kvcore_b200.weights.safetensors_io import write_safetensors

BACKENDS = [pytest.param("cpu", id="host"), pytest.param("cuda:0", id="gpu", marks=pytest.mark.gpu)]
# largest |difference| of a row over the request's largest |logit|; in bfloat16 also the root mean square of a
# row's difference (its mean taken off) over that of the request's logits.  A wrong key, a lost state or a
# window one position off moves a row by 1e-2 and more (test_each_mechanism_changes_the_logits); the 32-bit
# runs hold every position to 5e-5.  In bfloat16 a single row may stray further than the median row.
TOLERANCE = {"float32": 5e-5}
BF16_ROW_TOLERANCE = 1e-1
BF16_MEDIAN_RMS_TOLERANCE = 3.5e-2
# a position where a router's choice hangs on less than this is left out of the bfloat16 comparisons
BF16_ROUTER_MARGIN = 0.1


@pytest.fixture(params=BACKENDS)
def device(request, monkeypatch):
    if request.param == "cpu":
        plain_kernels.install(monkeypatch)
    return request.param


M, A = P.mamba_layer, P.attention_layer
CONFIGS = {
    # both mixers in turn, a loop over the middle layers that begins with a recurrence, layers without a feed-forward
    "all_kinds": P.model_config([
        A(heads=3, dim=16, vdim=24, kv_rank=40, window=11, mlp=P.moe(experts=6, top=2, ff=20, limit=1.5)),
        M(heads=4, vdim=12, state=20, groups=2, conv=3, norm_groups=3, mlp=P.moe(experts=5, top=3, ff=12, limit=0.8)),
        A(heads=2, dim=24, vdim=8, kv_rank=32, window=19, scale=0.3, mlp=None),
        M(heads=2, vdim=20, state=12, groups=1, conv=5, norm_groups=2, mlp=P.moe(experts=4, top=1, ff=24, limit=2.0)),
    ], vocab=83, width=40, loop=(1, 3, 3), bigram=(37, 5, 11), eps=1e-5, logit_scale=0.6, softcap=9.0),
    # what the first makes unequal is equal or 1 here and the other way round: one head, groups of one head, one tap,
    # one part in the norm, a window of one position and one longer than any request, every expert chosen, a single
    # expert, a loop over everything taken once, one bucket, no scale, sizes no 16-byte vector fits
    "coincide": P.model_config([
        M(heads=1, vdim=10, state=6, groups=1, conv=1, norm_groups=1, mlp=P.moe(experts=3, top=3, ff=6, limit=0.5)),
        A(heads=1, dim=10, vdim=6, kv_rank=14, window=1, mlp=P.moe(experts=1, top=1, ff=10, limit=4.0)),
        A(heads=3, dim=6, vdim=6, kv_rank=6, window=500, mlp=None),
        M(heads=3, vdim=7, state=9, groups=3, conv=9, norm_groups=7, mlp=None),
    ], vocab=61, width=42, loop=(0, 4, 1), bigram=(1, 1, 1), eps=1e-6, softcap=50.0),
    # sizes the tensor-core attention and the carried-up reading of long portions take, windows across several pages,
    # state sizes that are shared by several threads a column, a loop at the end
    "serving_sizes": P.model_config([
        M(heads=4, vdim=64, state=128, groups=2, conv=4, norm_groups=2, mlp=P.moe(experts=8, top=2, ff=32, limit=1.0)),
        A(heads=4, dim=32, vdim=32, kv_rank=64, window=44, mlp=P.moe(experts=8, top=2, ff=32, limit=1.0)),
        A(heads=4, dim=48, vdim=64, kv_rank=80, window=70, scale=0.2, mlp=P.moe(experts=16, top=4, ff=16, limit=3.0)),
    ], vocab=128, width=64, loop=(1, 3, 2), bigram=(211, 7, 3), eps=1e-5, logit_scale=0.4, softcap=12.0),
}
LENGTHS = {"all_kinds": (1, 23, 45, 70, 37, 2), "coincide": (64, 1, 30, 50), "serving_sizes": (150, 3, 97, 61)}


def write_folder(folder, cfg, seed, weights=None):
    weights = P.random_weights(cfg, seed) if weights is None else weights
    folder.mkdir(parents=True, exist_ok=True)
    (folder / "config.json").write_text(json.dumps(cfg))
    write_safetensors(folder / "model.safetensors", {k: v.to(torch.bfloat16) for k, v in weights.items()})
    return {k: v.to(torch.bfloat16).double() for k, v in weights.items()}


def references(cfg, weights, requests):
    reference, margins = {}, {}
    for rid, toks in requests.items():
        seen = []
        reference[rid] = P.forward(cfg, weights, toks, margins=seen).numpy()
        margins[rid] = seen[0].numpy()
    return reference, margins


@pytest.fixture(scope="module", params=list(CONFIGS))
def case(request, tmp_path_factory):
    name = request.param
    cfg = CONFIGS[name]
    folder = tmp_path_factory.mktemp(f"mamevik_{name}")
    weights = write_folder(folder, cfg, seed=len(name))
    requests = {f"q{i}": rc.random_tokens(cfg["vocab"], n, 30 + i) for i, n in enumerate(LENGTHS[name])}
    reference, margins = references(cfg, weights, requests)
    return dict(name=name, cfg=cfg, folder=folder, weights=weights, requests=requests, reference=reference,
                margins=margins)


def compare(rows, reference, dtype, margins=None):
    """32-bit: every row within TOLERANCE.  bfloat16: rows whose own router margin is small are left out; a row
    in front of which some router chose otherwise (these narrow models' streams carry a percent of rounding, and a
    state or a cached key hands a changed row on) may stray, so up to 6 % of the rows may lie beyond the row
    tolerance, while the median row must stay within BF16_MEDIAN_RMS_TOLERANCE: a kernel that is a little
    wrong everywhere fails the second, a wrong key or a lost state the 32-bit runs and the kernels' own tests."""
    assert rows
    spread, beyond = [], []
    for (rid, pos), row in sorted(rows.items()):
        assert np.isfinite(row).all(), f"non-finite logits for {rid}@{pos}"
        err = np.abs(row - reference[rid][pos]).max() / np.abs(reference[rid]).max()
        if dtype == "float32":
            assert err <= TOLERANCE[dtype], f"{rid}: first wrong position {pos} (error {err:.3e})"
            continue
        if margins is not None and margins[rid][pos] < BF16_ROUTER_MARGIN:
            continue
        diff = row - reference[rid][pos]
        rms = np.sqrt(np.mean((diff - diff.mean()) ** 2)) / reference[rid].std()
        spread.append(rms)
        if max(err, rms) > BF16_ROW_TOLERANCE:
            beyond.append((rid, pos, float(max(err, rms))))
    if spread:
        assert len(beyond) <= max(2, 0.06 * len(spread)), f"{len(beyond)} of {len(spread)} rows stray: {beyond[:8]}"
        assert np.median(spread) <= BF16_MEDIAN_RMS_TOLERANCE, f"median rms error {np.median(spread):.3e}"


# ---- configuration -----------------------------------------------------------------------------------
def test_config_names_the_tensors_of_the_plain_statement(case):
    from kvcore_b200.parts.model import build_model

    spec = model_spec_from_folder(case["folder"])
    assert spec.architecture == "Mamevik"
    model = build_model(spec, dtype=torch.float32, device="meta")
    assert {slot.name: slot.shape for slot in model.weight_slots()} == P.tensor_shapes(case["cfg"])


def test_config_gives_every_constant_to_the_parts():
    spec = model_spec_from_config(CONFIGS["all_kinds"])
    assert [(e.layer, e.ahead, e.cache_of) for e in spec.schedule] == [
        (0, None, None), (1, ("loop", 0), None), (2, None, None), (1, ("loop", 1), None), (2, None, None),
        (1, ("loop", 2), None), (2, None, None), (3, None, None)]
    step = spec.stream_steps["loop"]
    assert step.kind == "recall_origin" and (step.params["times"], step.params["hidden_size"]) == (3, 40)
    pairs, norm = spec.embedding.params["pairs"], spec.embedding.params["norm"]
    assert (pairs["buckets"], pairs["mul_prev"], pairs["mul_cur"]) == (37, 5, 11)
    assert (norm["eps"], norm["offset"]) == (1e-5, 1.0)
    p = spec.layers[1].mixer.params
    assert (p["num_heads"], p["value_dim"], p["state_dim"], p["num_groups"], p["conv_taps"], p["norm_groups"], p["eps"]) == \
        (4, 12, 20, 2, 3, 3, 1e-5)
    p = spec.layers[2].mixer.params
    assert (p["num_heads"], p["head_dim"], p["value_dim"], p["kv_rank"], p["window"], p["scale"], p["rot_dim"], p["sink"],
            p["gate"]) == (2, 24, 8, 32, 19, 0.3, 0, True, False)
    moe = spec.layers[1].feed_forward.params
    assert (moe["num_experts"], moe["top_k"], moe["expert_size"], moe["join"], moe["score"], moe["weight_on"],
            moe["router_bias"]) == (5, 3, 12, (1.702, 0.8, 1.0), "softmax_chosen", "output", True)
    assert spec.layers[2].feed_forward is None and set(spec.layers[2].norms) == {"mixer_norm"}
    assert all(n.params["offset"] == 1.0 and n.params["eps"] == 1e-5 for n in spec.layers[0].norms.values())
    assert spec.final_norm.params["offset"] == 1.0
    assert (spec.lm_head.params["logit_scale"], spec.lm_head.params["softcap"], spec.lm_head.params["tied_to"]) == (0.6, 9.0, "embed")
    # keys that a model may leave out
    bare = json.loads(json.dumps(CONFIGS["all_kinds"]))
    for key in ("loop", "embedding", "logit_scale", "logit_softcap"):
        bare.pop(key)
    bare["layers"][0]["mixer"].pop("mask")
    plain = model_spec_from_config(bare)
    assert [(e.layer, e.ahead) for e in plain.schedule] == [(i, None) for i in range(4)] and not plain.stream_steps
    assert "pairs" not in plain.embedding.params and plain.lm_head.params["softcap"] is None
    assert plain.layers[0].mixer.params["window"] is None


@pytest.mark.parametrize("change,message", [
    (lambda c: c["layers"][0].update(type="gla"), "mixer of this design"),
    (lambda c: c["layers"][0]["mlp"].update(kind="dense"), "feed-forward of this design"),
    (lambda c: c["layers"][1]["mixer"].update(groups=3), "multiple"),
    (lambda c: c["layers"][1]["mixer"].update(norm_groups=5), "norm_groups"),
    (lambda c: c["layers"][1]["mixer"].pop("state"), "state"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=6), "exceeds experts"),
    (lambda c: c["layers"][1]["mlp"]["expert"].update(limit=0.0), "limit"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(size=0), "size"),
    (lambda c: c["layers"][0]["mixer"].pop("scale"), "scale"),
    (lambda c: c["loop"].update(stop=5), "loop over layers"),
    (lambda c: c["loop"].update(start=3), "loop over layers"),
    (lambda c: c["loop"].update(times=0), "times"),
    (lambda c: c["embedding"]["bigram"].update(buckets=0), "buckets"),
    (lambda c: c["embedding"]["bigram"].pop("mul_cur"), "mul_cur"),
    (lambda c: c.update(logit_softcap=-1.0), "logit_softcap"),
    (lambda c: c.pop("norm"), "norm"),
])
def test_config_refuses(change, message):
    cfg = json.loads(json.dumps(CONFIGS["all_kinds"]))
    change(cfg)
    with pytest.raises(ConfigError, match=message):
        model_spec_from_config(cfg)


def test_cache_groups_and_state():
    """A pass of the loop has pages and states of its own; attention layers of one latent size and window share a page
    group; a state-space layer keeps no pages and one state row a request and pass; the embedding keeps one word."""
    from kvcore_b200.cache.kv_manager import group_entries
    from kvcore_b200.parts.model import build_model

    model = build_model(model_spec_from_config(CONFIGS["all_kinds"]), dtype=torch.float32, device="meta")
    requirements = model.entry_requirements()
    groups, entry_group = group_entries(requirements)
    assert [(g.planes, g.heads, g.width, g.window, g.entries) for g in groups] == [
        (1, 1, 40, 11, (0,)), (1, 1, 32, 19, (2, 4, 6))]
    assert entry_group == {0: 0, 2: 1, 4: 1, 6: 1}
    row = 4 * 12 * 20 + (4 * 12 + 2 * 2 * 20) * 2
    last = 2 * 20 * 12 + (2 * 20 + 2 * 12) * 4
    assert [None if r.state_spec is None else r.state_spec.shape for r in requirements] == [
        None, (row,), None, (row,), None, (row,), None, (last,)]
    spec = model.embedding_state_spec()
    assert spec.shape == (1,) and spec.dtype == torch.int32


def test_unused_tensors_of_a_checkpoint_are_accepted(device, tmp_path):
    """A layer without a feed-forward may carry the norm in front of one."""
    from kvcore_b200.engine.trace_replay import build_replay

    cfg = CONFIGS["coincide"]
    weights = P.random_weights(cfg, 3)
    weights["l2.norm2"] = torch.zeros(cfg["width"])
    write_folder(tmp_path / "m", cfg, 3, weights)
    build_replay(str(tmp_path / "m"), "float32", 64, device=device)


# ---- the cuttings ---------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_cuttings_match_the_plain_statement(case, dtype, device, tmp_path):
    cfg, requests = case["cfg"], case["requests"]
    traces = {
        "whole": rc.trace_whole(requests),
        "tail": rc.trace_decode_tail(requests, tail=26),
        "chunks": rc.trace_chunks(requests, sizes=(7, 3, 16, 2, 5, 1, 9, 2, 31)),
        "mixed": rc.trace_mixed(requests, max_live=4, seed=3),
    }
    results = {}
    for name, steps in traces.items():
        out = tmp_path / name
        rc.run_inprocess(case["folder"], dtype, steps, out, rc.peak_tokens(steps), device=device,
                         fill_freed_pages="poison" if name == "mixed" else None)
        rows = rc.collect(steps, out, cfg["vocab"])
        assert len(rows) == sum(len(t) for t in requests.values())
        compare(rows, case["reference"], dtype, case["margins"])
        results[name] = rows
    if dtype == "float32" and device != "cpu":
        # every kernel of the 32-bit path sums in an order that depends on the position only
        for name in ("tail", "chunks", "mixed"):
            for key, row in results["whole"].items():
                assert np.array_equal(row, results[name][key]), f"{name} differs from whole at {key}"


def test_residual_stream_after_every_layer(case, device):
    """Layer by layer, every pass of the loop counted: the 32-bit stream plus what the block leaves to the norm behind
    it, against the plain statement's, in two portions (the second begins inside a window, with a convolution and a
    state to carry over and a token in front that only the state knows)."""
    from kvcore_b200 import kernels as K
    from kvcore_b200.engine.step import StepEntry
    from kvcore_b200.engine.trace_replay import build_replay

    tokens = case["requests"]["q1"] if len(case["requests"]["q1"]) > 2 else case["requests"]["q2"]
    step_function, kv = build_replay(str(case["folder"]), "float32", 256, device=device)
    seen = []
    for block in step_function.model.blocks:
        original = block.forward

        def recording(h, residual, ctx, cache, original=original):
            out = original(h, residual, ctx, cache)
            seen.append(K.stream_add_rows(out[1].clone(), out[0])[0].cpu())
            return out
        block.forward = recording
    cut = len(tokens) // 3 + 1
    runs = len(step_function.model.schedule)
    assert kv.allocate_slots("x", cut)
    step_function.step([StepEntry("x", tokens[:cut], [])])
    assert kv.allocate_slots("x", len(tokens) - cut)
    step_function.step([StepEntry("x", tokens[cut:], [len(tokens) - cut - 1])])
    collected = []
    P.forward(case["cfg"], case["weights"], tokens, streams=collected)
    assert len(seen) == 2 * runs and len(collected) == runs
    for index, want in enumerate(collected):
        got = torch.cat([seen[index], seen[runs + index]])
        assert got.dtype == torch.float32
        torch.testing.assert_close(got.double(), want, rtol=5e-5, atol=5e-5, msg=lambda m: f"layer run {index}: {m}")


def test_pages_and_slots_are_used_again(case, device, tmp_path):
    """A pool for the largest live set only: the trace needs more pages over its life than the pool has and
    more requests than state slots in a row, so a new request finds a page and a state row that another has
    left (the row must read as zeros, the page must not be read before it is written)."""
    requests = dict(case["requests"])
    requests.update({f"again{i}": toks for i, toks in enumerate(case["requests"].values())})
    steps = rc.trace_mixed(requests, max_live=3, seed=11)
    peak = rc.peak_tokens(steps)
    assert sum(-(-len(t) // 16) * 16 for t in requests.values()) > peak
    out = tmp_path / "o"
    step_function, kv = rc.run_inprocess(case["folder"], "float32", steps, out, peak, device=device,
                                         fill_freed_pages="poison")
    assert all(pool.num_free == pool.num_usable for pool in kv.pools)
    reference = dict(case["reference"])
    reference.update({f"again{i}": ref for i, ref in enumerate(case["reference"].values())})
    compare(rc.collect(steps, out, case["cfg"]["vocab"]), reference, "float32")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding(dtype, device, tmp_path):
    """Two prompt tokens, then single tokens: the windows pass over decoded tokens only, pages behind them are
    handed back, the states and the token in front run on (on the GPU: decode graphs captured and replayed)."""
    cfg = CONFIGS["serving_sizes"] if device != "cpu" else CONFIGS["all_kinds"]
    folder = tmp_path / "m"
    weights = write_folder(folder, cfg, seed=5)
    tokens = rc.random_tokens(cfg["vocab"], 150 if device != "cpu" else 60, 77)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": tokens[:2], "want": [0, 1]}], "end": []}]
    for pos in range(2, len(tokens)):
        steps.append({"step": pos - 1, "entries": [{"id": "a", "tokens": [tokens[pos]], "want": [0]}],
                      "end": ["a"] if pos == len(tokens) - 1 else []})
    out = tmp_path / "o"
    rc.run_inprocess(folder, dtype, steps, out, 192, device=device, fill_freed_pages="poison")
    reference, margins = references(cfg, weights, {"a": tokens})
    compare(rc.collect(steps, out, cfg["vocab"]), reference, dtype, margins)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_portions_behind_earlier_ones(dtype, device, tmp_path):
    """Portions long enough to be read through per-head keys (on the GPU, bfloat16), behind a context whose early pages
    the window has handed back already, alone and beside short portions and single tokens."""
    cfg = CONFIGS["serving_sizes"]
    folder = tmp_path / "m"
    weights = write_folder(folder, cfg, seed=8)
    requests = {rid: rc.random_tokens(cfg["vocab"], n, 300 + n) for rid, n in (("long", 330), ("short", 40), ("one", 5))}
    parts = [("long", 140), ("long", 60), ("short", 30), ("one", 3)], [("long", 130), ("short", 9), ("one", 1)], [("short", 1), ("one", 1)]
    parts = ([parts[0][0]], parts[0][1:], parts[1], parts[2])
    at, steps = {rid: 0 for rid in requests}, []
    for portion in parts:
        entries = []
        for rid, n in portion:
            entries.append({"id": rid, "tokens": requests[rid][at[rid]:at[rid] + n], "want": list(range(n))})
            at[rid] += n
        steps.append({"step": len(steps), "entries": entries, "end": []})
    steps[-1]["end"] = list(requests)
    assert at == {rid: len(t) for rid, t in requests.items()}
    out = tmp_path / "o"
    rc.run_inprocess(folder, dtype, steps, out, rc.peak_tokens(steps), device=device, fill_freed_pages="poison")
    reference, margins = references(cfg, weights, requests)
    compare(rc.collect(steps, out, cfg["vocab"]), reference, dtype, margins)


# ---- faults that random weights would hide ----------------------------------------------------------------
def _standout_model(window: int):
    """One attention layer behind which everything is plain: the latent of one token (id 1) and the query of another
    (id 2) are made to meet in a score that takes the whole softmax, and the value of the first moves the logits."""
    cfg = P.model_config([A(heads=2, dim=16, vdim=16, kv_rank=32, window=window, scale=0.25)],
                         vocab=24, width=32, loop=(0, 1, 1), bigram=(5, 1, 2), softcap=100.0)
    w = {name: torch.zeros(shape) for name, shape in P.tensor_shapes(cfg).items()}
    g = torch.Generator().manual_seed(3)
    w["embed"] = torch.randn(24, 32, generator=g)
    w["embed"][:, :2] = 0.0
    w["embed"][1, 0], w["embed"][2, 1] = 12.0, 12.0            # two directions of their own
    w["loop.in"] = torch.cat([torch.eye(32), torch.zeros(32, 32)], 1)
    p = "l0.mix."
    w[p + "dkv"] = torch.eye(32)
    w[p + "dkv.norm"] = torch.ones(32)
    w[p + "q"][0, 1] = 6.0                                     # token 2 asks along the first latent entry,
    w[p + "uk"][0, 0] = 6.0                                    # which token 1 answers (head 0)
    w[p + "uv"] = torch.randn(32, 32, generator=g)
    w[p + "sink"] = torch.tensor([1.0, -1.0])
    w[p + "o"] = torch.randn(32, 32, generator=g)
    return cfg, w


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("window", [7, 16, 17, 33])
def test_key_just_inside_and_just_outside_the_window(window, dtype, device, tmp_path):
    """A dominating key one position inside and one outside the window (and far behind it), in prompts and decoded, on
    and off page borders."""
    cfg, w = _standout_model(window)
    folder = tmp_path / "m"
    weights = write_folder(folder, cfg, 0, w)
    requests = {}
    for distance in (window - 1, window, window + 20):
        for place in (0, 3, 15, 16):                           # where the key stands
            filler = rc.random_tokens(20, place + distance + 4, 7 * distance + place)
            tokens = [t + 3 for t in filler]
            tokens[place], tokens[place + distance] = 1, 2
            requests[f"d{distance}p{place}"] = tokens
    reference, _ = references(cfg, weights, requests)
    other = json.loads(json.dumps(cfg))
    other["layers"][0]["mixer"]["mask"]["size"] = window + 1
    moved = 0.0
    for rid, tokens in requests.items():
        if rid.startswith(f"d{window}p"):
            wrong = P.forward(other, weights, tokens).numpy()
            moved = max(moved, float(np.abs(wrong - reference[rid]).max() / np.abs(reference[rid]).max()))
    assert moved > 0.2                                         # a window one too long shows
    for name, steps in (("whole", rc.trace_whole(requests)), ("tail", rc.trace_decode_tail(requests, tail=5)),
                        ("chunks", rc.trace_chunks(requests, sizes=(5, 2, 16, 3)))):
        out = tmp_path / name
        rc.run_inprocess(folder, dtype, steps, out, rc.peak_tokens(steps), device=device, fill_freed_pages="poison")
        for (rid, pos), row in rc.collect(steps, out, cfg["vocab"]).items():
            err = np.abs(row - reference[rid][pos]).max() / np.abs(reference[rid]).max()
            assert err <= (TOLERANCE[dtype] if dtype == "float32" else 4e-2), f"{name}: {rid}@{pos}: {err:.3e}"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_token_far_back_that_only_the_state_carries(dtype, device, tmp_path):
    """A state-space layer that takes in one token (its step size is large there and next to nothing elsewhere, its
    decay slow) and reads it out at the end: a hundred tokens on, in prompts, portions and decoded steps."""
    cfg = P.model_config([M(heads=2, vdim=8, state=8, groups=1, conv=4, norm_groups=1)], vocab=24, width=16,
                         loop=(0, 1, 1), bigram=(5, 1, 2), softcap=100.0)
    w = {name: torch.zeros(shape) for name, shape in P.tensor_shapes(cfg).items()}
    g = torch.Generator().manual_seed(4)
    w["embed"] = torch.randn(24, 16, generator=g)
    w["embed"][:, 0] = 0.0
    w["embed"][1, 0] = 8.0
    w["loop.in"] = torch.cat([torch.eye(16), torch.zeros(16, 16)], 1)
    p = "l0.mix."
    inner, channels = 16, 32
    w[p + "in"] = torch.randn(inner + channels + 2, 16, generator=g) * 0.3
    w[p + "in"][-2:] = 0.0
    w[p + "in"][-2:, 0] = 3.0                                  # step sizes: token 1 alone is taken in
    w[p + "dt_bias"] = torch.full((2,), -6.0)
    w[p + "A_log"] = torch.full((2,), -5.0)
    w[p + "conv"] = torch.zeros(channels, 4)
    w[p + "conv"][:, -1], w[p + "conv"][:, 0] = 1.0, 0.7
    w[p + "conv.b"] = torch.full((channels,), 0.3)
    w[p + "norm"] = torch.ones(inner)
    w[p + "o"] = torch.randn(16, inner, generator=g)
    folder = tmp_path / "m"
    weights = write_folder(folder, cfg, 0, w)
    requests = {}
    for place in (0, 9):
        tokens = [t + 3 for t in rc.random_tokens(20, 110 + place, 50 + place)]
        tokens[place] = 1
        requests[f"p{place}"] = tokens
    reference, _ = references(cfg, weights, requests)
    for rid, tokens in requests.items():                       # without that token the last logits are others
        other = list(tokens)
        other[int(rid[1:])] = 3
        assert np.abs(P.forward(cfg, weights, other).numpy()[-1] - reference[rid][-1]).max() > 0.2 * np.abs(reference[rid]).max()
    for name, steps in (("whole", rc.trace_whole(requests)), ("tail", rc.trace_decode_tail(requests, tail=100)),
                        ("chunks", rc.trace_chunks(requests, sizes=(2, 13, 3, 1, 2))),
                        ("mixed", rc.trace_mixed(requests, max_live=2, seed=2))):
        out = tmp_path / name
        rc.run_inprocess(folder, dtype, steps, out, rc.peak_tokens(steps), device=device)
        for (rid, pos), row in rc.collect(steps, out, cfg["vocab"]).items():
            err = np.abs(row - reference[rid][pos]).max() / np.abs(reference[rid]).max()
            assert err <= (TOLERANCE[dtype] if dtype == "float32" else 8e-2), f"{name}: {rid}@{pos}: {err:.3e}"


def test_each_mechanism_changes_the_logits():
    """The plain statement itself: leaving a mechanism out moves the logits by far more than any tolerance
    here, so a test that passes has seen it.  (Guards the tests, not the product.)"""
    cfg = CONFIGS["all_kinds"]
    weights = P.random_weights(cfg, 9, dtype=torch.float64)
    tokens = rc.random_tokens(cfg["vocab"], 40, 3)
    base = P.forward(cfg, weights, tokens)

    def distance(logits):
        return float((logits - base).abs().max() / base.abs().max())

    def moved(config=None, **tensors):
        other = dict(weights)
        other.update(tensors)
        return distance(P.forward(config or cfg, other, tokens))

    def changed(change):
        other = json.loads(json.dumps(cfg))
        change(other)
        return other

    for mechanism in ("bigram", "loop.in", "loop.step", "conv", "D", "sink", "mask", "router.b", "limit", "softcap"):
        assert distance(P.forward(cfg, weights, tokens, leave_out=(mechanism,))) > 1e-3, mechanism
    zeros, ones = torch.zeros_like, torch.ones_like
    mixer = lambda c, i: c["layers"][i]["mixer"]
    for name in ("l1.mix.conv.b", "l1.mix.dt_bias", "l1.mix.A_log", "embed.norm", "l0.norm1", "l0.norm2", "final.norm"):
        assert moved(**{name: zeros(weights[name])}) > 1e-3, name
    for name in ("l1.mix.norm", "l0.mix.dkv.norm"):
        assert moved(**{name: ones(weights[name])}) > 1e-3, name
    first_row = weights["bigram"].clone()
    first_row[-1] = 0.0
    assert moved(bigram=first_row) > 1e-3                                                    # the first token's own row
    for size in (10, 12):                                                                     # one position either way
        assert moved(changed(lambda c: mixer(c, 0)["mask"].update(size=size))) > 1e-4
    for size in (18, 20):
        assert moved(changed(lambda c: mixer(c, 2)["mask"].update(size=size))) > 1e-4
    assert moved(changed(lambda c: mixer(c, 2).update(scale=0.2))) > 1e-3
    assert moved(changed(lambda c: mixer(c, 1).update(norm_groups=2))) > 1e-3
    assert moved(changed(lambda c: c["loop"].update(times=2)), **{"loop.step": weights["loop.step"][:2]}) > 1e-3
    assert moved(changed(lambda c: c["layers"][1]["mlp"]["router"].update(top=2))) > 1e-3
    assert moved(changed(lambda c: c["embedding"]["bigram"].update(mul_prev=6))) > 1e-3
    assert moved(changed(lambda c: c.update(logit_scale=0.5))) > 1e-3


# ---- configurations drawn at random ------------------------------------------------------------------------
def drawn_config(seed):
    """Another model of the design: sizes, head counts, order of layers, loop, windows and constants all drawn."""
    import random

    rng = random.Random(seed)
    fast = seed % 2 == 0                       # every other model has widths the tensor-core attention takes
    width = rng.choice([32, 48, 64, 96] if fast else [24, 40, 56, 72])
    layers = []
    for _ in range(rng.randrange(2, 6)):
        mlp = None
        if rng.random() < 0.8:
            count = rng.randrange(1, 10)
            mlp = P.moe(experts=count, top=rng.randrange(1, min(count, 4) + 1), ff=rng.choice([8, 16, 24] if fast else [6, 12, 20]),
                        limit=rng.choice([0.5, 1.0, 3.0, 7.0]))
        if rng.random() < 0.45:
            groups = rng.choice([1, 2, 3])
            heads = groups * rng.choice([1, 2, 3])
            vdim = rng.choice([8, 16, 32] if fast else [5, 6, 12])
            # (parts of a few entries may all lie near zero, and a norm then multiplies whatever rounding they carry)
            parts = rng.choice([n for n in range(1, 9) if heads * vdim % n == 0 and (n == 1 or heads * vdim // n >= 8)])
            layers.append(M(heads=heads, vdim=vdim, state=rng.choice([16, 32, 64] if fast else [4, 6, 10, 24]), groups=groups,
                            conv=rng.choice([1, 2, 3, 4, 5, 7]), norm_groups=parts, mlp=mlp))
            continue
        layers.append(A(heads=rng.choice([1, 2, 3, 4, 6]), dim=rng.choice([16, 32, 48] if fast else [6, 10, 20]),
                        vdim=rng.choice([8, 16, 40] if fast else [5, 7, 12]),
                        kv_rank=rng.choice([16, 32, 80, 128] if fast else [6, 10, 18, 30]),
                        window=rng.choice([1, 2, 5, 16, 17, 31, 40, 64, 300]), scale=rng.choice([None, 0.2, 0.5]), mlp=mlp))
    start = rng.randrange(0, len(layers))
    return P.model_config(layers, vocab=rng.randrange(40, 160), width=width,
                          loop=(start, rng.randrange(start + 1, len(layers) + 1), rng.choice([1, 2, 3])),
                          bigram=(rng.choice([1, 2, 17, 101]), rng.choice([1, 3, 29, 1009]), rng.choice([1, 2, 7, 2003])),
                          eps=rng.choice([1e-6, 1e-5]), logit_scale=rng.choice([1.0, 0.3]), softcap=rng.choice([5.0, 15.0, 40.0]))


@pytest.mark.parametrize("seed", range(8))
def test_configurations_drawn_at_random(seed, device, tmp_path):
    """Eight other models of the design through the framework: in 32-bit every position of every cutting against
    the plain statement (and, on the GPU, bit-equal between cuttings); in bfloat16 the mixed cutting."""
    cfg = drawn_config(seed)
    folder = tmp_path / "m"
    weights = write_folder(folder, cfg, seed=100 + seed)
    requests = {f"d{i}": rc.random_tokens(cfg["vocab"], n, 500 + 10 * seed + i) for i, n in enumerate((1, 2, 47, 90, 33))}
    reference, margins = references(cfg, weights, requests)
    traces = {"whole": rc.trace_whole(requests), "tail": rc.trace_decode_tail(requests, tail=40),
              "chunks": rc.trace_chunks(requests, sizes=(2, 13, 1, 5, 32, 3)),
              "mixed": rc.trace_mixed(requests, max_live=3, seed=seed)}
    if device == "cpu":        # the stand-in kernels are slow, and the other configurations run every cutting there
        traces.pop("whole")
        traces.pop("tail")
    results = {}
    for name, steps in traces.items():
        out = tmp_path / name
        rc.run_inprocess(folder, "float32", steps, out, rc.peak_tokens(steps), device=device,
                         fill_freed_pages="poison" if name == "mixed" else None)
        results[name] = rc.collect(steps, out, cfg["vocab"])
        compare(results[name], reference, "float32")
    if device != "cpu":
        for name in ("tail", "chunks", "mixed"):
            for key, row in results["whole"].items():
                assert np.array_equal(row, results[name][key]), f"{name} differs from whole at {key}"
        steps = traces["mixed"]
        rc.run_inprocess(folder, "bfloat16", steps, tmp_path / "b", rc.peak_tokens(steps), device=device, fill_freed_pages="poison")
        compare(rc.collect(steps, tmp_path / "b", cfg["vocab"]), reference, "bfloat16", margins)


# ---- the entry point and the scheduler -------------------------------------------------------------------
def plain_greedy(cfg, weights, prompt, steps):
    tokens = list(prompt)
    for _ in range(steps):
        tokens.append(int(P.forward(cfg, weights, tokens)[-1].argmax()))
    return tokens[len(prompt):]


def generate(folder, prompts, new_tokens, device, *, block_size, pages, seqs, budget, prefix=False):
    config = KVCoreConfig(
        model_config=ModelConfig(model=str(folder), dtype="float32", max_model_len=128 if block_size == 16 else 64),
        cache_config=CacheConfig(block_size=block_size, num_gpu_blocks=pages, enable_prefix_caching=prefix),
        scheduler_config=SchedulerConfig(max_num_seqs=seqs, max_num_scheduled_tokens=budget,
                                         max_num_partial_prefills=seqs, max_long_partial_prefills=seqs),
        device_config=DeviceConfig(device=device),
    )
    engine = LLMEngine(config)
    requests = [GenerationRequest(f"g{i}", SamplingParams(max_tokens=new_tokens, temperature=0.0), tuple(p))
                for i, p in enumerate(prompts)]
    outputs = [list(output.output_token_ids) for output in engine.generate(requests)]
    return engine, outputs


@pytest.mark.parametrize("name,budget", [("all_kinds", 16), ("coincide", 7)])
def test_greedy_generation_through_the_entry_point(device, tmp_path, name, budget):
    cfg = CONFIGS[name]
    folder = tmp_path / "m"
    weights = write_folder(folder, cfg, seed=21)
    prompts = [rc.random_tokens(cfg["vocab"], n, 60 + i) for i, n in enumerate((5, 19, 33))]
    engine, outputs = generate(folder, prompts, 12, device, block_size=16, pages=24, seqs=4, budget=budget)
    for prompt, output in zip(prompts, outputs):
        assert output == plain_greedy(cfg, weights, prompt, 12)
    kv = engine.engine_core.model_runner.kv_manager
    kv.check_invariants()
    assert not kv.live_requests()


def test_generation_with_few_pages_and_preemption(device, tmp_path):
    """So few pages that a running request is preempted and computed again from its first token: its state
    rows must read as new (an empty state, no token in front), not as what it left."""
    cfg = CONFIGS["all_kinds"]
    folder = tmp_path / "m"
    weights = write_folder(folder, cfg, seed=22)
    prompts = [rc.random_tokens(cfg["vocab"], n, 90 + i) for i, n in enumerate((30, 28, 26))]
    _, outputs = generate(folder, prompts, 10, device, block_size=4, pages=16, seqs=3, budget=32)
    for prompt, output in zip(prompts, outputs):
        assert output == plain_greedy(cfg, weights, prompt, 10)


def test_prefix_reuse_is_off_where_the_embedding_keeps_state(device, tmp_path):
    """A model whose only per-request state is the token in front: pages alone do not hold what a request needs, so none
    are taken over (all of its tokens stay visible, which by itself would allow it)."""
    cfg = P.model_config([A(heads=2, dim=8, vdim=8, kv_rank=16, window=1)], vocab=50, width=24, loop=(0, 1, 2), bigram=(13, 3, 7))
    cfg["layers"][0]["mixer"].pop("mask")
    folder = tmp_path / "m"
    weights = write_folder(folder, cfg, seed=23)
    prompt = rc.random_tokens(50, 40, 1)
    engine, outputs = generate(folder, [prompt, prompt + [3]], 4, device, block_size=16, pages=24, seqs=1, budget=64, prefix=True)
    kv = engine.engine_core.model_runner.kv_manager
    assert not kv.prefix_caching and kv.num_prefix_hits == 0
    assert outputs == [plain_greedy(cfg, weights, prompt, 4), plain_greedy(cfg, weights, prompt + [3], 4)]


# ---- the programs, each in a process of its own ------------------------------------------------------------
@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_program_on_a_mamevik_folder(case, dtype, tmp_path):
    """``bin/trace_run`` as a user drives it: a step, its ``done`` line, the next step."""
    if case["name"] != "serving_sizes":
        pytest.skip("one configuration is enough for the subprocess run")
    steps = rc.trace_mixed(case["requests"], max_live=3, seed=5)
    steps.insert(1, {"step": 1000, "entries": [], "end": []})      # a step that brings nothing
    out = tmp_path / "out"
    rc.run_subprocess(case["folder"], dtype, steps, out, rc.peak_tokens(steps))
    rows = rc.collect(steps, out, case["cfg"]["vocab"])
    assert len(rows) == sum(len(t) for t in case["requests"].values())
    compare(rows, case["reference"], dtype, case["margins"])


@pytest.mark.gpu
def test_offline_batch_program_on_a_mamevik_folder(tmp_path):
    import ast
    import re
    import subprocess
    import sys

    cfg = CONFIGS["serving_sizes"]
    folder = tmp_path / "m"
    weights = write_folder(folder, cfg, seed=4)
    prompts = {f"req-{i}": rc.random_tokens(cfg["vocab"], n, 80 + i) for i, n in enumerate((70, 9, 33))}
    (tmp_path / "requests.json").write_text(json.dumps(
        [dict(request_id=rid, prompt_token_ids=tokens) for rid, tokens in prompts.items()]))
    command = [sys.executable, str(rc.ROOT / "bin" / "kvcore_offline_batch"), "--model", str(folder), "--dtype", "float32",
               "--prompt-tokens-file", str(tmp_path / "requests.json"), "--max-tokens", "6", "--block-size", "16",
               "--num-gpu-blocks", "64", "--max-model-len", "256", "--max-num-seqs", "4",
               "--max-num-scheduled-tokens", "48", "--max-num-partial-prefills", "4", "--max-long-partial-prefills", "4",
               "--log-level", "WARNING"]
    result = subprocess.run(command, capture_output=True, text=True, timeout=300)
    assert result.returncode == 0, result.stderr[-2000:]
    found = {m["id"]: list(ast.literal_eval(m["ids"])) for m in re.finditer(
        r"^\[(?P<id>[^\]]+)\] finish_reason=\S+\ntoken_ids=(?P<ids>\(.*\))$", result.stdout, re.M)}
    assert list(found) == list(prompts)
    for rid, prompt in prompts.items():
        assert found[rid] == plain_greedy(cfg, weights, prompt, 6)
