"""Nufavik on the device against the plain implementation (``plain_nufavik``, float64).

Every test makes its own small configuration and random weights.  32-bit runs must agree within 1e-4 at every
token; bfloat16 runs within 4 % of the logits' spread in the root mean square.  The schedules cut the same requests
in different ways: a request's logits must not depend on the cut, on the rest of the batch, or on which pages and
slots it got."""

import numpy as np
import pytest
import torch

import nufavik_helpers as nf
import plain_nufavik as plain
from engine_helpers import (F32_ATOL, random_tokens, run_schedule, schedule_mixed, schedule_portions, schedule_tail_one_by_one,
                            schedule_whole)

pytestmark = pytest.mark.gpu


def engine_for(folder, dtype="float32", **options):
    from mini_llm_b200.engine import Engine
    options.setdefault("page_size", 8)
    options.setdefault("max_requests", 4)
    options.setdefault("cache_tokens", 1024)
    return Engine(folder, dtype=dtype, **options)


def check(engine, folder, requests, steps, atol=F32_ATOL):
    got = run_schedule(engine, requests, steps)
    for name, tokens in requests.items():
        expected = nf.plain_logits(folder, tokens)
        worst = np.abs(got[name] - expected).max(axis=1)
        assert worst.max() <= atol, f"request {name}: first wrong token {int(np.argmax(worst > atol))} of {len(tokens)}, off by {worst.max():.2e}"
    engine.cache.check()


def dev(values, dtype=torch.float32):
    return torch.tensor(np.asarray(values), dtype=dtype, device="cuda")


# ---- each mechanism alone ----------------------------------------------------------------------

LAYERS = {
    "attention": nf.layer(mlp=None),
    "one_kv_head_no_rotation_five_taps": nf.layer(mlp=None, heads=6, kv_heads=1, dim=8, vdim=40, rot_dims=0, taps=5),
    "all_entries_rotated_one_tap": nf.layer(mlp=None, heads=2, kv_heads=2, dim=24, vdim=24, rot_dims=24, taps=1, scale=1.0),
    "odd_sizes": nf.layer(mlp=None, heads=3, kv_heads=1, dim=10, vdim=7, rot_dims=6, taps=2),
    "window_of_one_and_one_kept": nf.layer(mlp=None, window=1, keep_first=1),
    "nothing_kept": nf.layer(mlp=None, window=9, keep_first=0),
    "window_never_full": nf.layer(mlp=None, window=100, keep_first=5),
    "more_kept_than_seen": nf.layer(mlp=None, window=2, keep_first=21),
    "all_kept": nf.layer(mlp=None, window=2, keep_first=300),
    "experts": nf.layer(),
    "one_expert_no_identity": nf.layer(mlp=nf.moe(6, 0, 1, 0.5, 12)),
    "all_chosen": nf.layer(mlp=nf.moe(3, 2, 5, 2.0, 40)),
    "identity_for_the_most": nf.layer(mlp=nf.moe(1, 6, 3, 1.3, 8)),
}


@pytest.mark.parametrize("name", LAYERS)
def test_one_layer_of_each_kind(tmp_path, name):
    folder = nf.make_model(str(tmp_path / "m"), nf.config([LAYERS[name]]), seed=3, matrix_scale=3.0)
    engine = engine_for(folder)
    requests = {"a": random_tokens(1, 37, 211), "b": random_tokens(2, 1, 211), "c": random_tokens(3, 2, 211)}
    check(engine, folder, requests, schedule_whole(requests))
    check(engine, folder, requests, schedule_portions(requests))
    check(engine, folder, requests, schedule_tail_one_by_one(requests, tail=37))


def test_residual_stream_after_every_layer(tmp_path):
    from mini_llm_b200.engine import StepEntry
    folder = nf.make_model(str(tmp_path / "m"), nf.full_stack(), seed=5, matrix_scale=2.0)
    engine = engine_for(folder)
    tokens = random_tokens(4, 29, 211)
    _, streams = nf.plain_logits(folder, tokens, keep_layers=True)
    slot = engine.open_request()
    engine.step([StepEntry(slot, tokens, [28])], dump_hidden=True)
    assert len(engine.hidden_dump) == len(streams) + 1
    model_config, tensors = plain.load_model(folder)
    np.testing.assert_allclose(engine.hidden_dump[0].cpu().numpy(), tensors["embed"][tokens] * model_config["embedding"]["scale"], atol=1e-6)
    for index, expected in enumerate(streams):
        np.testing.assert_allclose(engine.hidden_dump[index + 1].cpu().numpy(), expected, rtol=0,
                                   atol=1e-4 * np.abs(expected).max(), err_msg=f"after layer {index}")
    engine.close_request(slot)


@pytest.mark.parametrize("mechanism", ["keep_first", "sink", "correction", "identity", "taps"])
def test_every_mechanism_shows(tmp_path, mechanism):
    """The engine stands with the full model and apart from the one without the mechanism."""
    folder = nf.make_model(str(tmp_path / "m"), nf.full_stack(), seed=6, matrix_scale=2.0)
    requests = {"a": random_tokens(5, 40, 211)}
    got = run_schedule(engine_for(folder), requests, schedule_whole(requests))["a"]
    np.testing.assert_allclose(got, nf.plain_logits(folder, requests["a"]), atol=F32_ATOL)
    assert np.abs(got[-1] - nf.plain_logits(folder, requests["a"], drop=(mechanism,))[-1]).max() > 200 * F32_ATOL


# ---- the same tokens, cut differently -----------------------------------------------------------

def test_prompt_against_token_by_token_and_portions(tmp_path):
    folder = nf.make_model(str(tmp_path / "m"), nf.full_stack(), seed=7, matrix_scale=2.0)
    engine = engine_for(folder)
    requests = {"a": random_tokens(11, 45, 211), "b": random_tokens(12, 7, 211)}
    check(engine, folder, requests, schedule_whole(requests))
    check(engine, folder, requests, schedule_tail_one_by_one(requests, tail=45))        # every token alone, from the first
    check(engine, folder, requests, schedule_tail_one_by_one(requests, tail=5))
    check(engine, folder, requests, schedule_portions(requests))
    check(engine, folder, requests, schedule_portions(requests, sizes=(2, 2, 3, 2, 17)))
    assert engine.step_kinds["replayed"] > 0          # steps of one shape were replayed from a captured graph


@pytest.mark.parametrize("page_size", [8, 16, 3])
def test_mixed_batches_and_reuse_of_pages_and_slots(tmp_path, page_size):
    """Six requests through three slots and a page pool that holds less than their sum: pages and slots are given
    back and used again (and poisoned in between), portions run beside single tokens; every request must come out
    as it does alone.  The windows give pages back while their requests still run, the kept tokens' pages stay."""
    folder = nf.make_model(str(tmp_path / "m"), nf.full_stack(), seed=9, matrix_scale=2.0)
    lengths = {"a": 61, "b": 9, "c": 33, "d": 2, "e": 40, "f": 18}
    requests = {name: random_tokens(20 + i, n, 211) for i, (name, n) in enumerate(lengths.items())}
    prompts = {"a": 40, "b": 9, "c": 20, "d": 1, "e": 40, "f": 3}
    engine = engine_for(folder, max_requests=3, cache_tokens=160, debug_poison=True, page_size=page_size)
    check(engine, folder, requests, schedule_mixed(requests, prompts, max_live=3))
    check(engine, folder, requests, schedule_mixed(requests, prompts, max_live=2, portion_sizes=(2, 11, 3)))
    assert not any(engine.cache.pages_in_use()) and engine.cache.free_slots == 3
    assert engine.cache.freed_by_window > 0


# ---- single keys that decide: far away, among the kept ones, and at a window's edge -------------

def _marked_layer(window, keep_first):
    return nf.config([nf.layer(heads=2, kv_heads=1, dim=8, vdim=8, taps=3, rot_dims=4, base=50.0, scale=0.2, window=window,
                               keep_first=keep_first, mlp=None)], vocab=64, width=32, embedding_scale=1.5)


def _decides(folder, with_key, without):
    return np.abs(nf.plain_logits(folder, with_key)[-1] - nf.plain_logits(folder, without)[-1]).max()


def _rows_of_one_position(t):
    """The filter passes its input on, so that a key and a value are their own token's alone, and values weigh enough
    to show."""
    for name in "qkv":
        t[f"l0.mix.{name}.conv"][:] = 0.0
        t[f"l0.mix.{name}.conv"][:, -1] = 1.0
    t["l0.mix.v"] *= 3.0
    t["l0.mix.o"] *= 2.0


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("key_at, keep_first, seen", [(0, 1, True), (0, 0, False), (7, 8, True), (8, 8, False), (10, 11, True), (11, 11, False),
                                                      (15, 16, True), (16, 16, False), (39, 40, True), (40, 40, False)])
def test_the_last_kept_token_and_the_first_that_is_not(tmp_path, key_at, keep_first, seen, dtype):
    """The logits of the last token hang on one early key hundreds of places back, behind dozens of page borders and
    given-back pages, if it is among the kept ones, and do not notice it if it is the next one: in a prompt, in
    portions and decoded alone, with the border of the kept ones inside a page and on a page's edge."""
    folder = nf.make_model(str(tmp_path / "m"), _marked_layer(13, keep_first), seed=13, matrix_scale=2.0, bfloat16_values=True,
                           bend=lambda t: (nf.mark(t, "l0.mix", 8), _rows_of_one_position(t)))
    with_key, without = nf.marked_tokens(260, key_at)
    change = _decides(folder, with_key, without)
    assert change > 0.1 if seen else change < 1e-9
    engine = engine_for(folder, dtype=dtype, debug_poison=True)
    expected = nf.plain_logits(folder, with_key)[-1]
    for steps in (schedule_whole({"r": with_key}), schedule_tail_one_by_one({"r": with_key}, tail=3),
                  schedule_portions({"r": with_key}, sizes=(8, 7, 9, 64, 2)), schedule_tail_one_by_one({"r": with_key}, tail=240)):
        got = run_schedule(engine, {"r": with_key}, steps)["r"][-1]
        assert np.abs(got - expected).max() < (F32_ATOL if dtype == "float32" else 0.05 * expected.std() + 1e-3)
    assert engine.cache.freed_by_window > 0
    engine.cache.check()


@pytest.mark.parametrize("window", [1, 13, 16, 40])
@pytest.mark.parametrize("keep_first", [0, 5])
def test_keys_just_inside_and_just_outside_the_window(tmp_path, window, keep_first):
    """The marked key stands ``window - 1`` places before the last token (the oldest key it sees) or ``window`` places
    before it (the newest it does not).  Windows of one, shorter than, equal to and longer than two pages, in a
    prompt, in portions and decoded alone.  (In a window of one the oldest key is the query's own: only the second
    case is left.)"""
    folder = nf.make_model(str(tmp_path / "m"), _marked_layer(window, keep_first), seed=15, matrix_scale=2.0,
                           bend=lambda t: (nf.mark(t, "l0.mix", 8), _rows_of_one_position(t)))
    n = 90
    outside, without = nf.marked_tokens(n, n - 1 - window)
    np.testing.assert_allclose(nf.plain_logits(folder, outside)[-1], nf.plain_logits(folder, without)[-1], atol=1e-12)
    sequences = [outside]
    if window > 1:
        inside, _ = nf.marked_tokens(n, n - window)
        assert _decides(folder, inside, without) > 0.1
        sequences.append(inside)
    engine = engine_for(folder, cache_tokens=256)
    for tokens in sequences:
        requests = {"r": tokens}
        check(engine, folder, requests, schedule_whole(requests))
        check(engine, folder, requests, schedule_tail_one_by_one(requests, tail=window + 3))
        check(engine, folder, requests, schedule_portions(requests, sizes=(8, 7, 9, 33, 2)))
    assert engine.cache.freed_by_window > 0


def test_the_convolution_reaches_over_cuts(tmp_path):
    """Five taps of equal size: every one of a cut's four predecessors enters the next portion's first tokens, also
    where a portion has fewer tokens than the filter looks back."""
    folder = nf.make_model(str(tmp_path / "m"), nf.config([nf.layer(taps=5, mlp=None), nf.layer(taps=4)]), seed=21, matrix_scale=3.0)
    engine = engine_for(folder)
    requests = {"a": random_tokens(71, 50, 211), "b": random_tokens(72, 21, 211)}
    for sizes in ((2, 2, 2, 2, 2), (3, 2, 5, 4), (9, 2, 1, 1, 2)):
        check(engine, folder, requests, schedule_portions(requests, sizes=sizes))
    check(engine, folder, requests, schedule_mixed(requests, {"a": 30, "b": 11}, max_live=2, portion_sizes=(2, 5, 3)))
    check(engine, folder, requests, schedule_tail_one_by_one(requests, tail=12))


def test_long_decoding(tmp_path):
    """220 single tokens: the window passes over decoded tokens and gives their pages back, the first ones stay.
    A pool of eight pages a group serves a request of 28 pages' length: it holds the kept and the window's pages."""
    folder = nf.make_model(str(tmp_path / "m"), nf.config([nf.layer(window=20, keep_first=11), nf.layer(window=20, keep_first=11)], width=64, vocab=97),
                           seed=17, matrix_scale=2.0)
    engine = engine_for(folder)
    requests = {"long": random_tokens(31, 221, 97)}
    check(engine, folder, requests, schedule_tail_one_by_one(requests, tail=220))
    check(engine, folder, requests, schedule_whole(requests))
    check(engine, folder, requests, schedule_portions(requests, sizes=(16, 17, 15, 2, 33, 100)))
    slot = engine.open_request()
    from mini_llm_b200.engine import StepEntry
    for token in requests["long"][:100]:
        engine.step([StepEntry(slot, [token], [0])])
    # positions 0 .. 10 in two pages, and those from 81 on (the next query's window) in pages 10 .. 12
    assert engine.cache.pages_held(slot)[0] == 2 + 3
    engine.close_request(slot)
    assert not any(engine.cache.pages_in_use())


# ---- bfloat16 ------------------------------------------------------------------------------------

def all_experts(raw):
    """The same stack with every expert chosen for every token: no choice hangs on a near tie, which rounding to
    bfloat16 may turn (the 32-bit tests cover the choice itself)."""
    for one in raw["layers"]:
        if one["mlp"] is not None:
            one["mlp"]["router"]["top"] = one["mlp"]["router"]["experts"] + one["mlp"]["router"]["identity"]
    return raw


def check_rounding(engine, folder, requests, steps, share=0.04):
    got = run_schedule(engine, requests, steps)
    for name, tokens in requests.items():
        expected = nf.plain_logits(folder, tokens)
        ratio = float(np.sqrt(((got[name] - expected) ** 2).mean()) / expected.std())
        assert ratio <= share, f"request {name}: root mean square of the difference is {ratio:.3f} of the logits' spread"
    engine.cache.check()


def test_bfloat16_follows_within_its_rounding(tmp_path):
    folder = nf.make_model(str(tmp_path / "m"), all_experts(nf.full_stack(width=128)), seed=19, bfloat16_values=True)
    engine = engine_for(folder, dtype="bfloat16")
    requests = {"a": random_tokens(41, 140, 211), "b": random_tokens(42, 12, 211), "c": random_tokens(43, 70, 211)}
    check_rounding(engine, folder, requests, schedule_whole(requests))
    check_rounding(engine, folder, requests, schedule_mixed(requests, {"a": 100, "b": 6, "c": 64}, max_live=3))
    check_rounding(engine, folder, requests, schedule_tail_one_by_one(requests, tail=10))
    chosen = {kernel for key, kernel in engine.kernels.choices.items() if key[0] in ("capped_attention", "linear")}
    assert {"capped_attention_tiled", "split_attention", "gemm_tcgen05"} <= chosen


def test_bfloat16_on_freed_pages(tmp_path):
    """Values and keys of other sizes, windows that pass pages on, kept tokens, poisoned free pages."""
    folder = nf.make_model(str(tmp_path / "m"), all_experts(nf.full_stack(width=128)), seed=20, bfloat16_values=True)
    engine = engine_for(folder, dtype="bfloat16", max_requests=3, cache_tokens=320, debug_poison=True)
    lengths = {"a": 161, "b": 9, "c": 33, "d": 2, "e": 90, "f": 18}
    requests = {name: random_tokens(20 + i, n, 211) for i, (name, n) in enumerate(lengths.items())}
    check_rounding(engine, folder, requests, schedule_mixed(requests, {"a": 140, "b": 9, "c": 20, "d": 1, "e": 70, "f": 3}, max_live=3,
                                                            portion_sizes=(70, 3, 2, 9, 50)))
    assert engine.cache.freed_by_window > 0


def test_bfloat16_with_sizes_no_fast_kernel_takes(tmp_path):
    """A width that is no multiple of 8, key sizes of 6 and 10: every product and the attention fall back to kernels
    that take any size, in bfloat16 too."""
    raw = nf.config([nf.layer(heads=3, kv_heads=1, dim=10, vdim=14, rot_dims=6),
                     nf.layer(heads=2, kv_heads=2, dim=6, vdim=10, rot_dims=2, mlp=nf.moe(3, 1, 2, 1.5, 9))], width=100, vocab=203)
    folder = nf.make_model(str(tmp_path / "m"), all_experts(raw), seed=29, bfloat16_values=True)
    requests = {"a": random_tokens(61, 150, 203), "b": random_tokens(62, 3, 203), "c": random_tokens(63, 40, 203)}
    engine = engine_for(folder, dtype="bfloat16")
    check_rounding(engine, folder, requests, schedule_whole(requests))
    check_rounding(engine, folder, requests, schedule_mixed(requests, {"a": 130, "b": 2, "c": 33}, max_live=3))
    chosen = {kernel for key, kernel in engine.kernels.choices.items() if key[0] in ("capped_attention", "linear")}
    assert chosen == {"capped_attention_plain", "linear_plain"}
    check(engine_for(folder), folder, requests, schedule_portions(requests))


def test_greedy_generation_through_the_scheduler(tmp_path):
    from mini_llm_b200.generate import generate
    folder = nf.make_model(str(tmp_path / "m"), nf.full_stack(), seed=23, matrix_scale=3.0)
    model_config, tensors = plain.load_model(folder)
    prompts = [random_tokens(50 + i, n, 211) for i, n in enumerate((3, 19, 1, 30, 8))]
    got = generate(folder, prompts, max_new_tokens=12, temperature=0.0, dtype="float32", page_size=8, max_sessions=3,
                   cache_tokens=256, max_prefill_chunk=7)
    for prompt, generated in zip(prompts, got):
        tokens = list(prompt)
        for index, token in enumerate(generated):
            logits = plain.forward(model_config, tensors, tokens)[-1]
            ordered = np.sort(logits)
            if ordered[-1] - ordered[-2] < 1e-3:
                break                                   # a near tie: either token is right, and the paths part here
            assert token == int(np.argmax(logits)), f"generated token {index}"
            tokens.append(token)


# ---- the mechanisms' kernels by themselves ------------------------------------------------------

def _attention_case(rng, n_tokens, heads, kv_heads, dim, vdim, page_size, dtype, window, keep, start=0):
    """One request of ``n_tokens`` cached positions; the step's queries are its last ``n_tokens - start``.  Pages that
    neither the window of the first query nor the kept tokens reach are gone: their table entries name a page of NaN."""
    n_pages = -(-n_tokens // page_size)
    order = rng.permutation(n_pages + 3)[:n_pages + 1]
    gone, order = order[0], order[1:]
    k = rng.normal(0, 1, (n_tokens, kv_heads, dim))
    v = rng.normal(0, 1, (n_tokens, kv_heads, vdim))
    q = rng.normal(0, 1, (n_tokens, heads, dim))
    if dtype == torch.bfloat16:
        k, v, q = (nf.to_bfloat16_values(x).astype(np.float64) for x in (k, v, q))
    k_pages = torch.zeros((n_pages + 3, page_size, kv_heads, dim), dtype=dtype, device="cuda")
    v_pages = torch.zeros((n_pages + 3, page_size, kv_heads, vdim), dtype=dtype, device="cuda")
    for block in range(n_pages):
        part = slice(block * page_size, min(n_tokens, (block + 1) * page_size))
        k_pages[order[block], :part.stop - part.start] = dev(k[part], dtype)
        v_pages[order[block], :part.stop - part.start] = dev(v[part], dtype)
    k_pages[gone], v_pages[gone] = float("nan"), float("nan")
    table = order.copy()
    kept_blocks, first_needed = -(-keep // page_size), max(0, start - window + 1) // page_size
    table[kept_blocks:max(kept_blocks, first_needed)] = gone
    return (q, k, v, k_pages, v_pages, dev(table[None, :], torch.int32), dev(np.arange(start, n_tokens), torch.int32),
            torch.zeros(n_tokens - start, dtype=torch.int32, device="cuda"))


def _attend(q, k, v, scale, window, keep, first_position):
    out = np.zeros((q.shape[0], q.shape[1], v.shape[2]))
    for t in range(q.shape[0]):
        seen = plain.visible(first_position + t, window, keep)
        for h in range(q.shape[1]):
            g = h // (q.shape[1] // k.shape[1])
            out[t, h] = plain.sink_weights(k[seen, g] @ q[t, h] * scale) @ v[seen, g]
    return out


@pytest.mark.parametrize("heads, kv_heads, dim, vdim, window, keep, start", [
    (4, 2, 16, 24, 9, 5, 0), (4, 2, 16, 24, 9, 5, 60), (3, 1, 8, 8, 40, 33, 100), (2, 2, 64, 80, 33, 1, 130), (2, 1, 24, 200, 5, 64, 90),
    (6, 1, 16, 16, 1, 3, 77), (2, 2, 8, 16, 300, 7, 5), (2, 2, 8, 16, 10, 0, 70), (4, 1, 128, 64, 31, 32, 97)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_attention_kernels_with_kept_tokens(heads, kv_heads, dim, vdim, window, keep, start, dtype):
    """Tiles and the plain form against the formula, from the sequence's start and from far behind it, where the
    kept keys lie tiles ahead of the window's."""
    from mini_llm_b200.kernels import ops
    n = start + 70
    q, k, v, k_pages, v_pages, table, positions, items = _attention_case(np.random.default_rng(dim + start), n, heads, kv_heads, dim, vdim, 8,
                                                                        dtype, window, keep, start)
    m = n - start
    expected = _attend(q[start:], k, v, 0.4, window, keep, start).reshape(m, heads * vdim)
    for tiled in (False, True):
        out = torch.full((m, heads * vdim), float("nan"), dtype=dtype, device="cuda")
        ops.capped_attention(out, dev(q[start:].reshape(m, -1), dtype), k_pages, v_pages, table, positions, items, heads, kv_heads, dim, vdim, 8,
                             0.4, 0.0, window, tiled=tiled, sink=torch.zeros(heads, device="cuda"), keep=keep)
        np.testing.assert_allclose(out.float().cpu().numpy(), expected, atol=2e-5 if dtype == torch.float32 else 0.02, err_msg=f"tiled={tiled}")


@pytest.mark.parametrize("heads, kv_heads, dim, vdim, window, keep, dtype", [
    (6, 2, 64, 80, 50, 20, torch.float32), (6, 2, 64, 64, 100, 130, torch.bfloat16), (6, 1, 32, 128, 1, 64, torch.float32),
    (8, 4, 128, 72, 200, 1, torch.bfloat16), (8, 4, 24, 40, 64, 0, torch.float32), (6, 3, 96, 104, 600, 9, torch.bfloat16)])
def test_attention_in_register_tiles_with_kept_tokens(heads, kv_heads, dim, vdim, window, keep, dtype):
    """Steps of thousands of (token, head) rows: two requests whose border falls inside a tile, the second one's
    portion far into its sequence."""
    from mini_llm_b200.kernels import ops
    rng = np.random.default_rng(dim + vdim)
    page, n0, n1, start1 = 16, 333, 460, 240
    cases = [_attention_case(rng, n0, heads, kv_heads, dim, vdim, page, dtype, window, keep),
             _attention_case(rng, n1, heads, kv_heads, dim, vdim, page, dtype, window, keep, start=start1)]
    shift = cases[0][3].shape[0]
    k_pages, v_pages = torch.cat([cases[0][3], cases[1][3]]), torch.cat([cases[0][4], cases[1][4]])
    table = torch.zeros((2, max(c[5].shape[1] for c in cases)), dtype=torch.int32, device="cuda")
    table[0, :cases[0][5].shape[1]] = cases[0][5][0]
    table[1, :cases[1][5].shape[1]] = cases[1][5][0] + shift
    positions = torch.cat([cases[0][6], cases[1][6]])
    items = torch.cat([torch.zeros(n0), torch.ones(n1 - start1)]).to(torch.int32).cuda()
    q = np.concatenate([cases[0][0], cases[1][0][start1:]])
    n = q.shape[0]
    assert n * heads >= 2048
    expected = np.concatenate([_attend(cases[0][0], cases[0][1], cases[0][2], 0.3, window, keep, 0),
                               _attend(cases[1][0][start1:], cases[1][1], cases[1][2], 0.3, window, keep, start1)]).reshape(n, heads * vdim)
    zeros = torch.zeros(heads, device="cuda")
    out = torch.full((n, heads * vdim), float("nan"), dtype=dtype, device="cuda")
    ops.capped_attention(out, dev(q.reshape(n, -1), dtype), k_pages, v_pages, table, positions, items, heads, kv_heads, dim, vdim, page, 0.3,
                         0.0, window, tiled=True, sink=zeros, keep=keep)
    np.testing.assert_allclose(out.float().cpu().numpy(), expected, atol=2e-5 if dtype == torch.float32 else 0.02)


@pytest.mark.parametrize("dim, vdim", [(64, 64), (64, 80), (16, 24), (128, 40), (8, 256), (72, 8)])
@pytest.mark.parametrize("window, keep", [(70, 0), (70, 20), (1, 3), (150, 130), (400, 20), (33, 290)])
def test_split_attention_with_kept_tokens(dim, vdim, window, keep):
    """Single tokens over split keys (bfloat16): a step of several requests of one sequence's pages at different
    lengths, the kept keys numbered ahead of the window's, values of another size than the keys."""
    from mini_llm_b200.kernels import ops
    rng = np.random.default_rng(dim + window)
    heads, kv_heads, n, page = 4, 2, 300, 16
    lasts = (300, 1, 21, 65, 299)
    cases = {last: _attention_case(rng, last, heads, kv_heads, dim, vdim, page, torch.bfloat16, window, keep, start=last - 1) for last in lasts}
    k_pages, v_pages = torch.cat([cases[l][3] for l in lasts]), torch.cat([cases[l][4] for l in lasts])
    table, shift = torch.zeros((len(lasts), -(-n // page)), dtype=torch.int32, device="cuda"), 0
    for i, last in enumerate(lasts):
        table[i, :cases[last][5].shape[1]] = cases[last][5][0] + shift
        shift += cases[last][3].shape[0]
    q = np.stack([cases[last][0][last - 1] for last in lasts])
    expected = np.concatenate([_attend(cases[l][0][l - 1:], cases[l][1], cases[l][2], 0.3, window, keep, l - 1) for l in lasts])
    chunk = 64
    max_chunks = -(-min(table.shape[1] * page, window + keep) // chunk)
    row = ops.split_attention_row(dim, vdim)
    cells = len(lasts) * heads * max_chunks
    acc, ml = torch.empty(cells * row, device="cuda"), torch.empty(cells * 2, device="cuda")
    counters = torch.zeros(len(lasts) * heads, dtype=torch.int32, device="cuda")
    out = torch.full((len(lasts), heads * vdim), float("nan"), dtype=torch.bfloat16, device="cuda")
    ops.split_attention(out, dev(q.reshape(len(lasts), -1), torch.bfloat16), k_pages, v_pages, table, dev([l - 1 for l in lasts], torch.int32),
                        dev(range(len(lasts)), torch.int32), heads, kv_heads, dim, page, 0.3, window, chunk, max_chunks, acc, ml, counters,
                        sink=torch.zeros(heads, device="cuda"), value_size=vdim, keep=keep)
    np.testing.assert_allclose(out.float().cpu().numpy(), expected.reshape(len(lasts), -1), atol=0.02)
    assert int(counters.abs().sum()) == 0


@pytest.mark.parametrize("taps", [1, 2, 5])
@pytest.mark.parametrize("norm", [None, "head"])
def test_taps_rotation_and_store_in_one_kernel(taps, norm):
    """A sequence cut in portions down to one token, beside another request, through the kernel that filters, norms,
    turns and stores; the state it leaves; single tokens move it themselves."""
    from mini_llm_b200.kernels import ops
    rng = np.random.default_rng(taps)
    heads, kv_heads, dim, vdim, page, rot_dims, n = 4, 2, 16, 24, 8, 10, 31
    q_width, k_width, v_width = heads * dim, kv_heads * dim, kv_heads * vdim
    columns = q_width + k_width + v_width
    u, w = rng.normal(0, 1, (n, columns)), rng.normal(0, 1, (columns, taps))
    filtered = plain.short_convolution(u, w)
    q, k, v = filtered[:, :q_width], filtered[:, q_width:q_width + k_width], filtered[:, q_width + k_width:]
    gains = (rng.uniform(0.5, 1.5, dim), rng.uniform(0.5, 1.5, dim))

    def normed(x, gain):
        x = x.reshape(n, -1, dim)
        return plain.rms_norm(x, gain, 1e-3) if norm else x
    q_expected = plain.rotate_half(normed(q, gains[0]), np.arange(n), 70.0, rot_dims).reshape(n, -1)
    k_expected = plain.rotate_half(normed(k, gains[1]), np.arange(n), 70.0, rot_dims)
    inv_freq = torch.tensor([70.0 ** (-2.0 * i / rot_dims) for i in range(rot_dims // 2)], dtype=torch.float64, device="cuda")
    k_pages, v_pages = torch.zeros((8, page, kv_heads, dim), device="cuda"), torch.zeros((8, page, kv_heads, vdim), device="cuda")
    table = dev([[6, 6, 6, 6], [3, 1, 0, 5]], torch.int32)
    state = torch.zeros((3, taps - 1, columns), device="cuda")
    got, done = [], 0
    for cut in (1, 2, 1, 9, 1, 1, 3, 13):
        single = cut == 1
        other = 1 if single else 2                            # another request's tokens come first
        rows = np.concatenate([rng.normal(0, 1, (other, columns)), u[done:done + cut]])
        q_out = torch.full((other + cut, q_width), float("nan"), device="cuda")
        positions = dev(list(range(other)) + list(range(done, done + cut)), torch.int32)
        items = dev([0] * other + [1] * cut, torch.int32)
        ops.norm_rotary_store(dev(rows), q_width, q_width + k_width, heads, kv_heads, dim, vdim, q_out, dev(gains[0]) if norm else None,
                              dev(gains[1]) if norm else None, norm, 1e-3, rot_dims, "half", inv_freq, positions, items, table, page, k_pages,
                              v_pages, taps=(dev(w), state, dev([0, 2], torch.int32), dev([0, done], torch.int32),
                                             dev([0, other], torch.int32), dev([other, cut], torch.int32), single))
        got.append(q_out[other:].cpu().numpy())
        done += cut
    assert done == n
    np.testing.assert_allclose(np.concatenate(got), q_expected, atol=2e-5)
    order = [3, 1, 0, 5]
    for p in range(n):
        np.testing.assert_allclose(k_pages[order[p // page], p % page].cpu().numpy(), k_expected[p], atol=2e-5, err_msg=f"key {p}")
        np.testing.assert_allclose(v_pages[order[p // page], p % page].cpu().numpy(), v[p].reshape(kv_heads, vdim), atol=2e-5, err_msg=f"value {p}")
    if taps > 1:
        np.testing.assert_allclose(state[2].cpu().numpy(), u[n - taps + 1:], atol=1e-6)
        assert float(state[1].abs().max()) == 0.0


@pytest.mark.parametrize("experts, identity, top", [(5, 2, 3), (1, 3, 2), (6, 0, 6), (40, 9, 8), (3, 1, 1)])
def test_router_with_corrections_and_identity_experts(experts, identity, top):
    """The third rule of the router, with more outputs than a warp has lanes, and both ways through the experts (pair
    by pair, and all at once) with and without the sum written over what was there."""
    from mini_llm_b200.kernels import ops
    rng = np.random.default_rng(experts)
    n, width, inner, outputs = 9, 40, 16, experts + identity
    x, router, correction = rng.normal(0, 1, (n, width)), rng.normal(0, 0.4, (outputs, width)), rng.normal(0, 0.1, outputs)
    ups, downs = rng.normal(0, 0.3, (experts, inner, width)), rng.normal(0, 0.3, (experts, width, inner))
    before = rng.normal(0, 1, (n, width))
    choice = torch.zeros(n * top, dtype=torch.int32, device="cuda")
    in_weight, out_weight, passed = torch.zeros(n * top, device="cuda"), torch.zeros(n * top, device="cuda"), torch.full((n,), 7.0, device="cuda")
    ops.route(dev(x), dev(router), None, top, choice, in_weight, out_weight, rule="softmax_of_all", correction=dev(correction),
              n_identity=identity, scale=2.5, identity_weight=passed if identity else None)
    expected = np.zeros((n, width))
    for t in range(n):
        chosen, weights = plain.choose(x[t] @ router.T, correction, top, 2.5)
        assert choice[t * top:(t + 1) * top].tolist() == [e if e < experts else -1 for e in chosen]
        np.testing.assert_allclose(out_weight[t * top:(t + 1) * top].cpu().numpy(), np.where(chosen < experts, weights, 0.0), atol=2e-6)
        if identity:
            assert abs(float(passed[t]) - weights[chosen >= experts].sum()) < 2e-6
        for e, g in zip(chosen, weights):
            expected[t] += g * (x[t] if e >= experts else (np.maximum(x[t] @ ups[e].T, 0.0) ** 2) @ downs[e].T)
    up_matrix, down_matrix = dev(ups.reshape(-1, width)), dev(np.concatenate(list(downs), axis=1))
    up_of = torch.tensor([up_matrix[e * inner:].data_ptr() for e in range(experts)], dtype=torch.int64, device="cuda")
    down_of = torch.tensor([down_matrix.data_ptr() + 4 * e * inner for e in range(experts)], dtype=torch.int64, device="cuda")
    inner_of = torch.full((experts,), inner, dtype=torch.int32, device="cuda")
    for assign in (False, True):
        hidden, act = dev(before), torch.full((n * top, inner), float("nan"), device="cuda")
        ops.experts(hidden, act, dev(x), choice, in_weight, out_weight, None, up_of, down_of, inner_of, inner, top, ld_down=experts * inner,
                    assign=assign, identity_weight=passed if identity else None)
        np.testing.assert_allclose(hidden.cpu().numpy(), expected + (0.0 if assign else before), atol=3e-5)
        hidden, gu = dev(before), dev(x) @ up_matrix.T
        combined = torch.full((n, experts * inner), float("nan"), device="cuda")
        ops.expert_combine(combined, gu.contiguous(), choice, in_weight, out_weight, experts, inner, top, top, form="relu_squared", hidden=hidden,
                           x=dev(x), identity_weight=passed if identity else None, assign=assign)
        if assign and not identity:
            hidden.zero_()
        result = hidden.cpu().numpy() + combined.cpu().numpy().astype(np.float64) @ down_matrix.cpu().numpy().astype(np.float64).T
        np.testing.assert_allclose(result, expected + (0.0 if assign else before), atol=2e-4)
