"""Kerepel on the device against the plain implementation (``plain_kerepel``, float64).

Every test makes its own small configuration and random weights.  32-bit runs must agree within 1e-4 at every
token; bfloat16 runs within 4 % of the logits' spread in the root mean square.  The schedules cut the same requests
in different ways: a request's logits must not depend on the cut, on the rest of the batch, or on which pages and
slots it got."""

import numpy as np
import pytest
import torch

import kerepel_helpers as kp
import plain_kerepel as plain
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
        expected = kp.plain_logits(folder, tokens)
        worst = np.abs(got[name] - expected).max(axis=1)
        assert worst.max() <= atol, f"request {name}: first wrong token {int(np.argmax(worst > atol))} of {len(tokens)}, off by {worst.max():.2e}"
    engine.cache.check()


def dev(values, dtype=torch.float32):
    return torch.tensor(np.asarray(values), dtype=dtype, device="cuda")


# ---- each mechanism alone ----------------------------------------------------------------------

STACKS = {
    "attention": [kp.attention(mlp=None)],
    "one_kv_head_five_taps": [kp.attention(mlp=None, heads=6, kv_heads=1, dim=8, vdim=40, taps=5)],
    "one_tap_no_cap": [kp.attention(mlp=None, heads=2, kv_heads=2, dim=24, vdim=24, taps=1, softcap=None, scale=0.3)],
    "odd_sizes": [kp.attention(mlp=None, heads=3, kv_heads=1, dim=10, vdim=7, taps=2)],
    "values_of_one_entry": [kp.attention(mlp=None, heads=4, kv_heads=4, dim=4, vdim=1)],
    "window_of_one": [kp.attention(mlp=None, window=1)],
    "window_never_full": [kp.attention(mlp=None, window=100)],
    "shared_keys": [kp.attention(mlp=None), kp.attention(mlp=None, kv_from=0, window=20, taps=4), kp.attention(mlp=None, kv_from=0, window=3, heads=2)],
    "latent": [kp.latent(mlp=None)],
    "latent_one_head_no_scaling": [kp.latent(mlp=None, heads=1, dim=8, rot_dim=4, vdim=40, rank=16, scaling=None)],
    "latent_nothing_turns": [kp.latent(mlp=None, rot_dim=0, scaling=None)],
    "latent_odd_sizes": [kp.latent(mlp=None, heads=5, dim=7, rot_dim=6, vdim=9, rank=19, scaling=kp.yarn(1.0, 64.0, 2.0, 1.0))],
    "latent_narrow": [kp.latent(mlp=None, heads=2, dim=4, rot_dim=2, vdim=4, rank=6)],
    "dense": [kp.latent(mlp=kp.dense(33))],
    "experts": [kp.latent(mlp=kp.moe())],
    "experts_without_groups_or_shared": [kp.latent(mlp=kp.moe(7, 3, None, 20, 2.0, None))],
    "groups_of_one": [kp.latent(mlp=kp.moe(5, 2, (5, 3), 12, 0.7, (6, 1.1)))],
    "one_group": [kp.latent(mlp=kp.moe(4, 4, (1, 1), 12, 0.7, (50, 0.2)))],
    "many_experts": [kp.latent(mlp=kp.moe(72, 5, (9, 2), 8, 0.7, (16, 0.2)))],
}


@pytest.mark.parametrize("name", STACKS)
def test_one_stack_of_each_kind(tmp_path, name):
    folder = kp.make_model(str(tmp_path / "m"), kp.config(STACKS[name]), seed=3, matrix_scale=3.0)
    engine = engine_for(folder)
    requests = {"a": random_tokens(1, 37, 211), "b": random_tokens(2, 1, 211), "c": random_tokens(3, 2, 211)}
    check(engine, folder, requests, schedule_whole(requests))
    check(engine, folder, requests, schedule_portions(requests))
    check(engine, folder, requests, schedule_tail_one_by_one(requests, tail=37))


@pytest.mark.parametrize("more", [dict(side=None), dict(side=1), dict(side=5, width=100), dict(side=40, width=34), dict(buckets=1), dict(mul_prev=0),
                                  dict(mul_prev=1900000000, mul_cur=2100000000, buckets=1013), dict(logit_scale=1.0, eps=1e-2)])
def test_inputs_from_the_tokens(tmp_path, more):
    """The pair table and the tokens' own rows of several sizes, factors whose products need 64 bits, a constant of one."""
    folder = kp.make_model(str(tmp_path / "m"), kp.config([kp.attention(), kp.latent(mlp=None)], **more), seed=4, matrix_scale=2.0)
    engine = engine_for(folder)
    requests = {"a": random_tokens(1, 80, 211), "b": random_tokens(2, 1, 211), "c": random_tokens(3, 2, 211)}
    check(engine, folder, requests, schedule_whole(requests))
    check(engine, folder, requests, schedule_portions(requests, sizes=(2, 3, 2, 31)))
    check(engine, folder, requests, schedule_mixed(requests, {"a": 70, "b": 1, "c": 2}, max_live=3))


def test_without_a_pair_table(tmp_path):
    raw = kp.config([kp.attention(), kp.latent()])
    raw["embedding"] = {}
    folder = kp.make_model(str(tmp_path / "m"), raw, seed=4)
    requests = {"a": random_tokens(1, 30, 211)}
    check(engine_for(folder), folder, requests, schedule_portions(requests))


def test_residual_stream_after_every_layer(tmp_path):
    from mini_llm_b200.engine import StepEntry
    folder = kp.make_model(str(tmp_path / "m"), kp.full_stack(), seed=5, matrix_scale=2.0)
    engine = engine_for(folder)
    tokens = random_tokens(4, 29, 211)
    _, streams = kp.plain_logits(folder, tokens, keep_layers=True)
    slot = engine.open_request()
    engine.step([StepEntry(slot, tokens, [28])], dump_hidden=True)
    assert len(engine.hidden_dump) == len(streams) + 1
    model_config, tensors = plain.load_model(folder)
    np.testing.assert_allclose(engine.hidden_dump[0].cpu().numpy(), plain.embed(model_config, tensors, tokens), atol=1e-6)
    for index, expected in enumerate(streams):
        np.testing.assert_allclose(engine.hidden_dump[index + 1].cpu().numpy(), expected, rtol=0,
                                   atol=1e-4 * np.abs(expected).max(), err_msg=f"after layer {index}")
    engine.close_request(slot)


@pytest.mark.parametrize("mechanism", kp.MECHANISMS)
def test_every_mechanism_shows(tmp_path, mechanism):
    """The engine stands with the full model and apart from the one without the mechanism."""
    folder = kp.make_model(str(tmp_path / "m"), kp.full_stack(), seed=6, matrix_scale=2.0)
    requests = {"a": random_tokens(5, 40, 211)}
    got = run_schedule(engine_for(folder), requests, schedule_whole(requests))["a"]
    np.testing.assert_allclose(got, kp.plain_logits(folder, requests["a"]), atol=F32_ATOL)
    assert np.abs(got[-1] - kp.plain_logits(folder, requests["a"], drop=(mechanism,))[-1]).max() > 200 * F32_ATOL


# ---- the same tokens, cut differently -----------------------------------------------------------

def test_prompt_against_token_by_token_and_portions(tmp_path):
    folder = kp.make_model(str(tmp_path / "m"), kp.full_stack(), seed=7, matrix_scale=2.0)
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
    as it does alone.  The windows give pages back while their requests still run; a slot's last token and last
    projected rows are another request's when the slot is used again."""
    folder = kp.make_model(str(tmp_path / "m"), kp.full_stack(), seed=9, matrix_scale=2.0)
    lengths = {"a": 61, "b": 9, "c": 33, "d": 2, "e": 40, "f": 18}
    requests = {name: random_tokens(20 + i, n, 211) for i, (name, n) in enumerate(lengths.items())}
    prompts = {"a": 40, "b": 9, "c": 20, "d": 1, "e": 40, "f": 3}
    engine = engine_for(folder, max_requests=3, cache_tokens=160, debug_poison=True, page_size=page_size)
    check(engine, folder, requests, schedule_mixed(requests, prompts, max_live=3))
    check(engine, folder, requests, schedule_mixed(requests, prompts, max_live=2, portion_sizes=(2, 11, 3)))
    assert not any(engine.cache.pages_in_use()) and engine.cache.free_slots == 3
    assert engine.cache.freed_by_window > 0


def test_the_last_token_is_a_requests_state(tmp_path):
    """Pairs that cross a cut: the first token of every portion finds the one before it, also when another request
    ran in between, and the first token of a request finds none in a slot that was used before."""
    folder = kp.make_model(str(tmp_path / "m"), kp.config([kp.latent(mlp=None)], buckets=5003, side=None), seed=8)
    engine = engine_for(folder, max_requests=2, cache_tokens=256)
    requests = {"a": random_tokens(81, 23, 211), "b": random_tokens(82, 11, 211), "c": random_tokens(83, 5, 211)}
    steps = [[("a", 2)], [("b", 1), ("a", 3)], [("b", 2)], [("a", 1), ("b", 1)], [("a", 1)], [("b", 7), ("a", 1)], [("c", 1), ("a", 15)], [("c", 4)]]
    check(engine, folder, requests, steps)
    check(engine, folder, requests, steps)


# ---- single keys that decide: far away, and at a window's edge ----------------------------------

def _marked_attention(window, readers=()):
    one = dict(heads=2, kv_heads=1, dim=8, vdim=8, scale=1.0, softcap=60.0, mlp=None)
    return kp.config([kp.attention(taps=3, window=window, **one)] + [kp.attention(taps=1, window=w, kv_from=0, **one) for w in readers],
                     vocab=64, width=32, side=4)


def _decides(folder, with_key, without):
    return np.abs(kp.plain_logits(folder, with_key)[-1] - kp.plain_logits(folder, without)[-1]).max()


def _schedules(tokens, tail):
    requests = {"r": tokens}
    return (schedule_whole(requests), schedule_tail_one_by_one(requests, tail=tail), schedule_portions(requests, sizes=(8, 7, 9, 64, 2)))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("window", [1, 13, 16, 40])
def test_keys_just_inside_and_just_outside_the_window(tmp_path, window, dtype):
    """The marked key stands ``window - 1`` places before the last token (the oldest key it sees) or ``window`` places
    before it (the newest it does not).  Windows of one, shorter than, equal to and longer than two pages, in a
    prompt, in portions and decoded alone.  (In a window of one the oldest key is the query's own.)"""
    folder = kp.make_model(str(tmp_path / "m"), _marked_attention(window), seed=15, matrix_scale=2.0, bfloat16_values=True,
                           bend=lambda t: (kp.quiet_neighbours(t), kp.mark_attention(t, "l0.mix", 8, 2)))
    n = 90
    outside, without = kp.marked_tokens(n, n - 1 - window)
    np.testing.assert_allclose(kp.plain_logits(folder, outside)[-1], kp.plain_logits(folder, without)[-1], atol=1e-12)
    sequences = [outside]
    if window > 1:
        inside, _ = kp.marked_tokens(n, n - window)
        assert _decides(folder, inside, without) > 0.5
        sequences.append(inside)
    engine = engine_for(folder, dtype=dtype, cache_tokens=256, debug_poison=True)
    for tokens in sequences:
        expected = kp.plain_logits(folder, tokens)[-1]
        for steps in _schedules(tokens, window + 3):
            got = run_schedule(engine, {"r": tokens}, steps)["r"][-1]
            assert np.abs(got - expected).max() < (F32_ATOL if dtype == "float32" else 0.05 * expected.std() + 1e-3)
    assert engine.cache.freed_by_window > 0


@pytest.mark.parametrize("owner, reader", [(9, 30), (30, 9), (16, 17)])
def test_a_readers_own_window_over_shared_keys(tmp_path, owner, reader):
    """A layer reads another's keys through its own window: wider than the owner's (whose pages must wait for it) or
    narrower; the marked key lies just inside and just outside the reader's window."""
    def bend(t):
        kp.quiet_neighbours(t)
        kp.mark_attention(t, "l0.mix", 8, 2)
        t["l1.mix.q"][7] = 0.0
        t["l1.mix.q"][7, :8] = -6.0
        t["l1.mix.q.norm"][:], t["l1.mix.q.norm"][7] = 1.0, 2.0
        t["l1.mix.q.conv"][:] = 1.0
        t["l1.norm1"][:8] = 1.0
        t["l1.mix.o"] *= 6.0
        t["l0.mix.o"] *= 0.02                     # (what the owner itself makes of the key hardly shows)
    folder = kp.make_model(str(tmp_path / "m"), _marked_attention(owner, (reader,)), seed=16, matrix_scale=2.0, bend=bend)
    n = 80
    engine = engine_for(folder, cache_tokens=256, debug_poison=True)
    for key_at in (n - reader, n - 1 - reader, n - owner, n - 1 - owner):
        tokens, without = kp.marked_tokens(n, key_at)
        change = _decides(folder, tokens, without)
        assert change > 0.5 if key_at >= n - reader else change < 0.3
        for steps in _schedules(tokens, max(owner, reader) + 3):
            check(engine, folder, {"r": tokens}, steps)
    assert engine.cache.freed_by_window > 0


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("key_at", [0, 7, 8, 63, 64, 200])
def test_far_keys_through_the_latent(tmp_path, key_at, dtype):
    """The logits of the last token hang on one key hundreds of places back, at page and tile borders: in a prompt, in
    portions and decoded alone."""
    raw = kp.config([kp.latent(heads=2, dim=8, rot_dim=4, vdim=8, rank=16, scale=1.0, mlp=None)], vocab=64, width=32, side=4)
    folder = kp.make_model(str(tmp_path / "m"), raw, seed=13, matrix_scale=2.0, bfloat16_values=True,
                           bend=lambda t: (kp.quiet_neighbours(t), kp.mark_latent(t, "l0.mix", 16, 8)))
    tokens, without = kp.marked_tokens(331, key_at)
    assert _decides(folder, tokens, without) > 0.5
    engine = engine_for(folder, dtype=dtype, debug_poison=True)
    expected = kp.plain_logits(folder, tokens)[-1]
    for steps in _schedules(tokens, 5):
        got = run_schedule(engine, {"r": tokens}, steps)["r"][-1]
        assert np.abs(got - expected).max() < (F32_ATOL if dtype == "float32" else 0.05 * expected.std() + 1e-3)


def test_the_convolution_reaches_over_cuts(tmp_path):
    """Every one of a cut's four predecessors enters the next portion's first tokens, also where a portion has fewer
    tokens than the filter looks back; a reader filters its own queries only."""
    folder = kp.make_model(str(tmp_path / "m"), kp.config([kp.attention(taps=5, mlp=None), kp.attention(taps=4, kv_from=0)]), seed=21, matrix_scale=3.0)
    engine = engine_for(folder)
    requests = {"a": random_tokens(71, 50, 211), "b": random_tokens(72, 21, 211)}
    for sizes in ((2, 2, 2, 2, 2), (3, 2, 5, 4), (9, 2, 1, 1, 2)):
        check(engine, folder, requests, schedule_portions(requests, sizes=sizes))
    check(engine, folder, requests, schedule_mixed(requests, {"a": 30, "b": 11}, max_live=2, portion_sizes=(2, 5, 3)))
    check(engine, folder, requests, schedule_tail_one_by_one(requests, tail=12))


def test_long_decoding(tmp_path):
    """220 single tokens: the window passes over decoded tokens and gives their pages back, the latent keeps all."""
    folder = kp.make_model(str(tmp_path / "m"), kp.config([kp.attention(window=20), kp.latent(), kp.attention(window=12, kv_from=0)], width=64, vocab=97),
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
    # attention: positions from 81 on (the next query's window) in pages 10 .. 12; the latent: all thirteen
    held = [n for n, group in zip(engine.cache.pages_held(slot), engine.cache.groups) if group.paged]
    assert sorted(held) == [3, 13]
    engine.close_request(slot)
    assert not any(engine.cache.pages_in_use())


# ---- bfloat16 ------------------------------------------------------------------------------------

def all_experts(raw):
    """The same stack with every expert chosen for every token: no choice hangs on a near tie, which rounding to
    bfloat16 may turn (the 32-bit tests cover the choice itself)."""
    for one in raw["layers"]:
        if one["mlp"] is not None and one["mlp"]["kind"] == "moe":
            router = one["mlp"]["router"]
            router["top"] = router["experts"]
            if router.get("groups"):
                router["groups"]["keep"] = router["groups"]["count"]
    return raw


def check_rounding(engine, folder, requests, steps, share=0.04):
    got = run_schedule(engine, requests, steps)
    for name, tokens in requests.items():
        expected = kp.plain_logits(folder, tokens)
        ratio = float(np.sqrt(((got[name] - expected) ** 2).mean()) / expected.std())
        assert ratio <= share, f"request {name}: root mean square of the difference is {ratio:.3f} of the logits' spread"
    engine.cache.check()


def test_bfloat16_follows_within_its_rounding(tmp_path):
    folder = kp.make_model(str(tmp_path / "m"), all_experts(kp.full_stack(width=128, side=16)), seed=19, bfloat16_values=True)
    engine = engine_for(folder, dtype="bfloat16")
    requests = {"a": random_tokens(41, 140, 211), "b": random_tokens(42, 12, 211), "c": random_tokens(43, 70, 211)}
    check_rounding(engine, folder, requests, schedule_whole(requests))
    check_rounding(engine, folder, requests, schedule_mixed(requests, {"a": 100, "b": 6, "c": 64}, max_live=3))
    check_rounding(engine, folder, requests, schedule_tail_one_by_one(requests, tail=10))
    chosen = {kernel for key, kernel in engine.kernels.choices.items()}
    assert {"capped_attention_tiled", "split_attention", "gemm_tcgen05", "latent_attention_tiled", "latent_attention_tiled_parts",
            "token_gate", "token_gate_rows"} <= chosen


def test_bfloat16_on_freed_pages(tmp_path):
    folder = kp.make_model(str(tmp_path / "m"), all_experts(kp.full_stack(width=128)), seed=20, bfloat16_values=True)
    engine = engine_for(folder, dtype="bfloat16", max_requests=3, cache_tokens=320, debug_poison=True)
    lengths = {"a": 161, "b": 9, "c": 33, "d": 2, "e": 90, "f": 18}
    requests = {name: random_tokens(20 + i, n, 211) for i, (name, n) in enumerate(lengths.items())}
    check_rounding(engine, folder, requests, schedule_mixed(requests, {"a": 140, "b": 9, "c": 20, "d": 1, "e": 70, "f": 3}, max_live=3,
                                                            portion_sizes=(70, 3, 2, 9, 50)))
    assert engine.cache.freed_by_window > 0


def test_bfloat16_with_sizes_no_fast_kernel_takes(tmp_path):
    """A width that is no multiple of 8, odd key, latent and row sizes: every product and the attentions fall back to kernels
    that take any size, in bfloat16 too."""
    raw = kp.config([kp.attention(heads=3, kv_heads=1, dim=10, vdim=14, mlp=kp.dense(33)),
                     kp.latent(heads=2, dim=6, rot_dim=2, vdim=10, rank=21, mlp=kp.moe(3, 2, None, 9, 0.8, (7, 0.6)))], width=100, vocab=203, side=3)
    folder = kp.make_model(str(tmp_path / "m"), all_experts(raw), seed=29, bfloat16_values=True)
    requests = {"a": random_tokens(61, 150, 203), "b": random_tokens(62, 3, 203), "c": random_tokens(63, 40, 203)}
    engine = engine_for(folder, dtype="bfloat16")
    check_rounding(engine, folder, requests, schedule_whole(requests))
    check_rounding(engine, folder, requests, schedule_mixed(requests, {"a": 130, "b": 2, "c": 33}, max_live=3))
    chosen = {kernel for key, kernel in engine.kernels.choices.items() if key[0] in ("capped_attention", "latent_attention", "linear")}
    assert chosen == {"capped_attention_plain", "latent_attention_plain", "linear_plain"}
    check(engine_for(folder), folder, requests, schedule_portions(requests))


def test_greedy_generation_through_the_scheduler(tmp_path):
    """Tokens are taken on the device (the host reads them a step late): the pair of a sampled token and the one before
    it is made there.  Requests wait for one another's slots; prompts come in portions."""
    from mini_llm_b200.generate import generate
    folder = kp.make_model(str(tmp_path / "m"), kp.full_stack(), seed=23, matrix_scale=2.0)
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

def _attention_case(rng, n_tokens, heads, kv_heads, dim, vdim, page_size, dtype, window, start=0):
    """One request of ``n_tokens`` cached positions; the step's queries are its last ``n_tokens - start``.  Pages the window
    of the first query does not reach are gone: their table entries name a page of NaN."""
    n_pages = -(-n_tokens // page_size)
    order = rng.permutation(n_pages + 3)[:n_pages + 1]
    gone, order = order[0], order[1:]
    k, v = rng.normal(0, 1, (n_tokens, kv_heads, dim)), rng.normal(0, 1, (n_tokens, kv_heads, vdim))
    q = rng.normal(0, 1, (n_tokens, heads, dim))
    if dtype == torch.bfloat16:
        k, v, q = (kp.to_bfloat16_values(x).astype(np.float64) for x in (k, v, q))
    k_pages = torch.zeros((n_pages + 3, page_size, kv_heads, dim), dtype=dtype, device="cuda")
    v_pages = torch.zeros((n_pages + 3, page_size, kv_heads, vdim), dtype=dtype, device="cuda")
    for block in range(n_pages):
        part = slice(block * page_size, min(n_tokens, (block + 1) * page_size))
        k_pages[order[block], :part.stop - part.start] = dev(k[part], dtype)
        v_pages[order[block], :part.stop - part.start] = dev(v[part], dtype)
    k_pages[gone], v_pages[gone] = float("nan"), float("nan")
    table = order.copy()
    table[:max(0, start - window + 1) // page_size] = gone
    return (q, k, v, k_pages, v_pages, dev(table[None, :], torch.int32), dev(np.arange(start, n_tokens), torch.int32),
            torch.zeros(n_tokens - start, dtype=torch.int32, device="cuda"))


def _attend(q, k, v, gate, scale, cap, window, first_position, wide=True):
    heads, vdim = q.shape[1], v.shape[2]
    slopes = plain.slopes(heads)
    out = np.zeros((q.shape[0], heads, vdim))
    for t in range(q.shape[0]):
        p = first_position + t
        seen = np.arange(max(0, p - window + 1), p + 1)
        for h in range(heads):
            g = h // (heads // k.shape[1])
            s = cap * np.tanh(k[seen, g] @ q[t, h] * scale / cap) - slopes[h] * (p - seen)
            out[t, h] = plain.softmax(s) @ v[seen, g]
            out[t, h] *= plain.sigmoid(gate[t, h * vdim:(h + 1) * vdim] if wide else gate[t, h])
    return out.reshape(q.shape[0], -1)


@pytest.mark.parametrize("heads, kv_heads, dim, vdim, window, start", [
    (4, 2, 16, 24, 9, 0), (4, 2, 16, 24, 9, 60), (3, 1, 8, 8, 40, 100), (2, 2, 64, 80, 33, 130), (2, 1, 24, 200, 5, 90),
    (12, 1, 16, 16, 200, 7), (2, 2, 8, 16, 300, 5), (4, 1, 128, 64, 31, 97)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_attention_kernels_with_a_bias_by_distance_and_a_gate(heads, kv_heads, dim, vdim, window, start, dtype):
    """Tiles and the plain form against the formula, with a gate per entry and one per head that stand in a wider buffer."""
    from mini_llm_b200.kernels import ops
    n, m = start + 70, 70
    rng = np.random.default_rng(dim + start)
    q, k, v, k_pages, v_pages, table, positions, items = _attention_case(rng, n, heads, kv_heads, dim, vdim, 8, dtype, window, start)
    buffer = dev(rng.normal(0, 1.5, (m, 5 + heads * vdim)))
    slopes = dev(plain.slopes(heads))
    for wide in (True, False):
        expected = _attend(q[start:], k, v, buffer[:, 5:].cpu().numpy(), 0.4, 3.0, window, start, wide)
        for tiled in (False, True):
            out = torch.full((m, heads * vdim), float("nan"), dtype=dtype, device="cuda")
            ops.capped_attention(out, dev(q[start:].reshape(m, -1), dtype), k_pages, v_pages, table, positions, items, heads, kv_heads, dim, vdim, 8,
                                 0.4, 3.0, window, tiled=tiled, gate=buffer[:, 5:], gate_wide=wide, slopes=slopes)
            np.testing.assert_allclose(out.float().cpu().numpy(), expected, atol=2e-5 if dtype == torch.float32 else 0.02, err_msg=f"{tiled} {wide}")


@pytest.mark.parametrize("heads, kv_heads, dim, vdim, window, dtype", [
    (6, 2, 64, 80, 50, torch.float32), (6, 2, 64, 64, 100, torch.bfloat16), (6, 1, 32, 128, 1, torch.float32),
    (8, 4, 128, 72, 200, torch.bfloat16), (8, 4, 24, 40, 64, torch.float32), (7, 1, 96, 104, 600, torch.bfloat16)])
def test_attention_in_register_tiles_with_a_bias_by_distance_and_a_gate(heads, kv_heads, dim, vdim, window, dtype):
    """Steps of thousands of (token, head) rows: two requests whose border falls inside a tile, the second one's
    portion far into its sequence."""
    from mini_llm_b200.kernels import ops
    rng = np.random.default_rng(dim + vdim)
    page, n0, n1, start1 = 16, 333, 460, 240
    cases = [_attention_case(rng, n0, heads, kv_heads, dim, vdim, page, dtype, window),
             _attention_case(rng, n1, heads, kv_heads, dim, vdim, page, dtype, window, start=start1)]
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
    gate = rng.normal(0, 1.5, (n, heads * vdim))
    for wide in (True, False):
        expected = np.concatenate([_attend(cases[0][0], cases[0][1], cases[0][2], gate[:n0], 0.3, 4.0, window, 0, wide),
                                   _attend(cases[1][0][start1:], cases[1][1], cases[1][2], gate[n0:], 0.3, 4.0, window, start1, wide)])
        out = torch.full((n, heads * vdim), float("nan"), dtype=dtype, device="cuda")
        ops.capped_attention(out, dev(q.reshape(n, -1), dtype), k_pages, v_pages, table, positions, items, heads, kv_heads, dim, vdim, page, 0.3,
                             4.0, window, tiled=True, gate=dev(gate), gate_wide=wide, slopes=dev(plain.slopes(heads)))
        np.testing.assert_allclose(out.float().cpu().numpy(), expected, atol=2e-5 if dtype == torch.float32 else 0.02)


@pytest.mark.parametrize("dim, vdim", [(64, 64), (64, 80), (16, 24), (128, 40), (8, 256), (72, 8)])
@pytest.mark.parametrize("window", [1, 70, 150, 400])
def test_split_attention_with_a_bias_by_distance_and_a_gate(dim, vdim, window):
    """Single tokens over split keys (bfloat16): requests of different lengths, values of another size than the keys."""
    from mini_llm_b200.kernels import ops
    rng = np.random.default_rng(dim + window)
    heads, kv_heads, n, page = 4, 2, 300, 16
    lasts = (300, 1, 21, 65, 299)
    cases = {last: _attention_case(rng, last, heads, kv_heads, dim, vdim, page, torch.bfloat16, window, start=last - 1) for last in lasts}
    k_pages, v_pages = torch.cat([cases[l][3] for l in lasts]), torch.cat([cases[l][4] for l in lasts])
    table, shift = torch.zeros((len(lasts), -(-n // page)), dtype=torch.int32, device="cuda"), 0
    for i, last in enumerate(lasts):
        table[i, :cases[last][5].shape[1]] = cases[last][5][0] + shift
        shift += cases[last][3].shape[0]
    q = np.stack([cases[last][0][last - 1] for last in lasts])
    gate = rng.normal(0, 1.5, (len(lasts), heads * vdim))
    chunk = 64
    max_chunks = -(-min(table.shape[1] * page, window) // chunk)
    row = ops.split_attention_row(dim, vdim)
    cells = len(lasts) * heads * max_chunks
    acc, ml = torch.empty(cells * row, device="cuda"), torch.empty(cells * 2, device="cuda")
    counters = torch.zeros(len(lasts) * heads, dtype=torch.int32, device="cuda")
    for wide in (True, False):
        expected = np.concatenate([_attend(cases[l][0][l - 1:], cases[l][1], cases[l][2], gate[i:i + 1], 0.3, 4.0, window, l - 1, wide)
                                   for i, l in enumerate(lasts)])
        out = torch.full((len(lasts), heads * vdim), float("nan"), dtype=torch.bfloat16, device="cuda")
        ops.split_attention(out, dev(q.reshape(len(lasts), -1), torch.bfloat16), k_pages, v_pages, table, dev([l - 1 for l in lasts], torch.int32),
                            dev(range(len(lasts)), torch.int32), heads, kv_heads, dim, page, 0.3, window, chunk, max_chunks, acc, ml, counters,
                            cap=4.0, value_size=vdim, gate=dev(gate), gate_wide=wide, slopes=dev(plain.slopes(heads)))
        np.testing.assert_allclose(out.float().cpu().numpy(), expected, atol=0.02)
        assert int(counters.abs().sum()) == 0


@pytest.mark.parametrize("experts, top, groups, shared", [(6, 2, (3, 2), True), (5, 3, None, True), (72, 5, (9, 2), False), (8, 8, (4, 4), True),
                                                         (5, 2, (5, 2), False), (40, 4, (2, 1), True)])
def test_router_with_groups_and_clamped_experts(experts, top, groups, shared):
    """Sigmoid scores ranked with a correction of both signs within the best groups, and both ways through the experts
    (pair by pair, and all at once) with a limit for the routed ones and another for the shared one."""
    from mini_llm_b200.kernels import ops
    rng = np.random.default_rng(experts)
    n, width, inner, shared_inner = 9, 40, 16, 24
    limits = (0.6, 0.35)
    pairs = top + int(shared)
    x, router, correction = rng.normal(0, 1, (n, width)), rng.normal(0, 0.4, (experts, width)), rng.normal(-0.6, 0.5, experts)
    shared_gate = rng.normal(0, 0.3, (1, width))
    w = {}
    sizes = [inner] * experts + ([shared_inner] if shared else [])
    for e, size in enumerate(sizes):
        w[f"e{e}.gate"], w[f"e{e}.up"] = rng.normal(0, 0.3, (size, width)), rng.normal(0, 0.3, (size, width))
        w[f"e{e}.down"] = rng.normal(0, 0.3, (width, size))
    before = rng.normal(0, 1, (n, width))
    choice = torch.zeros(n * pairs, dtype=torch.int32, device="cuda")
    in_weight, out_weight = torch.zeros(n * pairs, device="cuda"), torch.zeros(n * pairs, device="cuda")
    ops.route(dev(x), dev(router), dev(shared_gate) if shared else None, top, choice, in_weight, out_weight, rule="sigmoid",
              correction=dev(correction), groups=groups[0] if groups else 0, keep_groups=groups[1] if groups else 0)
    expected = np.zeros((n, width))
    how = {"top": top, **({"groups": {"count": groups[0], "keep": groups[1]}} if groups else {})}
    for t in range(n):
        chosen, weights = plain.choose(x[t] @ router.T, correction, how)
        assert choice[t * pairs:t * pairs + top].tolist() == chosen.tolist()
        np.testing.assert_allclose(out_weight[t * pairs:t * pairs + top].cpu().numpy(), weights, atol=2e-6)
        for e, g in zip(chosen, weights):
            expected[t] += g * plain.expert(x[t], w, f"e{e}", limits[0])
        if shared:
            expected[t] += plain.sigmoid(shared_gate[0] @ x[t]) * plain.expert(x[t], w, f"e{experts}", limits[1])
    total, starts = sum(sizes), np.concatenate([[0], np.cumsum(sizes)[:-1]])
    up_matrix = dev(np.concatenate([w[f"e{e}.{which}"] for which in ("gate", "up") for e in range(len(sizes))]))
    down_matrix = dev(np.concatenate([w[f"e{e}.down"] for e in range(len(sizes))], axis=1))

    def table(base, offsets):
        return torch.tensor([base + 4 * int(o) for o in offsets], dtype=torch.int64, device="cuda")
    gate_of, up_of = table(up_matrix.data_ptr(), starts * width), table(up_matrix.data_ptr(), (total + starts) * width)
    down_of, inner_of = table(down_matrix.data_ptr(), starts), dev(sizes, torch.int32)
    form = dict(form="clamped_glu", limit=limits[0], shared_limit=limits[1], alpha=1.702)
    for assign in (False, True):
        hidden, act = dev(before), torch.full((n * pairs, max(sizes)), float("nan"), device="cuda")
        ops.experts(hidden, act, dev(x), choice, in_weight, out_weight, gate_of, up_of, down_of, inner_of, max(sizes), pairs, ld_down=total,
                    assign=assign, n_experts=experts, **form)
        np.testing.assert_allclose(hidden.cpu().numpy(), expected + (0.0 if assign else before), atol=3e-5)
    gu = (dev(x).double() @ up_matrix.double().T).float().contiguous()
    combined = torch.full((n, total), float("nan"), device="cuda")
    ops.expert_combine(combined, gu, choice, in_weight, out_weight, experts, inner, top, pairs, **form)
    result = combined.cpu().numpy().astype(np.float64) @ down_matrix.cpu().numpy().astype(np.float64).T
    np.testing.assert_allclose(result, expected, atol=2e-4)


@pytest.mark.parametrize("n, dim, width", [(1, 16, 64), (7, 5, 33), (40, 24, 128), (64, 8, 200)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_token_gate_kernels(n, dim, width, dtype):
    from mini_llm_b200.kernels import ops
    rng = np.random.default_rng(n)
    x, w, side = rng.normal(0, 1, (n, width)), rng.normal(0, 0.1, (dim, width)), rng.normal(0, 1, (31, 3 * dim))
    if dtype == torch.bfloat16:
        w, side = (kp.to_bfloat16_values(a).astype(np.float64) for a in (w, side))
    ids = rng.integers(0, 31, n)
    for index in range(3):
        expected = plain.gelu_tanh(x @ w.T) * side[ids][:, index * dim:(index + 1) * dim]
        out, again = (torch.full((n, dim), float("nan"), dtype=dtype, device="cuda") for _ in range(2))
        ops.token_gate(out, dev(x), dev(w, dtype), dev(side, dtype), dev(ids, torch.int32), index * dim)
        ops.token_gate_rows(again, dev(x @ w.T), dev(side, dtype), dev(ids, torch.int32), index * dim)
        for got in (out, again):
            np.testing.assert_allclose(got.float().cpu().numpy(), expected, atol=1e-5 if dtype == torch.float32 else 0.01 * np.abs(expected).max())


@pytest.mark.parametrize("n, width", [(3, 64), (5, 33), (9, 2048), (2, 5000)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_add_normed_norm_kernel(n, width, dtype):
    from mini_llm_b200.kernels import ops
    rng = np.random.default_rng(width)
    hidden, y = rng.normal(0, 3, (n, width)), rng.normal(0, 0.2, (n, width))
    gain, next_gain = rng.uniform(0.5, 1.5, width), rng.uniform(0.5, 1.5, width)
    stream, normed = dev(hidden), torch.full((n, width), float("nan"), dtype=dtype, device="cuda")
    ops.add_normed_norm(stream, dev(y), dev(gain), 1e-3, normed, dev(next_gain), 1e-5)
    expected = hidden + plain.rms_norm(y, gain, 1e-3)
    np.testing.assert_allclose(stream.cpu().numpy(), expected, atol=2e-5)
    np.testing.assert_allclose(normed.float().cpu().numpy(), plain.rms_norm(expected, next_gain, 1e-5), atol=1e-5 if dtype == torch.float32 else 0.03)
