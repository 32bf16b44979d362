"""The Sefelorn decoder inside the engine against the plain float64 implementation (tests/plain_sefelorn.py).

Every mechanism alone (one-layer models), whole prompts against token-by-token decoding, portions down to two tokens,
mixed batches against each request alone, pages and state slots that are freed and used again, keys just inside and just
outside every window and just kept or not kept at a sequence's start, in prompts and in decoding, far keys and page
borders with peaked attention, states that last, the first tokens of a sequence, long decoding, requests that outgrow the
cache pool, several sizes, the residual stream layer by layer, greedy generation through the scheduler, the command line,
and the new kernels against torch.
"""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import plain_sefelorn as P
import sefelorn_models as M
from helpers import ROOT

pytestmark = pytest.mark.gpu

TOL = {"float32": 2e-5, "bfloat16": 4e-2}         # max |difference| / max |reference logit|
# With peaked attention a rounding of a score moves the weights of the keys by as much more, and a state that lasts
# for hundreds of tokens adds up as many roundings.
TOL_SHARP = {"float32": 1.5e-3, "bfloat16": 8e-2}
SHARP = {"float32": 1.0, "bfloat16": 0.5}         # the bfloat16 engine rounds keys to 8 bits: half the sharpening
DTYPES = ["float32", "bfloat16"]


def rel_err(got, ref):
    ref = np.asarray(ref, dtype=np.float64)
    return float(np.max(np.abs(np.asarray(got, dtype=np.float64) - ref)) / np.max(np.abs(ref)))


def runner_for(path, dtype, page_size=16, pool_tokens=1024, max_seqs=4, max_batch_tokens=1024):
    from rustingstrata_b200.config import EngineConfig
    from rustingstrata_b200.engine import ModelRunner
    eng = EngineConfig(dtype=dtype, page_size=page_size, num_pages=(pool_tokens + page_size - 1) // page_size,
                       max_seqs=max_seqs, max_batch_tokens=max_batch_tokens, max_logit_rows=max_batch_tokens)
    return ModelRunner.from_dir(path, eng)


def tokens_for(cfg, n, seed):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], size=n).tolist()


def plain_logits(cfg, w, toks):
    return P.forward(toks, w, cfg).numpy()


_MODELS = {}


def model(tmp_path_factory, key, cfg, seed=0, sharp=0.0):
    key = f"{key}_{sharp}"
    if key not in _MODELS:
        path = str(tmp_path_factory.mktemp("sefelorn") / key)
        _MODELS[key] = (path,) + M.make(path, cfg, seed, sharp)
    return _MODELS[key]


def assert_rows_within(err, tol, what):
    """Per-position errors of a run with sharpened weights: none beyond one and a half times the tolerance and at most
    one position in fifty beyond the tolerance itself (where a query weighs two keys nearly alike, the rounding of a
    score tips the balance; a fault of a mask, a page or a state moves whole stretches of positions by far more)."""
    err = np.asarray(err)
    over = err > tol
    first = int(np.argmax(over)) if over.any() else -1
    assert err.max() <= 1.5 * tol and over.sum() <= max(1, 0.02 * len(err)), \
        f"{what}: worst {err.max():.3e}, {int(over.sum())} of {len(err)} positions over {tol}, the first at {first}"


def step_all(r, rid, toks, want=None):
    from rustingstrata_b200.engine import StepEntry
    out = r.step([StepEntry(rid, toks, list(range(len(toks))) if want is None else want)])
    r.check_status()
    return None if out is None else out.cpu().numpy()


# ----------------------------------------------------------------------------- each mechanism alone
R1 = M.right(1, 8, 8, 4.0, 4)           # a small second mixer beside the attention under test
L1 = M.left(1, 1, 16, 16, 8, 2)
ONE_LAYER = {
    "window_grouped_rotated_prefix": M.config(97, 64, [(M.parallel(M.left(6, 3, 16, 8, 11, 4, rot=(8, 50.0)), R1), None)]),
    "window_one_kv_head_no_rotation_nothing_kept": M.config(97, 64, [(M.parallel(M.left(3, 1, 24, 40, 7, 0, scale=0.3), R1), None)]),
    "window_all_rotated_heads_equal": M.config(97, 72, [(M.parallel(M.left(2, 2, 12, 12, 16, 16, rot=(12, 1000.0)), R1), None)], eps=1e-5),
    "window_of_one_key": M.config(97, 64, [(M.parallel(M.left(1, 1, 32, 16, 1, 3, rot=(4, 7.0)), R1), None)]),
    "more_kept_than_the_window_holds": M.config(97, 64, [(M.parallel(M.left(2, 1, 16, 32, 4, 19, rot=(16, 1e4)), R1), None)]),
    "window_longer_than_the_prompt": M.config(97, 64, [(M.parallel(M.left(2, 2, 16, 16, 300, 9, rot=(16, 1e4)), R1), None)]),
    "linear_attention_rows_that_need_padding": M.config(97, 64, [(M.parallel(L1, M.right(3, 18, 20, 5.0, 6)), None)]),
    "linear_attention_two_column_blocks": M.config(97, 64, [(M.parallel(L1, M.right(2, 40, 36, 16.0, 16)), None)], eps=1e-5),
    "linear_attention_one_head_fast_decay": M.config(97, 64, [(M.parallel(L1, M.right(1, 8, 4, 0.5, 1), scales=(0.2, 2.0)), None)]),
    "linear_attention_wide_rows": M.config(97, 64, [(M.parallel(L1, M.right(1, 132, 40, 1.0, 5)), None)]),
    "mamba2_groups_and_parts": M.config(97, 64, [(M.mamba2(4, 16, 24, groups=2, conv=4, norm_groups=2), None)]),
    "mamba2_group_per_head_part_per_head": M.config(97, 64, [(M.mamba2(3, 8, 16, groups=3, conv=3, norm_groups=3), None)]),
    "mamba2_parts_across_heads": M.config(97, 64, [(M.mamba2(2, 12, 8, conv=2, norm_groups=3), None)]),
    "mamba2_one_tap_odd_sizes": M.config(97, 72, [(M.mamba2(3, 5, 21, conv=1, norm_groups=5), None)], eps=1e-5),
    "mamba2_wide_state": M.config(97, 64, [(M.mamba2(1, 40, 132, conv=6), None)]),
    "clamped_feed_forward": M.config(97, 64, [(M.mamba2(1, 8, 8), M.dense(120, 0.6))], logit_scale=0.3, embedding_scale=3.0),
    "clamped_feed_forward_wide_limit": M.config(97, 64, [(M.parallel(L1, R1), M.dense(56, 40.0))]),
    "loop_of_one_layer": M.config(97, 64, [(M.mamba2(2, 16, 16, conv=3), M.dense(64))], loop=(0, 1, 4), embedding_scale=0.3),
    "loop_at_the_end": M.config(97, 64, [(M.mamba2(2, 16, 16), None), (M.parallel(L1, R1), M.dense(40))], loop=(1, 2, 2)),
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(ONE_LAYER))
def test_mechanism_alone(tmp_path_factory, name, dtype):
    """A small model per mechanism: the stream after every layer run and the logits of a whole prompt, the same
    prompt in portions, and token by token."""
    from rustingstrata_b200.engine import StepEntry
    path, cfg, w = model(tmp_path_factory, "one_" + name, ONE_LAYER[name], seed=len(name))
    toks = tokens_for(cfg, 45, 3)
    streams = []
    ref = P.forward(toks, w, cfg, streams).numpy()
    r = runner_for(path, dtype, page_size=8, pool_tokens=256)
    got_streams = []
    kinds = [r.model.blocks[c.layer].kind for c in r.model.calls]
    logits = r.step([StepEntry("a", toks, list(range(len(toks))))],
                    on_layer=lambda k, x: got_streams.append(x.float().cpu().numpy().copy()) if kinds[k] != "stream_reentry" else None)
    r.check_status()
    assert len(got_streams) == len(streams)
    for i, (g, s) in enumerate(zip(got_streams, streams)):
        assert rel_err(g, s.numpy()) <= TOL[dtype], f"{name} {dtype}: stream after layer run {i}"
    assert rel_err(logits.cpu().numpy(), ref) <= TOL[dtype]
    r.release("a")
    got, pos = [], 0
    for n in [2, 5, 1, 2, 17, 3, 2, 13]:
        got.append(step_all(r, "b", toks[pos:pos + n]))
        pos += n
    assert pos == len(toks)
    assert rel_err(np.concatenate(got), ref) <= TOL[dtype], f"{name} {dtype}: portions"
    r.release("b")
    got = [step_all(r, "c", [t]) for t in toks]
    assert rel_err(np.concatenate(got), ref) <= TOL[dtype], f"{name} {dtype}: token by token"


# ----------------------------------------------------------------------------- whole models, every cutting
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["P", "Q", "R", "S"])
def test_cuttings_of_a_prompt(tmp_path_factory, name, dtype):
    """Whole, last tokens one by one (captured steps), portions of several sizes down to two tokens."""
    path, cfg, w = model(tmp_path_factory, name, name, seed=11)
    toks = tokens_for(cfg, 150, 5)
    ref = plain_logits(cfg, w, toks)
    r = runner_for(path, dtype, page_size=16, pool_tokens=512)
    assert rel_err(step_all(r, "w", toks), ref) <= TOL[dtype], "whole"
    r.release("w")
    n = len(toks) - 40
    got = [step_all(r, "d", toks[:n])] + [step_all(r, "d", [t]) for t in toks[n:]]
    assert rel_err(np.concatenate(got), ref) <= TOL[dtype], "decoding"
    if r.model.capturable:
        assert r.graph_replays > 0
    r.release("d")
    got, pos, k = [], 0, 0
    sizes = [7, 2, 13, 2, 5, 3, 29, 2, 16, 4, 11, 2, 1, 1, 31]
    while pos < len(toks):
        m = min(sizes[k % len(sizes)], len(toks) - pos)
        got.append(step_all(r, "p", toks[pos:pos + m]))
        pos, k = pos + m, k + 1
    assert rel_err(np.concatenate(got), ref) <= TOL[dtype], "portions"


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["P", "R"])
def test_mixed_batches_with_pages_and_slots_used_again(tmp_path_factory, name, dtype):
    """Up to three live requests of unequal length in a pool that cannot hold all seven at once: portions of some
    beside single tokens of others, requests left out of steps, and every row equal to the request run alone.  A slot
    that a request with a long-lived state has left is taken by the next one, which must start from zero."""
    from rustingstrata_b200.engine import StepEntry
    path, cfg, w = model(tmp_path_factory, name + "_sharp", name, seed=21, sharp=SHARP[dtype])
    tol = TOL_SHARP[dtype]
    lengths = [70, 33, 121, 9, 64, 1, 47]
    toks = {f"r{i}": tokens_for(cfg, n, 40 + i) for i, n in enumerate(lengths)}
    ref = {k: plain_logits(cfg, w, t) for k, t in toks.items()}
    scale = max(np.max(np.abs(v)) for v in ref.values())      # one scale for all requests: a one-token request has no spread of its own
    r = runner_for(path, dtype, page_size=16, pool_tokens=256, max_seqs=3)
    rng = np.random.default_rng(9)
    waiting, live, pos = list(toks), [], {}
    worst, rows, slots_seen, errs = 0.0, 0, {}, []
    while waiting or live:
        while waiting and len(live) < 3 and sum((len(toks[x]) + 15) // 16 for x in live + [waiting[0]]) <= 16:
            live.append(waiting.pop(0))
            pos[live[-1]] = 0
        chosen = [x for x in live if rng.random() < 0.7] or [live[0]]
        entries, where = [], []
        for rid in chosen:
            left = len(toks[rid]) - pos[rid]
            n = 1 if left <= 12 else int(min(rng.choice([2, 3, 5, 9, 17, 31]), left - 12))
            want = list(range(n))
            entries.append(StepEntry(rid, toks[rid][pos[rid]:pos[rid] + n], want))
            where += [(rid, pos[rid] + j) for j in want]
            pos[rid] += n
        out = r.step(entries).cpu().numpy()
        r.check_status()
        for rid in chosen:
            slots_seen.setdefault(r.cache.slot(rid), set()).add(rid)
        for row, (rid, p) in zip(out, where):
            e = float(np.max(np.abs(row - ref[rid][p])) / scale)
            worst, rows = max(worst, e), rows + 1
            errs.append(e)
            assert e <= 1.5 * tol, f"{name} {dtype}: request {rid} position {p}: {e:.3e}"
        for rid in [x for x in live if pos[x] == len(toks[x])]:
            live.remove(rid)
            r.release(rid)
    r.cache.check()
    assert rows == sum(lengths)
    assert_rows_within(errs, tol, "mixed batches")
    print(f"mixed {name} {dtype}: worst {worst:.3e}")
    assert max(len(v) for v in slots_seen.values()) >= 2, "no state slot was used again"
    assert all(p.reuses > 0 for p in r.cache.pools), "no page was used again"


# ----------------------------------------------------------------------------- edges of windows and kept first tokens
EDGE_TOL = {"float32": 1.5e-4, "bfloat16": 2e-2}   # root mean square over the vocabulary, over that of the reference


def row_rms(d):
    d = d - d.mean(axis=1, keepdims=True)
    return np.sqrt((d * d).mean(axis=1))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["P", "R", "S"])
def test_edges_of_windows_and_kept_tokens(tmp_path_factory, name, dtype):
    """Peaked attention, so that a key more or a key less shows.  The premise first, on the plain implementation: with
    every window one key larger or smaller, or one first token more or less kept, the logits of several positions move by
    more than twice the tolerance.  Then the engine: the prompt whole, a short prompt followed by single tokens that pass
    every window's edge and the kept tokens' edge, and portions that start and end on and beside them."""
    path, cfg, w = model(tmp_path_factory, name + "_sharp", name, seed=21, sharp=SHARP[dtype])
    tol = EDGE_TOL[dtype]
    n = {"P": 150, "R": 330, "S": 120}[name]
    toks = tokens_for(cfg, n, 31)
    ref = plain_logits(cfg, w, toks)
    scale = row_rms(ref).mean()
    for size, keep in ((1, 0), (-1, 0), (0, 1), (0, -1)):
        if size < 0 and any(L["mixer"]["left"]["mask"]["size"] == 1 for L in cfg["layers"] if L["type"] == "parallel"):
            continue
        moved = row_rms(plain_logits(M.with_masks(cfg, size, keep), w, toks) - ref) / scale
        assert (moved > 2 * tol).sum() >= 5, f"premise: windows {size:+d}, kept {keep:+d}"
    r = runner_for(path, dtype, page_size=16, pool_tokens=512, max_batch_tokens=512)
    assert_rows_within(row_rms(step_all(r, "w", toks) - ref) / scale, tol, "whole")
    r.release("w")
    got = [step_all(r, "d", toks[:3])] + [step_all(r, "d", [t]) for t in toks[3:]]
    assert_rows_within(row_rms(np.concatenate(got) - ref) / scale, tol, "decoding")
    r.release("d")
    edges = {p + d for L in cfg["layers"] if L["type"] == "parallel" for e in L["mixer"]["left"]["mask"].values()
             for p in range(e, n, max(e, 16)) for d in (-1, 0, 1)}
    marks = sorted({0, n} | {p for p in edges if 0 < p < n})
    got = [step_all(r, "p", toks[a:b]) for a, b in zip(marks[:-1], marks[1:])]
    assert_rows_within(row_rms(np.concatenate(got) - ref) / scale, tol, "portions cut at the edges")


@pytest.mark.parametrize("dtype", DTYPES)
def test_far_keys_page_borders_and_long_state(tmp_path_factory, dtype):
    """A window wider than the sequence, peaked attention (each query looks at one or two keys, at any distance) and states
    that last for hundreds of tokens, over 700 positions: every position of the prompt, then decoding across page borders
    and the borders of the attention's key tiles, against the plain implementation."""
    path, cfg, w = model(tmp_path_factory, "R_far", M.with_masks(M.CONFIGS["R"], 900), seed=21, sharp=SHARP[dtype])
    toks = tokens_for(cfg, 700, 77)
    ref = plain_logits(cfg, w, toks)
    r = runner_for(path, dtype, page_size=16, pool_tokens=768, max_batch_tokens=768)
    n = 600
    got = [step_all(r, "a", toks[:n])] + [step_all(r, "a", [t]) for t in toks[n:n + 60]] + [step_all(r, "a", toks[n + 60:])]
    err = np.max(np.abs(np.concatenate(got) - ref), axis=1) / np.max(np.abs(ref))
    print(f"far keys {dtype}: worst {err.max():.3e}")
    assert_rows_within(err, TOL_SHARP[dtype], "far keys")


def test_sharp_weights_look_far_back_and_keep_state():
    """The premises of the tests with sharp weights, checked on the plain implementation: dropping the oldest 100 tokens
    changes the last logits by more than twice the widest tolerance (so a lost far key would show in either engine), and
    each recurrent mixer alone still feels tokens 200 back by ten times the 32-bit engine's tolerance."""
    cfg = M.with_masks(M.CONFIGS["R"], 900)
    w = M.draw_weights(cfg, 21, sharp=0.5)
    toks = tokens_for(cfg, 700, 77)
    full, cut = plain_logits(cfg, w, toks)[-20:], plain_logits(cfg, w, toks[100:])[-20:]
    assert np.max(np.abs(full - cut)) / np.max(np.abs(full)) > 2 * TOL_SHARP["bfloat16"]
    for key in ("linear_attention_two_column_blocks", "mamba2_groups_and_parts"):
        c1 = ONE_LAYER[key]
        w1 = M.draw_weights(c1, 5, sharp=1.0)
        t1 = tokens_for(c1, 400, 9)
        w1 = {k: torch.zeros_like(v) if k.endswith("left.o") else v for k, v in w1.items()}      # the recurrence alone
        a, b = plain_logits(c1, w1, t1)[-5:], plain_logits(c1, w1, t1[200:])[-5:]
        assert np.max(np.abs(a - b)) / np.max(np.abs(a)) > 10 * TOL_SHARP["float32"], key


@pytest.mark.parametrize("dtype", DTYPES)
def test_first_tokens_and_short_sequences(tmp_path_factory, dtype):
    """Sequences shorter than the convolutions' taps, single-token prompts, and a first step of one token beside
    longer ones in the same batch; then each grows token by token past the taps."""
    from rustingstrata_b200.engine import StepEntry
    path, cfg, w = model(tmp_path_factory, "R", "R", seed=11)
    r = runner_for(path, dtype, page_size=16, pool_tokens=256)
    seqs = {"one": tokens_for(cfg, 1, 1), "two": tokens_for(cfg, 2, 2), "three": tokens_for(cfg, 3, 3), "ten": tokens_for(cfg, 10, 4)}
    out = r.step([StepEntry(k, t, list(range(len(t)))) for k, t in seqs.items()]).cpu().numpy()
    r.check_status()
    at = 0
    for k, t in seqs.items():
        assert rel_err(out[at:at + len(t)], plain_logits(cfg, w, t)) <= TOL[dtype], k
        at += len(t)
    for _ in range(4):
        for k in seqs:
            seqs[k] = seqs[k] + tokens_for(cfg, 1, len(seqs[k]) + 50)
        out = r.step([StepEntry(k, t[-1:], [0]) for k, t in seqs.items()]).cpu().numpy()
        for row, (k, t) in zip(out, seqs.items()):
            assert rel_err(row, plain_logits(cfg, w, t)[-1]) <= TOL[dtype], k


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding(tmp_path_factory, dtype):
    """300 tokens one by one after a short prompt (replayed graphs, pages taken as it goes, states that last)."""
    path, cfg, w = model(tmp_path_factory, "P_sharp", "P", seed=21, sharp=SHARP[dtype])
    toks = tokens_for(cfg, 320, 8)
    ref = plain_logits(cfg, w, toks)
    r = runner_for(path, dtype, page_size=8, pool_tokens=384)
    got = [step_all(r, "a", toks[:20])] + [step_all(r, "a", [t]) for t in toks[20:]]
    err = np.max(np.abs(np.concatenate(got) - ref), axis=1) / np.max(np.abs(ref))
    print(f"long decoding {dtype}: worst {err.max():.3e}")
    assert_rows_within(err, TOL_SHARP[dtype], "long decoding")


@pytest.mark.parametrize("dtype", DTYPES)
def test_requests_that_outgrow_the_pool(tmp_path_factory, dtype):
    """Every layer's attention is windowed, so a request may hold more tokens than the cache pool: 400 tokens in a pool of
    128, two requests side by side, pages of the passed window taken again while the kept first ones stay."""
    from rustingstrata_b200.engine import StepEntry
    path, cfg, w = model(tmp_path_factory, "S", "S", seed=11)
    a, b = tokens_for(cfg, 400, 5), tokens_for(cfg, 300, 6)
    ra, rb = plain_logits(cfg, w, a), plain_logits(cfg, w, b)
    r = runner_for(path, dtype, page_size=8, pool_tokens=128 + 64, max_batch_tokens=64)
    at, got_a, got_b = 0, [], []
    while at < 400:
        n = min(17 if at < 200 else 1, 400 - at)
        entries = [StepEntry("a", a[at:at + n], list(range(n)))]
        m = min(n, 300 - at)
        if m > 0:
            entries.append(StepEntry("b", b[at:at + m], list(range(m))))
        out = r.step(entries).cpu().numpy()
        r.check_status()
        got_a.append(out[:n])
        got_b.append(out[n:])
        at += n
    assert rel_err(np.concatenate(got_a), ra) <= TOL[dtype] and rel_err(np.concatenate(got_b), rb) <= TOL[dtype]
    r.cache.check()
    assert all(p.reuses > 0 for p in r.cache.pools)


WIDE = {
    # 15 query heads over 5 kv heads with heads of 96 / 128, a window over several key tiles, state heads of 128 x 128,
    # widths that reach the 128 x 128 tiles of the tensor-core products
    "wide_heads": M.config(500, 512, [(M.parallel(M.left(15, 5, 96, 128, 150, 40, rot=(32, 1e5)), M.right(4, 128, 128, 16.0, 16)), M.dense(1024)),
                                      (M.mamba2(8, 64, 128, groups=2, conv=4), M.dense(768))], eps=1e-5, loop=(0, 2, 2)),
    # many small heads, state heads wider than they are tall, a norm part per head
    "many_heads": M.config(300, 256, [(M.parallel(M.left(32, 32, 16, 16, 70, 33, rot=(16, 1e4)), M.right(16, 16, 96, 8.0, 8)), None),
                                      (M.mamba2(16, 48, 16, groups=1, conv=3, norm_groups=16), M.dense(384))]),
    # single query heads of 256: the CUDA-core attention in both engines; state heads of 256 rows
    "heads_of_256": M.config(300, 256, [(M.parallel(M.left(2, 1, 256, 256, 90, 7, rot=(128, 1e4)), M.right(2, 256, 64, 16.0, 32)), M.dense(264)),
                                        (M.mamba2(2, 96, 256, conv=2), None)]),
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(WIDE))
def test_wider_shapes_and_long_portions(tmp_path_factory, name, dtype):
    """A portion of 500 tokens, 30 single tokens, a portion of 110: the forms of the kernels that only large steps and
    wide heads reach."""
    path, cfg, w = model(tmp_path_factory, "wide_" + name, WIDE[name], seed=7)
    toks = tokens_for(cfg, 640, 3)
    ref = plain_logits(cfg, w, toks)
    r = runner_for(path, dtype, page_size=16, pool_tokens=768, max_batch_tokens=768)
    got = [step_all(r, "a", toks[:500])] + [step_all(r, "a", [t]) for t in toks[500:530]] + [step_all(r, "a", toks[530:])]
    err = np.max(np.abs(np.concatenate(got) - ref), axis=1) / np.max(np.abs(ref))
    print(f"wide {name} {dtype}: worst {err.max():.3e}")
    assert err.max() <= TOL[dtype], f"first wrong position {int(np.argmax(err > TOL[dtype]))}"


# ----------------------------------------------------------------------------- the engine's own entry points
@pytest.mark.parametrize("chunk", [None, 7])
def test_greedy_generation_through_the_scheduler(tmp_path_factory, chunk):
    """Engine.generate (scheduler, admission, prompt portions of 7 tokens, decode steps launched ahead) gives the plain
    implementation's greedy tokens in 32-bit, for several prompts of unequal length at once."""
    from rustingstrata_b200 import Engine
    path, cfg, w = model(tmp_path_factory, "P", "P", seed=11)
    prompts = [tokens_for(cfg, n, 60 + n) for n in (5, 23, 1, 40)]
    want = []
    for p in prompts:
        seq = list(p)
        for _ in range(12):
            seq.append(int(np.argmax(plain_logits(cfg, w, seq)[-1])))
        want.append(seq[len(p):])
    eng = Engine(path, dtype="float32", page_size=8, max_tokens=512, max_batch_tokens=64, max_seqs=4, prefill_chunk=chunk)
    assert eng.generate(prompts, max_new_tokens=12) == want
    # and once more through the same engine: slots and pages of the finished requests are taken again
    assert eng.generate(prompts[::-1], max_new_tokens=12) == want[::-1]


def test_generation_without_any_cache(tmp_path_factory):
    """A model of state mixers only keeps no pages at all: the scheduler admits and decodes by slots alone."""
    from rustingstrata_b200 import Engine
    path, cfg, w = model(tmp_path_factory, "one_mamba2_groups_and_parts", ONE_LAYER["mamba2_groups_and_parts"], seed=5)
    prompts = [tokens_for(cfg, n, 60 + n) for n in (5, 40, 1)]
    want = []
    for p in prompts:
        seq = list(p)
        for _ in range(8):
            seq.append(int(np.argmax(plain_logits(cfg, w, seq)[-1])))
        want.append(seq[len(p):])
    eng = Engine(path, dtype="float32", page_size=8, max_tokens=64, max_batch_tokens=32, max_seqs=2, prefill_chunk=16)
    assert eng.generate(prompts, max_new_tokens=8) == want


def test_bfloat16_generation_picks_top_tokens(tmp_path_factory):
    from rustingstrata_b200 import Engine
    path, cfg, w = model(tmp_path_factory, "R", "R", seed=11)
    prompt = tokens_for(cfg, 30, 2)
    eng = Engine(path, dtype="bfloat16", page_size=16, max_tokens=256, max_batch_tokens=64, max_seqs=2)
    got = eng.generate(prompt, max_new_tokens=10)
    logits = plain_logits(cfg, w, prompt + got)
    for i, t in enumerate(got):
        row = logits[len(prompt) - 1 + i]
        assert row[t] >= row.max() - 0.08 * np.abs(logits).max()


def read_model_folder(folder):
    """A safetensors file read by hand: name → float64 tensor."""
    import struct
    with open(os.path.join(folder, "model.safetensors"), "rb") as f:
        n = struct.unpack("<Q", f.read(8))[0]
        header = json.loads(f.read(n))
        blob = f.read()
    out = {}
    for name, ent in header.items():
        if name == "__metadata__":
            continue
        lo, hi = ent["data_offsets"]
        bits = np.frombuffer(blob[lo:hi], dtype=np.uint16).astype(np.uint32) << 16
        out[name] = torch.from_numpy(bits.view(np.float32).astype(np.float64)).reshape(ent["shape"])
    return out


def test_trace_replay_and_command_line(tmp_path_factory, tmp_path):
    """bin/trace_run on a model folder (logits of a request cut in two steps beside a second request), and
    ``init-random`` + ``generate`` of the package's command line for this architecture."""
    path, cfg, w = model(tmp_path_factory, "Q", "Q", seed=11)
    toks = tokens_for(cfg, 40, 1)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": toks[:25], "want": [0, 24]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": toks[25:], "want": [14]}, {"id": "y", "tokens": toks[:3], "want": [2]}],
              "end": ["x", "y"]}]
    out = tmp_path / "out"
    res = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", path, "--dtype", "float32",
                          "--out", str(out), "--max-tokens", "128"], input="".join(json.dumps(s) + "\n" for s in steps),
                         capture_output=True, text=True, timeout=600)
    assert res.returncode == 0, res.stderr[-2000:]
    assert [ln for ln in res.stdout.splitlines() if ln.startswith("done")] == ["done 0", "done 1"]
    ref = plain_logits(cfg, w, toks)
    a = np.fromfile(out / "0.f32", dtype="<f4").reshape(2, cfg["vocab"])
    b = np.fromfile(out / "1.f32", dtype="<f4").reshape(2, cfg["vocab"])
    assert rel_err(a, ref[[0, 24]]) <= TOL["float32"] and rel_err(b, ref[[39, 2]]) <= TOL["float32"]
    cfg_path = tmp_path / "config.json"
    cfg_path.write_text(json.dumps(M.CONFIGS["P"]))
    made = tmp_path / "made"
    cli = [sys.executable, "-m", "rustingstrata_b200"]
    env = dict(os.environ, PYTHONPATH=ROOT)
    r1 = subprocess.run(cli + ["init-random", "--config", str(cfg_path), "--out", str(made), "--seed", "3"],
                        capture_output=True, text=True, timeout=600, env=env)
    assert r1.returncode == 0, r1.stderr[-2000:]
    r2 = subprocess.run(cli + ["generate", "--model", str(made), "--prompt", "1,2,3,4", "-n", "6", "--dtype", "float32"],
                        capture_output=True, text=True, timeout=600, env=env)
    assert r2.returncode == 0, r2.stderr[-2000:]
    # the folder it wrote, read by this file's own reader, generates the same tokens in the plain implementation
    w2 = read_model_folder(str(made))
    seq = [1, 2, 3, 4]
    for _ in range(6):
        seq.append(int(np.argmax(plain_logits(M.CONFIGS["P"], w2, seq)[-1])))
    assert ",".join(str(t) for t in seq[4:]) in r2.stdout.replace(" ", "") or " ".join(str(t) for t in seq[4:]) in r2.stdout, r2.stdout


# ----------------------------------------------------------------------------- kernels alone
@pytest.mark.parametrize("rows", [3, 8, 40, 200])
@pytest.mark.parametrize("shape", [(256, 320), (72, 40)])
def test_clamped_gate_in_every_product(rows, shape):
    """act(gate) * up as the epilogue of the bfloat16 products (skinny, stream-K, tiled) and as a pass of its own, against
    torch, with values on both sides of the limit."""
    from rustingstrata_b200.kernels import ops
    K, I = shape
    g = torch.Generator().manual_seed(rows)
    a = torch.randn(rows, K, generator=g).to(torch.bfloat16).cuda()
    gate, up = (torch.randn(I, K, generator=g).mul(K ** -0.5 * 2).to(torch.bfloat16).cuda() for _ in range(2))
    w = torch.stack([gate, up], dim=1).reshape(2 * I, K).contiguous()
    alpha, limit = 1.3, 0.9
    G, U = a.float() @ gate.float().T, a.float() @ up.float().T
    assert (G > limit).any() and (U > limit).any() and (U < -limit).any()
    Gc, Uc = G.clamp(max=limit), U.clamp(-limit, limit)
    ref = Gc * torch.sigmoid(alpha * Gc) * (Uc + 1)
    out = torch.empty(rows, I, dtype=torch.bfloat16, device="cuda")
    ops.linear_swiglu(a, w, out, rows, activation="clamped", gate=(alpha, limit))
    assert (out.float() - ref).abs().max() <= 2e-2
    both = torch.cat([G, U], dim=1).contiguous()
    f = torch.empty(rows, I, device="cuda")
    ops.silu_mul(both, f, rows, "clamped", (alpha, limit))
    assert (f - ref).abs().max() <= 1e-5


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("n", [96, 100, 1024, 4096, 5000])
def test_two_norms_of_a_row_are_the_two_kernels(n, dtype):
    """The pair form gives the bits of two single norms, also when it settles a product's owed sum on the way."""
    from rustingstrata_b200.kernels import ops
    g = torch.Generator().manual_seed(n)
    x = torch.randn(5, n, generator=g).cuda()
    w1, w2 = (torch.randn(n, generator=g).to(torch.bfloat16).cuda() for _ in range(2))
    a, b, c, d = (torch.empty(5, n, dtype=dtype, device="cuda") for _ in range(4))
    ops.rmsnorm(x, w1, 1e-6, a)
    ops.rmsnorm(x, w2, 1e-6, b)
    ops.rmsnorm(x, w1, 1e-6, c, weight2=w2, out2=d)
    assert torch.equal(a, c) and torch.equal(b, d)
    if dtype == torch.bfloat16 and n % 8 == 0:
        h = torch.randn(5, 512, generator=g).to(torch.bfloat16).cuda()
        m = torch.randn(n, 512, generator=g).mul(0.05).to(torch.bfloat16).cuda()
        y, z = x.clone(), x.clone()
        ops.linear(h, m, y, 5, accumulate=True)
        ops.rmsnorm(y, w1, 1e-6, a)
        ops.rmsnorm(y, w2, 1e-6, b)
        owed = ops.linear(h, m, z, 5, accumulate=True, may_defer=True)
        assert owed is not None
        ops.rmsnorm(z, w1, 1e-6, c, pending=owed, weight2=w2, out2=d)
        assert torch.equal(y, z) and torch.equal(a, c) and torch.equal(b, d)


@pytest.mark.parametrize("tau", [0.25, 1.0, 16.0])
@pytest.mark.parametrize("shape", [(3, 20, 20, 7), (2, 18, 32, 5), (4, 128, 128, 16)])
def test_low_rank_decay(shape, tau):
    """sigmoid(W u + b)^(1 / tau) over many magnitudes of the argument, padding zero, against float64."""
    from rustingstrata_b200.kernels import ops
    H, dim, rows, rank = shape
    g = torch.Generator().manual_seed(dim)
    T = 37
    u = torch.randn(T, rank + 3, generator=g).cuda()[:, :rank] * 4.0
    w = torch.randn(H * dim, rank, generator=g).to(torch.bfloat16).cuda()
    b = (10 * torch.randn(H * dim, generator=g)).cuda()
    out = torch.full((T, H * rows), 7.0, device="cuda")
    ops.low_rank_decay(u, w, b, tau, out, H, dim, rows, T)
    z = u.double() @ w.double().T + b.double()
    ref = torch.exp(torch.nn.functional.logsigmoid(z) / tau).view(T, H, dim)
    got = out.view(T, H, rows).double()
    assert (got[:, :, dim:] == 0).all()
    assert ((got[:, :, :dim] - ref).abs() / (ref + 1e-30)).max() < 2e-3 and (got[:, :, :dim] - ref).abs().max() < 2e-5


@pytest.mark.parametrize("shape", [(1, 8192), (1, 9000), (3, 120), (8, 64), (5, 33), (1, 4096), (2, 1200)])
def test_gated_group_norm(shape):
    from rustingstrata_b200.kernels import ops
    parts, width = shape
    g = torch.Generator().manual_seed(width)
    n, T = parts * width, 7
    y, z, w = torch.randn(T, n, generator=g).cuda(), torch.randn(T, n + 4, generator=g).cuda()[:, :n], torch.randn(n, generator=g).cuda()
    u = (y.double() * torch.nn.functional.silu(z.double())).view(T, parts, width)
    ref = (u / torch.sqrt((u * u).mean(-1, keepdim=True) + 1e-5)).view(T, n) * w.double()
    for dt, tol in ((torch.float32, 2e-6), (torch.bfloat16, 5e-3)):
        out = torch.empty(T, n, dtype=dt, device="cuda")
        ops.gated_group_norm(y, z, w, out, parts, 1e-5, T)
        assert (out.double() - ref).abs().max() / ref.abs().max() < tol


def test_joined_matrices_count_once(tmp_path_factory):
    """The roofline's bytes and flops of a model whose blocks join their parts' matrices: every matrix once."""
    from rustingstrata_b200.engine import roofline
    path, cfg, w = model(tmp_path_factory, "R", "R", seed=11)
    r = runner_for(path, "bfloat16", pool_tokens=64, max_batch_tokens=64)
    assert any(getattr(b, "join_out", False) for b in r.model.blocks)
    shapes = M.tensor_shapes(cfg)
    total = sum(int(np.prod(s)) for s in shapes.values()) * 2
    assert total <= roofline.weight_bytes(r.model) <= total * 1.05                   # small vectors are kept in float32
    mats = sum(2 * int(np.prod(s)) for n, s in shapes.items() if len(s) == 2 and n != "embed" and not n.endswith("conv"))
    state = 6.0 * (4 * 32 * 48 + 8 * 64 * 32)
    assert abs(roofline.flops_per_token(r.model) - mats - state) <= 0.02 * mats
