"""The Gemodra decoder inside the engine against the plain float64 implementation (tests/plain_gemodra.py).

Every mechanism alone (one-layer models), whole prompts against token-by-token decoding, portions down to two tokens, mixed
batches against each request alone, pages and slots that are freed and used again, far keys and page borders with peaked
attention, sinks that matter, the first tokens of a sequence, long decoding, several sizes, the residual stream layer by
layer, the new kernels against torch, greedy generation through the scheduler, and the command line.
"""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import gemodra_models as M
import plain_gemodra as P
from helpers import ROOT

pytestmark = pytest.mark.gpu

TOL = {"float32": 2e-5, "bfloat16": 4e-2}         # max |difference| / max |reference logit|
# With peaked attention a rounding of a score moves the weights of the keys by as much more.
TOL_SHARP = {"float32": 1.5e-3, "bfloat16": 8e-2}
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


def model(tmp_path_factory, key, cfg, seed=0, sharp=False, steady=False, shift=0.0):
    if key not in _MODELS:
        path = str(tmp_path_factory.mktemp("gemodra") / key)
        _MODELS[key] = (path,) + M.make(path, cfg, seed, sharp, steady, shift)
    return _MODELS[key]


def model_for(tmp_path_factory, dtype, key, cfg, seed=0, sharp=False):
    """The model a test runs in this element type.  The bfloat16 engine rounds the router's input, so its models get
    corrections that decide the choice alone; and half the sharpening: its queries and latents are rounded to 8 bits, and
    scores that are scaled up carry that rounding into the weights."""
    steady = dtype == "bfloat16"
    return model(tmp_path_factory, key + ("_steady" if steady else ""), cfg, seed, 0.5 * sharp if steady else sharp, steady)


def assert_rows_within(err, tol, what):
    """Per-position errors of a run with sharpened weights: none beyond one and a half times the tolerance and at most
    one position in fifty beyond the tolerance itself (where a query weighs two keys nearly alike, the rounding of a
    score tips the balance; a fault of a mask, a page or a slot moves whole stretches of positions by far more)."""
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
_A = M.unrotated(1, 8, 8, 16, 8)                  # a small mixer where the feed-forward is the matter
ONE_LAYER = {
    "rotated_all_sizes_unequal": M.config(97, 64, [(M.rotated(6, 16, 8, 24, 40, 20, base=50.0), None)], side=None),
    "rotated_one_head_padded_row": M.config(97, 72, [(M.rotated(1, 12, 6, 20, 21, 9, base=7.0, scale=0.5), None)], eps=1e-5, side=None),
    "rotated_part_wider_than_the_rest": M.config(97, 64, [(M.rotated(3, 8, 32, 8, 16, 40), None)], side=None),
    "rotated_twenty_heads": M.config(97, 64, [(M.rotated(20, 8, 8, 8, 24, 32), None)], side=None),
    "unrotated_all_sizes_unequal": M.config(97, 64, [(M.unrotated(3, 16, 24, 40, 28, scale=0.4), None)], side=None),
    "unrotated_padded_row": M.config(97, 64, [(M.unrotated(5, 8, 12, 21, 16), None)], side=None),
    "unrotated_one_head": M.config(97, 72, [(M.unrotated(1, 32, 8, 16, 64), None)], eps=1e-5, side=None),
    "residual_multiplier": M.config(97, 64, [(M.rotated(2, 16, 16, 16, 32, 24), None)], mult=0.1, side=None, cap=None),
    "logit_cap": M.config(97, 64, [(_A, None)], side=None, cap=0.75),
    "token_side": M.config(97, 64, [(_A, None), (_A, None)], mult=0.8, side=24),
    "token_side_odd_columns": M.config(97, 72, [(_A, None), (_A, M.moe(3, 1, 16))], side=13),
    "experts_in_groups": M.config(97, 64, [(_A, M.moe(10, 3, 24, identity=2, scale=2.0, groups=(4, 2), shared=40))], side=None),
    "experts_one_group_kept": M.config(97, 64, [(_A, M.moe(8, 4, 16, identity=2, scale=0.7, groups=(2, 1), shared=8))], side=None),
    "experts_all_groups_kept": M.config(97, 64, [(_A, M.moe(6, 2, 16, groups=(3, 3)))], side=None),
    "experts_without_groups_or_shared": M.config(97, 64, [(_A, M.moe(5, 1, 32, identity=1))], side=None),
    "experts_mostly_identity": M.config(97, 64, [(_A, M.moe(2, 4, 32, identity=10, shared=24))], side=None),
    "experts_all_chosen": M.config(97, 64, [(_A, M.moe(3, 4, 20, identity=1, shared=24))], mult=0.3, side=None),
    "experts_of_odd_width": M.config(97, 60, [(_A, M.moe(4, 2, 18, identity=1, shared=22))], mult=0.3, side=12),
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(ONE_LAYER))
def test_mechanism_alone(tmp_path_factory, name, dtype):
    """One mechanism per model: the stream after every layer run and the logits of every position, whole and in portions."""
    cfg = ONE_LAYER[name]
    path, cfg, w = model_for(tmp_path_factory, dtype, "one_" + name, cfg, seed=5)
    toks = tokens_for(cfg, 45, 3)
    streams = []
    ref = P.forward(toks, w, cfg, streams).numpy()
    r = runner_for(path, dtype, page_size=8, pool_tokens=256)
    from rustingstrata_b200.engine import StepEntry
    got_streams = []
    logits = r.step([StepEntry("a", toks, list(range(len(toks))))],
                    on_layer=lambda k, x: got_streams.append(x.float().cpu().numpy().copy()))
    r.check_status()
    assert len(got_streams) == len(streams) == len(cfg["layers"])
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


def test_groups_compare_negative_choice_scores(tmp_path_factory):
    """Corrections that push every choice score far below zero: the experts of dropped groups must count as minus infinity,
    not as zero."""
    path, cfg, w = model(tmp_path_factory, "negative", ONE_LAYER["experts_in_groups"], seed=5, shift=-4.0)
    toks = tokens_for(cfg, 40, 3)
    assert rel_err(step_all(runner_for(path, "float32"), "a", toks), plain_logits(cfg, w, toks)) <= TOL["float32"]


# ----------------------------------------------------------------------------- whole models, every cutting
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["P", "Q", "R", "S"])
def test_cuttings_of_a_prompt(tmp_path_factory, name, dtype):
    """Whole, last tokens one by one (captured steps), portions of several sizes down to two tokens."""
    path, cfg, w = model_for(tmp_path_factory, dtype, name, name, seed=11)
    toks = tokens_for(cfg, 150, 5)
    ref = plain_logits(cfg, w, toks)
    r = runner_for(path, dtype, page_size=16, pool_tokens=512)
    assert rel_err(step_all(r, "w", toks), ref) <= TOL[dtype], "whole"
    r.release("w")
    n = len(toks) - 40
    got = [step_all(r, "d", toks[:n])] + [step_all(r, "d", [t]) for t in toks[n:]]
    assert rel_err(np.concatenate(got), ref) <= TOL[dtype], "decoding"
    assert r.model.capturable and r.graph_replays > 0
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
    beside single tokens of others, requests left out of steps, and every row equal to the request run alone."""
    from rustingstrata_b200.engine import StepEntry
    path, cfg, w = model_for(tmp_path_factory, dtype, name + "_sharp", name, seed=21, sharp=True)
    tol = TOL_SHARP[dtype]
    lengths = [70, 33, 121, 9, 64, 1, 47]
    toks = {f"r{i}": tokens_for(cfg, n, 40 + i) for i, n in enumerate(lengths)}
    ref = {k: plain_logits(cfg, w, t) for k, t in toks.items()}
    scale = max(np.max(np.abs(v)) for v in ref.values())      # one scale for all requests: a one-token request has no spread of its own
    r = runner_for(path, dtype, page_size=16, pool_tokens=256, max_seqs=3)
    rng = np.random.default_rng(9)
    waiting, live, pos = list(toks), [], {}
    slots_seen, errs = {}, []
    while waiting or live:
        while waiting and len(live) < 3 and sum((len(toks[x]) + 15) // 16 for x in live + [waiting[0]]) <= 16:
            live.append(waiting.pop(0))
            pos[live[-1]] = 0
        chosen = [x for x in live if rng.random() < 0.7] or [live[0]]
        entries, where = [], []
        for rid in chosen:
            left = len(toks[rid]) - pos[rid]
            n = 1 if left <= 12 else int(min(rng.choice([2, 3, 5, 9, 17, 31]), left - 12))
            entries.append(StepEntry(rid, toks[rid][pos[rid]:pos[rid] + n], list(range(n))))
            where += [(rid, pos[rid] + j) for j in range(n)]
            pos[rid] += n
        out = r.step(entries).cpu().numpy()
        r.check_status()
        for rid in chosen:
            slots_seen.setdefault(r.cache.slot(rid), set()).add(rid)
        for row, (rid, p) in zip(out, where):
            errs.append(float(np.max(np.abs(row - ref[rid][p])) / scale))
            assert errs[-1] <= 1.5 * tol, f"{name} {dtype}: request {rid} position {p}: {errs[-1]:.3e}"
        for rid in [x for x in live if pos[x] == len(toks[x])]:
            live.remove(rid)
            r.release(rid)
    r.cache.check()
    assert len(errs) == sum(lengths)
    assert_rows_within(errs, tol, "mixed batches")
    print(f"mixed {name} {dtype}: worst {max(errs):.3e}")
    assert max(len(v) for v in slots_seen.values()) >= 2, "no slot was used again"
    assert all(p.reuses > 0 for p in r.cache.pools), "no page was used again"


# ----------------------------------------------------------------------------- far keys, first tokens, long decoding
@pytest.mark.parametrize("dtype", DTYPES)
def test_far_keys_and_page_borders(tmp_path_factory, dtype):
    """Peaked attention (each query looks at one or two keys, at any distance) and raised sinks over 700 positions: every
    position of the prompt, then decoding across page borders and the borders of the attention's key tiles and splits."""
    path, cfg, w = model_for(tmp_path_factory, dtype, "R_sharp", "R", seed=21, sharp=True)
    toks = tokens_for(cfg, 700, 77)
    ref = plain_logits(cfg, w, toks)
    r = runner_for(path, dtype, page_size=16, pool_tokens=768, max_batch_tokens=768)
    n = 600
    got = [step_all(r, "a", toks[:n])] + [step_all(r, "a", [t]) for t in toks[n:n + 60]] + [step_all(r, "a", toks[n + 60:])]
    err = np.max(np.abs(np.concatenate(got) - ref), axis=1) / np.max(np.abs(ref))
    print(f"far keys {dtype}: worst {err.max():.3e}")
    assert_rows_within(err, TOL_SHARP[dtype], "far keys")


def test_sharp_weights_look_far_back():
    """The premise of the tests with sharp weights, on the plain implementation: dropping the oldest 100 tokens changes the
    last logits by more than twice the widest tolerance, so a lost far key would show in either engine."""
    cfg = M.CONFIGS["R"]
    for sharp, steady in ((1.0, False), (0.5, True)):
        w = M.draw_weights(cfg, 21, sharp, steady)
        toks = tokens_for(cfg, 700, 77)
        full, cut = plain_logits(cfg, w, toks)[-20:], plain_logits(cfg, w, toks[100:])[-20:]
        assert np.max(np.abs(full - cut)) / np.max(np.abs(full)) > 2 * TOL_SHARP["bfloat16"]


@pytest.mark.parametrize("dtype", DTYPES)
def test_first_tokens_and_short_sequences(tmp_path_factory, dtype):
    """Single-token prompts and a first step of one token beside longer ones in the same batch; then each grows token
    by token."""
    from rustingstrata_b200.engine import StepEntry
    path, cfg, w = model_for(tmp_path_factory, dtype, "R", "R", seed=11)
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
    """300 tokens one by one after a short prompt (replayed graphs, pages taken as it goes)."""
    path, cfg, w = model_for(tmp_path_factory, dtype, "P_sharp", "P", seed=21, sharp=True)
    toks = tokens_for(cfg, 320, 8)
    ref = plain_logits(cfg, w, toks)
    r = runner_for(path, dtype, page_size=8, pool_tokens=384)
    got = [step_all(r, "a", toks[:20])] + [step_all(r, "a", [t]) for t in toks[20:]]
    err = np.max(np.abs(np.concatenate(got) - ref), axis=1) / np.max(np.abs(ref))
    print(f"long decoding {dtype}: worst {err.max():.3e}")
    assert_rows_within(err, TOL_SHARP[dtype], "long decoding")


WIDE = {
    # a latent row of 512 + 64, 24 heads, 40 outputs of the router in 8 groups, widths that reach the 128 x 128 tiles
    "wide_rows": M.config(500, 512, [
        (M.rotated(24, 64, 64, 128, 512, 320, base=1e6), M.moe(34, 4, 64, identity=6, scale=2.5, groups=(8, 3), shared=256)),
        (M.unrotated(8, 128, 96, 384, 256), M.moe(16, 6, 128, identity=2, scale=1.5, groups=(3, 2), shared=320))], eps=1e-5, side=128),
    "many_heads": M.config(300, 256, [
        (M.rotated(40, 16, 16, 24, 48, 72), M.moe(16, 8, 32, scale=1.0, groups=(2, 2))),
        (M.unrotated(33, 24, 16, 64, 48), None)], mult=0.4, side=40),
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(WIDE))
def test_wider_shapes_and_long_portions(tmp_path_factory, name, dtype):
    """A portion of 500 tokens, 30 single tokens, a portion of 110: the forms of the kernels that only large steps and
    wide heads reach."""
    path, cfg, w = model_for(tmp_path_factory, dtype, "wide_" + name, WIDE[name], seed=7)
    toks = tokens_for(cfg, 640, 3)
    ref = plain_logits(cfg, w, toks)
    r = runner_for(path, dtype, page_size=16, pool_tokens=768, max_batch_tokens=768)
    got = [step_all(r, "a", toks[:500])] + [step_all(r, "a", [t]) for t in toks[500:530]] + [step_all(r, "a", toks[530:])]
    err = np.max(np.abs(np.concatenate(got) - ref), axis=1) / np.max(np.abs(ref))
    print(f"wide {name} {dtype}: worst {err.max():.3e}")
    assert err.max() <= TOL[dtype], f"first wrong position {int(np.argmax(err > TOL[dtype]))}"


@pytest.mark.parametrize("n", [2, 9, 24, 64])
def test_many_single_tokens_at_once(tmp_path_factory, n):
    """Decode steps of many requests: the products' forms for few, some and many rows, the captured step of each size."""
    from rustingstrata_b200.engine import StepEntry
    path, cfg, w = model_for(tmp_path_factory, "bfloat16", "R", "R", seed=11)
    r = runner_for(path, "bfloat16", page_size=16, pool_tokens=n * 32, max_seqs=n)
    seqs = [tokens_for(cfg, 5 + i % 17, i) for i in range(n)]
    r.step([StepEntry(f"s{i}", t[:-3], []) for i, t in enumerate(seqs)])
    for k in (3, 2, 1):
        out = r.step([StepEntry(f"s{i}", [t[-k]], [0]) for i, t in enumerate(seqs)]).cpu().numpy()
        r.check_status()
    for i, t in enumerate(seqs):
        assert rel_err(out[i], plain_logits(cfg, w, t)[-1]) <= TOL["bfloat16"], i


# ----------------------------------------------------------------------------- kernels against torch
def _status():
    return torch.zeros(1, dtype=torch.int32, device="cuda")


def test_router_choice_with_groups_worth_their_best_score():
    """The router kernel with softmax scores and groups worth their largest choice score, corrections of both signs, against
    the same rule written with torch."""
    from rustingstrata_b200.kernels import ops
    g = torch.Generator().manual_seed(3)
    for E, top, groups, keep, scale, shift in [(12, 3, 4, 2, 2.0, 0.0), (20, 2, 2, 1, 2.5, -3.0), (64, 6, 8, 4, 1.0, -0.5),
                                               (6, 2, 6, 3, 1.5, 0.0), (40, 1, 0, 0, 3.0, -1.0), (5, 5, 1, 1, 1.0, 0.0)]:
        T = 70
        logits = torch.randn(T, E + 3, generator=g) * 2           # further columns of the product are not the router's
        corr = torch.randn(E, generator=g) * 0.3 + shift
        s = torch.softmax(logits[:, :E].double(), dim=-1)
        pick = s + corr.double()
        if groups:
            worth = pick.view(T, groups, E // groups).max(dim=-1).values
            ok = torch.zeros(T, groups, dtype=torch.bool).scatter_(1, worth.topk(keep, dim=-1).indices, True)
            pick = pick.masked_fill(~ok.repeat_interleave(E // groups, dim=1), -float("inf"))
        want = pick.topk(top, dim=-1).indices
        choice = torch.empty(T * top, dtype=torch.int32, device="cuda")
        weights = torch.empty(T * top, dtype=torch.float32, device="cuda")
        status = _status()
        ops.router_topk(logits.cuda()[:, :E], corr.cuda(), top, T, choice, weights, status, groups=groups, keep=keep,
                        scale=scale, renormalize=False, group_worth="max")
        assert int(status.item()) == 0
        got = choice.view(T, top).cpu().long()
        assert torch.equal(got.sort(dim=1).values, want.sort(dim=1).values), (E, top, groups, keep)
        assert torch.allclose(weights.view(T, top).cpu().double(), s.gather(1, got) * scale, rtol=1e-5, atol=1e-6)


@pytest.mark.parametrize("T", [1, 5, 32])
def test_choice_and_lists_in_one_launch(T):
    """The joint launch for small steps gives the two launches' choices, weights and tiles, and deals every pair once."""
    from rustingstrata_b200.kernels import ops
    g = torch.Generator().manual_seed(T)
    for E, identity, top, groups, keep in [(12, 4, 3, 4, 2), (40, 0, 5, 0, 0), (3, 9, 2, 2, 1)]:
        n = E + identity
        logits, corr = torch.randn(T, n + 1, generator=g).cuda()[:, :n], torch.randn(n, generator=g).cuda()
        outs = []
        for joint in (True, False):
            i32 = lambda k: torch.full((k,), -1, dtype=torch.int32, device="cuda")                  # noqa: E731
            choice, weights, order, tiles, n_tiles, status = i32(T * top), torch.zeros(T * top, device="cuda"), i32(T * top), i32(3 * (T * top + E)), i32(1), _status()
            kw = dict(groups=groups, keep=keep, scale=1.5, renormalize=False, group_worth="max")
            if joint:
                assert ops.core().rs_router_route_supported(T, n, groups, E)
                ops.router_route(logits, corr, top, T, choice, weights, E, 16, order, tiles, n_tiles, status, identity=identity, **kw)
            else:
                ops.router_topk(logits, corr, top, T, choice, weights, status, **kw)
                ops.moe_route(None, choice.view(T, top), E, T, 16, order, tiles, n_tiles, status, identity=identity)
            assert int(status.item()) == 0
            nt = int(n_tiles.item())
            outs.append((choice.tolist(), weights.tolist(), tiles[: 3 * nt].tolist()))
            rows = sum(outs[-1][2][2::3])
            assert sorted(order[:rows].tolist()) == [i for i, c in enumerate(outs[-1][0]) if c < E]
        assert outs[0] == outs[1]


def test_identity_choices_get_no_rows_in_the_lists():
    from rustingstrata_b200.kernels import ops
    T, top, E, identity, rows = 300, 3, 5, 4, 64
    choice = torch.from_numpy(np.stack([np.random.default_rng(t).permutation(E + identity)[:top] for t in range(T)]).astype(np.int32))
    order = torch.full((T * top,), -1, dtype=torch.int32, device="cuda")
    tiles = torch.zeros(3 * (T * top // rows + E), dtype=torch.int32, device="cuda")
    n_tiles, status = torch.zeros(1, dtype=torch.int32, device="cuda"), _status()
    ops.moe_route(None, choice.cuda(), E, T, rows, order, tiles, n_tiles, status, identity=identity)
    assert int(status.item()) == 0
    flat, order = choice.view(-1), order.cpu()
    seen = []
    for e, r0, n in tiles.cpu().view(-1, 3)[: int(n_tiles.item())].tolist():
        pairs = order[r0: r0 + n].tolist()
        assert all(int(flat[p]) == e for p in pairs)
        seen += pairs
    assert sorted(seen) == [i for i in range(T * top) if int(flat[i]) < E]
    # a choice beyond the identity experts is flagged
    bad = choice.clone()
    bad[0, 0] = E + identity
    ops.moe_route(None, bad.cuda(), E, T, rows, torch.empty(T * top, dtype=torch.int32, device="cuda"), tiles, n_tiles, status, identity=identity)
    assert int(status.item()) == ops.STATUS_BAD_PLAN


@pytest.mark.parametrize("n", [256, 70])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_combination_of_experts(n, dtype):
    """Weighted pairs, identity experts, a shared part behind a sigmoid, a factor on the whole, the sum into a stream and the
    copy of its new rows, with rows that allow 16-byte accesses and rows that do not."""
    from rustingstrata_b200.kernels import ops
    g = torch.Generator().manual_seed(1)
    T, top, E = 37, 3, 4
    pair, shared, x = (torch.randn(r, n, generator=g) for r in (T * top, T, T))
    h = torch.randn(T, n, generator=g).to(dtype)
    wts, z = torch.rand(T * top, generator=g), torch.randn(T, 5, generator=g)
    choice = torch.randint(0, E + 2, (T * top,), generator=g).to(torch.int32)
    rows = torch.where((choice >= E)[:, None], h.double().repeat_interleave(top, 0), pair.double())
    y = 0.3 * ((rows * wts.double()[:, None]).view(T, top, n).sum(1) + torch.sigmoid(z[:, 4:].double()) * shared.double())
    xs, copy = x.cuda(), torch.zeros(T, n, dtype=dtype, device="cuda")
    common = dict(shared=shared.cuda(), h=h.cuda(), pair_weights=wts.cuda(), choice=choice.cuda(), n_experts=E,
                  gate_logit=z.cuda()[:, 4:], scale=0.3)
    ops.moe_combine(pair.cuda(), top, 1.0, xs, T, accumulate=True, copy=copy, **common)
    assert torch.allclose(xs.cpu().double(), x.double() + y, rtol=1e-5, atol=1e-5)
    assert torch.equal(copy, xs.to(dtype))
    out = torch.empty(T, n, device="cuda")
    ops.moe_combine(pair.cuda(), top, 1.0, out, T, **common)
    assert torch.allclose(out.cpu().double(), y, rtol=1e-5, atol=1e-5)


@pytest.mark.parametrize("rows", [3, 40, 300])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("per", ["block", "column"])
def test_block_product_behind_a_gate(rows, dtype, per):
    """The block-diagonal product times factor * sigmoid(gate), in its form for few rows and its tiled forms."""
    from rustingstrata_b200.kernels import ops
    g = torch.Generator().manual_seed(2)
    B, O, I = 5, 24, 48
    x = torch.randn(rows, B * I, generator=g).to(dtype)
    w = (torch.randn(B, O, I, generator=g) / I ** 0.5).to(dtype)
    gates = torch.randn(rows, 7 + B * O, generator=g)
    gate = gates[:, 7: 7 + (B if per == "block" else B * O)]
    want = torch.einsum("tbi,boi->tbo", x.double().view(rows, B, I), w.double()).reshape(rows, B * O)
    f = torch.sigmoid(gate.double())
    want = want * 0.7 * (f.repeat_interleave(O, 1) if per == "block" else f)
    out = torch.zeros(rows, B * O, dtype=dtype, device="cuda")
    cut = gates.cuda()
    ops.block_linear(x.cuda(), w.cuda(), out, rows, I, O, gate=cut[:, 7: 7 + gate.shape[1]], out_scale=0.7)
    assert rel_err(out.float().cpu().numpy(), want.numpy()) <= (1e-5 if dtype == torch.float32 else 8e-3)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("window", [0, 37])
@pytest.mark.parametrize("H,lat,v", [(3, 48, 40), (20, 128, 128), (8, 576, 512), (70, 80, 72), (16, 320, 256), (33, 304, 304)])
def test_attention_over_latents_with_a_sink(dtype, H, lat, v, window):
    """The kernels of latent attention (narrow and wide portions, the split form over several splits) with sinks from next to nothing to
    far above every score, over scattered pages, against float64."""
    from rustingstrata_b200.kernels import ops
    from rustingstrata_b200.parts.attention import SPLIT_KEYS, decode_splits
    g = torch.Generator().manual_seed(4)
    page, kv_lens, q_lens = 16, [300, 241, 1], [1, 120, 1]
    pages = [(n + page - 1) // page for n in kv_lens]
    ids = torch.randperm(sum(pages) + 5, generator=g)[: sum(pages)].to(torch.int32)
    table = torch.full((3, max(pages)), -1, dtype=torch.int32)
    at = 0
    for s, n in enumerate(pages):
        table[s, :n], at = ids[at: at + n], at + n
    cache = torch.randn(sum(pages) + 5, 1, 1, page, lat, generator=g).to(dtype)
    T = sum(q_lens)
    q = (torch.randn(T, H * lat, generator=g) / lat ** 0.5 * 2).to(dtype)
    sink = torch.linspace(-20.0, 12.0, H)
    scale = 0.9
    want, q_start = torch.zeros(T, H, lat, dtype=torch.float64), [0]
    for s in range(3):
        keys = torch.stack([cache[table[s, p // page], 0, 0, p % page] for p in range(kv_lens[s])]).double()
        for j in range(q_lens[s]):
            t, end = q_start[-1] + j, kv_lens[s] - q_lens[s] + j + 1
            seen = slice(max(0, end - window) if window else 0, end)
            sc = q[t].double().view(H, lat) @ keys[seen].T * scale
            m = torch.maximum(sc.max(-1).values, sink.double())
            e = torch.exp(sc - m[:, None])
            want[t] = e @ keys[seen] / (e.sum(-1) + torch.exp(sink.double() - m))[:, None]
        q_start.append(q_start[-1] + q_lens[s])
    dev = lambda x: torch.as_tensor(x, dtype=torch.int32).cuda()                                    # noqa: E731
    out, status = torch.zeros(T, H * lat, dtype=dtype, device="cuda"), _status()
    singles = [s for s in range(3) if q_lens[s] == 1]
    splits = [int(n) for n in decode_splits(np.array([kv_lens[s] for s in singles]), window)]
    split_start = dev([0] + list(np.cumsum(splits)))
    partial = torch.zeros(1, (sum(splits) + 2) * H * (lat + 2), device="cuda")
    common = dict(q=q.cuda(), out=out, cache=cache.cuda(), block_table=table.cuda(), q_start=dev(q_start), kv_len=dev(kv_lens),
                  page_size=page, window=window, scale=scale, status=status, sink=sink.cuda())
    split = dict(split_keys=SPLIT_KEYS, max_splits=max(splits), split_start=split_start, total_splits=sum(splits), partial=partial)
    if dtype == torch.bfloat16:
        shape = dict(n_heads=H, lat=lat, split_weights=True, v_cols=v)
        outs = {}
        for wide in (False, True):
            qpc = ops.attention_latent_q_per_cta(H, wide)
            work = [(1, o) for o in range(0, q_lens[1], qpc)]
            outs[wide] = torch.zeros_like(out)
            ops.attention_latent(work=dev(work).view(-1), n_work=len(work), decode=False, wide=wide, **shape, **dict(common, out=outs[wide]))
            ops.attention_latent(work=dev(singles), n_work=len(singles), decode=True, **shape, **dict(common, out=outs[wide]), **split)
    else:
        qpc = ops.attention_q_per_cta(H, 1)
        work = [(1, o) for o in range(0, q_lens[1], qpc)]
        shape = dict(n_q=H, n_kv=1, head_dim=lat, one_plane=True)
        ops.attention_simt(work=dev(work).view(-1), n_work=len(work), decode=False, **shape, **common)
        ops.attention_simt(work=dev(singles), n_work=len(singles), decode=True, **shape, **common, **split)
        outs, v = {False: out}, lat
    assert int(status.item()) == 0
    for form, x in outs.items():
        got = x.float().cpu().double().view(T, H, lat)
        for h in range(H):
            assert rel_err(got[:, h, :v], want[:, h, :v]) <= (2e-5 if dtype == torch.float32 else 1.2e-2), (form, h, float(sink[h]))
        assert dtype == torch.float32 or not got[:, :, v:].any()


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("rows", [1, 6, 8, 30])
def test_queries_against_a_latent(rows, dtype):
    """The key map folded into the queries with the rotated parts behind it: one launch for few rows, two for many."""
    from rustingstrata_b200.kernels import ops
    g = torch.Generator().manual_seed(rows)
    for H, dim, rot, rank in [(3, 16, 8, 24), (5, 40, 32, 64), (2, 24, 0, 21), (4, 12, 6, 20), (2, 576, 16, 32), (2, 800, 16, 32)]:
        lat = (rank + rot + 15) // 16 * 16
        q = torch.randn(rows, H * (dim + rot), generator=g).to(dtype)
        w = (torch.randn(H, rank, dim, generator=g) / dim ** 0.5).to(torch.bfloat16 if dtype == torch.bfloat16 else dtype)
        pos = torch.randint(0, 50, (rows,), generator=g).to(torch.int32)
        ang = pos.double()[:, None] * 100.0 ** (-2.0 * torch.arange(max(rot, 2) // 2, dtype=torch.float64) / max(rot, 2))
        table = torch.arange(50, dtype=torch.float64)[:, None] * 100.0 ** (-2.0 * torch.arange(max(rot, 2) // 2, dtype=torch.float64) / max(rot, 2))
        cos_sin = torch.cat([table.cos(), table.sin()], 1).float().cuda() if rot else None
        out, status = torch.full((rows, H * lat), 7.0, dtype=dtype, device="cuda"), _status()
        zero = torch.zeros(rows, dtype=torch.int32, device="cuda")
        ops.latent_queries(q.cuda(), w.cuda(), out, rows, dim + rot, lat, cos_sin, rot, rot, pos.cuda()[:, None], zero, zero[:1, None], 16, status)
        assert int(status.item()) == 0
        x = q.double().view(rows, H, dim + rot)
        want = torch.zeros(rows, H, lat, dtype=torch.float64)
        want[..., :rank] = torch.einsum("thd,hrd->thr", x[..., :dim], w.double())
        if rot:
            c, s = ang.cos()[:, None], ang.sin()[:, None]
            u, v = x[..., dim::2], x[..., dim + 1::2]
            want[..., rank: rank + rot: 2], want[..., rank + 1: rank + rot: 2] = u * c - v * s, v * c + u * s
        assert rel_err(out.float().cpu(), want.view(rows, -1)) <= (1e-5 if dtype == torch.float32 else 6e-3), (H, dim, rot, rank)


@pytest.mark.parametrize("n", [256, 1028, 4096, 8192, 75])
def test_norm_of_a_sublayer_into_the_stream(n):
    """x += norm(delta) and the next reader's norm, in the form that keeps rows in registers and the one for other widths."""
    from rustingstrata_b200.kernels import ops
    g = torch.Generator().manual_seed(n)
    x, d = torch.randn(5, n, generator=g), torch.randn(5, n, generator=g)
    gain, w2 = torch.randn(n, generator=g), torch.randn(n, generator=g).to(torch.bfloat16)
    want = x.double() + P.rms_norm(d.double(), gain.double(), 1e-5)
    for dtype, tol in ((torch.float32, 2e-6), (torch.bfloat16, 5e-3)):
        xs, out = x.cuda(), torch.zeros(5, n, dtype=dtype, device="cuda")
        ops.rmsnorm_add(xs, d.cuda(), gain.cuda(), 1e-5, 5, w2.cuda(), 1e-3, out)
        assert rel_err(xs.cpu(), want) <= 2e-6 and rel_err(out.float().cpu(), P.rms_norm(want, w2.double(), 1e-3)) <= tol
    xs = x.cuda()
    ops.rmsnorm_add(xs, d.cuda(), gain[:1].cuda(), 1e-5, 5)
    assert rel_err(xs.cpu(), x.double() + P.rms_norm(d.double(), gain[:1].double(), 1e-5)) <= 2e-6


def test_small_row_kernels():
    """The normed embedding, the projection gated by a table row, the capped logits and the cast against torch; a token id
    outside the table is flagged."""
    from rustingstrata_b200.kernels import ops
    g = torch.Generator().manual_seed(6)
    T, V, D, n = 9, 50, 75, 13
    ids = torch.randint(0, V, (T,), generator=g).to(torch.int32)
    table, w = torch.randn(V, D, generator=g).to(torch.bfloat16), torch.randn(D, generator=g).to(torch.bfloat16)
    status, out = _status(), torch.zeros(T, D, device="cuda")
    ops.embed_rmsnorm(table.cuda(), ids.cuda(), w.cuda(), 1e-3, out, T, status)
    e = table.double()[ids.long()]
    assert rel_err(out.cpu(), P.rms_norm(e, w.double(), 1e-3)) <= 1e-6
    z = torch.randn(T, n, generator=g) * 3
    for dtype, tol in ((torch.float32, 1e-6), (torch.bfloat16, 5e-3)):
        act = torch.zeros(T, n, dtype=dtype, device="cuda")
        ops.gelu_table_gate(z.cuda(), table.cuda(), 20, ids.cuda(), act, T, status)
        assert rel_err(act.float().cpu(), P.gelu_tanh(z.double()) * e[:, 20:20 + n]) <= tol
    logits = torch.randn(T, D, generator=g) * 5
    x = logits.cuda()
    ops.softcap_rows(x, T, 3.0, 0.5)
    assert rel_err(x.cpu(), 3.0 * torch.tanh(logits.double() * 0.5 / 3.0)) <= 1e-6
    copy = torch.zeros(T, D, dtype=torch.bfloat16, device="cuda")
    ops.cast_rows(logits.cuda(), copy, T)
    assert torch.equal(copy.cpu(), logits.to(torch.bfloat16))
    assert int(status.item()) == 0
    ops.embed_rmsnorm(table.cuda(), torch.full((T,), V, dtype=torch.int32, device="cuda"), w.cuda(), 1e-3, out, T, status)
    assert int(status.item()) == ops.STATUS_BAD_TOKEN


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


def test_bfloat16_generation_picks_top_tokens(tmp_path_factory):
    from rustingstrata_b200 import Engine
    path, cfg, w = model(tmp_path_factory, "R_steady", "R", seed=11, steady=True)
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
