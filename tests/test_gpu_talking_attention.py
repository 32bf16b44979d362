"""The tensor-core form of talking-heads attention against a plain float64 computation over the same bfloat16 cache, and
against the CUDA-core form: head counts with and without grouping, head sizes up to 128, windows, unequal sequences on
shuffled pages, every query tile size, and key tiles dealt out over several CTAs (with parts that get no tile at all)."""
import numpy as np
import pytest
import torch

pytestmark = pytest.mark.gpu


def plain(q, k, v, talk, sink, gate, scale, window, first_pos):
    """q [n, H, dk] float64 at positions first_pos.., k [L, G, dk], v [L, G, dv]: out [n, H, dv]."""
    n, H, _ = q.shape
    L, G, dv = v.shape
    r = H // G
    raw = torch.stack([(q[:, h] @ k[:, h // r].T) * scale for h in range(H)])            # [H, n, L]
    mixed = torch.einsum("hg,gij->hij", talk, raw) if talk is not None else raw
    out = torch.zeros(n, H, dv, dtype=torch.float64)
    for i in range(n):
        pos = first_pos + i
        lo = max(0, pos - window + 1) if window else 0
        for h in range(H):
            s = mixed[h, i, lo:pos + 1]
            top = s.max() if sink is None else torch.maximum(s.max(), sink[h])
            e = torch.exp(s - top)
            den = e.sum() + (torch.exp(sink[h] - top) if sink is not None else 0.0)
            out[i, h] = (e / den) @ v[lo:pos + 1, h // r]
    return out * gate[:, :, None] if gate is not None else out


CASES = [
    # H, G, dk, dv, window, talk, sink, gate
    (16, 4, 64, 64, 0, True, True, True),
    (8, 8, 32, 16, 0, True, True, False),
    (32, 4, 16, 64, 0, True, True, True),
    (4, 1, 128, 128, 0, True, False, True),
    (6, 3, 48, 32, 37, True, True, True),
    (2, 2, 16, 16, 0, False, True, True),
    (12, 2, 32, 80, 70, True, False, False),
]


@pytest.mark.parametrize("case", CASES, ids=lambda c: "h{}g{}k{}v{}w{}".format(*c[:5]))
@pytest.mark.parametrize("qt,parts", [(16, 1), (8, 3), (4, 1), (4, 7), (16, 2)])
def test_tensor_core_form(case, qt, parts):
    from rustingstrata_b200.kernels import ops
    H, G, dk, dv, window, has_talk, has_sink, has_gate = case
    most = ops.talking_attention_mma_q_per_cta(H, G, dk, dv)
    assert most >= 4, "a shape the tensor-core form is meant to take"
    qt = min(qt, most)
    dev = torch.device("cuda")
    gen = torch.Generator().manual_seed(H * 1000 + dk + qt + parts)
    page, hdp = 16, (max(dk, dv) + 7) // 8 * 8
    # sequences: (keys after the step, queries in the step): a portion from the start, a portion after 150 keys, a
    # single token far in, a single token that is the sequence's first
    seqs = [(77, 77), (150 + 41, 41), (333, 1), (1, 1)]
    n_pages = sum((kv + page - 1) // page for kv, _ in seqs) + 3
    order = torch.randperm(n_pages, generator=gen).tolist()
    cache = torch.zeros(n_pages, 2, G, page, hdp, dtype=torch.bfloat16)
    table = torch.full((len(seqs), max((kv + page - 1) // page for kv, _ in seqs)), -1, dtype=torch.int32)
    ks, vs = [], []
    for s, (kv, _) in enumerate(seqs):
        k = torch.randn(kv, G, dk, generator=gen).to(torch.bfloat16)
        v = torch.randn(kv, G, dv, generator=gen).to(torch.bfloat16)
        ks.append(k), vs.append(v)
        for b in range((kv + page - 1) // page):
            pg = order.pop()
            table[s, b] = pg
            n = min(page, kv - b * page)
            cache[pg, 0, :, :n, :dk] = k[b * page:b * page + n].transpose(0, 1)
            cache[pg, 1, :, :n, :dv] = v[b * page:b * page + n].transpose(0, 1)
    T = sum(n for _, n in seqs)
    q = torch.randn(T, H * dk, generator=gen) * 1.5
    gate = torch.rand(T, H, generator=gen) if has_gate else None
    talk = (torch.eye(H) * 0.7 + torch.randn(H, H, generator=gen) * 0.3) if has_talk else None
    sink = torch.randn(H, generator=gen) * 2 if has_sink else None
    scale = dk ** -0.5
    q_start = np.concatenate([[0], np.cumsum([n for _, n in seqs])]).astype(np.int32)
    kv_len = np.array([kv for kv, _ in seqs], dtype=np.int32)
    ref = torch.cat([plain(q[q_start[s]:q_start[s + 1]].double().view(-1, H, dk), ks[s].double(), vs[s].double(),
                           None if talk is None else talk.double(), None if sink is None else sink.double(),
                           None if gate is None else gate[q_start[s]:q_start[s + 1]].double(), scale, window, kv - n)
                     for s, (kv, n) in enumerate(seqs)]).view(T, H * dv)
    work, rows = [], 0
    for s, (kv, n) in enumerate(seqs):
        for q0 in range(0, n, qt):
            nq = min(qt, n - q0)
            for p in range(parts):
                work.append((s, q0, p, parts, rows))
            rows += parts * nq if parts > 1 else 0
    work = torch.tensor(work, dtype=torch.int32).flatten()
    d = lambda t: None if t is None else t.to(dev)                                  # noqa: E731
    status = torch.zeros(1, dtype=torch.int32, device=dev)
    out = torch.full((T, H * dv), float("nan"), dtype=torch.float32, device=dev)
    partial = torch.full((max(rows, 1), H * (dv + 2)), float("nan"), dtype=torch.float32, device=dev)
    ops.talking_attention_mma(d(q), d(gate), d(cache), d(table), page, d(torch.from_numpy(q_start)), d(torch.from_numpy(kv_len)),
                              d(work), len(work) // 5, parts > 1, d(talk), d(sink), out, partial if parts > 1 else None,
                              H, G, dk, dv, window, qt, scale, status)
    torch.cuda.synchronize()
    assert int(status.item()) == 0
    err = (out.cpu().double() - ref).abs().max().item() / ref.abs().max().item()
    assert err < 3e-5, err
    # the CUDA-core form over the same cache
    simt_q = min(qt, ops.talking_attention_q_per_cta(H, dk, dv))
    w2 = torch.tensor([(s, q0) for s, (kv, n) in enumerate(seqs) for q0 in range(0, n, simt_q)], dtype=torch.int32).flatten()
    out2 = torch.full((T, H * dv), float("nan"), dtype=torch.float32, device=dev)
    ops.talking_attention(d(q), d(gate), d(cache), d(table), page, d(torch.from_numpy(q_start)), d(torch.from_numpy(kv_len)),
                          d(w2), len(w2) // 2, d(talk), d(sink), out2, H, G, dk, dv, window, simt_q, scale, status)
    torch.cuda.synchronize()
    assert (out2.cpu().double() - ref).abs().max().item() / ref.abs().max().item() < 3e-5
    # a bfloat16 result is the rounding of the same numbers
    out3 = torch.zeros((T, H * dv), dtype=torch.bfloat16, device=dev)
    ops.talking_attention_mma(d(q), d(gate), d(cache), d(table), page, d(torch.from_numpy(q_start)), d(torch.from_numpy(kv_len)),
                              d(work), len(work) // 5, parts > 1, d(talk), d(sink), out3, partial if parts > 1 else None,
                              H, G, dk, dv, window, qt, scale, status)
    torch.cuda.synchronize()
    assert (out3.float() - out).abs().max().item() <= 2 ** -8 * out.abs().max().item()


# ----------------------------------------------------------------------------- heads that do not mix, kept first keys
def plain_masked(q, k, v, sink, gate, scale, window, chunk, keep, first_pos, out_scale):
    n, H, _ = q.shape
    r = H // k.shape[1]
    i, j = torch.arange(first_pos, first_pos + n)[:, None], torch.arange(k.shape[0])[None, :]
    near = torch.ones(n, k.shape[0], dtype=torch.bool)
    if window:
        near &= i - j < window
    if chunk:
        near &= i // chunk == j // chunk
    seen = (j <= i) & (near | (j < keep))
    out = torch.zeros(n, H, v.shape[2], dtype=torch.float64)
    for h in range(H):
        s = torch.where(seen, (q[:, h] @ k[:, h // r].T) * scale, torch.tensor(-float("inf"), dtype=torch.float64))
        if sink is not None:
            s = torch.cat([s, sink[h].expand(n, 1)], dim=1)
        w = torch.softmax(s, dim=1)[:, : k.shape[0]]
        out[:, h] = w @ v[:, h // r]
    return out_scale * (out if gate is None else out * gate[:, :, None])


GROUPED = [
    # H, G, dk, dv, window, chunk, keep, sink, gate
    (16, 4, 64, 64, 0, 0, 0, True, True),
    (6, 3, 48, 32, 37, 0, 20, False, False),
    (4, 4, 128, 128, 70, 0, 5, False, False),
    (3, 1, 16, 112, 1, 0, 3, False, True),
    (8, 1, 112, 16, 64, 0, 64, True, False),
    (32, 2, 32, 48, 5, 0, 130, False, False),
    (5, 1, 96, 128, 200, 0, 1, False, False),
    (4, 2, 64, 80, 0, 48, 0, True, False),
    (40, 2, 32, 32, 100, 0, 17, False, False),        # twenty heads a group: no tile of one query
]


@pytest.mark.parametrize("case", GROUPED, ids=lambda c: "h{}g{}k{}v{}w{}c{}f{}".format(*c[:7]))
@pytest.mark.parametrize("parts", [1, 3])
def test_grouped_form_and_kept_keys(case, parts):
    """The grouped kernel (tiles of several queries and of one), the all-heads tensor-core form and the CUDA-core form without
    a mix, over one cache: windows, kept first keys, blocks; pages that nobody sees are not in the table."""
    from rustingstrata_b200.kernels import ops
    H, G, dk, dv, window, chunk, keep, has_sink, has_gate = case
    dev = torch.device("cuda")
    gen = torch.Generator().manual_seed(H * 100 + dk + parts)
    page, hdp, scale, out_scale = 16, (max(dk, dv) + 7) // 8 * 8, 1.5 * dk ** -0.5, 0.6
    seqs = [(77, 77), (150 + 141, 141), (333, 1), (1, 1), (500, 2)]                  # (keys after the step, queries in it)
    n_pages = sum((kv + page - 1) // page for kv, _ in seqs) + 3
    order = torch.randperm(n_pages, generator=gen).tolist()
    cache = torch.full((n_pages, 2, G, page, hdp), float("nan"), dtype=torch.bfloat16)
    table = torch.full((len(seqs), max((kv + page - 1) // page for kv, _ in seqs)), -1, dtype=torch.int32)
    ks, vs = [], []
    for s, (kv, n) in enumerate(seqs):
        k, v = (torch.randn(kv, G, d, generator=gen).to(torch.bfloat16) for d in (dk, dv))
        ks.append(k), vs.append(v)
        lo = max(0, kv - n - window + 1) if window else 0
        lo = max(lo, (kv - n) // chunk * chunk) if chunk else lo
        for b in range((kv + page - 1) // page):
            if (b + 1) * page <= lo and b * page >= keep:
                continue                                                             # a page the window has passed
            pg = order.pop()
            table[s, b] = pg
            m = min(page, kv - b * page)
            cache[pg, 0, :, :m, :dk], cache[pg, 1, :, :m, :dv] = k[b * page:b * page + m].transpose(0, 1), v[b * page:b * page + m].transpose(0, 1)
    T = sum(n for _, n in seqs)
    q = torch.randn(T, H * dk, generator=gen) * 1.5
    gate = torch.rand(T, H, generator=gen) if has_gate else None
    sink = torch.randn(H, generator=gen) * 2 if has_sink else None
    q_start = np.concatenate([[0], np.cumsum([n for _, n in seqs])]).astype(np.int32)
    kv_len = np.array([kv for kv, _ in seqs], dtype=np.int32)
    ref = torch.cat([plain_masked(q[q_start[s]:q_start[s + 1]].double().view(-1, H, dk), ks[s].double(), vs[s].double(),
                                  None if sink is None else sink.double(),
                                  None if gate is None else gate[q_start[s]:q_start[s + 1]].double(), scale, window, chunk, keep, kv - n,
                                  out_scale) for s, (kv, n) in enumerate(seqs)]).view(T, H * dv)
    d = lambda t: None if t is None else (torch.from_numpy(t) if isinstance(t, np.ndarray) else t).to(dev)       # noqa: E731
    status = torch.zeros(1, dtype=torch.int32, device=dev)
    q_d, gate_d, cache_d, table_d, qs_d, kv_d, sink_d = d(q), d(gate), d(cache), d(table), d(q_start), d(kv_len), d(sink)

    def tiles(which, qt, n_parts):
        work, rows = [], 0
        for s in which:
            n = seqs[s][1]
            for q0 in range(0, n, qt):
                nq = min(qt, n - q0)
                work += [(s, q0, p, n_parts, rows) for p in range(n_parts)]
                rows += n_parts * nq if n_parts > 1 else 0
        return d(torch.tensor(work, dtype=torch.int32).flatten()), len(work), rows

    def close(out, what):
        torch.cuda.synchronize()
        assert int(status.item()) == 0
        err = (out.cpu().double() - ref).abs().max().item() / ref.abs().max().item()
        assert err < 3e-5, f"{what}: {err}"
    masks = dict(chunk=chunk, keep=keep, out_scale=out_scale)
    qt = ops.grouped_attention_q_per_cta(H, G, dk, dv)
    assert qt == 64 // (H // G)
    out = torch.full((T, H * dv), float("nan"), device=dev)
    alone = [s for s, (_, n) in enumerate(seqs) if n == 1] if ops.grouped_attention_single_ok(H, G, dk, dv) else []
    assert bool(alone) == (H // G <= 16)
    for which, tile, single in ((sorted(set(range(len(seqs))) - set(alone)), qt, False), (alone, 1, True)):
        if which:
            work, n, rows = tiles(which, tile, parts)
            partial = torch.full((max(rows, 1), H * (dv + 2)), float("nan"), device=dev) if parts > 1 else None
            ops.grouped_attention_mma(q_d, gate_d, cache_d, table_d, page, qs_d, kv_d, work, n, parts > 1, single, sink_d, out, partial,
                                      H, G, dk, dv, window, tile, scale, status, **masks)
    close(out, "grouped")
    small = torch.zeros((T, H * dv), dtype=torch.bfloat16, device=dev)
    work, n, rows = tiles(range(len(seqs)), min(qt, 7), 1)
    ops.grouped_attention_mma(q_d, gate_d, cache_d, table_d, page, qs_d, kv_d, work, n, False, False, sink_d, small, None,
                              H, G, dk, dv, window, min(qt, 7), scale, status, **masks)
    assert (small.float() - out).abs().max().item() <= 2 ** -7 * out.abs().max().item()
    most = ops.talking_attention_mma_q_per_cta(H, G, dk, dv)
    if most:
        out2 = torch.full((T, H * dv), float("nan"), device=dev)
        work, n, rows = tiles(range(len(seqs)), 4, parts)
        partial = torch.full((max(rows, 1), H * (dv + 2)), float("nan"), device=dev) if parts > 1 else None
        ops.talking_attention_mma(q_d, gate_d, cache_d, table_d, page, qs_d, kv_d, work, n, parts > 1, None, sink_d, out2, partial,
                                  H, G, dk, dv, window, 4, scale, status, **masks)
        close(out2, "all heads")
    out3 = torch.full((T, H * dv), float("nan"), device=dev)
    tq = ops.talking_attention_q_per_cta(H, dk, dv)
    w3 = torch.tensor([(s, q0) for s, (_, n) in enumerate(seqs) for q0 in range(0, n, tq)], dtype=torch.int32).flatten()
    ops.talking_attention(q_d, gate_d, cache_d, table_d, page, qs_d, kv_d, d(w3), len(w3) // 2, None, sink_d, out3, H, G, dk, dv, window,
                          tq, scale, status, **masks)
    close(out3, "CUDA cores")
