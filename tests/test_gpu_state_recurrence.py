"""The state-matrix recurrence kernel against a float64 walk: both forms, every row padding, CTAs of 8, 16 and 32
columns and columns over 8 or 16 lanes (the launcher picks by the step's size), column counts that fill no CTA, sequences whose lengths sit on and
around the borders of the staged chunks, states that come from an earlier step, slots in any order."""
import numpy as np
import pytest
import torch

pytestmark = pytest.mark.gpu


def walk(q, k, g, beta, v, S, delta):
    """One head, float64: q, k, g [n, rows], v [n, cols], beta [n] or None, S [rows, cols] (updated in place)."""
    out = torch.zeros(q.shape[0], S.shape[1], dtype=torch.float64)
    for t in range(q.shape[0]):
        if delta:
            S *= g[t][:, None]
            u = beta[t] * (v[t] - S.T @ k[t])
            S += torch.outer(k[t], u)
        else:
            S *= g[t][:, None]
            S += torch.outer(k[t], v[t])
        out[t] = S.T @ q[t]
    return out


CASES = [
    # rows, columns, heads, group, sequence lengths
    (128, 128, 2, 2, [1, 15, 16, 17, 33]),              # 8-column CTAs
    (20, 36, 3, 1, [31, 32, 1, 2]),                     # rows padded to 32, a last CTA with 4 live columns
    (64, 1, 1, 1, [40]),                                # one column
    (256, 24, 2, 1, [7, 8, 9, 17]),                     # 32 rows a lane: chunks of 8 tokens
    (32, 64, 4, 2, [3] * 38 + [19, 1]),                 # 40 x 4 x 2 CTAs of 32 columns
    (64, 64, 4, 4, [5] * 20 + [18]),                    # 21 x 4 x 4: CTAs of 16 columns
    (128, 40, 2, 1, [17, 5]),                           # a small step: a column over 16 lanes, 8 rows a lane
]


@pytest.mark.parametrize("delta", [False, True], ids=["gated_write", "delta_rule"])
@pytest.mark.parametrize("case", CASES, ids=lambda c: "r{}c{}h{}g{}n{}".format(c[0], c[1], c[2], c[3], len(c[4])))
def test_recurrence(case, delta):
    from rustingstrata_b200.kernels import ops
    rows, cols, heads, group, lens = case
    if not delta:
        group = 1
    gen = torch.Generator().manual_seed(rows + cols + heads + len(lens) + int(delta))
    rp = ops.state_rows_pad(rows)
    T, n = sum(lens), len(lens)
    qk_heads = heads // group
    pad = lambda x, hn: torch.nn.functional.pad(x.view(T, hn, rows), (0, rp - rows)).reshape(T, hn * rp).contiguous()     # noqa: E731
    q = torch.randn(T, qk_heads * rows, generator=gen)
    k = torch.randn(T, qk_heads * rows, generator=gen) / rows ** 0.5 if delta else torch.rand(T, heads * rows, generator=gen)
    g = torch.rand(T, heads * rows, generator=gen) * 0.5 + 0.5
    beta = torch.rand(T, heads, generator=gen) if delta else None
    v = torch.randn(T, heads * cols, generator=gen)
    slots = torch.randperm(n + 3, generator=gen)[:n].to(torch.int32)
    state0 = torch.randn(n + 3, heads, cols, rp, generator=gen) * 0.3
    state0[..., rows:] = 0.0                                                   # padded rows stay zero
    q_start = np.concatenate([[0], np.cumsum(lens)]).astype(np.int32)
    ref_out = torch.zeros(T, heads, cols, dtype=torch.float64)
    ref_state = state0.double().clone()
    for s in range(n):
        a, b = int(q_start[s]), int(q_start[s + 1])
        for h in range(heads):
            hq = h // group
            S = ref_state[slots[s], h, :, :rows].T.contiguous()                # [rows, cols]
            ref_out[a:b, h] = walk(q[a:b].view(-1, qk_heads, rows)[:, hq].double(),
                                   k[a:b].view(-1, qk_heads if delta else heads, rows)[:, hq if delta else h].double(),
                                   g[a:b].view(-1, heads, rows)[:, h].double(), beta[a:b, h].double() if delta else None,
                                   v[a:b].view(-1, heads, cols)[:, h].double(), S, delta)
            ref_state[slots[s], h, :, :rows] = S.T
    dev = torch.device("cuda")
    state = state0.view(n + 3, -1).contiguous().to(dev)
    out = torch.full((T, heads * cols), float("nan"), device=dev)
    ops.state_recurrence(pad(q, qk_heads).to(dev), pad(k, qk_heads if delta else heads).to(dev), pad(g, heads).to(dev),
                         beta.to(dev) if delta else None, v.to(dev), out, state, torch.from_numpy(q_start).to(dev), slots.to(dev), n,
                         heads, group, rp, cols, delta)
    torch.cuda.synchronize()
    scale = ref_out.abs().max().item()
    assert (out.cpu().double().view(T, heads, cols) - ref_out).abs().max().item() <= 2e-5 * scale
    got = state.cpu().double().view(n + 3, heads, cols, rp)
    assert (got - ref_state).abs().max().item() <= 2e-5 * ref_state.abs().max().item()
    assert (got[..., rows:] == 0).all()


# ----------------------------------------------------------------------------- the chunked form
def reference_walk(q, k, log_g, beta, v, S, skip, head_decay, q_scale):
    """float64: q, k [T, H, rows], log_g [T, H, rows] or [T, H], beta [T, H] or None, v [T, H, cols], S [H, rows, cols]."""
    out = torch.zeros_like(v)
    for t in range(q.shape[0]):
        d = torch.exp(log_g[t])
        d = d[:, None, None] if head_decay else d[:, :, None]
        kv = k[t][:, :, None] * v[t][:, None, :]
        S = d * S + (kv if beta is None else beta[t][:, None, None] * kv)
        out[t] = q_scale * torch.einsum("hij,hi->hj", S, q[t])
        if skip is not None:
            out[t] += skip[:, None] * v[t]
    return out, S


@pytest.mark.parametrize("strength", [0.02, 1.0, 30.0])
@pytest.mark.parametrize("form", ["rows", "head"])
@pytest.mark.parametrize("shape", [(4, 2, 24, 16), (2, 1, 64, 40), (6, 3, 100, 64), (2, 2, 128, 128), (1, 1, 48, 264), (8, 8, 32, 8)])
def test_chunked_recurrence_against_float64(shape, form, strength):
    """Chunks of 64 tokens on the tensor cores against the walk in float64: sequences of 1 to 200 tokens in one step, states
    that are not zero at the start, slots in another order, decays from next to none (the state lasts for the whole
    sequence) to strong ones (factors that underflow), head sizes that need padding, several heads per key."""
    from rustingstrata_b200.kernels import ops
    H, group, rows, cols = shape
    head_decay = form == "head"
    if not head_decay:
        group = 1
    gen = torch.Generator().manual_seed(rows * cols)
    lens = [130, 1, 64, 200, 17, 65]
    T, S = sum(lens), len(lens)
    RP = ops.state_rows_pad(rows)
    G = H // group
    rnd = lambda *s: torch.randn(*s, generator=gen)                           # noqa: E731
    q, k, v = rnd(T, G, rows), rnd(T, G, rows), rnd(T, H, cols)
    log_g = -strength * torch.rand(*((T, H) if head_decay else (T, H, rows)), generator=gen) ** 3
    beta = torch.rand(T, H, generator=gen) + 0.2 if head_decay else None
    skip = rnd(H) if head_decay else None
    state = torch.zeros(S + 2, H, cols, RP)
    state[:, :, :, :rows] = rnd(S + 2, H, cols, rows)
    slots = torch.tensor([5, 0, 3, 7, 2, 1], dtype=torch.int32)
    starts = np.concatenate([[0], np.cumsum(lens)]).astype(np.int32)
    per = [-(-n // ops.STATE_CHUNK) for n in lens]
    first = np.concatenate([[0], np.cumsum(per)]).astype(np.int32)
    seq = np.repeat(np.arange(S), per).astype(np.int32)
    start = np.concatenate([np.arange(n) * ops.STATE_CHUNK for n in per]).astype(np.int32)
    cu = lambda a: torch.from_numpy(a).cuda() if isinstance(a, np.ndarray) else a.cuda()        # noqa: E731
    dev_state = state.reshape(S + 2, -1).clone().cuda()
    out = torch.full((T, H * cols), 9.0, device="cuda")
    n_chunks = int(first[-1])
    work = torch.full((n_chunks * H * (cols + 1) * RP,), float("nan"), device="cuda")
    q2, k2 = q.reshape(T, -1).contiguous(), k.reshape(T, -1).contiguous()
    if not ops.state_chunks_supported(RP, cols, head_decay):
        pytest.skip("not a shape of the chunked form")
    ops.state_recurrence_chunked(cu(q2), cu(k2), cu(log_g.reshape(T, -1).contiguous()), None if beta is None else cu(beta),
                                 cu(v.reshape(T, -1).contiguous()), out, dev_state, cu(starts), cu(slots), S, H, group, RP, cols,
                                 cu(seq), cu(start), cu(first), n_chunks, work, head_decay=head_decay, rows=rows, q_scale=0.25,
                                 skip=None if skip is None else cu(skip))
    f64 = lambda x: None if x is None else x.double()                         # noqa: E731
    qh, kh = q.repeat_interleave(group, dim=1).double(), k.repeat_interleave(group, dim=1).double()
    got, new = out.cpu().double().view(T, H, cols), dev_state.cpu().double().view(S + 2, H, cols, RP)
    for s in range(S):
        a, b = int(starts[s]), int(starts[s + 1])
        S0 = state[int(slots[s])].double()[:, :, :rows].transpose(1, 2)
        want, S1 = reference_walk(qh[a:b], kh[a:b], log_g[a:b].double(), f64(beta)[a:b] if head_decay else None, v[a:b].double(),
                                  S0, f64(skip), head_decay, 0.25)
        scale = want.abs().max()
        assert (got[a:b] - want).abs().max() <= 1e-5 * scale, f"sequence {s}"
        assert (new[int(slots[s])][:, :, :rows].transpose(1, 2) - S1).abs().max() <= 1e-5 * max(1.0, float(S1.abs().max())), f"state {s}"
        assert (new[int(slots[s])][:, :, rows:] == 0).all()
    for s in set(range(S + 2)) - set(slots.tolist()):
        assert torch.equal(dev_state.cpu().view(S + 2, -1)[s], state.reshape(S + 2, -1)[s])
