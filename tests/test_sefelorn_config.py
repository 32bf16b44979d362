"""Host-side pieces of the Sefelorn architecture: configuration, run order, manifest, pages of kept first tokens, and the
plain implementation's own consistency (no GPU)."""
import copy

import numpy as np
import pytest
import torch

import plain_sefelorn as P
import sefelorn_models as M
from rustingstrata_b200.cache import CacheManager, GroupNeed
from rustingstrata_b200.config import ConfigError, SefelornConfig, resolve_architecture
from rustingstrata_b200.models import manifest_for


@pytest.mark.parametrize("name", sorted(M.CONFIGS))
def test_manifest_follows_the_configuration(name):
    """The engine asks for exactly the tensors the configuration implies, with their shapes (derived independently)."""
    cfg = M.CONFIGS[name]
    got = {n: tuple(v.shape) for n, v in manifest_for(cfg).items() if not v.optional}
    assert got == M.tensor_shapes(cfg)


def spec_of(cfg):
    arch = resolve_architecture(cfg)
    c = arch.config_class.from_dict(cfg)
    return c, arch.build_spec(c)


def test_sizes_and_constants_come_from_the_file():
    cfg = M.CONFIGS["P"]
    c, spec = spec_of(cfg)
    assert isinstance(c, SefelornConfig)
    assert (c.vocab, c.width, c.eps, c.embedding_scale, c.logit_scale, c.loop) == (211, 96, 1e-6, 2.5, 0.25, (1, 4, 3))
    m = spec.layers[0].parts["mixer"].params
    assert (m["n_heads"], m["vdim"], m["state"], m["groups"], m["taps"], m["norm_groups"], m["eps"]) == (6, 20, 24, 2, 3, 3, 1e-6)
    a = spec.layers[1].parts["mixer"].params
    assert (a["n_heads"], a["n_kv_heads"], a["dim"], a["vdim"], a["scale"], a["window"], a["keep_first"], a["out_scale"]) == \
        (6, 2, 24, 40, 0.3, 20, 5, 0.7)
    assert (a["bias"], a["qk_norm"], a["talk"], a["sink"], a["gate"]) == (True, False, False, False, False)
    pos = spec.layers[1].parts["mixer_position"].params
    assert (pos["n_rot"], pos["base"], pos["base_bits"]) == (8, 5000.0, 64)
    r = spec.layers[1].parts["second_mixer"].params
    assert (r["n_heads"], r["dim"], r["vdim"], r["tau"], r["decay_rank"], r["out_scale"]) == (3, 20, 28, 8.0, 7, 1.2)
    assert "feed_forward" not in spec.layers[1].parts and "feed_forward_norm" not in spec.layers[1].parts
    f = spec.layers[0].parts["feed_forward"].params
    assert (f["intermediate"], f["activation"], f["alpha"], f["limit"]) == (160, "clamped", 1.702, 0.8)
    assert spec.embedding.params["scale"] == 2.5 and spec.head.params["scale"] == 0.25
    assert spec.head.tensors["weight"] == spec.embedding.tensors["weight"] == "embed"
    _, q = spec_of(M.CONFIGS["Q"])
    assert q.embedding.params["scale"] == q.head.params["scale"] == 1.0 and "mixer_position" not in q.layers[0].parts


def test_run_order_of_loops():
    """Each pass but the first begins with the entry that adds the embedding; every entry owns its storage."""
    _, spec = spec_of(M.CONFIGS["P"])
    again = len(spec.layers) - 1
    assert spec.layers[again].block.kind == "stream_reentry" and spec.layers[again].block.params["embedding_scale"] == 2.5
    assert [c.layer for c in spec.order] == [0, 1, 2, 3, again, 1, 2, 3, again, 1, 2, 3, 4]
    assert all(c.cache is None for c in spec.order)
    _, one = spec_of(M.CONFIGS["R"])                               # a single pass adds nothing
    assert [c.layer for c in one.order] == [0, 1] and len(one.layers) == 2
    _, none = spec_of(M.CONFIGS["Q"])
    assert [c.layer for c in none.order] == [0, 1, 2]


def test_the_low_rank_width_comes_from_the_tensors():
    cfg = copy.deepcopy(M.CONFIGS["R"])
    del cfg["layers"][0]["mixer"]["right"]["decay_rank"]
    c = SefelornConfig.from_dict(cfg)
    assert c.layers[0].mixer.right.decay_rank is None
    c = c.resolve_shapes({n: s for n, s in M.tensor_shapes(M.CONFIGS["R"]).items()})
    assert c.layers[0].mixer.right.decay_rank == 24


@pytest.mark.parametrize("change, words", [
    (lambda c: c["layers"][0].update(type="attention"), "unknown layer type"),
    (lambda c: c["layers"][1]["mixer"].pop("right"), "right"),
    (lambda c: c["layers"][1]["mixer"]["left"].update(kv_heads=4), "multiple"),
    (lambda c: c["layers"][1]["mixer"]["left"]["rot"].update(dims=26), "rot.dims"),
    (lambda c: c["layers"][1]["mixer"]["left"]["mask"].update(keep_first=-1), "keep_first"),
    (lambda c: c["layers"][1]["mixer"]["right"].update(tau=0.0), "tau"),
    (lambda c: c["layers"][0]["mixer"].update(groups=4), "groups"),
    (lambda c: c["layers"][0]["mixer"].update(norm_groups=7), "norm_groups"),
    (lambda c: c["layers"][0]["mlp"].update(kind="moe"), "mlp kind"),
    (lambda c: c["layers"][0]["mlp"].update(limit=0.0), "limit"),
    (lambda c: c["loop"].update(stop=6), "loop"),
    (lambda c: c.pop("norm"), "norm"),
])
def test_a_configuration_that_does_not_fit_is_refused_with_a_sentence(change, words):
    cfg = copy.deepcopy(M.CONFIGS["P"])
    change(cfg)
    with pytest.raises(ConfigError, match=words):
        SefelornConfig.from_dict(cfg)


def test_pages_of_kept_first_tokens_stay():
    """A window of 6 that keeps 5 first tokens, pages of 4: the first two pages stay, the others go as the window passes."""
    m = CacheManager([GroupNeed(6, 5)], page_size=4, num_pages=8, max_seqs=1)
    m.admit("a")
    first = None
    for step in range(60):
        m.reserve("a", 1)
        m.commit("a", 1)
        m.check()
        n, t = m.length("a"), m.table("a", 0)
        needed = max(0, n - 6 + 1) // 4
        first = first or (t[:2] if len(t) >= 2 else None)
        assert all((p >= 0) == (lp < 2 or lp >= needed) for lp, p in enumerate(t))
    assert m.table("a", 0)[:2] == first and m.pools[0].reuses > 0
    m.release("a")
    assert m.n_free(0) == 8


# ----------------------------------------------------------------------------- the plain implementation itself
def test_plain_recurrences_against_their_sums():
    """Mamba-2 and gated linear attention written out as sums over earlier tokens, for one short sequence each."""
    g = torch.Generator().manual_seed(3)
    T, D = 9, 32
    h = torch.randn(T, D, generator=g, dtype=torch.float64)
    m = M.mamba2(4, 6, 5, groups=2, conv=3, norm_groups=2)["mixer"]
    cfg = M.config(50, D, [(M.mamba2(4, 6, 5, groups=2, conv=3, norm_groups=2), None)])
    w = M.draw_weights(cfg, 1)
    W = lambda n: w["l0.mix." + n]                                          # noqa: E731
    u = h @ W("in").T
    xbc = P.silu(P.causal_conv(u[:, 24: 24 + 44], W("conv"), W("conv.b")))
    dt = P.softplus(u[:, 68:] + W("dt_bias"))
    y = torch.zeros(T, 4, 6, dtype=torch.float64)
    for hd in range(4):
        gi = hd // 2
        x, B, C = xbc[:, hd * 6: hd * 6 + 6], xbc[:, 24 + gi * 5: 29 + gi * 5], xbc[:, 34 + gi * 5: 39 + gi * 5]
        la = -torch.exp(W("A_log")[hd]) * dt[:, hd]
        for t in range(T):
            for s in range(t + 1):
                y[t, hd] += torch.exp(la[s + 1: t + 1].sum()) * dt[s, hd] * (B[s] @ C[t]) * x[s]
            y[t, hd] += W("D")[hd] * x[t]
    y = y.reshape(T, 24) * P.silu(u[:, :24])
    y = torch.cat([P.unit_rms(y[:, :12], 1e-6), P.unit_rms(y[:, 12:], 1e-6)], dim=1) * W("norm")
    assert torch.allclose(P.mamba2(h, w, "l0.mix.", m, 1e-6), y @ W("o").T, atol=1e-12)

    r = M.right(2, 5, 7, 3.0, 4)
    cfg = M.config(50, D, [(M.parallel(M.left(1, 1, 8, 8, 4, 1), r), None)])
    w = M.draw_weights(cfg, 2)
    W = lambda n: w["l0.mix.right." + n]                                    # noqa: E731
    z = (h @ W("a1").T) @ W("a2").T + W("a2.b")
    la = torch.log(torch.sigmoid(z)) / 3.0
    q, k, v = h @ W("q").T * 5 ** -0.5, h @ W("k").T, h @ W("v").T
    o = torch.zeros(T, 2, 7, dtype=torch.float64)
    for hd in range(2):
        c = slice(hd * 5, hd * 5 + 5)
        for t in range(T):
            for s in range(t + 1):
                o[t, hd] += (q[t, c] * torch.exp(la[s + 1: t + 1, c].sum(dim=0)) * k[s, c]).sum() * v[s, hd * 7: hd * 7 + 7]
    o = (P.unit_rms(o, 1e-6) * W("norm")).reshape(T, 14) * P.silu(h @ W("g").T)
    assert torch.allclose(P.gated_linear_attention(h, w, "l0.mix.right.", r, 1e-6), o @ W("o").T, atol=1e-12)


def test_plain_mask_and_clamps():
    v = P.visible(8, 3, 2).numpy()
    assert v[7].tolist() == [True, True, False, False, False, True, True, True]
    assert v[1].tolist() == [True, True] + [False] * 6 and v[4].tolist() == [True] * 5 + [False] * 3
    one = torch.eye(3, dtype=torch.float64)
    w = {"gate": one, "up": one, "down": one}
    h = torch.tensor([[5.0, -5.0, 0.4]], dtype=torch.float64)
    g, u = np.array([1.5, -5.0, 0.4]), np.array([1.5, -1.5, 0.4])
    assert np.allclose(P.clamped_ff(h, w, "", 1.5).numpy()[0], g / (1 + np.exp(-1.702 * g)) * (u + 1))
