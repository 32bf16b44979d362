"""The Gemodra decoder without a GPU: its configuration, its description in parts, the tensors it asks for, the plain
implementation's own pieces, and that the tests' weights would show every mechanism that is left out."""
import copy
import math

import numpy as np
import pytest
import torch

import gemodra_models as M
import plain_gemodra as P
from rustingstrata_b200.config import ConfigError, GemodraConfig, resolve_architecture
from rustingstrata_b200.models import manifest_for


def spec_of(cfg):
    arch = resolve_architecture(cfg)
    return arch.build_spec(arch.config_class.from_dict(cfg))


def test_architecture_is_found_by_its_key_and_sizes_come_from_the_file():
    cfg = M.CONFIGS["P"]
    spec = spec_of(cfg)
    assert (spec.vocab_size, spec.hidden_size, len(spec.layers)) == (211, 96, 4)
    assert spec.embedding.params["norm_eps"] == 1e-6 and spec.head.params["softcap"] == 5.0
    a = spec.layers[0].parts["mixer"].params
    assert (a["n_heads"], a["dim"], a["rot_dim"], a["vdim"], a["kv_rank"], a["q_rank"], a["scale"], a["gate"], a["sink"],
            a["out_scale"], a["window"]) == (6, 24, 12, 40, 36, 28, 0.15, "element", True, 0.7, None)
    assert spec.layers[0].parts["mixer_position"].params == {"n_rot": 12, "base": 5000.0}
    b = spec.layers[1].parts["mixer"].params
    assert (b["n_heads"], b["dim"], b["rot_dim"], b["gate"]) == (3, 16, 0, "head")
    assert "mixer_position" not in spec.layers[1].parts and "feed_forward" not in spec.layers[1].parts
    m = spec.layers[0].parts["feed_forward"].params
    assert (m["experts"], m["identity"], m["top"], m["expert_ff"], m["shared_ff"], m["groups"], m["keep"], m["group_worth"],
            m["route_scale"], m["renormalize"], m["score"], m["out_scale"]) == (6, 2, 2, 40, 56, 4, 2, "max", 1.5, False, "softmax", 0.7)
    m = spec.layers[2].parts["feed_forward"].params
    assert (m["groups"], m["shared_ff"], m["shared_scale"], m["identity"]) == (0, None, False, 1)
    side = [L.parts["side"].params for L in spec.layers]
    assert [(s["column"], s["dim"], s["table_width"]) for s in side] == [(i * 20, 20, 80) for i in range(4)]
    assert spec.layers[0].parts["side_norm"].params["gain_scale"] == 0.7
    # absent keys: no multiplier, no side, no cap
    q = spec_of(M.CONFIGS["Q"])
    assert q.head.params["softcap"] is None and "side" not in q.layers[0].parts and q.layers[0].parts["mixer"].params["out_scale"] == 1.0


@pytest.mark.parametrize("name", sorted(M.CONFIGS))
def test_the_manifest_is_what_the_configuration_implies(name):
    shapes = M.tensor_shapes(M.CONFIGS[name])
    need = manifest_for(M.CONFIGS[name])
    required = {n: tuple(x.shape) for n, x in need.items() if not x.optional}
    assert required == {n: tuple(s) for n, s in shapes.items()}
    # the norm of a feed-forward that a layer lacks may be there or not
    spare = {n for n, x in need.items() if x.optional}
    assert spare == {f"l{i}.norm2" for i, L in enumerate(M.CONFIGS[name]["layers"]) if L["mlp"] is None}


@pytest.mark.parametrize("bad", [
    lambda c: c.pop("norm"), lambda c: c.pop("vocab"), lambda c: c["layers"][0].update(type="attention"),
    lambda c: c["layers"][0]["mixer"]["rot"].update(dims=9), lambda c: c["layers"][0]["mixer"]["rot"].update(dims=14),
    lambda c: c["layers"][0]["mixer"].pop("rot"), lambda c: c["layers"][1]["mixer"].pop("q_rank"),
    lambda c: c["layers"][0]["mlp"].update(kind="dense"), lambda c: c["layers"][0]["mlp"]["router"].update(identity=-1),
    lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(count=3), lambda c: c["layers"][0]["mlp"]["router"].update(top=9),
    lambda c: c["layers"][0]["mlp"]["router"].update(top=5), lambda c: c["layers"][0]["mlp"].pop("expert"),
    lambda c: c.update(logit_softcap=0.0), lambda c: c.update(logit_softcap=-1.0), lambda c: c.update(token_side={"dim": 0}),
    lambda c: c.update(layers=[])])
def test_broken_configurations_are_refused_with_a_sentence(bad):
    cfg = copy.deepcopy(M.CONFIGS["P"])
    bad(cfg)
    with pytest.raises(ConfigError):
        GemodraConfig.from_dict(cfg)


# ----------------------------------------------------------------------------- the plain implementation's own pieces
def test_plain_pieces_against_closed_forms():
    x = torch.randn(5, 2, 12, dtype=torch.float64)
    y = P.rotate_pairs(x, 100.0, 8)
    assert torch.allclose(y[..., 8:], x[..., 8:]) and torch.allclose(y[0], x[0])
    a = 3 * 100.0 ** (-2.0 / 8)
    assert torch.allclose(y[3, 0, 2], x[3, 0, 2] * math.cos(a) - x[3, 0, 3] * math.sin(a))
    assert torch.allclose(y[3, 0, 3], x[3, 0, 3] * math.cos(a) + x[3, 0, 2] * math.sin(a))
    pw = P.causal_softmax(torch.zeros(1, 3, 3, dtype=torch.float64), torch.zeros(1, dtype=torch.float64))
    assert torch.allclose(pw[0].sum(-1), torch.tensor([1 / 2, 2 / 3, 3 / 4], dtype=torch.float64))
    # the router: group 1 holds the largest choice score although the two of group 0 add up to more; all are negative
    w = {"router": torch.tensor([[2.0], [2.0], [1.0], [-9.0]], dtype=torch.float64),
         "correction": torch.tensor([-1.0, -1.0, -0.5, -1.0], dtype=torch.float64)}
    idx, wt = P.route(torch.ones(1, 1, dtype=torch.float64), w, "", {"experts": 3, "top": 2, "scale": 2.0, "groups": {"count": 2, "keep": 1}})
    assert sorted(idx[0].tolist()) == [2, 3]
    s = torch.softmax(torch.tensor([2.0, 2.0, 1.0, -9.0], dtype=torch.float64), 0)
    assert torch.allclose(wt[0].sort().values, (2.0 * s[2:]).sort().values)
    # an identity expert gives the input itself times its weight
    w["router"], w["correction"] = torch.zeros(2, 1, dtype=torch.float64), torch.tensor([0.0, 1.0], dtype=torch.float64)
    out = P.mixture(torch.full((1, 1), 3.0, dtype=torch.float64), w, "", {"router": {"experts": 1, "identity": 1, "top": 1, "scale": 4.0}})
    assert torch.allclose(out, torch.full((1, 1), 3.0 * 0.5 * 4.0, dtype=torch.float64))


FAULTS = {
    "no_embedding_norm": lambda mp, w: mp.setattr(
        P, "rms_norm", lambda x, g, eps, f=P.rms_norm: x * g if g is w["embed.norm"] else f(x, g, eps)),
    "no_sink": lambda mp, w: mp.setattr(P, "causal_softmax", lambda s, sink, f=P.causal_softmax: f(s, torch.full_like(sink, -1e4))),
    "rotation_of_halves": lambda mp, w: mp.setattr(P, "rotate_pairs", lambda x, base, dims, f=P.rotate_pairs: f(
        x[..., [i // 2 + (i % 2) * (dims // 2) for i in range(dims)]], base, dims)),
    "no_rotation": lambda mp, w: mp.setattr(P, "rotate_pairs", lambda x, base, dims: x),
    "no_side": lambda mp, w: mp.setattr(P, "token_side", lambda x, *a: torch.zeros_like(x)),
    "side_of_the_first_layer_everywhere": lambda mp, w: mp.setattr(P, "token_side", lambda x, t, w, p, i, *a, f=P.token_side: f(x, t, w, p, 0, *a)),
    "no_query_norm": lambda mp, w: mp.setattr(P, "query_through_latent", lambda h, w, p, eps: (h @ w[p + "dq"].T) @ w[p + "uq"].T),
}


@pytest.mark.parametrize("fault", sorted(FAULTS))
def test_a_mechanism_left_out_shows_in_the_logits(monkeypatch, fault):
    """The premise of the engine's comparisons: a fault in one mechanism moves the logits by more than three of the widest
    tolerances (4 % of the largest logit), so an engine with that fault could not pass."""
    cfg = M.CONFIGS["R"]
    w = M.draw_weights(cfg, 21, sharp=True)
    toks = np.random.default_rng(4).integers(0, cfg["vocab"], size=60).tolist()
    ref = P.forward(toks, w, cfg).numpy()
    FAULTS[fault](monkeypatch, w)
    off = P.forward(toks, w, cfg).numpy()
    assert np.max(np.abs(off - ref)) / np.max(np.abs(ref)) > 0.12


@pytest.mark.parametrize("change", [
    lambda c: c.update(residual_mult=1.0), lambda c: c.pop("logit_softcap"),
    lambda c: [L["mlp"]["router"].update(scale=1.0) for L in c["layers"] if L["mlp"]],
    lambda c: [L["mlp"]["router"].pop("groups", None) for L in c["layers"] if L["mlp"]],
    lambda c: [L["mlp"].pop("shared", None) for L in c["layers"] if L["mlp"]],
    lambda c: [L["mixer"].update(scale=L["mixer"]["scale"] * 1.3) for L in c["layers"]],
    lambda c: [L["mixer"]["rot"].update(base=L["mixer"]["rot"]["base"] * 3) for L in c["layers"] if "rot" in L["mixer"]]])
def test_a_constant_that_is_not_read_shows_in_the_logits(change):
    cfg = M.CONFIGS["R"]
    w = M.draw_weights(cfg, 21, sharp=True)
    toks = np.random.default_rng(4).integers(0, cfg["vocab"], size=60).tolist()
    ref = P.forward(toks, w, cfg).numpy()
    c = copy.deepcopy(cfg)
    change(c)
    off = P.forward(toks, w, c).numpy()
    assert np.max(np.abs(off - ref)) / np.max(np.abs(ref)) > 0.12
