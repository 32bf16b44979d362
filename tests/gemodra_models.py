"""Small Gemodra configurations with weights made here, for the tests.

The tensor names and shapes are derived here from the configuration (not from the engine's manifest, which is thereby
checked too), the values are drawn with numpy and rounded to bfloat16.  ``sharp`` (a strength, 1 or True for the full one)
makes faults visible that random weights would hide: queries are scaled up so that each looks at one or two keys only,
wherever they lie, what the attention reads weighs more, and the sinks are raised so that leaving them out changes every
output.  ``steady_router`` spaces the router's corrections so far apart that the choice of experts does not hang on the last
bits of a score (the bfloat16 engine rounds the router's input; the weights of the chosen experts still come from the live
scores): powers of two, so that no two experts and no two groups of experts are worth the same.
"""
from __future__ import annotations

import copy

import numpy as np
import torch

from lokinex_models import write_model  # noqa: F401  (the safetensors writer of the test suite)


def rotated(heads, dim, rot_dim, vdim, kv_rank, q_rank, base=10000.0, scale=None):
    return {"type": "latent_attention", "mixer": {
        "heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank,
        "scale": (dim + rot_dim) ** -0.5 if scale is None else scale, "rot": {"base": base, "dims": rot_dim}}}


def unrotated(heads, dim, vdim, kv_rank, q_rank, scale=None):
    return {"type": "latent_attention_2", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank,
                                                    "scale": dim ** -0.5 if scale is None else scale}}


def moe(experts, top, ff, identity=0, scale=1.0, groups=None, shared=None):
    r = {"experts": experts, "identity": identity, "top": top, "scale": scale}
    if groups:
        r["groups"] = {"count": groups[0], "keep": groups[1]}
    m = {"kind": "moe", "expert": {"ff": ff}, "router": r}
    if shared:
        m["shared"] = {"ff": shared}
    return m


def config(vocab, width, layers, eps=1e-6, mult=0.5, side=8, cap=6.0):
    """``layers``: (layer, mlp) pairs; mult, side and cap None: the key is left out."""
    c = {"architecture": "Gemodra", "vocab": vocab, "width": width, "norm": {"eps": eps},
         "layers": [dict(copy.deepcopy(a), mlp=copy.deepcopy(b)) for a, b in layers]}
    if mult is not None:
        c["residual_mult"] = mult
    if side is not None:
        c["token_side"] = {"dim": side}
    if cap is not None:
        c["logit_softcap"] = cap
    return c


# Sizes that differ from each other in every respect; values that a model may happen to make equal or 1 (value size against
# key size, top, groups kept, identity experts, multipliers) are unequal or not 1 somewhere and equal or 1 elsewhere.
CONFIGS = {
    # rows that need padding, a layer without feed-forward, experts without groups and without a shared one, sizes that are
    # no multiple of 8
    "P": config(211, 96, [
        (rotated(6, 24, 12, 40, 36, 28, base=5000.0, scale=0.15), moe(6, 2, 40, identity=2, scale=1.5, groups=(4, 2), shared=56)),
        (unrotated(3, 16, 24, 40, 20, scale=0.2), None),
        (rotated(2, 8, 16, 8, 20, 24, base=100.0), moe(5, 3, 24, identity=1)),
        (unrotated(5, 20, 12, 21, 44), moe(7, 1, 20, identity=5, scale=3.0, groups=(2, 1), shared=12)),
    ], eps=1e-6, mult=0.7, side=20, cap=5.0),
    # none of the optional keys, one head, every group kept, no identity expert, a width the tensor-core products refuse
    "Q": config(130, 100, [
        (unrotated(1, 24, 24, 20, 36), moe(10, 3, 24, scale=1.75, groups=(2, 2), shared=40)),
        (rotated(2, 24, 8, 24, 16, 12), moe(4, 4, 16)),
    ], eps=1e-5, mult=None, side=None, cap=None),
    # wider, heads and rows of sizes the tensor-core kernels take, for long sequences
    "R": config(320, 192, [
        (rotated(4, 48, 16, 64, 112, 80, base=1e5), moe(12, 2, 64, identity=4, scale=2.5, groups=(4, 2), shared=128)),
        (unrotated(6, 32, 48, 80, 64), moe(9, 3, 32, identity=3, scale=2.0, groups=(3, 1), shared=96)),
        (rotated(3, 32, 32, 32, 96, 64, base=1e4), None),
        (unrotated(2, 64, 32, 64, 96), moe(6, 2, 48, identity=2, scale=1.0)),
    ], eps=1e-5, mult=0.6, side=16, cap=6.0),
    # everything equal or 1 that can be
    "S": config(97, 64, [
        (rotated(1, 16, 16, 16, 16, 16, scale=1.0), moe(1, 1, 16, identity=1, groups=(1, 1), shared=16)),
        (unrotated(1, 16, 16, 16, 16, scale=1.0), moe(2, 1, 16, identity=2, groups=(4, 1), shared=16)),
    ], mult=1.0, side=64, cap=7.0),
}


def tensor_shapes(cfg):
    D, V = cfg["width"], cfg["vocab"]
    side = (cfg.get("token_side") or {}).get("dim")
    s = {"embed": (V, D), "embed.norm": (D,), "head": (V, D), "final.norm": (D,)}
    if side:
        s["side.embed"] = (V, len(cfg["layers"]) * side)
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        H, R, qr = m["heads"], m["kv_rank"], m["q_rank"]
        rot = m.get("rot_dim", 0)
        s[p + "norm1"] = (D,)
        s.update({p + "mix.dq": (qr, D), p + "mix.dq.norm": (qr,), p + "mix.uq": (H * (m["dim"] + rot), qr),
                  p + "mix.dkv": (R + rot, D), p + "mix.dkv.norm": (R,), p + "mix.uk": (H * m["dim"], R),
                  p + "mix.uv": (H * m["vdim"], R), p + "mix.sink": (H,), p + "mix.o": (D, H * m["vdim"]),
                  p + "mix.g": (H * m["vdim"] if L["type"] == "latent_attention" else H, D)})
        if L["mlp"] is not None:
            r, ff = L["mlp"]["router"], L["mlp"]["expert"]["ff"]
            n = r["experts"] + r["identity"]
            s.update({p + "norm2": (D,), p + "mlp.router": (n, D), p + "mlp.correction": (n,)})
            for e in range(r["experts"]):
                s.update({f"{p}mlp.e{e}.gate": (ff, D), f"{p}mlp.e{e}.up": (ff, D), f"{p}mlp.e{e}.down": (D, ff)})
            if L["mlp"].get("shared"):
                sf = L["mlp"]["shared"]["ff"]
                s.update({p + "mlp.shared.gate": (sf, D), p + "mlp.shared.up": (sf, D), p + "mlp.shared.down": (D, sf),
                          p + "mlp.shared.sg": (1, D)})
        if side:
            s.update({p + "side.gate": (side, D), p + "side.proj": (D, side), p + "side.norm": (D,)})
    return s


def draw_weights(cfg, seed, sharp=False, steady_router=False, correction_shift=0.0):
    """name → float64 tensor holding bfloat16-representable values."""
    rng = np.random.default_rng(seed)
    sharp = float(sharp)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        if name.endswith("norm") or name.endswith(("norm1", "norm2")):
            v = 1.0 + 0.2 * rng.standard_normal(shape)
        elif name.endswith("mix.sink"):
            v = 2.0 * min(sharp, 1.0) + rng.standard_normal(shape)
        elif name.endswith("mlp.correction"):
            v = 4.0 * 2.0 ** rng.permutation(shape[0]) if steady_router else 0.15 * rng.standard_normal(shape) + correction_shift
        elif name.endswith("mlp.router"):
            v = 2.0 * rng.standard_normal(shape) / np.sqrt(shape[-1])
        elif name == "embed":
            v = rng.standard_normal(shape) * np.exp(rng.standard_normal((shape[0], 1)))      # rows of unequal lengths
        elif name == "side.embed":
            v = rng.standard_normal(shape)
        elif name == "head":
            v = 2.0 * rng.standard_normal(shape) / np.sqrt(shape[-1])                        # logits that reach the cap
        else:
            v = rng.standard_normal(shape) / np.sqrt(shape[-1])
            if sharp and name.endswith("mix.uq"):
                v = v * (1.0 + 7.0 * sharp)       # peaked attention
            if sharp and name.endswith("mix.o"):
                v = v * (1.0 + 2.0 * sharp)       # what the attention reads far back weighs on the logits
        out[name] = torch.from_numpy(np.asarray(v, dtype=np.float32)).to(torch.bfloat16).to(torch.float64)
    return out


def make(path, name_or_cfg, seed=0, sharp=False, steady_router=False, correction_shift=0.0):
    cfg = CONFIGS[name_or_cfg] if isinstance(name_or_cfg, str) else name_or_cfg
    w = draw_weights(cfg, seed, sharp, steady_router, correction_shift)
    write_model(path, cfg, w)
    return cfg, w
