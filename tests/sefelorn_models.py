"""Small Sefelorn configurations with weights made here, for the tests.

The tensor names and shapes are derived here from the configuration (not from the engine's manifest, which is thereby
checked too), the values are drawn with numpy and rounded to bfloat16.  ``sharp`` (a factor, or True for 1) makes faults
visible that random weights would hide: the attention's queries are scaled up so that each query looks at one or two keys
only, wherever they lie, and its output weighs more; the decays of both recurrent mixers sit just below one, so that their
states last for hundreds of tokens.
"""
from __future__ import annotations

import copy

import numpy as np
import torch

from lokinex_models import write_model  # noqa: F401  (the safetensors writer of the test suite)


def mamba2(heads, vdim, state, groups=1, conv=4, norm_groups=1):
    return {"type": "mamba2", "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv,
                                        "norm_groups": norm_groups}}


def left(heads, kv_heads, dim, vdim, size, keep, rot=None, scale=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": dim ** -0.5 if scale is None else scale,
         "mask": {"size": size, "keep_first": keep}}
    if rot is not None:
        m["rot"] = {"dims": rot[0], "base": rot[1]}
    return m


def right(heads, dim, vdim, tau, decay_rank):
    return {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau, "decay_rank": decay_rank}


def parallel(l, r, scales=(0.7, 1.2)):
    return {"type": "parallel", "mixer": {"left": l, "right": r, "left_scale": scales[0], "right_scale": scales[1]}}


def dense(ff, limit=1.2):
    return {"kind": "dense", "ff": ff, "limit": limit}


def config(vocab, width, layers, eps=1e-6, loop=None, logit_scale=None, embedding_scale=None):
    c = {"architecture": "Sefelorn", "vocab": vocab, "width": width, "norm": {"eps": eps},
         "layers": [dict(copy.deepcopy(l), mlp=m) for l, m in layers]}
    if loop is not None:
        c["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    if logit_scale is not None:
        c["logit_scale"] = logit_scale
    if embedding_scale is not None:
        c["embedding"] = {"scale": embedding_scale}
    return c


# Sizes that differ from each other in every respect; values that a model may happen to make equal or 1 (kv heads against
# heads, vdim against dim, rot.dims against dim, groups, norm groups, taps, times, scales) are unequal or not 1 somewhere
# and equal or 1 elsewhere.
CONFIGS = {
    # a loop in the middle (start > 0, stop < layers), three passes, a layer without feed-forward, rows that need padding
    "P": config(211, 96, [
        (mamba2(6, 20, 24, groups=2, conv=3, norm_groups=3), dense(160, 0.8)),
        (parallel(left(6, 2, 24, 40, 20, 5, rot=(8, 5000.0), scale=0.3), right(3, 20, 28, 8.0, 7)), None),
        (mamba2(2, 12, 40, conv=5), dense(48, 2.0)),
        (parallel(left(4, 4, 16, 16, 33, 18, rot=(16, 300.0)), right(2, 40, 12, 2.0, 9), scales=(1.3, 0.4)), dense(72)),
        (mamba2(4, 8, 16, groups=4, conv=2, norm_groups=4), dense(64, 0.5)),
    ], eps=1e-6, loop=(1, 4, 3), logit_scale=0.25, embedding_scale=2.5),
    # no loop, no rotation, one kv head, no kept tokens, one tap, widths that neither the tensor-core products nor 16-byte
    # rows take, scales absent
    "Q": config(130, 100, [
        (parallel(left(5, 1, 32, 8, 12, 0), right(1, 18, 6, 1.0, 5), scales=(1.0, 1.0)), dense(54, 0.9)),
        (mamba2(3, 9, 21, conv=1), dense(40)),
        (mamba2(1, 30, 7, conv=4), None),
    ], eps=1e-5),
    # wider, one pass of a loop over everything, for long sequences
    "R": config(320, 256, [
        (parallel(left(4, 2, 48, 32, 100, 20, rot=(24, 1e5)), right(4, 32, 48, 16.0, 24)), dense(384)),
        (mamba2(8, 32, 64, groups=4, conv=4, norm_groups=8), dense(256, 3.0)),
    ], eps=1e-5, loop=(0, 2, 1), logit_scale=1.5, embedding_scale=0.5),
    # windows and kept tokens of a page, more kept tokens than the window holds, a window of one key; a loop from the start
    "S": config(150, 128, [
        (parallel(left(2, 1, 32, 48, 16, 16, rot=(32, 1e4)), right(2, 16, 16, 4.0, 8)), dense(96)),
        (parallel(left(3, 3, 16, 32, 5, 37, rot=(4, 50.0)), right(1, 64, 32, 16.0, 16)), None),
        (parallel(left(2, 2, 16, 16, 1, 3, rot=(16, 100.0)), right(4, 8, 24, 3.0, 4)), dense(80)),
    ], loop=(0, 2, 2), logit_scale=0.5, embedding_scale=4.0),
}


def tensor_shapes(cfg):
    D, V = cfg["width"], cfg["vocab"]
    s = {"embed": (V, D), "final.norm": (D,)}
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        s[p + "norm1"] = (D,)
        if L["type"] == "mamba2":
            H, inner, bc = m["heads"], m["heads"] * m["vdim"], 2 * m["groups"] * m["state"]
            s.update({p + "mix.in": (2 * inner + bc + H, D), p + "mix.conv": (inner + bc, m["conv"]), p + "mix.conv.b": (inner + bc,),
                      p + "mix.dt_bias": (H,), p + "mix.A_log": (H,), p + "mix.D": (H,), p + "mix.norm": (inner,),
                      p + "mix.o": (D, inner)})
        else:
            a, r = m["left"], m["right"]
            q, k, v = a["heads"] * a["dim"], a["kv_heads"] * a["dim"], a["kv_heads"] * a["vdim"]
            lp, rp = p + "mix.left.", p + "mix.right."
            s.update({lp + "q": (q, D), lp + "q.b": (q,), lp + "k": (k, D), lp + "k.b": (k,), lp + "v": (v, D), lp + "v.b": (v,),
                      lp + "o": (D, a["heads"] * a["vdim"])})
            k, v, n = r["heads"] * r["dim"], r["heads"] * r["vdim"], r["decay_rank"]
            s.update({rp + "q": (k, D), rp + "k": (k, D), rp + "v": (v, D), rp + "g": (v, D), rp + "o": (D, v), rp + "norm": (r["vdim"],),
                      rp + "a1": (n, D), rp + "a2": (k, n), rp + "a2.b": (k,)})
        if L["mlp"] is not None:
            ff = L["mlp"]["ff"]
            s.update({p + "norm2": (D,), p + "mlp.gate": (ff, D), p + "mlp.up": (ff, D), p + "mlp.down": (D, ff)})
    return s


def draw_weights(cfg, seed, sharp=0.0):
    """name → float64 tensor holding bfloat16-representable values."""
    sharp = float(sharp)
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        layer = name[: name.index(".") + 1] if name.startswith("l") and name[1].isdigit() else ""
        rest = name[len(layer):]
        z = rng.standard_normal(shape)
        if rest in ("norm1", "norm2", "final.norm", "mix.norm", "mix.right.norm"):
            v = 1.0 + 0.2 * z
        elif rest in ("mix.left.q", "mix.left.q.b"):
            v = (1.0 + 5.0 * sharp) * (0.3 * z if rest.endswith(".b") else z / np.sqrt(shape[-1]))
        elif rest in ("mix.left.k.b", "mix.left.v.b", "mix.conv.b"):
            v = 0.3 * z
        elif rest == "mix.right.a2.b":
            v = 6.0 * sharp + z
        elif rest == "mix.A_log":
            v = -5.0 * sharp + 0.5 * z
        elif rest in ("mix.dt_bias", "mix.D"):
            v = 0.7 * z
        elif rest == "mix.conv":
            v = 0.6 * z
        elif name == "embed":
            v = z
        elif rest in ("mlp.gate", "mlp.up"):
            v = 1.5 * z / np.sqrt(shape[-1])                   # reaches both sides of the clamps
        else:
            v = z / np.sqrt(shape[-1])
            if sharp and rest == "mix.left.o":
                v = v * (1.0 + 3.0 * sharp)                    # what the attention reads weighs on the logits
        out[name] = torch.from_numpy(np.asarray(v, dtype=np.float32)).to(torch.bfloat16).to(torch.float64)
    return out


def with_masks(cfg, size=0, keep=0):
    """The same configuration with every window ``size`` keys larger and ``keep`` more first tokens kept."""
    c = copy.deepcopy(cfg)
    for L in c["layers"]:
        if L["type"] == "parallel":
            m = L["mixer"]["left"]["mask"]
            m["size"], m["keep_first"] = m["size"] + size, max(0, m["keep_first"] + keep)
    return c


def make(path, name_or_cfg, seed=0, sharp=0.0):
    cfg = CONFIGS[name_or_cfg] if isinstance(name_or_cfg, str) else name_or_cfg
    w = draw_weights(cfg, seed, sharp)
    on_disk = copy.deepcopy(cfg)
    for L in on_disk["layers"]:          # the low-rank map's inner width is read from its tensor's shape
        if L["type"] == "parallel":
            del L["mixer"]["right"]["decay_rank"]
    write_model(path, on_disk, w)
    return cfg, w
