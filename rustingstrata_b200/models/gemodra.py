"""Gemodra: a pre-norm decoder of latent-attention layers with routed experts and a per-layer input from the token, as a
description in parts.

* Embedding ``token_table`` followed by an RMS norm; every layer is a ``pre_norm`` block whose sublayers' outputs are
  multiplied by the residual multiplier m (``out_scale`` of the mixer and the feed-forward, ``gain_scale`` of the norm that
  the per-token sublayer's output passes).
* Mixer ``latent_attention`` in two forms, both with queries through a latent of their own and a sink per head: with rotated
  parts (neighbouring pairs) and a gate per value, or without positions and a gate per head.
* Feed-forward ``routed_moe``: softmax scores over experts and identity experts, a correction that steers the choice only,
  groups worth their best choice score, scaled weights that are not renormalised, SiLU-gated experts, a shared expert behind
  a sigmoid; or none.
* ``side``: ``token_gate`` reads the stream after the feed-forward and the layer's columns of a table by token id.
* Head ``linear`` with a soft cap.
* Tensor names: embed, embed.norm, side.embed, final.norm, head, and per layer l<i>.{norm1, norm2, mix.*, mlp.*,
  side.{gate, proj, norm}}.
"""
from __future__ import annotations

from ..config.gemodra_config import LATENT_ATTENTION, GemodraConfig
from ..config.registry import register_architecture
from ..parts.spec import LayerCall, LayerSpec, ModelSpec, PartSpec


def build_gemodra_spec(cfg: GemodraConfig) -> ModelSpec:
    D, mult = cfg.width, cfg.residual_mult
    norm = lambda name, **more: PartSpec("rmsnorm", {"width": D, "eps": cfg.eps, **more}, {"weight": name})      # noqa: E731
    layers = []
    for i, L in enumerate(cfg.layers):
        p = f"l{i}."
        m = L.mixer
        parts = {"mixer_norm": norm(p + "norm1")}
        parts["mixer"] = PartSpec("latent_attention", {
            "hidden": D, "n_heads": m.heads, "dim": m.dim, "rot_dim": m.rot_dim, "vdim": m.vdim, "kv_rank": m.kv_rank,
            "q_rank": m.q_rank, "scale": m.scale, "eps": cfg.eps, "window": None, "sink": True,
            "gate": "element" if L.type == LATENT_ATTENTION else "head", "out_scale": mult, "weights_bits": 32}, {
            "dq_proj": p + "mix.dq", "q_latent_norm": p + "mix.dq.norm", "q_proj": p + "mix.uq", "dkv_proj": p + "mix.dkv",
            "latent_norm": p + "mix.dkv.norm", "uk_proj": p + "mix.uk", "uv_proj": p + "mix.uv", "sink": p + "mix.sink",
            "g_proj": p + "mix.g", "o_proj": p + "mix.o"})
        if m.rot_dim:
            parts["mixer_position"] = PartSpec("rope_interleaved", {"n_rot": m.rot_dims, "base": m.rot_base})
        ff = L.mlp
        if ff is not None:
            parts["feed_forward_norm"] = norm(p + "norm2")
            t = {"router": p + "mlp.router", "correction": p + "mlp.correction", "expert_gate": p + "mlp.e{e}.gate",
                 "expert_up": p + "mlp.e{e}.up", "expert_down": p + "mlp.e{e}.down"}
            if ff.shared_ff:
                t.update(shared_gate=p + "mlp.shared.gate", shared_up=p + "mlp.shared.up", shared_down=p + "mlp.shared.down",
                         shared_scale=p + "mlp.shared.sg")
            parts["feed_forward"] = PartSpec("routed_moe", {
                "hidden": D, "experts": ff.experts, "identity": ff.identity, "top": ff.top, "expert_ff": ff.expert_ff,
                "shared_ff": ff.shared_ff, "shared_scale": bool(ff.shared_ff), "correction": True, "score": "softmax",
                "groups": ff.groups[0] if ff.groups else 0, "keep": ff.groups[1] if ff.groups else 0, "group_worth": "max",
                "route_scale": ff.route_scale, "renormalize": False, "expert": "gated_silu", "out_scale": mult}, t)
        if cfg.side_dim is not None:
            parts["side"] = PartSpec("token_gate", {"hidden": D, "dim": cfg.side_dim, "vocab": cfg.vocab, "column": i * cfg.side_dim,
                                                    "table_width": len(cfg.layers) * cfg.side_dim},
                                     {"gate_proj": p + "side.gate", "out_proj": p + "side.proj", "table": "side.embed"})
            parts["side_norm"] = norm(p + "side.norm", gain_scale=mult)
        unused = () if ff is not None else (p + "norm2",)
        layers.append(LayerSpec(PartSpec("pre_norm", {"hidden": D, "ignored_norms": unused}), parts))
    return ModelSpec(
        name="gemodra", vocab_size=cfg.vocab, hidden_size=D, max_positions=cfg.max_positions,
        embedding=PartSpec("token_table", {"vocab": cfg.vocab, "width": D, "norm_eps": cfg.eps},
                           {"weight": "embed", "norm": "embed.norm"}),
        layers=tuple(layers), order=tuple(LayerCall(i) for i in range(len(layers))), final_norm=norm("final.norm"),
        head=PartSpec("linear", {"vocab": cfg.vocab, "width": D, "softcap": cfg.logit_softcap}, {"weight": "head"}))


register_architecture("Gemodra", GemodraConfig, build_gemodra_spec, aliases=("gemodra",), replace=True)
