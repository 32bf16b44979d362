"""Sefelorn: a decoder of parallel layers (mixer and feed-forward read the same x through norms of their own and join the
stream together) whose mixers are Mamba-2 or softmax attention beside gated linear attention, and which may repeat a run
of layers, as a description in parts.

* Every layer is a ``parallel`` block with an ``rmsnorm`` for the mixers and one for the feed-forward.
* A "parallel" layer has two mixers in that block: ``talking_attention`` without mix, norms, sink or gate (biased
  projections, rotated halves, a window that keeps the sequence's first tokens), and ``gated_linear_attention``; each
  brings its factor as ``out_scale``.  A "mamba2" layer has one, ``mamba2``.
* Feed-forward: ``gated_mlp`` with the clamped gate, or none.
* ``loop``: layers start .. stop - 1 run ``times`` times in a row with the same weights; each pass has caches and state of
  its own (every entry of the run order owns its storage), and each pass but the first begins with a ``stream_reentry``
  block that adds the embedding output to the stream.
* Embedding: ``table_sum`` with a scale; the head is the token table (without that scale), the logits times ``logit_scale``.
* Tensor names: embed, final.norm, and per layer l<i>.{norm1, norm2, mix.*, mlp.{gate, up, down}}.
"""
from __future__ import annotations

from ..config.registry import register_architecture
from ..config.sefelorn_config import MAMBA2, PARALLEL, SefelornConfig
from ..parts.spec import LayerCall, LayerSpec, ModelSpec, PartSpec

GATE_ALPHA = 1.702           # slope of the clamped gate's sigmoid
DEFAULT_LOW_RANK = 16        # inner width of the decay's low-rank map when neither configuration nor checkpoint says
ROTATION_ROWS = 1 << 16      # positions the rotation table holds at least: a window lets requests outgrow the cache pool


def build_sefelorn_spec(cfg: SefelornConfig) -> ModelSpec:
    D = cfg.width
    norm = lambda name: PartSpec("rmsnorm", {"width": D, "eps": cfg.eps}, {"weight": name})     # noqa: E731
    layers = []
    for i, L in enumerate(cfg.layers):
        p = f"l{i}."
        m = L.mixer
        parts = {"norm": norm(p + "norm1")}
        if L.type == MAMBA2:
            parts["mixer"] = PartSpec("mamba2", {
                "hidden": D, "n_heads": m.heads, "vdim": m.vdim, "state": m.state, "groups": m.groups, "taps": m.conv,
                "norm_groups": m.norm_groups, "eps": cfg.eps}, {
                "in_proj": p + "mix.in", "conv": p + "mix.conv", "conv_bias": p + "mix.conv.b", "dt_bias": p + "mix.dt_bias",
                "a_log": p + "mix.A_log", "d_skip": p + "mix.D", "norm": p + "mix.norm", "o_proj": p + "mix.o"})
        elif L.type == PARALLEL:
            a, r, lp, rp = m.left, m.right, p + "mix.left.", p + "mix.right."
            parts["mixer"] = PartSpec("talking_attention", {
                "hidden": D, "n_heads": a.heads, "n_kv_heads": a.kv_heads, "dim": a.dim, "vdim": a.vdim, "scale": a.scale,
                "window": a.window, "keep_first": a.keep_first, "out_scale": m.left_scale, "bias": True, "qk_norm": False,
                "talk": False, "sink": False, "gate": False}, {
                "q_proj": lp + "q", "k_proj": lp + "k", "v_proj": lp + "v", "o_proj": lp + "o", "q_bias": lp + "q.b",
                "k_bias": lp + "k.b", "v_bias": lp + "v.b"})
            if a.rot_dims:
                parts["mixer_position"] = PartSpec("rope_neox", {"n_rot": a.rot_dims, "base": a.rot_base, "base_bits": 64,
                                                                 "min_rows": ROTATION_ROWS if a.window else 0})
            parts["second_mixer"] = PartSpec("gated_linear_attention", {
                "hidden": D, "n_heads": r.heads, "dim": r.dim, "vdim": r.vdim, "tau": r.tau,
                "decay_rank": r.decay_rank or DEFAULT_LOW_RANK, "eps": cfg.eps, "out_scale": m.right_scale}, {
                "q_proj": rp + "q", "k_proj": rp + "k", "v_proj": rp + "v", "g_proj": rp + "g", "o_proj": rp + "o",
                "norm": rp + "norm", "a1_proj": rp + "a1", "a2_proj": rp + "a2", "a2_bias": rp + "a2.b"})
        else:
            raise ValueError(f"layer {i}: unknown type {L.type!r}")
        block = {"hidden": D}
        if L.ff is not None:
            parts["feed_forward_norm"] = norm(p + "norm2")
            parts["feed_forward"] = PartSpec("gated_mlp", {
                "hidden": D, "intermediate": L.ff, "activation": "clamped", "alpha": GATE_ALPHA, "limit": L.limit}, {
                "gate_proj": p + "mlp.gate", "up_proj": p + "mlp.up", "down_proj": p + "mlp.down"})
        else:
            block["ignored_norms"] = (p + "norm2",)
        layers.append(LayerSpec(PartSpec("parallel", block), parts))

    n = len(cfg.layers)
    if cfg.loop is None:
        order = [LayerCall(i) for i in range(n)]
    else:
        start, stop, times = cfg.loop
        order = [LayerCall(i) for i in range(start)]
        if times > 1:
            layers.append(LayerSpec(PartSpec("stream_reentry", {
                "hidden": D, "vocab": cfg.vocab, "n_passes": 1, "index": 0, "embedding_scale": cfg.embedding_scale},
                {"embedding": "embed"})))
        for k in range(times):
            if k:
                order.append(LayerCall(len(layers) - 1))
            order += [LayerCall(i) for i in range(start, stop)]
        order += [LayerCall(i) for i in range(stop, n)]
    return ModelSpec(
        name="sefelorn", vocab_size=cfg.vocab, hidden_size=D, max_positions=cfg.max_positions,
        embedding=PartSpec("table_sum", {"vocab": cfg.vocab, "width": D, "scale": cfg.embedding_scale}, {"weight": "embed"}),
        layers=tuple(layers), order=tuple(order), final_norm=norm("final.norm"),
        head=PartSpec("linear", {"vocab": cfg.vocab, "width": D, "scale": cfg.logit_scale}, {"weight": "embed"}))


register_architecture("Sefelorn", SefelornConfig, build_sefelorn_spec, aliases=("sefelorn",), replace=True)
