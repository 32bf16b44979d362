"""Arrangement of a layer's parts around the residual stream.

Reference ``block`` (src/model.rs:587-599): x += mixer(norm(x)); x += ffn(norm(x)).
The residual stream is float32 in both engines; the norm writes the activation type.
"""
from __future__ import annotations

import torch

from ..kernels import ops
from .base import Block, Norm
from .registry import register_part
from .spec import TensorNeed


@register_part("block", "pre_norm")
class PreNormBlock(Block):
    """x += mixer(norm(x)); x += feed_forward(norm(x)); x += norm(side(x)).

    params: hidden, ignored_norms (names of norm weights a checkpoint may carry for a sublayer that the layer lacks).
    Made of: mixer_norm, mixer; optionally feed_forward_norm with feed_forward (both or neither), and side with
    side_norm: a per-token sublayer that reads the stream as it is (in the activation type) and whose output is normed before
    it joins; and a position encoding for the mixer, if the layer lists one.

    The side's norm adds to the stream and, in the same kernel, applies the next layer's first norm where that layer is of
    this kind."""
    chain_safe = True
    roles = {"mixer_norm": "norm", "mixer": "mixer", "feed_forward_norm": "norm", "feed_forward": "feed_forward",
             "side": "feed_forward", "side_norm": "norm"}
    optional = ("feed_forward_norm", "feed_forward", "side", "side_norm")
    side = side_norm = None

    def __init__(self, spec, runtime, parts):
        super().__init__(spec, runtime, parts)
        self.mixer_norm, self.mixer = parts["mixer_norm"], parts["mixer"]
        self.ff_norm, self.feed_forward = parts.get("feed_forward_norm"), parts.get("feed_forward")
        self.side, self.side_norm = parts.get("side"), parts.get("side_norm")
        if (self.ff_norm is None) != (self.feed_forward is None):
            raise ValueError("block 'pre_norm' has a feed-forward with its norm or neither")
        if (self.side is None) != (self.side_norm is None):
            raise ValueError("block 'pre_norm' has a side sublayer with its norm or neither")
        if self.side_norm is not None and type(self.side_norm).forward_add is Norm.forward_add:
            raise ValueError("block 'pre_norm': the side_norm part cannot norm a sublayer's output into the stream")
        self.hidden = int(spec.params["hidden"])
        runtime.scratch("normed", runtime.max_batch_tokens, self.hidden)
        if self.side is not None:
            runtime.scratch("stream_rows", runtime.max_batch_tokens, self.hidden)
            runtime.scratch("sublayer_out", runtime.max_batch_tokens, self.hidden, torch.float32)

    def tensor_needs(self):
        return {name: TensorNeed((self.hidden,), "norm", optional=True) for name in self.spec.params.get("ignored_norms", ())}

    @property
    def first_reader_takes_owed(self):
        return getattr(self.mixer_norm, "takes_owed", False)

    def stream_reader(self):
        """The norm a block before this one may apply for it (see StepContext.next_reader)."""
        return self.mixer_norm

    def forward(self, residual, ctx, call):
        T = ctx.n_tokens
        h = self.runtime.get_scratch("normed")[:, : self.hidden]
        if getattr(ctx, "normed_ready", False):
            ctx.normed_ready = False             # the block before this one left the normed stream in h
        else:
            self.norm_of_stream(self.mixer_norm, residual, h, ctx)
        # a sublayer may leave its last sum to the norm that reads the stream next
        last = ctx.next_block_takes_owed and self.side is None
        ctx.may_owe = getattr(self.ff_norm, "takes_owed", False) if self.ff_norm is not None else last
        self.mixer.forward(h, residual, ctx, call.mixers["mixer"])
        ctx.may_owe = False
        copy = None
        if self.side is not None:
            # the product that reads the stream takes it in the activation type: the stream itself, or a rounded copy
            copy = None if self.runtime.precise else self.runtime.get_scratch("stream_rows")[:, : self.hidden]
        if self.feed_forward is not None:
            self.norm_of_stream(self.ff_norm, residual, h, ctx)
            ctx.may_owe, ctx.stream_copy = last, copy
            self.feed_forward.forward(h, residual, ctx)
            ctx.may_owe = False
            copied, ctx.stream_copy = copy is not None and ctx.stream_copy is None, None
        else:
            copied = False
        if self.side is None:
            return
        if ctx.owed is not None:
            ctx.owed.finish()
            ctx.owed = None
        if copy is not None and not copied:
            ops.cast_rows(residual[:, : self.hidden], copy, T)
        delta = self.runtime.get_scratch("sublayer_out", torch.float32)[:, : self.hidden]
        ctx.store_output = True
        try:
            self.side.forward(residual[:, : self.hidden] if copy is None else copy, delta, ctx)
        finally:
            ctx.store_output = False
        nxt = ctx.next_reader if isinstance(ctx.next_reader, Norm) else None
        self.side_norm.forward_add(delta, residual, T, then=nxt, out=h if nxt is not None else None)
        ctx.normed_ready = nxt is not None


@register_part("block", "parallel")
class ParallelBlock(Block):
    """Sublayers that all read the same x: x += mixer(norm(x)) + second_mixer(norm(x)) + feed_forward(ff_norm(x)), where the
    feed-forward reads norm(x) too if it has no norm of its own.

    params: hidden, ignored_norms (names of norm weights a checkpoint may carry for a sublayer that the layer lacks).
    Made of: norm, mixer, and optionally second_mixer, feed_forward, feed_forward_norm (position encodings for the mixers,
    if the layer lists any).  The outputs join the float32 stream in this order.

    Products are joined where the parts allow it (``joinable``): two mixers that read the same rows project them with one
    matrix, and if every sublayer can hand over the rows its output matrix multiplies, the rows lie side by side and one
    product [W_mixer | W_second | W_ff] adds all of them to the stream."""
    roles = {"norm": "norm", "mixer": "mixer", "second_mixer": "mixer", "feed_forward": "feed_forward", "feed_forward_norm": "norm"}
    optional = ("second_mixer", "feed_forward", "feed_forward_norm")

    def __init__(self, spec, runtime, parts):
        super().__init__(spec, runtime, parts)
        self.norm, self.feed_forward = parts["norm"], parts.get("feed_forward")
        self.ff_norm = parts.get("feed_forward_norm")
        if self.ff_norm is not None and self.feed_forward is None:
            raise ValueError("block 'parallel': a feed-forward norm without a feed-forward")
        self.mixer_roles = [r for r in ("mixer", "second_mixer") if r in parts]
        mixers = [parts[r] for r in self.mixer_roles]
        self.hidden = int(spec.params["hidden"])
        runtime.scratch("normed", runtime.max_batch_tokens, self.hidden)
        if self.ff_norm is not None:
            runtime.scratch("normed_ff", runtime.max_batch_tokens, self.hidden)
        sublayers = mixers + ([self.feed_forward] if self.feed_forward is not None else [])
        self.join_in = all(m.joinable for m in mixers)
        # (rows that start on 16 bytes in both element types: what the products and the rows' writers ask for)
        self.join_out = (self.join_in and len(sublayers) > 1 and all(s.joinable and s.row_cols % 8 == 0 for s in sublayers))
        self.in_cols = sum(m.in_cols for m in mixers) if self.join_in else 0
        self.row_cols = sum(s.row_cols for s in sublayers) if self.join_out else 0
        if self.join_out:
            runtime.scratch("joint_proj", runtime.max_batch_tokens, (self.in_cols + 3) // 4 * 4, torch.float32)
            runtime.scratch("joint_rows", runtime.max_batch_tokens, self.row_cols)       # a multiple of 8 columns

    def tensor_needs(self):
        return {name: TensorNeed((self.hidden,), "norm", optional=True) for name in self.spec.params.get("ignored_norms", ())}

    def finish_load(self):
        if not self.join_out:
            return
        mixers = [self.parts[r] for r in self.mixer_roles]
        ff = self.feed_forward
        outs = [m.w_o for m in mixers] + ([ff.w_down] if ff is not None else [])
        if len({m.w_in.dtype for m in mixers}) != 1 or len({w.dtype for w in outs}) != 1:
            self.join_out = False                          # matrices of different element types stay apart
            return
        self.w_in = mixers[0].w_in
        if len(mixers) > 1:
            self.w_in = torch.cat([m.w_in for m in mixers], dim=0).contiguous()
            at = 0
            for m in mixers:                               # one copy: the parts keep views
                m.w_in, at = self.w_in[at: at + m.in_cols], at + m.in_cols
        self.w_out = torch.cat(outs, dim=1).contiguous()
        at = 0
        for m in mixers:
            m.w_o, at = self.w_out[:, at: at + m.row_cols], at + m.row_cols
        if ff is not None:
            ff.w_down = self.w_out[:, at: at + ff.row_cols]

    def flops_per_token(self) -> float:
        return 0.0                           # the joined matrices are the parts', which count them

    @property
    def first_reader_takes_owed(self):
        return getattr(self.norm, "takes_owed", False)

    def forward(self, residual, ctx, call):
        rt, T = self.runtime, ctx.n_tokens
        h = h_ff = rt.get_scratch("normed")[:, : self.hidden]
        if self.ff_norm is None:
            self.norm_of_stream(self.norm, residual, h, ctx)
        else:
            h_ff = rt.get_scratch("normed_ff")[:, : self.hidden]
            owed, ctx.owed = ctx.owed, None
            if owed is not None and not getattr(self.norm, "takes_owed", False):
                owed.finish()
                owed = None
            self.norm.forward_pair(residual, h, self.ff_norm, h_ff, T, owed=owed)
        if self.join_out:
            proj = rt.get_scratch("joint_proj", torch.float32)[:, : self.in_cols]
            rows = rt.get_scratch("joint_rows")[:, : self.row_cols]
            ops.linear(h, self.w_in, proj, T, status=ctx.status)
            p_at = r_at = 0
            for r in self.mixer_roles:
                m = self.parts[r]
                m.forward_rows(proj[:, p_at: p_at + m.in_cols], rows[:, r_at: r_at + m.row_cols], ctx, call.mixers[r])
                p_at, r_at = p_at + m.in_cols, r_at + m.row_cols
            if self.feed_forward is not None:
                self.feed_forward.forward_rows(h_ff, rows[:, r_at:], ctx)
            ctx.owed = ops.linear(rows, self.w_out, residual, T, accumulate=True, status=ctx.status,
                                  may_defer=ctx.next_block_takes_owed)
            return
        # no sublayer may leave a sum owed to the stream: the next one adds into it right after
        ctx.may_owe = False
        for r in self.mixer_roles:
            self.parts[r].forward(h, residual, ctx, call.mixers[r])
        if self.feed_forward is not None:
            self.feed_forward.forward(h_ff, residual, ctx)


@register_part("block", "sandwich_norm")
class SandwichNormBlock(Block):
    """A layer whose sublayers are normed on both sides: x += post(mixer(conv(pre(x)))), x += post'(ff(pre'(x))).

    params: hidden, ignored_tensors (names of scalar tensors a checkpoint may carry for a sublayer the layer lacks).
    Made of: mixer_norm, mixer, mixer_post_norm; optionally input_conv (a convolution over time that
    what the mixer reads passes first; it keeps state like a mixer, hence its category), and feed_forward_norm,
    feed_forward, feed_forward_post_norm (all three or none).  The mixer and the feed-forward store their output in a
    float32 buffer of the block (``ctx.store_output``); the post-norm adds it to the stream and, in the same kernel,
    applies the norm of the stream's next reader inside the layer."""
    roles = {"mixer_norm": "norm", "input_conv": "mixer", "mixer": "mixer", "mixer_post_norm": "norm",
             "feed_forward_norm": "norm", "feed_forward": "feed_forward", "feed_forward_post_norm": "norm"}
    optional = ("input_conv", "feed_forward_norm", "feed_forward", "feed_forward_post_norm")

    def __init__(self, spec, runtime, parts):
        super().__init__(spec, runtime, parts)
        self.hidden = int(spec.params["hidden"])
        ff = [r for r in ("feed_forward_norm", "feed_forward", "feed_forward_post_norm") if r in parts]
        if len(ff) not in (0, 3):
            raise ValueError(f"block 'sandwich_norm' has a feed-forward with both of its norms or none; got {ff}")
        self.has_ff = bool(ff)
        for r in ("mixer_post_norm", "feed_forward_post_norm"):
            if r in parts and type(parts[r]).forward_add is Norm.forward_add:
                raise ValueError(f"block 'sandwich_norm': the {r} part cannot norm a sublayer's output into the stream")
        self.ignored = tuple(spec.params.get("ignored_tensors", ()))
        runtime.scratch("normed", runtime.max_batch_tokens, self.hidden)
        runtime.scratch("conv_out", runtime.max_batch_tokens, self.hidden)
        runtime.scratch("sublayer_out", runtime.max_batch_tokens, self.hidden, torch.float32)

    def tensor_needs(self):
        # gains of norms that a layer without a feed-forward has no use for: taken if the checkpoint has them
        return {name: TensorNeed((), "norm", optional=True) for name in self.ignored}

    def forward(self, residual, ctx, call):
        rt, p, T = self.runtime, self.parts, ctx.n_tokens
        h = rt.get_scratch("normed")[:, : self.hidden]
        delta = rt.get_scratch("sublayer_out", torch.float32)[:, : self.hidden]
        self.norm_of_stream(p["mixer_norm"], residual, h, ctx)
        if "input_conv" in p:
            h2 = rt.get_scratch("conv_out")[:, : self.hidden]
            p["input_conv"].forward(h, h2, ctx, call.mixers["input_conv"])
            h = h2
        ctx.store_output = True
        try:
            p["mixer"].forward(h, delta, ctx, call.mixers["mixer"])
            if not self.has_ff:
                p["mixer_post_norm"].forward_add(delta, residual, T)
                return
            h = rt.get_scratch("normed")[:, : self.hidden]
            p["mixer_post_norm"].forward_add(delta, residual, T, then=p["feed_forward_norm"], out=h)
            p["feed_forward"].forward(h, delta, ctx)
            p["feed_forward_post_norm"].forward_add(delta, residual, T)
        finally:
            ctx.store_output = False


@register_part("block", "stream_reentry")
class StreamReentryBlock(Block):
    """The start of a pass over a run of layers that is repeated with the same weights: the stream is mixed with the
    embedding output again, x <- W [x ; embedding(token)] + step, ``step`` one row of a [passes, hidden] table, or, without
    a matrix, x <- x + embedding_scale * embedding(token).

    params: hidden, vocab, n_passes, index (which row of the table), embedding_scale (1; for the form without a matrix).
    tensors: in_proj [hidden, 2 * hidden] (x first; left out: the plain sum), step [n_passes, hidden] (left out of the
    tensors: no such term), embedding [vocab, hidden] (the model's token table).
    No parts, no cache, no state."""
    roles = {}

    def __init__(self, spec, runtime, parts):
        super().__init__(spec, runtime, parts)
        p = spec.params
        self.hidden, self.vocab = int(p["hidden"]), int(p["vocab"])
        self.n_passes, self.index = int(p["n_passes"]), int(p["index"])
        if not 0 <= self.index < self.n_passes:
            raise ValueError(f"stream_reentry: pass {self.index} of {self.n_passes}")
        self.scale = float(p.get("embedding_scale", 1.0))
        self.mixes = "in_proj" in spec.tensors
        if self.mixes:
            runtime.scratch("stream_cat", runtime.max_batch_tokens, 2 * self.hidden)
        if (self.mixes and self.scale != 1.0) or ("step" in spec.tensors and not self.mixes):
            raise ValueError("stream_reentry: embedding_scale belongs to the form without a matrix, step to the one with it")

    def tensor_needs(self):
        t = self.spec.tensors
        needs = {t["embedding"]: TensorNeed((self.vocab, self.hidden), "embedding")}
        if self.mixes:
            needs[t["in_proj"]] = TensorNeed((self.hidden, 2 * self.hidden))
        if "step" in t:
            needs[t["step"]] = TensorNeed((self.n_passes, self.hidden))
        return needs

    def load(self, tensors):
        t = self.spec.tensors
        self.w_in = tensors[t["in_proj"]].contiguous() if self.mixes else None
        self.step_row = tensors[t["step"]][self.index].contiguous() if "step" in t else None
        self.table = tensors[t["embedding"]]

    def flops_per_token(self) -> float:
        return 4.0 * self.hidden * self.hidden if self.mixes else 0.0

    def forward(self, residual, ctx, call):
        T = ctx.n_tokens
        if ctx.owed is not None:
            ctx.owed.finish()
            ctx.owed = None
        if not self.mixes:
            ops.add_embed(residual, self.table, ctx.token_ids, self.scale, T, ctx.status)
            return
        cat = self.runtime.get_scratch("stream_cat")[:, : 2 * self.hidden]
        # cat = [x | embedding]; the stream is preset to the pass's row, and the product adds W cat onto it
        ops.concat_embed(residual, self.table, ctx.token_ids, self.step_row, cat, T, ctx.status)
        ops.linear(cat, self.w_in, residual, T, accumulate=True, status=ctx.status)
