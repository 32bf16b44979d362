"""Mixers that keep a matrix of state per head in place of a cache of keys: HGRN2, the gated delta rule with a decay
per key channel, retention with one fixed decay per head, gated linear attention with a decay per key channel, and
Mamba-2 with a decay per head that the input sets.  All walk a float32 state S [dim, vdim] per (request, head)
token by token and read it out with a query.

``hgrn2`` (gated linear recurrence whose forget gate also decides what is written).  From the mixer's input h:
q = silu(W_q h), v = W_v h, f = l + (1 - l) sigmoid(W_f h + b_f) per head and channel, l a learned lower bound;

    S_t = diag(f_t) S_(t-1) + (1 - f_t) v_t^T,        o_t = S_t^T q_t        (no key, no other scale);

each head's o_t is divided by its root mean square over vdim and multiplied by a weight [vdim] shared by the heads,
the heads are joined and W_o maps them back.

``gated_delta`` (delta rule with a decay per head and key channel).  q = W_q h, k = W_k h (qk heads x dim), v = W_v h
(heads x vdim), state head i reading q/k head i // (heads / qk heads); each channel of q, k, v passes a short causal
convolution over time and silu; q and k heads become unit vectors x / sqrt(sum x^2 + unit_eps), q times dim^-1/2;
beta = sigmoid(W_b h) per head; g = exp(-exp(A_h) softplus(W_a2 (W_a1 h) + dt)) per head and key channel;

    S <- diag(g_t) S;    u = beta_t (v_t - S^T k_t);    S <- S + k_t u^T;    o_t = S^T q_t

(the read-out sees the token's own write); each head's o_t divided by its root mean square over vdim, times a weight
[vdim] shared by the heads, times sigmoid(W_g2 (W_g1 h)) laid out heads x vdim; then W_o.

``retention`` (linear attention with a fixed decay per head, no softmax and no denominator).  q = W_q h, k = W_k h
(heads x dim), v = W_v h (heads x vdim), no biases; the layer's position part rotates a prefix of every q and k head;
k times dim^-1/2 after the rotation;

    S_t = decay_h S_(t-1) + k_t v_t^T,        o_t = S_t^T q_t;

each head's o_t is divided by its root mean square over vdim (no weight), the heads are joined, multiplied by
silu(W_g h) coordinate by coordinate, and W_o maps them back.

``gated_linear_attention``.  q = W_q h * q_scale (dim^-1/2), k = W_k h (heads x dim), v = W_v h (heads x vdim),
alpha = sigmoid(W_a2 (W_a1 h) + b)^(1 / tau) per head and key channel;

    S_t = diag(alpha_t) S_(t-1) + k_t v_t^T,        o_t = S_t^T q_t;

each head's o_t is divided by its root mean square over vdim and multiplied by a weight [vdim] shared by the heads, the
heads are joined, multiplied by silu(W_g h), and W_o maps them back.

``mamba2`` (state-space duality; N = state rows, G = groups, inner = heads x vdim).  W_in h = [z | x | B | C | dt] with
widths inner, inner, G N, G N, heads; x, B and C pass a short causal convolution over time with a bias, and silu;
dt <- softplus(dt + dt_bias); head h reads B and C of group h // (heads / G):

    S_t = exp(-exp(A_h) dt) S_(t-1) + dt B_t x_t^T,        y_t = S_t^T C_t + D_h x_t;

the joined y is multiplied by silu(z), each of ``norm_groups`` equal parts divided by its own root mean square, times a
weight [inner]; then W_o.

Per request the state slot holds S for every head (zero at admission) and, for a convolution, the last taps - 1
projected rows.  The projections follow the engine's element type with float32 results; gates, decays, norms, the
state and the recurrence are float32 in both engines.
"""
from __future__ import annotations

import numpy as np
import torch

from ..kernels import ops
from .base import CallInfo, HostBatch, Mixer, StepContext
from .registry import register_part
from .spec import StateNeed, TensorNeed


@register_part("mixer", "hgrn2")
class Hgrn2(Mixer):
    """params: hidden, n_heads, dim, vdim, eps (of the read-out norm), f_bias (bool, default True).
    tensors: q_proj, f_proj, f_bias, lower [heads * dim], v_proj, norm [vdim], o_proj."""

    def __init__(self, spec, runtime, position=None):
        super().__init__(spec, runtime)
        p = spec.params
        self.hidden, self.n_heads = int(p["hidden"]), int(p["n_heads"])
        self.dk, self.dv = int(p["dim"]), int(p["vdim"])
        self.eps = float(p.get("eps", 0.0))
        self.has_f_bias = bool(p.get("f_bias", True))
        self.rows_pad = ops.state_rows_pad(self.dk)
        self.qf_cols, self.v_cols = self.n_heads * self.dk, self.n_heads * self.dv
        self.in_cols = 2 * self.qf_cols + self.v_cols
        rt = runtime
        rt.scratch("state_proj", rt.max_batch_tokens, self.in_cols, torch.float32)
        rt.scratch("state_rows", 1, 3 * rt.max_batch_tokens * self.n_heads * self.rows_pad, torch.float32)
        rt.scratch("state_read", rt.max_batch_tokens, self.v_cols, torch.float32)
        rt.scratch("state_out", rt.max_batch_tokens, self.v_cols)

    def tensor_needs(self):
        t = self.spec.tensors
        needs = {t["q_proj"]: TensorNeed((self.qf_cols, self.hidden)), t["f_proj"]: TensorNeed((self.qf_cols, self.hidden)),
                 t["lower"]: TensorNeed((self.qf_cols,)), t["v_proj"]: TensorNeed((self.v_cols, self.hidden)),
                 t["norm"]: TensorNeed((self.dv,), "norm"), t["o_proj"]: TensorNeed((self.hidden, self.v_cols))}
        if self.has_f_bias:
            needs[t["f_bias"]] = TensorNeed((self.qf_cols,))
        return needs

    def load(self, tensors):
        t = self.spec.tensors
        mats = [tensors[t["q_proj"]], tensors[t["f_proj"]], tensors[t["v_proj"]]]
        if len({m.dtype for m in mats}) != 1:
            raise ValueError("hgrn2: the input projections must share an element type")
        self.w_in = torch.cat(mats, dim=0).contiguous()              # [q | f | v]
        self.f_bias = tensors[t["f_bias"]].to(torch.float32).contiguous() if self.has_f_bias else None
        self.lower = tensors[t["lower"]].to(torch.float32).contiguous()
        self.norm_w = tensors[t["norm"]].to(torch.float32).contiguous()
        self.w_o = tensors[t["o_proj"]].contiguous()

    def state_need(self):
        return StateNeed(self.n_heads * self.dv * self.rows_pad, "float32")

    def flops_per_token(self) -> float:
        return 2.0 * self.hidden * (self.in_cols + self.v_cols) + 6.0 * self.n_heads * self.dk * self.dv

    def forward(self, h, residual, ctx: StepContext, call: CallInfo):
        rt, T, H, RP = self.runtime, ctx.n_tokens, self.n_heads, self.rows_pad
        proj = rt.get_scratch("state_proj", torch.float32)[:, : self.in_cols]
        n = rt.max_batch_tokens * H * RP
        rows = rt.get_scratch("state_rows", torch.float32)[0]
        q, g, w = (rows[i * n:(i + 1) * n].view(rt.max_batch_tokens, H * RP) for i in range(3))
        read = rt.get_scratch("state_read", torch.float32)[:, : self.v_cols]
        out = rt.get_scratch("state_out")[:, : self.v_cols]
        ops.linear(h, self.w_in, proj, T, status=ctx.status)
        ops.hgrn2_prep(proj, self.f_bias, self.lower, q, g, w, H, self.dk, RP, T)
        ops.state_recurrence(q, w, g, None, proj[:, 2 * self.qf_cols:], read, call.state, ctx.q_start, ctx.state_slots,
                             ctx.n_seqs, H, 1, RP, self.dv, delta=False)
        ops.head_norm_gate(read, self.norm_w, None, out, H, self.dv, self.eps, T)
        ops.linear(out, self.w_o, residual, T, accumulate=not ctx.store_output, status=ctx.status)


@register_part("mixer", "gated_delta")
class GatedDelta(Mixer):
    """params: hidden, n_heads, n_qk_heads, dim, vdim, taps (0: no convolution), decay_rank, gate_rank, eps (of the
    read-out norm), unit_eps (inside the root of the unit vectors, default 1e-6).
    tensors: q_proj, k_proj, v_proj, q_conv, k_conv, v_conv [channels, taps], b_proj [heads, hidden], a_log [heads],
    a1_proj [decay_rank, hidden], a2_proj [heads * dim, decay_rank], dt_bias [heads * dim], g1_proj [gate_rank, hidden],
    g2_proj [heads * vdim, gate_rank], norm [vdim], o_proj."""

    def __init__(self, spec, runtime, position=None):
        super().__init__(spec, runtime)
        p = spec.params
        self.hidden, self.n_heads, self.n_qk = int(p["hidden"]), int(p["n_heads"]), int(p["n_qk_heads"])
        self.dk, self.dv = int(p["dim"]), int(p["vdim"])
        self.taps = int(p.get("taps") or 0)
        self.decay_rank, self.gate_rank = int(p["decay_rank"]), int(p["gate_rank"])
        self.eps, self.unit_eps = float(p.get("eps", 0.0)), float(p.get("unit_eps", 1e-6))
        if self.n_heads % self.n_qk:
            raise ValueError(f"gated_delta: {self.n_heads} heads are not a multiple of {self.n_qk} q/k heads")
        if self.taps > 64:
            raise ValueError(f"gated_delta: {self.taps} taps (up to 64 are supported)")
        self.rows_pad = ops.state_rows_pad(self.dk)
        self.qk_cols, self.v_cols = self.n_qk * self.dk, self.n_heads * self.dv
        self.channels = 2 * self.qk_cols + self.v_cols                   # what the convolution runs over
        self.beta_off = self.channels
        self.a1_off = self.beta_off + self.n_heads
        self.g1_off = self.a1_off + self.decay_rank
        self.in_cols = self.g1_off + self.gate_rank
        self.tail = max(0, self.taps - 1) * self.channels
        self.state_cols = self.n_heads * self.dv * self.rows_pad
        rt, mbt = runtime, runtime.max_batch_tokens
        rt.scratch("state_proj", mbt, self.in_cols, torch.float32)
        rt.scratch("state_rows", 1, mbt * (2 * self.n_qk + self.n_heads) * self.rows_pad, torch.float32)
        rt.scratch("delta_step", mbt, self.n_heads * self.dk, torch.float32)
        rt.scratch("delta_gate", mbt, self.v_cols, torch.float32)
        rt.scratch("delta_v", 1, mbt * (self.v_cols + self.n_heads), torch.float32)
        rt.scratch("state_read", mbt, self.v_cols, torch.float32)
        rt.scratch("state_out", mbt, self.v_cols)

    def tensor_needs(self):
        t, D = self.spec.tensors, self.hidden
        needs = {t["q_proj"]: TensorNeed((self.qk_cols, D)), t["k_proj"]: TensorNeed((self.qk_cols, D)),
                 t["v_proj"]: TensorNeed((self.v_cols, D)), t["b_proj"]: TensorNeed((self.n_heads, D)),
                 t["a_log"]: TensorNeed((self.n_heads,)), t["a1_proj"]: TensorNeed((self.decay_rank, D)),
                 t["a2_proj"]: TensorNeed((self.n_heads * self.dk, self.decay_rank)),
                 t["dt_bias"]: TensorNeed((self.n_heads * self.dk,)), t["g1_proj"]: TensorNeed((self.gate_rank, D)),
                 t["g2_proj"]: TensorNeed((self.v_cols, self.gate_rank)), t["norm"]: TensorNeed((self.dv,), "norm"),
                 t["o_proj"]: TensorNeed((D, self.v_cols))}
        if self.taps >= 1:
            needs.update({t["q_conv"]: TensorNeed((self.qk_cols, self.taps)), t["k_conv"]: TensorNeed((self.qk_cols, self.taps)),
                          t["v_conv"]: TensorNeed((self.v_cols, self.taps))})
        return needs

    def load(self, tensors):
        t = self.spec.tensors
        mats = [tensors[t[n]] for n in ("q_proj", "k_proj", "v_proj", "b_proj", "a1_proj", "g1_proj")]
        if len({m.dtype for m in mats}) != 1:
            raise ValueError("gated_delta: the input projections must share an element type")
        self.w_in = torch.cat(mats, dim=0).contiguous()              # [q | k | v | beta | a1 | g1]: h is read by one product
        self.w_a2, self.w_g2 = tensors[t["a2_proj"]].contiguous(), tensors[t["g2_proj"]].contiguous()
        self.w_o = tensors[t["o_proj"]].contiguous()
        f32 = lambda name: tensors[t[name]].to(torch.float32).contiguous()                        # noqa: E731
        self.a_log, self.dt_bias, self.norm_w = f32("a_log"), f32("dt_bias"), f32("norm")
        self.w_conv = None
        if self.taps >= 1:
            conv = torch.cat([tensors[t["q_conv"]], tensors[t["k_conv"]], tensors[t["v_conv"]]], dim=0)
            self.w_conv = conv.to(torch.float32).t().contiguous()    # tap-major, as the kernel reads it

    def state_need(self):
        # the slot's pitch stays a multiple of 16 bytes: the recurrence moves a state's rows in runs of four values
        return StateNeed(self.state_cols + (self.tail + 3) // 4 * 4, "float32")

    def flops_per_token(self) -> float:
        low_rank = self.decay_rank * self.n_heads * self.dk + self.gate_rank * self.v_cols
        return 2.0 * (self.hidden * (self.in_cols + self.v_cols) + low_rank) + 10.0 * self.n_heads * self.dk * self.dv

    def forward(self, h, residual, ctx: StepContext, call: CallInfo):
        rt, T, H, G, RP = self.runtime, ctx.n_tokens, self.n_heads, self.n_qk, self.rows_pad
        mbt = rt.max_batch_tokens
        proj = rt.get_scratch("state_proj", torch.float32)[:, : self.in_cols]
        rows = rt.get_scratch("state_rows", torch.float32)[0]
        q = rows[: mbt * G * RP].view(mbt, G * RP)
        k = rows[mbt * G * RP: 2 * mbt * G * RP].view(mbt, G * RP)
        g = rows[2 * mbt * G * RP: mbt * (2 * G + H) * RP].view(mbt, H * RP)
        step = rt.get_scratch("delta_step", torch.float32)[:, : H * self.dk]
        gate = rt.get_scratch("delta_gate", torch.float32)[:, : self.v_cols]
        vb = rt.get_scratch("delta_v", torch.float32)[0]
        v = vb[: mbt * self.v_cols].view(mbt, self.v_cols)
        beta = vb[mbt * self.v_cols: mbt * (self.v_cols + H)].view(mbt, H)
        read = rt.get_scratch("state_read", torch.float32)[:, : self.v_cols]
        out = rt.get_scratch("state_out")[:, : self.v_cols]
        ops.linear(h, self.w_in, proj, T, status=ctx.status)
        # the second halves of the two low-rank maps: decay steps and output gates, float32 in and out
        ops.linear(proj[:, self.a1_off: self.a1_off + self.decay_rank], self.w_a2, step, T, status=ctx.status)
        ops.linear(proj[:, self.g1_off: self.g1_off + self.gate_rank], self.w_g2, gate, T, status=ctx.status)
        state = call.state
        tail = state[:, self.state_cols:] if self.tail else None
        ops.delta_prep(proj, self.w_conv, tail, step, self.dt_bias, self.a_log, q, k, g, v, beta, ctx.seq_of_token, ctx.q_start,
                       ctx.state_slots, G, H, self.dk, self.dv, RP, self.beta_off, self.unit_eps, float(self.dk) ** -0.5, T,
                       ctx.n_seqs)
        ops.state_recurrence(q, k, g, beta, v, read, state, ctx.q_start, ctx.state_slots, ctx.n_seqs, H, H // G, RP, self.dv,
                             delta=True)
        ops.head_norm_gate(read, self.norm_w, gate, out, H, self.dv, self.eps, T)
        ops.linear(out, self.w_o, residual, T, accumulate=not ctx.store_output, status=ctx.status)


@register_part("mixer", "retention")
class Retention(Mixer):
    """params: hidden, n_heads, dim, vdim, decay (one number per head), eps (of the read-out norm), k_scale (default
    dim^-1/2), gate (bool, default True: the normed heads times silu(g_proj h)).
    tensors: q_proj, k_proj, v_proj, o_proj, and g_proj [heads * vdim, hidden] with a gate.  The layer's position part,
    if it has a rotation, must pair halves (coordinate i with i + n_rot / 2)."""

    def __init__(self, spec, runtime, position=None):
        super().__init__(spec, runtime)
        p = spec.params
        self.hidden, self.n_heads = int(p["hidden"]), int(p["n_heads"])
        self.dk, self.dv = int(p["dim"]), int(p["vdim"])
        self.decay = [float(d) for d in p["decay"]]
        if len(self.decay) != self.n_heads:
            raise ValueError(f"retention: {len(self.decay)} decays for {self.n_heads} heads")
        self.eps = float(p.get("eps", 0.0))
        self.k_scale = float(p["k_scale"]) if p.get("k_scale") is not None else float(self.dk) ** -0.5
        self.has_gate = bool(p.get("gate", True))
        self.position = position
        self.n_rot = int(getattr(position, "n_rot", 0) or 0)
        if self.n_rot and getattr(position, "pairing", "half") != "half":
            raise ValueError("retention: its kernel pairs the halves of the rotated prefix; the position part pairs otherwise")
        if self.n_rot > self.dk:
            raise ValueError(f"retention: {self.n_rot} rotated coordinates in heads of {self.dk}")
        self.rows_pad = ops.state_rows_pad(self.dk)
        self.qk_cols, self.v_cols = self.n_heads * self.dk, self.n_heads * self.dv
        self.in_cols = 2 * self.qk_cols + self.v_cols * (2 if self.has_gate else 1)
        rt = runtime
        rt.scratch("state_proj", rt.max_batch_tokens, self.in_cols, torch.float32)
        rt.scratch("state_rows", 1, 2 * rt.max_batch_tokens * self.n_heads * self.rows_pad, torch.float32)
        rt.scratch("state_read", rt.max_batch_tokens, self.v_cols, torch.float32)
        rt.scratch("state_out", rt.max_batch_tokens, self.v_cols)
        self.decay_rows = None

    def tensor_needs(self):
        t = self.spec.tensors
        needs = {t["q_proj"]: TensorNeed((self.qk_cols, self.hidden)), t["k_proj"]: TensorNeed((self.qk_cols, self.hidden)),
                 t["v_proj"]: TensorNeed((self.v_cols, self.hidden)), t["o_proj"]: TensorNeed((self.hidden, self.v_cols))}
        if self.has_gate:
            needs[t["g_proj"]] = TensorNeed((self.v_cols, self.hidden))
        return needs

    def load(self, tensors):
        t = self.spec.tensors
        mats = [tensors[t[n]] for n in ("q_proj", "k_proj", "v_proj")] + ([tensors[t["g_proj"]]] if self.has_gate else [])
        if len({m.dtype for m in mats}) != 1:
            raise ValueError("retention: the input projections must share an element type")
        self.w_in = torch.cat(mats, dim=0).contiguous()              # [q | k | v | gate]: h is read by one product
        self.w_o = tensors[t["o_proj"]].contiguous()
        # the decay of every row of every head, one row that all tokens read
        d = torch.tensor(self.decay, dtype=torch.float32).view(self.n_heads, 1).expand(self.n_heads, self.rows_pad)
        self.decay_rows = d.reshape(1, -1).contiguous().to(self.w_o.device)

    def state_need(self):
        return StateNeed(self.n_heads * self.dv * self.rows_pad, "float32")

    def flops_per_token(self) -> float:
        return 2.0 * self.hidden * (self.in_cols + self.v_cols) + 6.0 * self.n_heads * self.dk * self.dv

    def forward(self, h, residual, ctx: StepContext, call: CallInfo):
        rt, T, H, RP = self.runtime, ctx.n_tokens, self.n_heads, self.rows_pad
        proj = rt.get_scratch("state_proj", torch.float32)[:, : self.in_cols]
        n = rt.max_batch_tokens * H * RP
        rows = rt.get_scratch("state_rows", torch.float32)[0]
        q, k = (rows[i * n:(i + 1) * n].view(rt.max_batch_tokens, H * RP) for i in range(2))
        read = rt.get_scratch("state_read", torch.float32)[:, : self.v_cols]
        out = rt.get_scratch("state_out")[:, : self.v_cols]
        ops.linear(h, self.w_in, proj, T, status=ctx.status)
        rot = getattr(self.position, "cos_sin", None) if self.n_rot else None
        ops.retention_prep(proj, rot, self.n_rot, ctx.positions, self.k_scale, q, k, H, self.dk, RP, T, ctx.status)
        g = self.decay_rows.expand(T, H * RP)                        # pitch 0: the same decays for every token
        v_off = 2 * self.qk_cols
        ops.state_recurrence(q, k, g, None, proj[:, v_off: v_off + self.v_cols], read, call.state, ctx.q_start,
                             ctx.state_slots, ctx.n_seqs, H, 1, RP, self.dv, delta=False)
        gate = proj[:, v_off + self.v_cols:] if self.has_gate else None
        ops.head_norm_gate(read, None, gate, out, H, self.dv, self.eps, T, gate_silu=True)
        ops.linear(out, self.w_o, residual, T, accumulate=not ctx.store_output, status=ctx.status)


CHUNKED_FROM = 32      # the longest portion of a step from which on the bfloat16 engine walks it in chunks


class ChunkedRecurrence(Mixer):
    """What mixers share whose recurrence the chunked kernels take (csrc/state_chunks.cu): the step's list of chunks and the
    workspace.  The 32-bit engine, captured steps and steps of short portions walk token by token."""

    def _chunk_setup(self, n_heads: int, rows_pad: int, columns: int, head_decay: bool) -> None:
        rt = self.runtime
        self.chunks_ok = not rt.precise
        self._chunk_shape = (rows_pad, columns, head_decay)
        if self.chunks_ok:
            most = rt.max_batch_tokens // ops.STATE_CHUNK + rt.max_seqs
            rt.scratch("state_chunks", 1, most * n_heads * (columns + 1) * rows_pad, torch.float32)

    def plan_key(self):
        return ("state_chunks", ops.STATE_CHUNK) if self.chunks_ok else None

    def build_plan(self, batch: HostBatch):
        if batch.bucketed or int(batch.q_lens.max()) < CHUNKED_FROM:
            return {"n_chunks": 0}
        per_seq = -(-batch.q_lens // ops.STATE_CHUNK)
        first = np.zeros(batch.n_seqs + 1, np.int32)
        np.cumsum(per_seq, out=first[1:])
        seq = np.repeat(np.arange(batch.n_seqs, dtype=np.int32), per_seq)
        start = (np.arange(int(first[-1]), dtype=np.int32) - np.repeat(first[:-1], per_seq)) * ops.STATE_CHUNK
        return {"chunk_seq": seq, "chunk_start": start.astype(np.int32), "seq_first_chunk": first, "n_chunks": int(first[-1])}

    def _chunks(self, ctx: StepContext):
        """The step's chunk lists as keywords of ``ops.state_recurrence_chunked``, or None: token by token."""
        if not self.chunks_ok:
            return None
        plan = ctx.plans[self.plan_key()]
        if not plan["n_chunks"] or not ops.state_chunks_supported(*self._chunk_shape):
            return None
        return dict(plan, work=self.runtime.get_scratch("state_chunks", torch.float32))


def _on_16_bytes(dim: int, *ts) -> bool:
    """Whether every head of ``dim`` values in these float32 rows starts on 16 bytes (the recurrence can read them in place)."""
    return dim % 4 == 0 and all(t.stride(0) % 4 == 0 and t.data_ptr() % 16 == 0 for t in ts)


@register_part("mixer", "gated_linear_attention")
class GatedLinearAttention(ChunkedRecurrence):
    """params: hidden, n_heads, dim, vdim, tau, decay_rank (inner width of the decay's low-rank map), eps (of the read-out
    norm), q_scale (default dim^-1/2), out_scale (default 1: multiplies the mixer's output).
    tensors: q_proj, k_proj, v_proj, g_proj [heads * vdim, hidden], a1_proj [decay_rank, hidden], a2_proj [heads * dim,
    decay_rank], a2_bias [heads * dim], norm [vdim], o_proj."""
    joinable = True

    def __init__(self, spec, runtime, position=None):
        super().__init__(spec, runtime)
        p = spec.params
        self.hidden, self.n_heads = int(p["hidden"]), int(p["n_heads"])
        self.dk, self.dv = int(p["dim"]), int(p["vdim"])
        self.tau, self.rank = float(p["tau"]), int(p["decay_rank"])
        self.eps = float(p.get("eps", 0.0))
        self.q_scale = float(p["q_scale"]) if p.get("q_scale") is not None else float(self.dk) ** -0.5
        self.out_scale = float(p.get("out_scale", 1.0))
        if not self.tau > 0 or self.rank < 1:
            raise ValueError(f"gated_linear_attention: tau {self.tau} and decay_rank {self.rank} must be positive")
        self.rows_pad = ops.state_rows_pad(self.dk)
        self.qk_cols, self.v_cols = self.n_heads * self.dk, self.n_heads * self.dv
        self.v_off = 2 * self.qk_cols
        self.g_off = self.v_off + self.v_cols
        self.a1_off = self.g_off + self.v_cols
        self.in_cols = self.a1_off + self.rank
        self.row_cols = self.v_cols
        rt = runtime
        rt.scratch("state_proj", rt.max_batch_tokens, self.in_cols, torch.float32)
        # decays, and where heads do not start on 16 bytes the padded queries and keys
        rt.scratch("state_rows", 1, 3 * rt.max_batch_tokens * self.n_heads * self.rows_pad, torch.float32)
        rt.scratch("state_read", rt.max_batch_tokens, self.v_cols, torch.float32)
        rt.scratch("state_out", rt.max_batch_tokens, self.v_cols)
        self._chunk_setup(self.n_heads, self.rows_pad, self.dv, False)

    def tensor_needs(self):
        t, D = self.spec.tensors, self.hidden
        return {t["q_proj"]: TensorNeed((self.qk_cols, D)), t["k_proj"]: TensorNeed((self.qk_cols, D)),
                t["v_proj"]: TensorNeed((self.v_cols, D)), t["g_proj"]: TensorNeed((self.v_cols, D)),
                t["a1_proj"]: TensorNeed((self.rank, D)), t["a2_proj"]: TensorNeed((self.qk_cols, self.rank)),
                t["a2_bias"]: TensorNeed((self.qk_cols,)), t["norm"]: TensorNeed((self.dv,), "norm"),
                t["o_proj"]: TensorNeed((D, self.v_cols))}

    def load(self, tensors):
        t = self.spec.tensors
        mats = [tensors[t[n]] for n in ("q_proj", "k_proj", "v_proj", "g_proj", "a1_proj")]
        if len({m.dtype for m in mats}) != 1:
            raise ValueError("gated_linear_attention: the input projections must share an element type")
        self.w_in = torch.cat(mats, dim=0).contiguous()              # [q | k | v | gate | a1]: h is read by one product
        self.w_a2 = tensors[t["a2_proj"]].contiguous()
        self.a2_bias = tensors[t["a2_bias"]].to(torch.float32).contiguous()
        # the output's factor rides on the read-out norm's weight, in float32
        self.norm_w = (tensors[t["norm"]].to(torch.float32) * self.out_scale).contiguous()
        self.w_o = tensors[t["o_proj"]].contiguous()

    def state_need(self):
        return StateNeed(self.n_heads * self.dv * self.rows_pad, "float32")

    def flops_per_token(self) -> float:
        return 2.0 * (self.hidden * (self.in_cols + self.v_cols) + self.qk_cols * self.rank) + 6.0 * self.n_heads * self.dk * self.dv

    def forward(self, h, residual, ctx: StepContext, call: CallInfo):
        rt, T = self.runtime, ctx.n_tokens
        proj = rt.get_scratch("state_proj", torch.float32)[:, : self.in_cols]
        out = rt.get_scratch("state_out")[:, : self.v_cols]
        ops.linear(h, self.w_in, proj, T, status=ctx.status)
        self.forward_rows(proj, out, ctx, call)
        ops.linear(out, self.w_o, residual, T, accumulate=not ctx.store_output, status=ctx.status)

    def forward_rows(self, proj, out, ctx: StepContext, call: CallInfo):
        rt, T, H, RP = self.runtime, ctx.n_tokens, self.n_heads, self.rows_pad
        mbt = rt.max_batch_tokens
        n = mbt * H * RP
        flat = rt.get_scratch("state_rows", torch.float32)[0]
        q_buf, k_buf = flat[:n].view(mbt, H * RP), flat[n: 2 * n].view(mbt, H * RP)
        read = rt.get_scratch("state_read", torch.float32)[:, : self.v_cols]
        q, k, rows = proj[:, : self.qk_cols], proj[:, self.qk_cols: self.v_off], self.dk
        if not _on_16_bytes(self.dk, q, k):
            ops.pad_heads(q, q_buf, H, self.dk, RP, T)
            ops.pad_heads(k, k_buf, H, self.dk, RP, T)
            q, k, rows = q_buf, k_buf, RP
        g = flat[2 * n: 2 * n + mbt * H * rows].view(mbt, H * rows)
        chunks = self._chunks(ctx)
        ops.low_rank_decay(proj[:, self.a1_off: self.a1_off + self.rank], self.w_a2, self.a2_bias, self.tau, g, H, self.dk, rows, T,
                           log_decay=chunks is not None)
        walk = ops.state_recurrence if chunks is None else ops.state_recurrence_chunked
        walk(q, k, g, None, proj[:, self.v_off: self.g_off], read, call.state, ctx.q_start, ctx.state_slots, ctx.n_seqs, H, 1, RP,
             self.dv, rows=rows, q_scale=self.q_scale, **(chunks or {}))
        ops.head_norm_gate(read, self.norm_w, proj[:, self.g_off: self.a1_off], out, H, self.dv, self.eps, T, gate_silu=True)


@register_part("mixer", "mamba2")
class Mamba2(ChunkedRecurrence):
    """params: hidden, n_heads, vdim, state (rows of a head's state), groups (of B and C), taps, norm_groups, eps (of the
    read-out norm), out_scale (default 1: multiplies the mixer's output).
    tensors: in_proj [2 * inner + 2 * groups * state + heads, hidden], conv [inner + 2 * groups * state, taps], conv_bias,
    dt_bias [heads], a_log [heads], d_skip [heads], norm [inner], o_proj [hidden, inner], inner = heads * vdim."""
    joinable = True

    def __init__(self, spec, runtime, position=None):
        super().__init__(spec, runtime)
        p = spec.params
        self.hidden, self.n_heads, self.dv = int(p["hidden"]), int(p["n_heads"]), int(p["vdim"])
        self.rows, self.groups, self.taps = int(p["state"]), int(p["groups"]), int(p["taps"])
        self.norm_groups, self.eps = int(p["norm_groups"]), float(p.get("eps", 0.0))
        self.out_scale = float(p.get("out_scale", 1.0))
        if self.n_heads % self.groups:
            raise ValueError(f"mamba2: {self.n_heads} heads are not a multiple of {self.groups} groups")
        self.inner = self.row_cols = self.n_heads * self.dv
        if self.inner % self.norm_groups:
            raise ValueError(f"mamba2: {self.inner} inner channels do not divide into {self.norm_groups} norm groups")
        if not 1 <= self.taps <= 64:
            raise ValueError(f"mamba2: {self.taps} taps (1 to 64 are supported)")
        self.rows_pad = ops.state_rows_pad(self.rows)
        self.bc_cols = self.groups * self.rows
        self.channels = self.inner + 2 * self.bc_cols
        self.dt_off = self.inner + self.channels
        self.in_cols = self.dt_off + self.n_heads
        self.tail = (self.taps - 1) * self.channels
        self.state_cols = self.n_heads * self.dv * self.rows_pad
        rt, mbt = runtime, runtime.max_batch_tokens
        rt.scratch("state_proj", mbt, self.in_cols, torch.float32)
        self.conv_pitch = (self.channels + 3) // 4 * 4
        rt.scratch("mamba_conv", mbt, self.conv_pitch, torch.float32)
        rt.scratch("mamba_step", 1, 2 * mbt * self.n_heads, torch.float32)
        if self.rows % 4 or self.inner % 4:
            rt.scratch("state_rows", 1, 2 * mbt * self.groups * self.rows_pad, torch.float32)
        rt.scratch("state_read", mbt, self.inner, torch.float32)
        rt.scratch("state_out", mbt, self.inner)
        self._chunk_setup(self.n_heads, self.rows_pad, self.dv, True)

    def tensor_needs(self):
        t, D, H = self.spec.tensors, self.hidden, self.n_heads
        return {t["in_proj"]: TensorNeed((self.in_cols, D)), t["conv"]: TensorNeed((self.channels, self.taps)),
                t["conv_bias"]: TensorNeed((self.channels,)), t["dt_bias"]: TensorNeed((H,)), t["a_log"]: TensorNeed((H,)),
                t["d_skip"]: TensorNeed((H,)), t["norm"]: TensorNeed((self.inner,), "norm"),
                t["o_proj"]: TensorNeed((D, self.inner))}

    def load(self, tensors):
        t = self.spec.tensors
        f32 = lambda name: tensors[t[name]].to(torch.float32).contiguous()                        # noqa: E731
        self.w_in, self.w_o = tensors[t["in_proj"]].contiguous(), tensors[t["o_proj"]].contiguous()
        self.w_conv = f32("conv").t().contiguous()                   # tap-major, as the kernel reads it
        self.conv_bias, self.dt_bias, self.a_log, self.d_skip = f32("conv_bias"), f32("dt_bias"), f32("a_log"), f32("d_skip")
        self.norm_w = (f32("norm") * self.out_scale).contiguous()

    def state_need(self):
        # the slot's pitch stays a multiple of 16 bytes: the recurrence moves a state's rows in runs of four values
        return StateNeed(self.state_cols + (self.tail + 3) // 4 * 4, "float32")

    def flops_per_token(self) -> float:
        return 2.0 * self.hidden * (self.in_cols + self.inner) + 6.0 * self.n_heads * self.rows * self.dv

    def forward(self, h, residual, ctx: StepContext, call: CallInfo):
        rt, T = self.runtime, ctx.n_tokens
        proj = rt.get_scratch("state_proj", torch.float32)[:, : self.in_cols]
        out = rt.get_scratch("state_out")[:, : self.inner]
        ops.linear(h, self.w_in, proj, T, status=ctx.status)
        self.forward_rows(proj, out, ctx, call)
        ops.linear(out, self.w_o, residual, T, accumulate=not ctx.store_output, status=ctx.status)

    def forward_rows(self, proj, out, ctx: StepContext, call: CallInfo):
        rt, T, H, G, RP = self.runtime, ctx.n_tokens, self.n_heads, self.groups, self.rows_pad
        mbt = rt.max_batch_tokens
        conv = rt.get_scratch("mamba_conv", torch.float32)[:, : self.channels]
        flat = rt.get_scratch("mamba_step", torch.float32)[0]
        dt, decay = flat[: mbt * H].view(mbt, H), flat[mbt * H: 2 * mbt * H].view(mbt, H)
        read = rt.get_scratch("state_read", torch.float32)[:, : self.inner]
        state, chunks = call.state, self._chunks(ctx)
        ops.mamba2_prep(proj, self.inner, self.dt_off, self.w_conv, self.conv_bias, state[:, self.state_cols:] if self.tail else None,
                        self.dt_bias, self.a_log, conv, dt, decay, ctx.seq_of_token, ctx.q_start, ctx.state_slots, H, T, ctx.n_seqs,
                        log_decay=chunks is not None)
        k, q, rows = conv[:, self.inner: self.inner + self.bc_cols], conv[:, self.inner + self.bc_cols:], self.rows
        if not _on_16_bytes(self.rows, k, q):
            n = mbt * G * RP
            pads = rt.get_scratch("state_rows", torch.float32)[0]
            k_buf, q_buf = pads[:n].view(mbt, G * RP), pads[n: 2 * n].view(mbt, G * RP)
            ops.pad_heads(k, k_buf, G, self.rows, RP, T)
            ops.pad_heads(q, q_buf, G, self.rows, RP, T)
            k, q, rows = k_buf, q_buf, RP
        walk = ops.state_recurrence if chunks is None else ops.state_recurrence_chunked
        walk(q, k, decay, dt, conv[:, : self.inner], read, state, ctx.q_start, ctx.state_slots, ctx.n_seqs, H, H // G, RP, self.dv,
             head_decay=True, rows=rows, skip=self.d_skip, **(chunks or {}))
        ops.gated_group_norm(read, proj[:, : self.inner], self.norm_w, out, self.norm_groups, self.eps, T)
