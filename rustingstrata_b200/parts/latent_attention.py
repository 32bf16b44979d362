"""Attention whose keys and values are expanded from a cached low-rank latent (multi-head latent attention).

Per token the mixer's input h gives q = W_q h, laid out head by head as [dim unrotated | rot_dim rotated], and
W_dkv h = [latent part (kv_rank) | one rotated key part (rot_dim) shared by all heads].  c = RMSNorm(latent part) is
the latent; head k's key is [W_uk,k c | rotated part], its value W_uv,k c, and a score is
(q_unrotated . k_unrotated + q_rotated . k_rotated) * scale over the causal keys, softmax, W_o on the joined heads.

``rot_dim`` may be 0 (no rotated parts, no position part).  With ``q_rank`` the queries come through a latent of their own,
q = W_uq RMSNorm(W_dq h).  With ``sink`` the softmax's denominator of head k also holds exp(sink[k]), which has no key and no
value.  With ``gate`` the joined heads are multiplied by sigmoid(W_g h) before W_o, one number per token and head ("head") or
one per value ("element").  ``out_scale`` multiplies the mixer's output (a residual multiplier, say).

The projections that read h are one product [latent | rotated key part | query latent | gates]; gate and out_scale ride in
the value map's epilogue, in float32.

Only [c | rotated key part] is cached: one row per token (a one-plane cache, one "kv head" that every query head
reads).  The expansion is folded into the query and the result, which gives the same numbers:

    q_unrotated . (W_uk,k c) = (W_uk,k^T q_unrotated) . c         so the query of head k becomes [W_uk,k^T q_unrotated | q_rotated],
    sum_j p_j (W_uv,k c_j)   = W_uv,k (sum_j p_j c_j)             so attention returns latent sums and W_uv,k follows,

i.e. attention with ``heads`` query heads over one shared key/value row of kv_rank + rot_dim values (rounded up to
the kernels' multiple of 16, the padding zero).  The work lists, split form and partial-result workspace are those
of :class:`~rustingstrata_b200.parts.attention.PagedAttention`; the per-head maps are block-diagonal products.
"""
from __future__ import annotations

import torch

from ..kernels import ops
from .attention import SPLIT_KEYS, PagedAttention
from .base import CallInfo, StepContext
from .registry import register_part
from .spec import CacheNeed, PartSpec, TensorNeed


WIDE_TILES = 64        # tiles of 64 query rows from which a step's portions take the wide kernel


@register_part("mixer", "latent_attention")
class LatentAttention(PagedAttention):
    """params: hidden, n_heads, dim (unrotated query/key size per head), rot_dim, vdim, kv_rank, scale, eps (of the
    latents' norms), window (None: every key), q_rank (None: q = W_q h), sink (bool, default False), gate (None, "head" or True, or
    "element"), out_scale (default 1), weights_bits (16, the default: the tensor-core kernel rounds the softmax weights to
    bfloat16 for the weighted sum; 32: it multiplies them in two bfloat16 terms).  tensors: q_proj [heads * (dim + rot_dim),
    hidden], or with q_rank dq_proj [q_rank, hidden], q_latent_norm [q_rank] and q_proj [heads * (dim + rot_dim), q_rank];
    dkv_proj, latent_norm, uk_proj [heads * dim, kv_rank], uv_proj [heads * vdim, kv_rank], o_proj; g_proj [heads or
    heads * vdim, hidden] with a gate; sink [heads].  The layer's position part rotates the first ``n_rot`` <= rot_dim
    coordinates of the rotated parts (pairs (2i, 2i + 1): a part whose ``pairing`` is "interleaved")."""
    chain_safe = False
    one_plane = True
    max_head_dim = 576     # what the CUDA-core attention takes: a 512-wide latent with a 64-wide rotated part

    def __init__(self, spec, runtime, position=None):
        p = spec.params
        self.dim, self.rot_dim, self.vdim = int(p["dim"]), int(p["rot_dim"]), int(p["vdim"])
        self.rank = int(p["kv_rank"])
        self.q_head = self.dim + self.rot_dim
        self.lat = (self.rank + self.rot_dim + 15) // 16 * 16            # width of a cache row and of an absorbed query head
        if self.lat > 576:
            raise ValueError(f"latent_attention: kv_rank + rot_dim = {self.rank + self.rot_dim} exceeds the 576 values "
                             f"the attention kernels take per head")
        inner = PartSpec(spec.kind, {"hidden": p["hidden"], "n_heads": p["n_heads"], "n_kv_heads": 1, "head_dim": self.lat,
                                     "window": p.get("window"), "scale": p["scale"], "qk_norm": False}, spec.tensors)
        super().__init__(inner, runtime, position)
        self.spec = spec
        self._tensor_cores = None
        self.latent_eps = float(p["eps"])
        self.gate = {True: "head"}.get(p.get("gate"), p.get("gate") or None)
        if self.gate not in (None, "head", "element"):
            raise ValueError(f"latent_attention: gate {self.gate!r} (known: None, 'head', 'element')")
        self.gate_cols = {None: 0, "head": self.n_heads, "element": self.n_heads * self.vdim}[self.gate]
        self.q_rank = int(p.get("q_rank") or 0)
        self.has_sink = bool(p.get("sink", False))
        self.out_scale = float(p.get("out_scale", 1.0))
        self.split_weights = int(p.get("weights_bits", 16)) == 32
        # columns of the projection that reads h
        self.cq_at = self.rank + self.rot_dim
        self.gate_at = self.cq_at + self.q_rank
        self.dkv_cols = self.gate_at + self.gate_cols
        self.sink = None
        if position is not None and getattr(position, "cos_sin", None) is not None:
            if getattr(position, "pairing", "") != "interleaved":
                raise ValueError("latent_attention rotates neighbouring pairs: its position part must be an interleaved rotation")
            if position.n_rot > self.rot_dim:
                raise ValueError(f"latent_attention: {position.n_rot} rotated coordinates exceed rot_dim {self.rot_dim}")
        rt = runtime
        rt.scratch("latent_q", rt.max_batch_tokens, self.n_heads * self.q_head)
        rt.scratch("latent_dkv", rt.max_batch_tokens, self.dkv_cols, torch.float32)
        if self.q_rank:
            # the row pitch is the row's own width (rounded up), so that the rows stay 16-byte aligned whatever other layers ask for
            self.cq_name = f"latent_cq_{(self.q_rank + 7) // 8 * 8}"
            rt.scratch(self.cq_name, rt.max_batch_tokens, (self.q_rank + 7) // 8 * 8)
        rt.scratch("latent_o", rt.max_batch_tokens, self.n_heads * self.vdim)

    def tensor_needs(self):
        t, H = self.spec.tensors, self.n_heads
        needs = {t["q_proj"]: TensorNeed((H * self.q_head, self.q_rank or self.hidden)),
                 t["dkv_proj"]: TensorNeed((self.rank + self.rot_dim, self.hidden)),
                 t["latent_norm"]: TensorNeed((self.rank,), "norm"),
                 t["uk_proj"]: TensorNeed((H * self.dim, self.rank)),
                 t["uv_proj"]: TensorNeed((H * self.vdim, self.rank)),
                 t["o_proj"]: TensorNeed((self.hidden, H * self.vdim))}
        if self.q_rank:
            needs[t["dq_proj"]] = TensorNeed((self.q_rank, self.hidden))
            needs[t["q_latent_norm"]] = TensorNeed((self.q_rank,), "norm")
        if self.gate:
            needs[t["g_proj"]] = TensorNeed((self.gate_cols, self.hidden))
        if self.has_sink:
            needs[t["sink"]] = TensorNeed((H,))
        return needs

    def load(self, tensors):
        t, H = self.spec.tensors, self.n_heads
        self.w_q = tensors[t["q_proj"]].contiguous()
        down = [tensors[t["dkv_proj"]]]
        if self.q_rank:
            down.append(tensors[t["dq_proj"]])
            self.q_latent_norm = tensors[t["q_latent_norm"]].contiguous()
        if self.gate:
            down.append(tensors[t["g_proj"]])
        if len({w.dtype for w in down}) != 1:
            raise ValueError("latent_attention: the gate's and the latents' projections must share an element type")
        self.w_dkv = torch.cat(down, dim=0).contiguous()      # [latent | rotated key part | query latent | gates]: one product
        if self.has_sink:
            self.sink = tensors[t["sink"]].to(torch.float32).contiguous()
        self.latent_norm = tensors[t["latent_norm"]].contiguous()
        # head k's key expansion transposed: [rank, dim], the map from its unrotated query to the latent's coordinates
        self.w_uk_t = tensors[t["uk_proj"]].reshape(H, self.dim, self.rank).transpose(1, 2).contiguous()
        self.w_uv = tensors[t["uv_proj"]].reshape(H, self.vdim, self.rank).contiguous()
        self.w_o = tensors[t["o_proj"]].contiguous()

    def cache_need(self):
        return CacheNeed(1, self.lat, self.window or None, planes=1)

    def _sink(self):
        return self.sink

    @property
    def tensor_cores(self) -> bool:
        """Whether the tensor-core kernel of latent attention runs (the bfloat16 engine); else the CUDA-core kernel."""
        if self._tensor_cores is None:
            self._tensor_cores = ops.attention_latent_ok(self.runtime.dtype, self.n_heads, self.lat, self.runtime.page_size)
        return self._tensor_cores

    def plan_key(self):
        if not self.tensor_cores:
            return super().plan_key()
        if self.q_per_cta is None:
            self.q_per_cta = ops.attention_latent_q_per_cta(self.n_heads)
            self.q_per_wide_cta = ops.attention_latent_q_per_cta(self.n_heads, wide=True)
        return ("latent_attention", self.n_heads, self.window)

    def _tile_tokens(self, q_lens):
        """Wide tiles (64 query rows) where the step's portions give the device enough of them, else narrow ones (16)."""
        if not self.tensor_cores:
            return super()._tile_tokens(q_lens)
        head_parts = -(-self.n_heads // ops.LATENT_WIDE_ROWS)
        tiles = int(sum(-(-int(n) // self.q_per_wide_cta) for n in q_lens)) * head_parts
        return self.q_per_wide_cta if tiles >= WIDE_TILES else self.q_per_cta

    def _attend(self, q, ctx: StepContext, call: CallInfo):
        if not self.tensor_cores:
            return super()._attend(q, ctx, call)
        rt = self.runtime
        out = rt.get_scratch("attn_out")[:, : self.q_width]
        plan = ctx.plans[self.plan_key()]
        common = dict(q=q, out=out, cache=call.cache, block_table=ctx.block_tables[call.cache_group], q_start=ctx.q_start,
                      kv_len=ctx.kv_len, n_heads=self.n_heads, lat=self.lat, page_size=rt.page_size, window=self.window,
                      scale=self.scale, status=ctx.status, split_weights=self.split_weights, sink=self.sink,
                      v_cols=(self.rank + 7) // 8 * 8)
        if plan["n_prefill"]:
            ops.attention_latent(work=plan["prefill_work"], n_work=plan["n_prefill"], decode=False,
                                 wide=plan["tile_tokens"] != self.q_per_cta, **common)
        if plan["n_decode"]:
            ops.attention_latent(work=plan["decode_work"], n_work=plan["n_decode"], decode=True, split_keys=SPLIT_KEYS,
                                 max_splits=plan["max_splits"], split_start=plan["split_start"],
                                 total_splits=plan["total_splits"], partial=rt.get_scratch("attn_partial", torch.float32),
                                 **common)
        return out

    def flops_per_token(self) -> float:
        """Multiply-add flops of the products one token passes (the folded form the kernels run)."""
        H = self.n_heads
        return 2.0 * (H * self.q_head * (self.q_rank or self.hidden) + self.dkv_cols * self.hidden + H * self.rank * self.dim
                      + H * self.vdim * self.rank + self.hidden * H * self.vdim)

    def forward(self, h, residual, ctx: StepContext, call: CallInfo):
        rt, T, H = self.runtime, ctx.n_tokens, self.n_heads
        if not call.writes_cache:
            raise RuntimeError("latent_attention: every call owns its cache")
        q = rt.get_scratch("latent_q")[:, : H * self.q_head]
        dkv = rt.get_scratch("latent_dkv", torch.float32)[:, : self.dkv_cols]
        q_lat = rt.get_scratch("qkv")[:, : H * self.lat]
        o = rt.get_scratch("latent_o")[:, : H * self.vdim]
        pos = self.position
        rot = getattr(pos, "cos_sin", None) if pos is not None else None
        where = (rot, pos.n_rot if rot is not None else 0, ctx.positions, ctx.seq_of_token, ctx.block_tables[call.cache_group],
                 rt.page_size)
        sizes = (self.rank, self.rot_dim, self.lat, H, T, ctx.status)
        row = (dkv, self.latent_norm, self.latent_eps)
        query = (q, self.q_head, self.dim, q_lat)
        ops.linear(h, self.w_dkv, dkv, T, status=ctx.status)
        if not self.q_rank:
            ops.linear(h, self.w_q, q, T, status=ctx.status)
            ops.block_linear(q, self.w_uk_t, q_lat, T, self.q_head, self.lat)
            ops.latent_kv_write(*row, *query, *where, call.cache, *sizes)
        else:
            cq = rt.get_scratch(self.cq_name)[:, : self.q_rank]
            ops.latent_kv_write(*row, None, 0, 0, None, *where, call.cache, *sizes, cq=dkv[:, self.cq_at: self.gate_at],
                                cq_weight=self.q_latent_norm, cq_out=cq)
            ops.linear(cq, self.w_q, q, T, status=ctx.status)
            rot, n_rot, *place = where
            ops.latent_queries(q, self.w_uk_t, q_lat, T, self.q_head, self.lat, rot, n_rot, self.rot_dim, *place, ctx.status)
        out = self._attend(q_lat, ctx, call)
        ops.block_linear(out, self.w_uv, o, T, self.lat, self.vdim, gate=dkv[:, self.gate_at:] if self.gate else None,
                         out_scale=self.out_scale)
        ctx.owed = ops.linear(o, self.w_o, residual, T, accumulate=not ctx.store_output, status=ctx.status,
                              may_defer=ctx.may_owe and not ctx.store_output)
