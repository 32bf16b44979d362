"""A plain, slow implementation of the Gemodra decoder in float64, one function per mechanism.

It runs a whole sequence at once, keeps no cache, expands every key and value from the latent and shares no code with
the engine: the engine's kernels, parts and step function are compared with it.  ``weights`` maps checkpoint tensor names
to float64 torch tensors on the CPU; ``config`` is the parsed config.json.

Notation: every matrix is stored [out, in] and applied as x @ W.T; positions are 0 .. T - 1.
"""
from __future__ import annotations

import math

import torch

F64 = torch.float64


# ----------------------------------------------------------------------------- small pieces
def rms_norm(x, w, eps):
    """x over the root of (its mean square + eps) along the last axis, times w."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps) * w


def silu(z):
    return z * torch.sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def rotate_pairs(x, base, dims):
    """x [T, n, width]: coordinates 2i and 2i + 1 < dims form a pair that is turned by t * base^(-2i/dims)."""
    T = x.shape[0]
    i = torch.arange(dims // 2, dtype=F64)
    ang = torch.arange(T, dtype=F64)[:, None] * torch.pow(torch.tensor(base, dtype=F64), -2.0 * i / dims)[None, :]
    c, s = torch.cos(ang)[:, None, :], torch.sin(ang)[:, None, :]
    out = x.clone()
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out[..., 0:dims:2] = u * c - v * s
    out[..., 1:dims:2] = v * c + u * s
    return out


def causal_softmax(scores, sink):
    """Weights over the keys j <= i whose denominator also holds exp(sink) of the head.  scores [H, T, T], sink [H]."""
    T = scores.shape[-1]
    later = torch.arange(T)[None, :] > torch.arange(T)[:, None]
    s = scores.masked_fill(later[None], -math.inf)
    m = torch.maximum(s.max(dim=-1, keepdim=True).values, sink[:, None, None])
    e = torch.exp(s - m)
    return e / (e.sum(dim=-1, keepdim=True) + torch.exp(sink[:, None, None] - m))


# ----------------------------------------------------------------------------- mixers
def query_through_latent(h, w, p, eps):
    """W_uq RMSNorm(W_dq h)."""
    return rms_norm(h @ w[p + "dq"].T, w[p + "dq.norm"], eps) @ w[p + "uq"].T


def latent_attention(h, w, p, m, eps):
    """Heads with an unrotated and a rotated score part, the rotated key part shared by all heads; the joined heads are
    gated element by element."""
    T = h.shape[0]
    H, dn, dr, dv, rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = query_through_latent(h, w, p, eps).view(T, H, dn + dr)
    down = h @ w[p + "dkv"].T
    c = rms_norm(down[:, :rank], w[p + "dkv.norm"], eps)
    rot = m["rot"]
    k_rot = rotate_pairs(down[:, None, rank:], rot["base"], rot["dims"])[:, 0]
    q_rot = rotate_pairs(q[..., dn:], rot["base"], rot["dims"])
    k = (c @ w[p + "uk"].T).view(T, H, dn)
    v = (c @ w[p + "uv"].T).view(T, H, dv)
    scores = (torch.einsum("ihd,jhd->hij", q[..., :dn], k) + torch.einsum("ihd,jd->hij", q_rot, k_rot)) * m["scale"]
    o = torch.einsum("hij,jhd->ihd", causal_softmax(scores, w[p + "sink"]), v).reshape(T, H * dv)
    return (o * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def latent_attention_unrotated(h, w, p, m, eps):
    """Latent attention without positions; each head's result is gated by one number."""
    T = h.shape[0]
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    q = query_through_latent(h, w, p, eps).view(T, H, d)
    c = rms_norm(h @ w[p + "dkv"].T, w[p + "dkv.norm"], eps)
    k = (c @ w[p + "uk"].T).view(T, H, d)
    v = (c @ w[p + "uv"].T).view(T, H, dv)
    scores = torch.einsum("ihd,jhd->hij", q, k) * m["scale"]
    o = torch.einsum("hij,jhd->ihd", causal_softmax(scores, w[p + "sink"]), v)
    return (o * torch.sigmoid(h @ w[p + "g"].T)[:, :, None]).reshape(T, H * dv) @ w[p + "o"].T


MIXERS = {"latent_attention": latent_attention, "latent_attention_2": latent_attention_unrotated}


# ----------------------------------------------------------------------------- feed-forward
def route(h, w, p, router):
    """(chosen indices [T, top], weights [T, top]) of a token's outputs among experts and identity experts."""
    T = h.shape[0]
    z = h @ w[p + "router"].T
    s = torch.softmax(z, dim=-1)
    choice = s + w[p + "correction"]
    groups = router.get("groups")
    if groups:
        per = choice.shape[1] // groups["count"]
        worth = choice.view(T, groups["count"], per).max(dim=-1).values
        kept = worth.topk(groups["keep"], dim=-1).indices
        ok = torch.zeros(T, groups["count"], dtype=torch.bool).scatter_(1, kept, True)
        choice = choice.masked_fill(~ok.repeat_interleave(per, dim=1), -math.inf)
    idx = choice.topk(router["top"], dim=-1).indices
    return idx, torch.gather(s, 1, idx) * router.get("scale", 1.0)


def gated_ff(h, w, p):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def mixture(h, w, p, mlp):
    router = mlp["router"]
    idx, weight = route(h, w, p, router)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for k in range(router["top"]):
            e = int(idx[t, k])
            y = h[t] if e >= router["experts"] else gated_ff(h[t], w, f"{p}e{e}.")
            out[t] = out[t] + weight[t, k] * y
    if mlp.get("shared"):
        out = out + torch.sigmoid(h @ w[p + "shared.sg"].T) * gated_ff(h, w, p + "shared.")
    return out


# ----------------------------------------------------------------------------- the layer and the model
def token_side(x, tokens, w, p, i, dim, eps):
    """RMSNorm(W_proj (gelu(W_gate x) * e)) with e the layer's part of the token's row in the side table."""
    e = w["side.embed"][tokens][:, i * dim: (i + 1) * dim]
    y = (gelu_tanh(x @ w[p + "side.gate"].T) * e) @ w[p + "side.proj"].T
    return rms_norm(y, w[p + "side.norm"], eps)


def layer(x, tokens, w, config, i):
    L, eps, m = config["layers"][i], config["norm"]["eps"], config.get("residual_mult", 1.0)
    p = f"l{i}."
    x = x + m * MIXERS[L["type"]](rms_norm(x, w[p + "norm1"], eps), w, p + "mix.", L["mixer"], eps)
    if L.get("mlp"):
        x = x + m * mixture(rms_norm(x, w[p + "norm2"], eps), w, p + "mlp.", L["mlp"])
    if config.get("token_side"):
        x = x + m * token_side(x, tokens, w, p, i, config["token_side"]["dim"], eps)
    return x


def forward(tokens, w, config, layers_out=None):
    """Logits [T, vocab] of a whole sequence; ``layers_out`` collects the stream after every layer."""
    tokens = torch.as_tensor(tokens, dtype=torch.long)
    eps = config["norm"]["eps"]
    x = rms_norm(w["embed"][tokens], w["embed.norm"], eps)
    for i in range(len(config["layers"])):
        x = layer(x, tokens, w, config, i)
        if layers_out is not None:
            layers_out.append(x)
    z = rms_norm(x, w["final.norm"], eps) @ w["head"].T
    cap = config.get("logit_softcap")
    return cap * torch.tanh(z / cap) if cap else z
