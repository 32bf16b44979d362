"""A plain, slow implementation of the Sefelorn decoder in float64, one function per mechanism.

It runs a whole sequence at once, keeps no cache and no state (recurrences start from zero and walk every token) and
shares no code with the engine: the engine's kernels, parts and step function are compared with it.  ``weights``
maps checkpoint tensor names to float64 torch tensors on the CPU; ``config`` is the parsed config.json.

Notation: every matrix is stored [out, in] and applied as x @ W.T; x is the residual stream [T, D].
"""
from __future__ import annotations

import torch

F64 = torch.float64


# ----------------------------------------------------------------------------- small pieces
def unit_rms(x, eps):
    """x over the root of its mean square along the last axis, eps inside the root."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def silu(z):
    return z * torch.sigmoid(z)


def softplus(z):
    return torch.where(z > 30.0, z, torch.log1p(torch.exp(torch.clamp(z, max=30.0))))


def causal_conv(u, w, b):
    """out[t] = b + sum_j w[:, j] * u[t - (taps - 1) + j], zeros before the start.  u [T, C], w [C, taps], b [C]."""
    T, C = u.shape
    taps = w.shape[1]
    out = torch.zeros(T, C, dtype=u.dtype) + b
    for j in range(taps):
        back = taps - 1 - j
        if back < T:
            out[back:] += w[:, j] * u[: T - back]
    return out


def rotate_halves(x, dims, base):
    """x [T, heads, dim]: coordinate i turns with i + dims / 2 by position * base^(-2i / dims), i < dims / 2."""
    half = dims // 2
    f = torch.tensor([float(base) ** (-2.0 * i / dims) for i in range(half)], dtype=F64)
    ang = torch.arange(x.shape[0], dtype=F64)[:, None] * f[None, :]
    c, s = torch.cos(ang)[:, None, :], torch.sin(ang)[:, None, :]
    out = x.clone()
    u, v = x[..., :half], x[..., half:dims]
    out[..., :half] = u * c - v * s
    out[..., half:dims] = v * c + u * s
    return out


def visible(T, size, keep_first):
    """[T, T] booleans: query i sees key j if j <= i and (i - j < size or j < keep_first)."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    return (j <= i) & ((i - j < size) | (j < keep_first))


# ----------------------------------------------------------------------------- mixers
def softmax_attention(h, weights, prefix, m):
    """Biased, rotated softmax attention over a window and the sequence's first tokens."""
    H, G, dk, dv = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    T = h.shape[0]
    W = lambda n: weights[prefix + n]                                       # noqa: E731
    q = (h @ W("q").T + W("q.b")).reshape(T, H, dk)
    k = (h @ W("k").T + W("k.b")).reshape(T, G, dk)
    v = (h @ W("v").T + W("v.b")).reshape(T, G, dv)
    if m.get("rot"):
        q, k = (rotate_halves(z, int(m["rot"]["dims"]), m["rot"]["base"]) for z in (q, k))
    mask = visible(T, int(m["mask"]["size"]), int(m["mask"]["keep_first"]))
    out = torch.zeros(T, H, dv, dtype=F64)
    for hd in range(H):
        g = hd // (H // G)
        s = (q[:, hd] @ k[:, g].T) * float(m["scale"])
        s = torch.where(mask, s, torch.full_like(s, -float("inf")))
        e = torch.exp(s - s.max(dim=1, keepdim=True).values)
        out[:, hd] = (e / e.sum(dim=1, keepdim=True)) @ v[:, g]
    return out.reshape(T, H * dv) @ W("o").T


def gated_linear_attention(h, weights, prefix, m, eps):
    """S = diag(alpha) S + k v^T, o = S^T q, with alpha = sigmoid(z)^(1 / tau) per key channel."""
    H, dk, dv = int(m["heads"]), int(m["dim"]), int(m["vdim"])
    T = h.shape[0]
    W = lambda n: weights[prefix + n]                                       # noqa: E731
    q = (h @ W("q").T).reshape(T, H, dk) * dk ** -0.5
    k = (h @ W("k").T).reshape(T, H, dk)
    v = (h @ W("v").T).reshape(T, H, dv)
    z = ((h @ W("a1").T) @ W("a2").T + W("a2.b")).reshape(T, H, dk)
    alpha = torch.sigmoid(z) ** (1.0 / float(m["tau"]))
    out = torch.zeros(T, H, dv, dtype=F64)
    S = torch.zeros(H, dk, dv, dtype=F64)
    for t in range(T):
        S = alpha[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = torch.einsum("hij,hi->hj", S, q[t])
    out = (unit_rms(out, eps) * W("norm")).reshape(T, H * dv)
    return (out * silu(h @ W("g").T)) @ W("o").T


def side_by_side(h, weights, prefix, m, eps):
    """The weighted sum of both mixers, which read the same input."""
    left = softmax_attention(h, weights, prefix + "left.", m["left"])
    right = gated_linear_attention(h, weights, prefix + "right.", m["right"], eps)
    return float(m["left_scale"]) * left + float(m["right_scale"]) * right


def mamba2(h, weights, prefix, m, eps):
    """State space layer with one decay per head: S = exp(-exp(A) dt) S + dt B x^T, y = S^T C + D x."""
    H, P, N, G = int(m["heads"]), int(m["vdim"]), int(m["state"]), int(m["groups"])
    T, inner = h.shape[0], int(m["heads"]) * int(m["vdim"])
    W = lambda n: weights[prefix + n]                                       # noqa: E731
    u = h @ W("in").T
    z, xbc, dt = u[:, :inner], u[:, inner: 2 * inner + 2 * G * N], u[:, 2 * inner + 2 * G * N:]
    xbc = silu(causal_conv(xbc, W("conv"), W("conv.b")))
    x = xbc[:, :inner].reshape(T, H, P)
    B = xbc[:, inner: inner + G * N].reshape(T, G, N)
    C = xbc[:, inner + G * N:].reshape(T, G, N)
    dt = softplus(dt + W("dt_bias"))
    a = torch.exp(-torch.exp(W("A_log")) * dt)
    group = torch.arange(H) // (H // G)
    y = torch.zeros(T, H, P, dtype=F64)
    S = torch.zeros(H, N, P, dtype=F64)
    for t in range(T):
        S = a[t][:, None, None] * S + dt[t][:, None, None] * B[t][group][:, :, None] * x[t][:, None, :]
        y[t] = torch.einsum("hnp,hn->hp", S, C[t][group]) + W("D")[:, None] * x[t]
    y = y.reshape(T, inner) * silu(z)
    parts = int(m["norm_groups"])
    y = unit_rms(y.reshape(T, parts, inner // parts), eps).reshape(T, inner) * W("norm")
    return y @ W("o").T


# ----------------------------------------------------------------------------- feed-forward
def clamped_ff(h, weights, prefix, limit):
    """g = min(gate, limit), u = clamp(up, -limit, limit): down(g sigmoid(1.702 g) (u + 1))."""
    g = torch.clamp(h @ weights[prefix + "gate"].T, max=float(limit))
    u = torch.clamp(h @ weights[prefix + "up"].T, min=-float(limit), max=float(limit))
    return (g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ weights[prefix + "down"].T


# ----------------------------------------------------------------------------- the model
def run_order(config):
    """The layers in the order they run, with True where a pass but the first begins."""
    n = len(config["layers"])
    loop = config.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    start, stop, times = int(loop["start"]), int(loop["stop"]), int(loop["times"])
    order = [(i, False) for i in range(start)]
    for p in range(times):
        order += [(i, p > 0 and i == start) for i in range(start, stop)]
    return order + [(i, False) for i in range(stop, n)]


def layer(x, i, weights, config):
    """One parallel layer: mixer and feed-forward read norms of the same x, and both join it together."""
    L = config["layers"][i]
    eps = float(config["norm"]["eps"])
    p = f"l{i}."
    mixer = {"mamba2": mamba2, "parallel": side_by_side}[L["type"]]
    y = mixer(unit_rms(x, eps) * weights[p + "norm1"], weights, p + "mix.", L["mixer"], eps)
    if L.get("mlp") is not None:
        y = y + clamped_ff(unit_rms(x, eps) * weights[p + "norm2"], weights, p + "mlp.", L["mlp"]["limit"])
    return x + y


def forward(tokens, weights, config, layers_out=None):
    """Logits [T, vocab] of a token sequence; ``layers_out`` (a list) receives the stream after every layer run."""
    x0 = weights["embed"][torch.tensor(tokens)] * float(config.get("embedding", {}).get("scale", 1.0))
    x = x0.clone()
    for i, again in run_order(config):
        if again:
            x = x + x0
        x = layer(x, i, weights, config)
        if layers_out is not None:
            layers_out.append(x.clone())
    x = unit_rms(x, float(config["norm"]["eps"])) * weights["final.norm"]
    return (x @ weights["embed"].T) * float(config.get("logit_scale", 1.0))
