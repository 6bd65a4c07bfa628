"""A plain statement of the Degavik decoder in float64: whole sequences, no cache, no batching, one function per
mechanism.  It shares no code with the engine; the tests compare the engine with it.

`config` is the dict of config.json, `w` maps tensor names to float64 tensors, matrices stored [out, in].
"""
from __future__ import annotations

import math

import torch

F64 = torch.float64
UNIT_EPS = 1e-6


def rms_unit(x: torch.Tensor, eps: float) -> torch.Tensor:
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def softplus(z: torch.Tensor) -> torch.Tensor:
    return torch.log1p(torch.exp(-z.abs())) + z.clamp(min=0.0)


def rotate(x: torch.Tensor, positions: torch.Tensor, rot, layout: str) -> torch.Tensor:
    """x [T, heads, d]: the first rot.dims numbers of every head turned by the token's position."""
    if not rot or not rot.get("dims"):
        return x
    dims, base = int(rot["dims"]), float(rot["base"])
    f = torch.tensor([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=F64)
    ang = positions.to(F64)[:, None] * f[None, :]
    cos, sin = torch.cos(ang)[:, None, :], torch.sin(ang)[:, None, :]
    out = x.clone()
    if layout == "interleaved":
        first, second = slice(0, dims, 2), slice(1, dims, 2)
    else:
        first, second = slice(0, dims // 2), slice(dims // 2, dims)
    u, v = x[..., first], x[..., second]
    out[..., first] = u * cos - v * sin
    out[..., second] = v * cos + u * sin
    return out


def short_conv(x: torch.Tensor, taps: torch.Tensor) -> torch.Tensor:
    """x [T, C], taps [C, n]: y_t = sum_j taps[:, n-1-j] x_(t-j), zeros before the start."""
    T, n = x.shape[0], taps.shape[1]
    y = torch.zeros_like(x)
    for back in range(n):
        if back < T:
            y[back:] += x[:T - back] * taps[:, n - 1 - back]
    return y


def unit_vector(x: torch.Tensor) -> torch.Tensor:
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + UNIT_EPS)


def delta_steps(q, k, v, g, beta):
    """The gated delta rule a token at a time: q, k, g [T, H, dim], v [T, H, vdim], beta [T, H] -> o [T, H, vdim]."""
    T, H, dim = q.shape
    S = torch.zeros(H, dim, v.shape[-1], dtype=F64)
    out = torch.empty(T, H, v.shape[-1], dtype=F64)
    for t in range(T):
        S = g[t][:, :, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hdc,hd->hc", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out[t] = torch.einsum("hdc,hd->hc", S, q[t])
    return out


def channel_delta(h, w, p, m, eps):
    H, dim, vdim = int(m["heads"]), int(m["dim"]), int(m["vdim"])
    G = int(m.get("kv_heads", H))
    T = h.shape[0]
    rep = H // G
    q, k, v = (silu(short_conv(h @ w[p + n].T, w[p + n + ".conv"])) for n in ("q", "k", "v"))
    q = unit_vector(q.reshape(T, G, dim)) * dim ** -0.5
    k = unit_vector(k.reshape(T, G, dim))
    q, k = q.repeat_interleave(rep, 1), k.repeat_interleave(rep, 1)
    beta = torch.sigmoid(h @ w[p + "b"].T)
    step = softplus((h @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "dt_bias"]).reshape(T, H, dim)
    g = torch.exp(-torch.exp(w[p + "A_log"])[None, :, None] * step)
    o = delta_steps(q, k, v.reshape(T, H, vdim), g, beta)
    gate = torch.sigmoid((h @ w[p + "g1"].T) @ w[p + "g2"].T).reshape(T, H, vdim)
    o = rms_unit(o, eps) * w[p + "norm"] * gate
    return o.reshape(T, H * vdim) @ w[p + "o"].T


def visible(T: int, mask) -> torch.Tensor:
    """[T, T] of bool: whether row i sees key j."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    see = j <= i
    if mask and mask.get("size"):
        see = see & ((i - j < int(mask["size"])) | (j < int(mask.get("keep_first") or 0)))
    return see


def attention(h, w, p, m, positions, eps):
    H, dim, vdim = int(m["heads"]), int(m["dim"]), int(m["vdim"])
    G = int(m.get("kv_heads", H))
    T = h.shape[0]
    rep = H // G
    q = rms_unit((h @ w[p + "q"].T).reshape(T, H, dim), eps) * w[p + "q.norm"]
    k = rms_unit((h @ w[p + "k"].T).reshape(T, G, dim), eps) * w[p + "k.norm"]
    v = (h @ w[p + "v"].T).reshape(T, G, vdim).repeat_interleave(rep, 1)
    q = rotate(q, positions, m.get("rot"), "interleaved")
    k = rotate(k, positions, m.get("rot"), "interleaved").repeat_interleave(rep, 1)
    s = torch.einsum("ihd,jhd->hij", q, k) * float(m["scale"]) * w[p + "temp"][:, None, None]
    if m.get("softcap"):
        s = float(m["softcap"]) * torch.tanh(s / float(m["softcap"]))
    pr = torch.softmax(s.masked_fill(~visible(T, m.get("mask")), -math.inf), -1)
    pr = torch.einsum("hg,gij->hij", w[p + "talk"], pr)
    return torch.einsum("hij,jhd->ihd", pr, v).reshape(T, H * vdim) @ w[p + "o"].T


def retention(h, w, p, m, positions, eps):
    H, dim, vdim = int(m["heads"]), int(m["dim"]), int(m["vdim"])
    T = h.shape[0]
    q = rotate((h @ w[p + "q"].T).reshape(T, H, dim), positions, m.get("rot"), "split_half")
    k = rotate((h @ w[p + "k"].T).reshape(T, H, dim), positions, m.get("rot"), "split_half") * dim ** -0.5
    v = (h @ w[p + "v"].T).reshape(T, H, vdim)
    decay = torch.tensor([float(d) for d in m["decay"]], dtype=F64)
    S = torch.zeros(H, dim, vdim, dtype=F64)
    o = torch.empty(T, H, vdim, dtype=F64)
    for t in range(T):
        S = decay[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        o[t] = torch.einsum("hdc,hd->hc", S, q[t])
    return (rms_unit(o, eps).reshape(T, H * vdim) * silu(h @ w[p + "g"].T)) @ w[p + "o"].T


def gated(h, w, p):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def feed_forward(h, w, p, f, closeness=None):
    """`closeness`, a list, gets per token how far the last chosen logit lies above the first one left out."""
    if f["kind"] == "dense":
        return gated(h, w, p)
    n, top = int(f["router"]["experts"]), int(f["router"]["top"])
    z = h @ w[p + "router"].T + w[p + "router.b"]
    order = torch.sort(z, -1, descending=True)
    if closeness is not None:
        closeness.append(order.values[:, top - 1] - order.values[:, top] if top < n else torch.full((h.shape[0],), 1e9, dtype=F64))
    weights = torch.softmax(order.values[:, :top], -1)
    out = torch.zeros_like(h)
    for e in range(n):
        share = (weights * (order.indices[:, :top] == e)).sum(-1)
        rows = share > 0
        if rows.any():
            out[rows] += share[rows, None] * gated(h[rows], w, f"{p}e{e}.")
    if f.get("shared"):
        out = out + gated(h, w, p + "shared.")
    return out


def forward(config: dict, w: dict, tokens, return_layers: bool = False, closeness=None):
    """Logits [T, vocab] of one sequence from position 0."""
    eps = float(config["norm"]["eps"])
    ids = torch.as_tensor(tokens, dtype=torch.long)
    positions = torch.arange(len(ids))
    x = w["embed"][ids]
    layers = []
    for i, layer in enumerate(config["layers"]):
        own = layer.get("weights_of")
        p, m, kind = f"l{i if own is None else own}.", layer["mixer"], layer["type"]
        if kind == "channel_delta":
            y = channel_delta(x, w, p + "mix.", m, eps)
        elif kind == "attention":
            y = attention(x, w, p + "mix.", m, positions, eps)
        elif kind == "retention":
            y = retention(x, w, p + "mix.", m, positions, eps)
        else:
            raise ValueError(f"unknown layer type {kind!r}")
        x = x + rms_unit(y, eps) * w[p + "norm1"]
        if layer.get("mlp") is not None:
            y = feed_forward(x, w, p + "mlp.", layer["mlp"], closeness)
            x = x + rms_unit(y, eps) * w[p + "norm2"]
        layers.append(x)
    logits = rms_unit(x, eps) * w["final.norm"] @ w["head"].T
    return (logits, layers) if return_layers else logits
