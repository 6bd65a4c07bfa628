"""A plain statement of the Salipel decoder in float64: whole sequences, no cache, no batching, one function per
mechanism.  It shares no code with the engine; the tests compare the engine with it.

`config` is the dict of config.json, `w` maps tensor names to float64 tensors, matrices stored [out, in].
"""
from __future__ import annotations

import math

import torch

F64 = torch.float64


def rms_unit(x: torch.Tensor, eps: float) -> torch.Tensor:
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def frequencies(rot) -> torch.Tensor:
    """How far each pair turns per position; `rot.scaling` stretches the slow pairs."""
    dims, base = int(rot["dims"]), float(rot["base"])
    out = []
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        s = rot.get("scaling")
        if s:
            wave = 2.0 * math.pi / f
            turns = float(s["original"]) / wave
            if turns < float(s["low"]):
                f = f / float(s["factor"])
            elif turns <= float(s["high"]):
                share = (turns - float(s["low"])) / (float(s["high"]) - float(s["low"]))
                f = (1.0 - share) * f / float(s["factor"]) + share * f
        out.append(f)
    return torch.tensor(out, dtype=F64)


def rotate(x: torch.Tensor, rot) -> torch.Tensor:
    """x [T, heads, d] at positions 0..T-1: numbers i and i + dims/2 of every head are a pair."""
    if not rot or not rot.get("dims"):
        return x
    half = int(rot["dims"]) // 2
    ang = torch.arange(x.shape[0], dtype=F64)[:, None, None] * frequencies(rot)
    c, s = torch.cos(ang), torch.sin(ang)
    u, v = x[..., :half], x[..., half:2 * half]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., 2 * half:]], -1)


def causal(T: int) -> torch.Tensor:
    i = torch.arange(T)
    return i[None, :] <= i[:, None]


def window_sees(T: int, size: int, keep_first: int) -> torch.Tensor:
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    return causal(T) & ((i - j < size) | (j < keep_first))


def chunk_sees(T: int, size: int) -> torch.Tensor:
    i = torch.arange(T)
    return causal(T) & (i[:, None] // size == i[None, :] // size)


def attend(q, k, v, scale, sees, cap=None, slopes=None, sinks=None):
    """q [T, H, D], k [T, G, D], v [T, G, V] -> [T, H, V]."""
    T, H, _ = q.shape
    rep = H // k.shape[1]
    s = torch.einsum("ihd,jhd->hij", q, k.repeat_interleave(rep, 1)) * scale
    if cap:
        s = cap * torch.tanh(s / cap)
    if slopes is not None:
        i = torch.arange(T, dtype=F64)
        s = s - slopes[:, None, None] * (i[:, None] - i[None, :])
    s = s.masked_fill(~sees, -math.inf)
    if sinks is not None:
        s = torch.cat([s, sinks[:, None, None].expand(H, T, 1)], -1)
    p = torch.softmax(s, -1)[..., :T]
    return torch.einsum("hij,jhd->ihd", p, v.repeat_interleave(rep, 1))


def slopes_of(heads: int) -> torch.Tensor:
    return torch.tensor([2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)], dtype=F64)


def sizes(m):
    H, D = int(m["heads"]), int(m["dim"])
    return H, int(m.get("kv_heads", H)), D, int(m.get("vdim", D))


def heads_of(h, W, n):
    y = h @ W.T
    return y.reshape(h.shape[0], n, -1)


def chunked(h, w, p, m, eps):
    """Attention within chunks, a distance penalty, unit values, a sink."""
    H, G, D, V = sizes(m)
    q, k = heads_of(h, w[p + "q"], H), heads_of(h, w[p + "k"], G)
    v = rms_unit(heads_of(h, w[p + "v"], G), eps)
    mask = m.get("mask")
    sees = chunk_sees(len(h), int(mask["size"])) if mask and mask.get("size") else causal(len(h))
    o = attend(q, k, v, float(m["scale"]), sees, slopes=slopes_of(H), sinks=w[p + "sink"])
    return o.flatten(1) @ w[p + "o"].T


def lambda_of(w, p, m) -> torch.Tensor:
    return torch.exp(w[p + "lq1"] @ w[p + "lk1"]) - torch.exp(w[p + "lq2"] @ w[p + "lk2"]) + float(m["diff"])


def differential(h, w, p, m, eps):
    """Two softmax maps per head over the same values, one taken off the other."""
    H, G, D, V = sizes(m)
    q = rotate(rms_unit(heads_of(h, w[p + "q"], 2 * H), eps) * w[p + "q.norm"], m.get("rot"))
    k = rotate(rms_unit(heads_of(h, w[p + "k"], 2 * G), eps) * w[p + "k.norm"], m.get("rot"))
    v = heads_of(h, w[p + "v"], G)
    maps = [attend(q[:, j::2], k[:, j::2], v, float(m["scale"]), causal(len(h)), cap=m.get("softcap")) for j in (0, 1)]
    o = rms_unit(maps[0] - lambda_of(w, p, m) * maps[1], eps) * (1.0 - float(m["diff"]))
    return (o.flatten(1) * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def keys_as_values(h, w, p, m, eps):
    """Windowed attention whose values are the keys' projections; the first tokens stay visible."""
    H, G, D, V = sizes(m)
    raw = heads_of(h, w[p + "k"], G)
    q = rotate(rms_unit(heads_of(h, w[p + "q"], H), eps) * w[p + "q.norm"], m.get("rot"))
    k = rotate(rms_unit(raw, eps) * w[p + "k.norm"], m.get("rot"))
    mask = m.get("mask")
    sees = window_sees(len(h), int(mask["size"]), int(mask.get("keep_first") or 0)) if mask and mask.get("size") else causal(len(h))
    o = attend(q, k, raw, float(m["scale"]), sees)
    return (o.flatten(1) * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def log_sigmoid(z):
    return torch.clamp(z, max=0.0) - torch.log1p(torch.exp(-z.abs()))


def matrix_memory_steps(q, k, v, li, lf):
    """A token at a time: q, k [T, H, D], v [T, H, V], log gates li, lf [T, H] -> [T, H, V]."""
    T, H, D = q.shape
    S, n, top = torch.zeros(H, D, v.shape[-1], dtype=F64), torch.zeros(H, D, dtype=F64), torch.zeros(H, dtype=F64)
    out = torch.empty_like(v)
    for t in range(T):
        new = torch.maximum(lf[t] + top, li[t])
        keep, take = torch.exp(lf[t] + top - new), torch.exp(li[t] - new)
        S = keep[:, None, None] * S + take[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = keep[:, None] * n + take[:, None] * k[t]
        top = new
        size = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-top)) + 1e-6
        out[t] = torch.einsum("hdc,hd->hc", S, q[t]) / size[:, None]
    return out


def matrix_memory(h, w, p, m, eps):
    H, _, D, V = sizes(m)
    q = heads_of(h, w[p + "q"], H) * D ** -0.5
    k, v = heads_of(h, w[p + "k"], H), heads_of(h, w[p + "v"], H)
    cap = float(m["gate_cap"])
    li = cap * torch.tanh((h @ w[p + "i"].T + w[p + "i.b"]) / cap)
    lf = log_sigmoid(cap * torch.tanh((h @ w[p + "f"].T + w[p + "f.b"]) / cap))
    o = rms_unit(matrix_memory_steps(q, k, v, li, lf), eps).flatten(1)
    return (o * w[p + "norm"] * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def pair(h, w, p, m, eps):
    return (float(m["left_scale"]) * keys_as_values(h, w, p + "left.", m["left"], eps)
            + float(m["right_scale"]) * matrix_memory(h, w, p + "right.", m["right"], eps))


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def feed_forward(h, w, p, f, closeness=None):
    """`closeness`, a list, gets per token how far the last chosen score lies above the first one left out."""
    if f["kind"] == "dense":
        return (gelu_tanh(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T
    r = f["router"]
    n, top = int(r["experts"]), int(r["top"])
    s = torch.softmax(h @ w[p + "router"].T, -1)
    order = torch.sort(s + w[p + "correction"], -1, descending=True)
    if closeness is not None:
        closeness.append(order.values[:, top - 1] - order.values[:, top] if top < n else torch.full((h.shape[0],), 1e9, dtype=F64))
    chosen = order.indices[:, :top]
    share = torch.gather(s, 1, chosen)
    share = share / (share.sum(-1, keepdim=True) + 1e-20) * float(r["scale"])
    out = torch.zeros_like(h)
    for e in range(n):
        mine = (share * (chosen == e)).sum(-1)
        rows = (chosen == e).any(-1)
        if rows.any():
            y = torch.relu(h[rows] @ w[f"{p}e{e}.up"].T) ** 2 @ w[f"{p}e{e}.down"].T
            out[rows] += mine[rows, None] * y
    return out


MIXERS = {"attention": chunked, "attention_2": differential, "parallel": pair}


def forward(config: dict, w: dict, tokens, return_layers: bool = False, closeness=None):
    """Logits [T, vocab] of one sequence from position 0."""
    eps, mult = float(config["norm"]["eps"]), float(config["residual_mult"])
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    layers = []
    for i, layer in enumerate(config["layers"]):
        p = f"l{i}."
        h = rms_unit(x, eps) * w[p + "norm1"]
        y = MIXERS[layer["type"]](h, w, p + "mix.", layer["mixer"], eps)
        if layer.get("mlp") is not None:
            y = y + feed_forward(h, w, p + "mlp.", layer["mlp"], closeness)
        x = x + mult * y
        layers.append(x)
    logits = rms_unit(x, eps) * w["final.norm"] @ w["head"].T
    return (logits, layers) if return_layers else logits
