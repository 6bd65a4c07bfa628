"""The Salipel decoder as a `ModelSpec`.

Every layer is the "parallel" arrangement with a multiplier: with h = norm(x), x <- x + m (mixer(h) + feed_forward(h)), the
feed-forward optional.  Three mixers, all but one half of the last attention with different options of one part
(`general_attention`): within chunks of positions, with a distance penalty, normed values and a sink ("attention"); two
maps per head whose difference is normed, with normed and turned query and key heads, a soft cap and an output gate
("attention_2"); and a pair side by side ("parallel"): attention over a window that keeps the first tokens, whose values
are the keys' projections, and a matrix memory with exponential gates, each result times a constant.  The feed-forward is
dense and gated (tanh form of GELU), or routed: softmax scores over all experts, choice by corrected scores, weights that
add up to a constant, experts without a gate (squared ReLU).

The multiplier costs nothing: the stream is kept divided by it.  With y = x / m the layer is y <- y + mixer + feed_forward,
the embedding's rows are multiplied by 1 / m, and a norm of x is the norm of y with eps / m^2 under the root
(`ModelSpec.stream_unit` = m tells who wants to see x itself).

Tensor names: `embed`, `final.norm`, `head`, and per layer i `l<i>.norm1`, `l<i>.mix.q|k|v|sink|o`,
`l<i>.mix.q|k[.norm]|v|g|lq1|lk1|lq2|lk2|o` or `l<i>.mix.left.q|k[.norm]|g|o` and `l<i>.mix.right.q|k|v|g|i|f[.b]|norm|o`, and
`l<i>.mlp.gate|up|down` or `l<i>.mlp.router|correction`, `l<i>.mlp.e<j>.up|down`.
"""
from __future__ import annotations

from ..registry import ARCHITECTURES
from ..spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry
from .salipel import SalipelChunked, SalipelConfig, SalipelDifferential, SalipelFeedForward, SalipelPair

SLOPE_POWER = 8.0        # slope of head h: 2^(-8 (h + 1) / heads)


def _norm(c: SalipelConfig, name: str) -> PartSpec:
    # of the stream divided by residual_mult
    return PartSpec("rmsnorm", dict(width=c.width, eps=c.eps / c.residual_mult ** 2), aliases={"weight": name})


def _rotary(head: int, rot):
    if rot is None:
        return None
    return PartSpec("rotary", dict(head_dim=head, rotary_dim=rot.dims, theta=rot.base, layout="split_half", scaling=rot.scaling))


def _mixer(c: SalipelConfig, m, prefix: str) -> PartSpec:
    if isinstance(m, SalipelChunked):
        return PartSpec("general_attention",
                        dict(hidden_size=c.width, num_heads=m.heads, num_kv_heads=m.kv_heads, head_dim=m.dim, v_dim=m.vdim,
                             scale=m.scale, eps=c.eps, chunk=m.chunk, slope_power=SLOPE_POWER, v_norm=True, sink=True), prefix=prefix)
    if isinstance(m, SalipelDifferential):
        return PartSpec("general_attention",
                        dict(hidden_size=c.width, num_heads=m.heads, num_kv_heads=m.kv_heads, head_dim=m.dim, v_dim=m.vdim,
                             scale=m.scale, eps=c.eps, differential=m.diff, softcap=m.softcap, qk_norm=True, gate=True,
                             position=_rotary(m.dim, m.rot)), prefix=prefix)
    assert isinstance(m, SalipelPair)
    a, b = m.left, m.right
    left = PartSpec("general_attention",
                    dict(hidden_size=c.width, num_heads=a.heads, num_kv_heads=a.kv_heads, head_dim=a.dim, v_dim=a.dim, scale=a.scale,
                         eps=c.eps, window=a.window, keep_first=a.keep_first, values="keys", qk_norm=True, gate=True,
                         position=_rotary(a.dim, a.rot)), prefix=prefix + "left.")
    right = PartSpec("matrix_memory", dict(hidden_size=c.width, num_heads=b.heads, head_dim=b.dim, v_dim=b.vdim, gate_cap=b.gate_cap,
                                           eps=c.eps), prefix=prefix + "right.")
    return PartSpec("side_by_side", dict(hidden_size=c.width, left=left, right=right, left_scale=m.left_scale,
                                         right_scale=m.right_scale), prefix=prefix)


def _feed_forward(c: SalipelConfig, f: SalipelFeedForward, prefix: str) -> PartSpec:
    if f.kind == "dense":
        return PartSpec("gated_mlp", dict(hidden_size=c.width, intermediate_size=f.ff, activation="gelu_tanh"), prefix=prefix,
                        aliases={f"{n}_proj.weight": prefix + n for n in ("gate", "up", "down")})
    return PartSpec("routed_mlp", dict(hidden_size=c.width, intermediate_size=f.ff, experts=f.experts, top=f.top, correction=True,
                                       gated=False, activation="relu_squared", weight_scale=f.scale), prefix=prefix)


def describe_salipel(c: SalipelConfig) -> ModelSpec:
    layers = []
    for i, layer in enumerate(c.layers):
        p = f"l{i}."
        ffn = None if layer.mlp is None else _feed_forward(c, layer.mlp, p + "mlp.")
        layers.append(LayerSpec("parallel", _norm(c, p + "norm1"), _mixer(c, layer.mixer, p + "mix."), None, ffn))
    return ModelSpec(
        hidden_size=c.width, vocab_size=c.vocab, max_positions=c.max_context,
        embedding=PartSpec("embedding", dict(vocab_size=c.vocab, width=c.width, scale=1.0 / c.residual_mult), aliases={"weight": "embed"}),
        layers=layers, schedule=[ScheduleEntry(i) for i in range(len(layers))], final_norm=_norm(c, "final.norm"),
        lm_head=PartSpec("lm_head", dict(vocab_size=c.vocab, width=c.width), aliases={"weight": "head"}),
        stop_token_ids=tuple(c.eos_token_id), stream_unit=c.residual_mult)


def _register() -> None:
    from . import Architecture
    ARCHITECTURES.register("Salipel", Architecture("Salipel", SalipelConfig.from_dict, describe_salipel), replace=True)


_register()
