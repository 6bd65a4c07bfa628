"""The Degavik decoder as a `ModelSpec`.

Every layer is the "postnorm" arrangement: the sublayers read the residual stream itself and an RMS norm lies on each
one's result only, x += norm1(mixer(x)); x += norm2(feed_forward(x)) (the second may be absent).  Three mixers: a gated
delta rule with a decay per key channel, short convolutions on q, k and v, unit vectors for q and k, and a gated norm
per head ("channel_delta"); grouped-query attention with normed query and key heads, turned in interleaved pairs, a
learned number per head on the scores, a soft cap on them, a sliding window that keeps the first tokens, and the heads'
softmax weights mixed by a learned matrix ("attention"); linear attention with a fixed decay per head on turned q and k
and a norm per head ("retention").  The feed-forward is dense and gated, or routed: `top` experts with the largest
biased logits, weighted by the softmax over the chosen logits, and a shared expert for every token.  A layer may use
another layer's tensors: it is then another run of that layer in the schedule, with a cache and state of its own.

Tensor names: `embed`, `final.norm`, `head`, and per layer i that has tensors `l<i>.norm1|norm2`,
`l<i>.mix.q|k|v[.conv]|b|A_log|norm|a1|a2|dt_bias|g1|g2|o`, `l<i>.mix.q|k[.norm]|v|talk|temp|o` or
`l<i>.mix.q|k|v|g|o`, and `l<i>.mlp.gate|up|down` or `l<i>.mlp.router[.b]`, `l<i>.mlp.e<j>.gate|up|down`,
`l<i>.mlp.shared.gate|up|down`.
"""
from __future__ import annotations

from ..registry import ARCHITECTURES
from ..spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry
from .degavik import DegavikAttention, DegavikConfig, DegavikDelta, DegavikFeedForward, DegavikRetention, sizes_from_shapes

UNIT_EPS = 1e-6          # under the root of the delta rule's unit vectors


def _norm(c: DegavikConfig, name: str) -> PartSpec:
    return PartSpec("rmsnorm", dict(width=c.width, eps=c.eps), aliases={"weight": name})


def _rotary(head: int, dims: int, base: float, layout: str):
    if not dims:
        return None
    return PartSpec("rotary", dict(head_dim=head, rotary_dim=dims, theta=base, layout=layout))


def _mixer(c: DegavikConfig, m, prefix: str) -> PartSpec:
    if isinstance(m, DegavikDelta):
        return PartSpec("channel_delta",
                        dict(hidden_size=c.width, num_heads=m.heads, num_kv_heads=m.kv_heads, head_dim=m.dim, v_dim=m.vdim,
                             conv=m.conv, decay_rank=m.decay_rank, gate_rank=m.gate_rank, eps=c.eps, unit_eps=UNIT_EPS),
                        prefix=prefix)
    if isinstance(m, DegavikAttention):
        return PartSpec("talking_attention",
                        dict(hidden_size=c.width, num_heads=m.heads, num_kv_heads=m.kv_heads, head_dim=m.dim, v_dim=m.vdim,
                             scale=m.scale, eps=c.eps, position=_rotary(m.dim, m.rot_dims, m.rot_base, "interleaved"),
                             qk_norm=True, talk="weights", temp=True, softcap=m.softcap, window=m.window,
                             keep_first=m.keep_first), prefix=prefix)
    assert isinstance(m, DegavikRetention)
    return PartSpec("linear_attention",
                    dict(hidden_size=c.width, num_heads=m.heads, head_dim=m.dim, v_dim=m.vdim, decay=list(m.decay), eps=c.eps,
                         activation="none", position=_rotary(m.dim, m.rot_dims, m.rot_base, "split_half"),
                         k_scale=m.dim ** -0.5, norm="head", gate="silu"), prefix=prefix)


def _feed_forward(c: DegavikConfig, f: DegavikFeedForward, prefix: str) -> PartSpec:
    if f.kind == "dense":
        return PartSpec("gated_mlp", dict(hidden_size=c.width, intermediate_size=f.ff, activation="silu"), prefix=prefix,
                        aliases={f"{n}_proj.weight": prefix + n for n in ("gate", "up", "down")})
    return PartSpec("routed_mlp",
                    dict(hidden_size=c.width, intermediate_size=f.ff, experts=f.experts, top=f.top, correction=False,
                         logit_bias=True, shared_ff=f.shared_ff, shared_gate=False, activation="silu"), prefix=prefix)


def describe_degavik(c: DegavikConfig) -> ModelSpec:
    place, layers, schedule = {}, [], []
    for i, layer in enumerate(c.layers):
        if layer.weights_of is not None:
            continue
        p = f"l{i}."
        extras = {"mixer_post_norm": _norm(c, p + "norm1")}
        ffn = None
        if layer.mlp is not None:
            ffn = _feed_forward(c, layer.mlp, p + "mlp.")
            extras["ffn_post_norm"] = _norm(c, p + "norm2")
        place[i] = len(layers)
        layers.append(LayerSpec("postnorm", None, _mixer(c, layer.mixer, p + "mix."), None, ffn, extras))
    for i, layer in enumerate(c.layers):
        schedule.append(ScheduleEntry(place[i if layer.weights_of is None else layer.weights_of]))
    return ModelSpec(
        hidden_size=c.width, vocab_size=c.vocab, max_positions=c.max_context,
        embedding=PartSpec("embedding", dict(vocab_size=c.vocab, width=c.width), aliases={"weight": "embed"}),
        layers=layers, schedule=schedule, final_norm=_norm(c, "final.norm"),
        lm_head=PartSpec("lm_head", dict(vocab_size=c.vocab, width=c.width), aliases={"weight": "head"}),
        stop_token_ids=tuple(c.eos_token_id))


def _register() -> None:
    from . import Architecture
    ARCHITECTURES.register("Degavik", Architecture("Degavik", DegavikConfig.from_dict, describe_degavik, sizes_from_shapes),
                           replace=True)


_register()
