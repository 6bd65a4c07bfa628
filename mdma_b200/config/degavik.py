"""Typed configuration of the Degavik decoder, read from config.json.

Keys: `vocab`, `width`, `norm` {`eps`}, `layers` (a list; each entry has `type`, `mixer`, the mixer's sizes, `mlp`, the
feed-forward's description or null, and optionally `weights_of`, the number of a layer whose tensors this layer uses
instead of having its own).

Layer type "channel_delta" (a gated delta rule with a decay per key channel): {`heads`, `kv_heads`, `dim`, `vdim`,
`conv`: taps of the short convolutions, `decay_rank`, `gate_rank`: the inner sizes of the two low-rank projections;
where config.json does not give these two they are read off the tensors' shapes}.
Layer type "attention" (grouped queries, normed heads, mixed weights): {`heads`, `kv_heads`, `dim`, `vdim`, `scale`,
`softcap` (absent or null: none), `mask`: {`size`, `keep_first`} (absent or null: every earlier token is seen), `rot`:
{`base`, `dims`} (absent, null, or dims 0: no rotation)}.
Layer type "retention" (linear attention with a decay per head): {`heads`, `dim`, `vdim`, `decay`: a number per head,
`rot`}.
Feed-forward: {`kind`: "dense", `ff`} or {`kind`: "moe", `expert`: {`ff`}, `router`: {`experts`, `top`}, `shared`:
{`ff`} or null}.

Every size and every constant that can differ between models comes from here.  A layer kind or a feed-forward kind
the engine does not know rejects the file (it would change what is computed); other keys it does not know are named
in a warning and left alone.
"""
from __future__ import annotations

import copy
import sys
from dataclasses import dataclass
from typing import Optional

from .llama import ConfigError
from .mogevik import DEFAULT_CONTEXT, _count, _number, _positive_int

_TOP_KEYS = {"architecture", "architectures", "model_type", "torch_dtype", "dtype", "vocab", "width", "layers", "norm",
             "eos_token_id", "max_context"}
LAYER_KINDS = ("attention", "channel_delta", "retention")


def _warn_unknown(where: str, have, known) -> None:
    unknown = sorted(set(have) - set(known))
    if unknown:
        print(f"[mdma_b200] {where} has keys the Degavik reader does not know and leaves alone: {unknown}", file=sys.stderr)


def _object(where: str, v) -> dict:
    if not isinstance(v, dict):
        raise ConfigError(f"{where} must be an object")
    return v


@dataclass(frozen=True)
class DegavikDelta:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int
    decay_rank: int
    gate_rank: int


@dataclass(frozen=True)
class DegavikAttention:
    """`softcap` 0, `window` 0, `rot_dims` 0: without."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    softcap: float
    window: int
    keep_first: int
    rot_dims: int
    rot_base: float


@dataclass(frozen=True)
class DegavikRetention:
    heads: int
    dim: int
    vdim: int
    decay: tuple
    rot_dims: int
    rot_base: float


@dataclass(frozen=True)
class DegavikFeedForward:
    """`kind` "dense": `ff`.  `kind` "moe": `experts` experts of `ff`, `top` per token, a shared one of `shared_ff` (0: none)."""
    kind: str
    ff: int
    experts: int = 0
    top: int = 0
    shared_ff: int = 0


@dataclass(frozen=True)
class DegavikLayer:
    type: str
    mixer: object                          # DegavikDelta | DegavikAttention | DegavikRetention
    mlp: Optional[DegavikFeedForward]
    weights_of: Optional[int] = None       # the layer whose tensors this one uses (never itself one with `weights_of`)


@dataclass(frozen=True)
class DegavikConfig:
    vocab: int
    width: int
    layers: tuple
    eps: float
    eos_token_id: tuple = ()
    max_context: int = DEFAULT_CONTEXT

    @classmethod
    def from_dict(cls, raw: dict) -> "DegavikConfig":
        _warn_unknown("config.json", raw, _TOP_KEYS)
        for key in ("vocab", "width", "layers", "norm"):
            if key not in raw:
                raise ConfigError(f"config.json lacks {key!r}")
        vocab, width = _positive_int("vocab", raw["vocab"]), _positive_int("width", raw["width"])
        norm = _object("norm", raw["norm"])
        _warn_unknown("norm", norm, {"eps"})
        if "eps" not in norm:
            raise ConfigError("`norm` must have `eps`")
        eps = _number("norm.eps", norm["eps"])
        if eps < 0:
            raise ConfigError(f"norm.eps must be >= 0, got {eps!r}")
        if not isinstance(raw["layers"], list) or not raw["layers"]:
            raise ConfigError("`layers` must be a list with at least one layer")
        sources = weight_sources(raw["layers"])
        layers = []
        for i, entry in enumerate(raw["layers"]):
            own = cls._layer(f"layers[{i}]", entry)
            src = sources[i]
            if src != i:
                other = cls._layer(f"layers[{src}]", raw["layers"][src])
                if (own.type, own.mixer, own.mlp) != (other.type, other.mixer, other.mlp):
                    raise ConfigError(f"layers[{i}] uses the tensors of layer {src}, but is described otherwise")
                own = DegavikLayer(own.type, own.mixer, own.mlp, src)
            layers.append(own)
        eos = raw.get("eos_token_id", ())
        eos = (eos,) if isinstance(eos, int) else tuple(eos or ())
        max_context = _positive_int("max_context", raw.get("max_context", DEFAULT_CONTEXT))
        return cls(vocab, width, tuple(layers), eps, eos, max_context)

    @staticmethod
    def _layer(where: str, entry) -> DegavikLayer:
        if not isinstance(entry, dict) or "type" not in entry or "mixer" not in entry:
            raise ConfigError(f"{where} must have `type`, `mixer` and `mlp`")
        _warn_unknown(where, entry, {"type", "mixer", "mlp", "weights_of"})
        kind = entry["type"]
        if kind not in LAYER_KINDS:
            raise ConfigError(f"{where}.type {kind!r} is not implemented (have {sorted(LAYER_KINDS)})")
        w = f"{where}.mixer"
        m = _object(w, entry["mixer"])
        read = {"attention": DegavikConfig._attention, "channel_delta": DegavikConfig._delta,
                "retention": DegavikConfig._retention}[kind]
        return DegavikLayer(kind, read(w, m), DegavikConfig._mlp(f"{where}.mlp", entry.get("mlp")))

    @staticmethod
    def _heads(w: str, m: dict):
        heads, dim = _positive_int(f"{w}.heads", m.get("heads")), _positive_int(f"{w}.dim", m.get("dim"))
        kv_heads = _positive_int(f"{w}.kv_heads", m.get("kv_heads", heads))
        if heads % kv_heads:
            raise ConfigError(f"{w}: {heads} heads do not divide over {kv_heads} kv heads")
        return heads, kv_heads, dim, _positive_int(f"{w}.vdim", m.get("vdim", dim))

    @staticmethod
    def _rotation(w: str, m: dict, dim: int):
        rot = m.get("rot")
        if rot is None:
            return 0, 1.0
        _warn_unknown(f"{w}.rot", _object(f"{w}.rot", rot), {"base", "dims"})
        dims = _count(f"{w}.rot.dims", rot.get("dims", dim))
        if not dims:
            return 0, 1.0
        base = _number(f"{w}.rot.base", rot.get("base"))
        if dims % 2 or dims > dim or base <= 0:
            raise ConfigError(f"{w}.rot: {dims} turned numbers of a head of {dim} with base {base}")
        return dims, base

    @staticmethod
    def _delta(w: str, m: dict) -> DegavikDelta:
        _warn_unknown(w, m, {"heads", "kv_heads", "dim", "vdim", "conv", "decay_rank", "gate_rank"})
        heads, kv_heads, dim, vdim = DegavikConfig._heads(w, m)
        # a description without tensors (a plan, random weights) may leave the ranks out: a head's size
        return DegavikDelta(heads, kv_heads, dim, vdim, _positive_int(f"{w}.conv", m.get("conv")),
                            _positive_int(f"{w}.decay_rank", m.get("decay_rank", dim)),
                            _positive_int(f"{w}.gate_rank", m.get("gate_rank", dim)))

    @staticmethod
    def _attention(w: str, m: dict) -> DegavikAttention:
        _warn_unknown(w, m, {"heads", "kv_heads", "dim", "vdim", "scale", "softcap", "mask", "rot"})
        heads, kv_heads, dim, vdim = DegavikConfig._heads(w, m)
        scale = _number(f"{w}.scale", m.get("scale", dim ** -0.5))
        cap = 0.0 if m.get("softcap") is None else _number(f"{w}.softcap", m["softcap"])
        if cap < 0:
            raise ConfigError(f"{w}.softcap must be positive (or absent), got {cap!r}")
        window = keep = 0
        mask = m.get("mask")
        if mask is not None:
            _warn_unknown(f"{w}.mask", _object(f"{w}.mask", mask), {"size", "keep_first"})
            if mask.get("size") is not None:
                window = _positive_int(f"{w}.mask.size", mask["size"])
                keep = _count(f"{w}.mask.keep_first", mask.get("keep_first") or 0)
        dims, base = DegavikConfig._rotation(w, m, dim)
        return DegavikAttention(heads, kv_heads, dim, vdim, scale, cap, window, keep, dims, base)

    @staticmethod
    def _retention(w: str, m: dict) -> DegavikRetention:
        _warn_unknown(w, m, {"heads", "dim", "vdim", "decay", "rot"})
        heads, _, dim, vdim = DegavikConfig._heads(w, m)
        decay = m.get("decay")
        if isinstance(decay, (int, float)) and not isinstance(decay, bool):
            decay = [decay] * heads
        if not isinstance(decay, list) or len(decay) != heads:
            raise ConfigError(f"{w}.decay must give one number per head ({heads})")
        dims, base = DegavikConfig._rotation(w, m, dim)
        return DegavikRetention(heads, dim, vdim, tuple(_number(f"{w}.decay[{i}]", d) for i, d in enumerate(decay)), dims, base)

    @staticmethod
    def _mlp(where: str, raw) -> Optional[DegavikFeedForward]:
        if raw is None:
            return None
        kind = _object(where, raw).get("kind")
        if kind == "dense":
            _warn_unknown(where, raw, {"kind", "ff"})
            return DegavikFeedForward("dense", _positive_int(f"{where}.ff", raw.get("ff")))
        if kind != "moe":
            raise ConfigError(f"{where}.kind {kind!r} is not implemented (have ['dense', 'moe'])")
        _warn_unknown(where, raw, {"kind", "expert", "router", "shared"})
        expert, router = _object(f"{where}.expert", raw.get("expert")), _object(f"{where}.router", raw.get("router"))
        _warn_unknown(f"{where}.expert", expert, {"ff"})
        _warn_unknown(f"{where}.router", router, {"experts", "top"})
        ff = _positive_int(f"{where}.expert.ff", expert.get("ff"))
        experts = _positive_int(f"{where}.router.experts", router.get("experts"))
        top = _positive_int(f"{where}.router.top", router.get("top"))
        if top > experts:
            raise ConfigError(f"{where}: top {top} of {experts} experts")
        shared_ff = 0
        if raw.get("shared") is not None:
            _warn_unknown(f"{where}.shared", _object(f"{where}.shared", raw["shared"]), {"ff"})
            shared_ff = _positive_int(f"{where}.shared.ff", raw["shared"].get("ff"))
        return DegavikFeedForward("moe", ff, experts, top, shared_ff)


def weight_sources(layers: list) -> list:
    """Per layer the number of the layer whose tensors it uses (itself, unless `weights_of` says otherwise; a chain of
    `weights_of` is followed to its end)."""
    out = []
    for i in range(len(layers)):
        seen, j = {i}, i
        while isinstance(layers[j], dict) and layers[j].get("weights_of") is not None:
            k = layers[j]["weights_of"]
            if isinstance(k, bool) or not isinstance(k, int) or not 0 <= k < len(layers) or k in seen:
                raise ConfigError(f"layers[{j}].weights_of must name another layer with tensors of its own, got {k!r}")
            seen.add(k)
            j = k
        out.append(j)
    return out


def sizes_from_shapes(raw: dict, shapes: dict) -> dict:
    """The two low-rank sizes of every "channel_delta" layer, which config.json leaves to the shapes of `a1` and `g1`,
    filled in from `shapes` (tensor name -> shape); what config.json gives itself stays."""
    layers = raw.get("layers")
    if not isinstance(layers, list):
        return raw
    raw = copy.deepcopy(raw)
    for src, entry in zip(weight_sources(layers), raw["layers"]):
        if not isinstance(entry, dict) or entry.get("type") != "channel_delta" or not isinstance(entry.get("mixer"), dict):
            continue
        for key, tensor in (("decay_rank", "a1"), ("gate_rank", "g1")):
            shape = shapes.get(f"l{src}.mix.{tensor}")
            if key not in entry["mixer"] and shape is not None and len(shape) == 2:
                entry["mixer"][key] = int(shape[0])
    return raw
