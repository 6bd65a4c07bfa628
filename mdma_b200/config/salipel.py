"""Typed configuration of the Salipel decoder, read from config.json.

Keys: `vocab`, `width`, `norm` {`eps`}, `residual_mult` (what a layer's result is multiplied by before it joins the residual
stream), `layers` (a list; each entry has `type`, `mixer`, the mixer's sizes, and `mlp`, the feed-forward's description or
null).

Layer type "attention" (within chunks, a distance penalty, normed values, a sink): {`heads`, `kv_heads`, `dim`, `vdim`,
`scale`, `mask`: {`size`: positions of a chunk} (absent or null: every earlier token is seen)}.
Layer type "attention_2" (two maps per head, one taken off the other): {`heads`, `kv_heads`, `dim`, `vdim`, `scale`, `diff`,
`softcap` (absent or null: none), `rot`: {`base`, `dims`} (absent, null, or dims 0: no rotation)}.
Layer type "parallel": {`left`, `right`, `left_scale`, `right_scale`}, two mixers that read the same rows.
  left  (attention over a window with kept first tokens, values that are the keys' projections): {`heads`, `kv_heads`, `dim`,
        `vdim` (the same as `dim`), `scale`, `mask`: {`size`, `keep_first`} (absent or null: every earlier token is seen),
        `rot`: {`base`, `dims`, `scaling`: {`factor`, `low`, `high`, `original`} or null}}
  right (matrix memory with exponential gates): {`heads`, `dim`, `vdim`, `gate_cap`}
Feed-forward: {`kind`: "dense", `ff`} or {`kind`: "moe", `expert`: {`ff`}, `router`: {`experts`, `top`, `scale`}}.

Every size and every constant that can differ between models comes from here.  A layer kind or a feed-forward kind the
engine does not know rejects the file (it would change what is computed); other keys it does not know are named in a
warning and left alone.
"""
from __future__ import annotations

import sys
from dataclasses import dataclass
from typing import Optional

from .llama import ConfigError, RopeScaling
from .mogevik import DEFAULT_CONTEXT, _count, _number, _positive_int

_TOP_KEYS = {"architecture", "architectures", "model_type", "torch_dtype", "dtype", "vocab", "width", "layers", "norm",
             "residual_mult", "eos_token_id", "max_context"}
LAYER_KINDS = ("attention", "attention_2", "parallel")


def _warn_unknown(where: str, have, known) -> None:
    unknown = sorted(set(have) - set(known))
    if unknown:
        print(f"[mdma_b200] {where} has keys the Salipel reader does not know and leaves alone: {unknown}", file=sys.stderr)


def _object(where: str, v) -> dict:
    if not isinstance(v, dict):
        raise ConfigError(f"{where} must be an object")
    return v


def _positive(where: str, v) -> float:
    x = _number(where, v)
    if x <= 0:
        raise ConfigError(f"{where} must be positive, got {v!r}")
    return x


@dataclass(frozen=True)
class SalipelRotation:
    dims: int
    base: float
    scaling: Optional[RopeScaling] = None


@dataclass(frozen=True)
class SalipelChunked:
    """`chunk` 0: every earlier token is seen."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    chunk: int


@dataclass(frozen=True)
class SalipelDifferential:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    diff: float
    softcap: float                       # 0: none
    rot: Optional[SalipelRotation]


@dataclass(frozen=True)
class SalipelWindowed:
    """`window` 0: every earlier token is seen."""
    heads: int
    kv_heads: int
    dim: int
    scale: float
    window: int
    keep_first: int
    rot: Optional[SalipelRotation]


@dataclass(frozen=True)
class SalipelMemory:
    heads: int
    dim: int
    vdim: int
    gate_cap: float


@dataclass(frozen=True)
class SalipelPair:
    left: SalipelWindowed
    right: SalipelMemory
    left_scale: float
    right_scale: float


@dataclass(frozen=True)
class SalipelFeedForward:
    """`kind` "dense": `ff`.  `kind` "moe": `experts` experts of `ff`, `top` per token, their weights times `scale`."""
    kind: str
    ff: int
    experts: int = 0
    top: int = 0
    scale: float = 1.0


@dataclass(frozen=True)
class SalipelLayer:
    type: str
    mixer: object                        # SalipelChunked | SalipelDifferential | SalipelPair
    mlp: Optional[SalipelFeedForward]


@dataclass(frozen=True)
class SalipelConfig:
    vocab: int
    width: int
    layers: tuple
    eps: float
    residual_mult: float = 1.0
    eos_token_id: tuple = ()
    max_context: int = DEFAULT_CONTEXT

    @classmethod
    def from_dict(cls, raw: dict) -> "SalipelConfig":
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
        mult = 1.0 if raw.get("residual_mult") is None else _positive("residual_mult", raw["residual_mult"])
        if not isinstance(raw["layers"], list) or not raw["layers"]:
            raise ConfigError("`layers` must be a list with at least one layer")
        layers = tuple(cls._layer(f"layers[{i}]", entry) for i, entry in enumerate(raw["layers"]))
        eos = raw.get("eos_token_id", ())
        eos = (eos,) if isinstance(eos, int) else tuple(eos or ())
        max_context = _positive_int("max_context", raw.get("max_context", DEFAULT_CONTEXT))
        return cls(vocab, width, layers, eps, mult, eos, max_context)

    @staticmethod
    def _layer(where: str, entry) -> SalipelLayer:
        if not isinstance(entry, dict) or "type" not in entry or "mixer" not in entry:
            raise ConfigError(f"{where} must have `type`, `mixer` and `mlp`")
        _warn_unknown(where, entry, {"type", "mixer", "mlp"})
        kind = entry["type"]
        if kind not in LAYER_KINDS:
            raise ConfigError(f"{where}.type {kind!r} is not implemented (have {sorted(LAYER_KINDS)})")
        w = f"{where}.mixer"
        read = {"attention": SalipelConfig._chunked, "attention_2": SalipelConfig._differential, "parallel": SalipelConfig._pair}[kind]
        return SalipelLayer(kind, read(w, _object(w, entry["mixer"])), SalipelConfig._mlp(f"{where}.mlp", entry.get("mlp")))

    @staticmethod
    def _heads(w: str, m: dict):
        """(heads, kv heads, dim, vdim, scale)"""
        heads, dim = _positive_int(f"{w}.heads", m.get("heads")), _positive_int(f"{w}.dim", m.get("dim"))
        kv_heads = _positive_int(f"{w}.kv_heads", m.get("kv_heads", heads))
        if heads % kv_heads:
            raise ConfigError(f"{w}: {heads} heads do not divide over {kv_heads} kv heads")
        return heads, kv_heads, dim, _positive_int(f"{w}.vdim", m.get("vdim", dim)), _positive(f"{w}.scale", m.get("scale", dim ** -0.5))

    @staticmethod
    def _mask(w: str, m: dict, keys: set) -> dict:
        """The mask's description; empty where every earlier token is seen."""
        mask = m.get("mask")
        if mask is None:
            return {}
        _warn_unknown(f"{w}.mask", _object(f"{w}.mask", mask), keys)
        return {} if mask.get("size") is None else dict(mask, size=_positive_int(f"{w}.mask.size", mask["size"]))

    @staticmethod
    def _rotation(w: str, m: dict, dim: int) -> Optional[SalipelRotation]:
        rot = m.get("rot")
        if rot is None:
            return None
        _warn_unknown(f"{w}.rot", _object(f"{w}.rot", rot), {"base", "dims", "scaling"})
        dims = _count(f"{w}.rot.dims", rot.get("dims", dim))
        if not dims:
            return None
        base = _number(f"{w}.rot.base", rot.get("base"))
        if dims % 2 or dims > dim or base <= 0:
            raise ConfigError(f"{w}.rot: {dims} turned numbers of a head of {dim} with base {base}")
        scaling = None
        raw = rot.get("scaling")
        if raw is not None:
            s = f"{w}.rot.scaling"
            _warn_unknown(s, _object(s, raw), {"factor", "low", "high", "original"})
            factor, low, high = (_positive(f"{s}.{k}", raw.get(k)) for k in ("factor", "low", "high"))
            original = _positive(f"{s}.original", raw.get("original"))
            if high <= low:
                raise ConfigError(f"{s}: `high` {high} must be above `low` {low}")
            scaling = RopeScaling("llama3", factor=factor, low_freq_factor=low, high_freq_factor=high, original_max_position_embeddings=original)
        return SalipelRotation(dims, base, scaling)

    @staticmethod
    def _chunked(w: str, m: dict) -> SalipelChunked:
        _warn_unknown(w, m, {"heads", "kv_heads", "dim", "vdim", "scale", "mask"})
        mask = SalipelConfig._mask(w, m, {"size"})
        return SalipelChunked(*SalipelConfig._heads(w, m), mask.get("size", 0))

    @staticmethod
    def _differential(w: str, m: dict) -> SalipelDifferential:
        _warn_unknown(w, m, {"heads", "kv_heads", "dim", "vdim", "scale", "diff", "softcap", "rot"})
        heads, kv_heads, dim, vdim, scale = SalipelConfig._heads(w, m)
        cap = 0.0 if m.get("softcap") is None else _positive(f"{w}.softcap", m["softcap"])
        return SalipelDifferential(heads, kv_heads, dim, vdim, scale, _number(f"{w}.diff", m.get("diff")), cap,
                                   SalipelConfig._rotation(w, m, dim))

    @staticmethod
    def _pair(w: str, m: dict) -> SalipelPair:
        _warn_unknown(w, m, {"left", "right", "left_scale", "right_scale"})
        if "left" not in m or "right" not in m:
            raise ConfigError(f"{w} must have `left` and `right`")
        lw, rw = f"{w}.left", f"{w}.right"
        left, right = _object(lw, m["left"]), _object(rw, m["right"])
        _warn_unknown(lw, left, {"heads", "kv_heads", "dim", "vdim", "scale", "mask", "rot"})
        heads, kv_heads, dim, vdim, scale = SalipelConfig._heads(lw, left)
        if vdim != dim:
            raise ConfigError(f"{lw}: the values are the keys' projections; vdim {vdim} must be dim {dim}")
        mask = SalipelConfig._mask(lw, left, {"size", "keep_first"})
        windowed = SalipelWindowed(heads, kv_heads, dim, scale, mask.get("size", 0), _count(f"{lw}.mask.keep_first", mask.get("keep_first") or 0),
                                   SalipelConfig._rotation(lw, left, dim))
        _warn_unknown(rw, right, {"heads", "dim", "vdim", "gate_cap"})
        r_heads, r_dim = _positive_int(f"{rw}.heads", right.get("heads")), _positive_int(f"{rw}.dim", right.get("dim"))
        memory = SalipelMemory(r_heads, r_dim, _positive_int(f"{rw}.vdim", right.get("vdim", r_dim)), _positive(f"{rw}.gate_cap", right.get("gate_cap")))
        return SalipelPair(windowed, memory, _number(f"{w}.left_scale", m.get("left_scale", 1.0)), _number(f"{w}.right_scale", m.get("right_scale", 1.0)))

    @staticmethod
    def _mlp(where: str, raw) -> Optional[SalipelFeedForward]:
        if raw is None:
            return None
        kind = _object(where, raw).get("kind")
        if kind == "dense":
            _warn_unknown(where, raw, {"kind", "ff"})
            return SalipelFeedForward("dense", _positive_int(f"{where}.ff", raw.get("ff")))
        if kind != "moe":
            raise ConfigError(f"{where}.kind {kind!r} is not implemented (have ['dense', 'moe'])")
        _warn_unknown(where, raw, {"kind", "expert", "router"})
        expert, router = _object(f"{where}.expert", raw.get("expert")), _object(f"{where}.router", raw.get("router"))
        _warn_unknown(f"{where}.expert", expert, {"ff"})
        _warn_unknown(f"{where}.router", router, {"experts", "top", "scale"})
        ff = _positive_int(f"{where}.expert.ff", expert.get("ff"))
        experts = _positive_int(f"{where}.router.experts", router.get("experts"))
        top = _positive_int(f"{where}.router.top", router.get("top"))
        if top > experts:
            raise ConfigError(f"{where}: top {top} of {experts} experts")
        return SalipelFeedForward("moe", ff, experts, top, _number(f"{where}.router.scale", router.get("scale", 1.0)))
