"""Small Degavik configurations and weights for the tests.  The sizes differ from one another in every respect.
Weights are made here, tensor kind by tensor kind, so that every mechanism carries signal: decays from fast to slow,
scores large enough for the soft cap to bend them, mixing matrices far from the identity, norm weights and temperatures
that are not trivial, router logits that lie apart."""
import json
import os
import tempfile

import torch


def delta(heads, kv_heads, dim, vdim, conv, mlp=None, ranks=None):
    """`ranks`: the inner sizes of the two low-rank projections; kept beside the configuration, not in it."""
    out = {"type": "channel_delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv},
           "mlp": mlp}
    return out if ranks is None else dict(out, _ranks=ranks)


def attention(heads, kv_heads, dim, vdim, scale, softcap, window, keep, rot, mlp=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if softcap:
        m["softcap"] = softcap
    if window:
        m["mask"] = {"size": window, "keep_first": keep}
    if rot:
        m["rot"] = {"dims": rot[0], "base": rot[1]}
    return {"type": "attention", "mixer": m, "mlp": mlp}


def retention(heads, dim, vdim, decay, rot, mlp=None):
    m = {"heads": heads, "dim": dim, "vdim": vdim, "decay": list(decay)}
    if rot:
        m["rot"] = {"dims": rot[0], "base": rot[1]}
    return {"type": "retention", "mixer": m, "mlp": mlp}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, shared=None):
    out = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared:
        out["shared"] = {"ff": shared}
    return out


def again(j):
    """A run of layer j's tensors with a cache and state of its own."""
    return {"weights_of": j}


def config(vocab, width, eps, layers):
    """(config.json's dict, {layer: (decay rank, gate rank)})."""
    out, ranks = [], {}
    for i, e in enumerate(layers):
        if "type" not in e:
            e = dict({k: v for k, v in layers[e["weights_of"]].items()}, weights_of=e["weights_of"])
        e = dict(e)
        r = e.pop("_ranks", None)
        if r is not None and "weights_of" not in e:
            ranks[i] = r
        out.append(e)
    return {"architecture": "Degavik", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": out}, ranks


# grouped q/k heads in the delta rule, value heads wider than key heads, three taps and a first low-rank size that is no
# multiple of eight; attention with a window and kept first tokens, a third of a head turned; a layer without a
# feed-forward; layers run again with other layers' tensors; experts with and without a shared one
CFG_A, RANKS_A = config(97, 60, 1e-5, [
    delta(4, 2, 12, 20, 3, dense(44), ranks=(11, 7)),
    attention(6, 2, 24, 16, 0.3, 6.0, 19, 3, (8, 100.0), moe(5, 2, 28, shared=36)),
    retention(3, 20, 28, (0.6, 0.93, 0.995), (20, 1000.0), None),
    again(0),
    again(2),
    again(1),
])

# widths no tensor-core product takes; one key/value head for all; one tap (no convolution); attention without a window,
# a cap or a turn; a retention head partly turned with a decay of one; top one of three experts
CFG_B, RANKS_B = config(53, 35, 1e-6, [
    retention(2, 10, 6, (1.0, 0.8), (4, 7.0), moe(3, 1, 20)),
    attention(5, 1, 10, 6, 0.35, 0, 0, 0, None, dense(30)),
    delta(3, 3, 9, 13, 1, moe(4, 4, 12, shared=10), ranks=(5, 13)),
    again(1),
])

# sizes all tensor-core kernels take; the single-token kernel of the delta rule; a window of whole pages with kept
# tokens beyond a page; layers in another order
CFG_C, RANKS_C = config(160, 128, 1e-5, [
    attention(8, 4, 32, 48, 0.2, 12.0, 64, 18, (16, 5000.0), dense(192)),
    delta(4, 4, 64, 32, 4, moe(8, 3, 64, shared=64), ranks=(16, 24)),
    retention(2, 64, 64, (0.9, 0.99), None, dense(128)),
    delta(2, 2, 48, 96, 2, None, ranks=(24, 8)),
    again(1),
])

# one layer: heads four to a kv head, a window of two tokens and one kept
CFG_D, RANKS_D = config(61, 48, 1e-5, [attention(8, 2, 16, 8, 0.4, 3.0, 2, 1, (16, 10000.0), dense(40))])

CONFIGS = {"A": (CFG_A, RANKS_A), "B": (CFG_B, RANKS_B), "C": (CFG_C, RANKS_C), "D": (CFG_D, RANKS_D)}


def with_ranks(cfg, ranks):
    """The configuration with the low-rank sizes written into it (what a reader makes of the tensors' shapes)."""
    layers = []
    for i, e in enumerate(cfg["layers"]):
        src = e.get("weights_of", i)
        if src in ranks:
            e = dict(e, mixer=dict(e["mixer"], decay_rank=ranks[src][0], gate_rank=ranks[src][1]))
        layers.append(e)
    return dict(cfg, layers=layers)


def make_tensors(cfg, ranks, seed):
    """name -> float32 tensor, for every tensor the architecture declares."""
    from mdma_b200.config import load_config
    from mdma_b200.engine.model import expected_tensors
    arch, typed = load_config(with_ranks(cfg, ranks))
    g = torch.Generator().manual_seed(seed)
    rn = lambda *shape: torch.randn(tuple(shape), generator=g)
    kinds = {f"l{i}.": e["type"] for i, e in enumerate(cfg["layers"]) if "weights_of" not in e}
    out = {}
    for name, ts in expected_tensors(arch.describe(typed)).items():
        shape = tuple(ts.shape)
        last = name.split(".")[-1]
        kind = kinds.get(name.split(".")[0] + ".")
        if name == "embed":
            t = rn(*shape)
        elif name == "head":
            t = rn(*shape) * (1.6 / shape[1] ** 0.5)
        elif last in ("norm1", "norm2"):
            t = 0.7 + 0.2 * rn(*shape)                         # a sublayer's result has unit size before this weight
        elif last == "norm":
            t = 1.0 + 0.3 * rn(*shape)
        elif last == "conv":
            t = rn(*shape) * 0.6
            t[:, -1] += 0.5
        elif last == "A_log":
            t = rn(*shape) * 1.5 - 1.0                         # decays of a step from a few percent to none
        elif last == "dt_bias":
            t = rn(*shape) - 1.5
        elif last == "talk":
            t = torch.eye(shape[0]) + 0.4 * rn(*shape)
        elif last == "temp":
            t = 1.0 + 0.4 * rn(*shape).abs()
        elif name.endswith("router.b"):
            t = torch.randperm(shape[0], generator=g).float() * 2.5 + 0.2 * rn(*shape)     # logits lie apart
        elif last == "router":
            t = rn(*shape) * (0.25 / shape[1] ** 0.5)
        elif last == "b":
            t = rn(*shape) * (1.0 / shape[1] ** 0.5)
        elif last == "g" or last in ("a2", "g2"):
            t = rn(*shape) * (1.5 / shape[1] ** 0.5)
        elif last in ("q", "k") and kind == "retention":
            t = rn(*shape) * (0.8 / shape[1] ** 0.5)
        elif len(shape) == 2:
            t = rn(*shape) * (1.2 / shape[1] ** 0.5)
        else:
            raise AssertionError(f"no recipe for {name} {shape}")
        out[name] = t.to(torch.float32)
    return out


def make_model(cfg, ranks, seed, dtype=torch.float32, root=None):
    """Write a folder (config.json without the low-rank sizes + model.safetensors in `dtype`); returns (dir, tensors as
    stored, in float64)."""
    from mdma_b200.weights import write_safetensors
    d = tempfile.mkdtemp(prefix="degavik_tiny_", dir=root)
    with open(os.path.join(d, "config.json"), "w") as f:
        json.dump(cfg, f)
    tensors = {n: t.to(dtype) for n, t in make_tensors(cfg, ranks, seed).items()}
    write_safetensors(os.path.join(d, "model.safetensors"), tensors)
    return d, {n: t.double() for n, t in tensors.items()}
