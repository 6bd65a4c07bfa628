"""Small Salipel configurations and weights for the tests.  The sizes differ from one another in every respect.  Weights are
made here, tensor kind by tensor kind, so that every mechanism carries signal: scores large enough for caps, sinks and
masks to matter, two maps that differ, gates from open to closed, router scores that lie apart."""
import json
import os
import tempfile

import torch


def rot(dims, base, scaling=None):
    """`scaling`: (factor, low, high, original)."""
    out = {"dims": dims, "base": base}
    if scaling:
        out["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return out


def chunked(heads, kv_heads, dim, vdim, scale, chunk, mlp=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if chunk:
        m["mask"] = {"size": chunk}
    return {"type": "attention", "mixer": m, "mlp": mlp}


def differential(heads, kv_heads, dim, vdim, scale, diff, softcap, turn, mlp=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "diff": diff}
    if softcap:
        m["softcap"] = softcap
    if turn:
        m["rot"] = turn
    return {"type": "attention_2", "mixer": m, "mlp": mlp}


def windowed(heads, kv_heads, dim, scale, window, keep, turn):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale}
    if window:
        m["mask"] = {"size": window, "keep_first": keep}
    if turn:
        m["rot"] = turn
    return m


def memory(heads, dim, vdim, cap):
    return {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}


def pair(left, right, left_scale, right_scale, mlp=None):
    return {"type": "parallel", "mixer": {"left": left, "right": right, "left_scale": left_scale, "right_scale": right_scale}, "mlp": mlp}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, scale):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top, "scale": scale}}


def config(vocab, width, eps, mult, layers):
    return {"architecture": "Salipel", "vocab": vocab, "width": width, "norm": {"eps": eps}, "residual_mult": mult, "layers": layers}


# chunks and windows that are no page's size; three query heads to a kv head; a partly turned head whose slow pairs are
# stretched; value heads wider than the maps' keys; a layer without a feed-forward; memory heads that are not square
CFG_A = config(97, 60, 1e-5, 0.37, [
    chunked(6, 2, 24, 16, 0.3, 19, dense(44)),
    differential(4, 2, 12, 20, 0.4, 0.35, 3.0, rot(8, 100.0), moe(5, 2, 28, 1.7)),
    pair(windowed(4, 2, 20, 0.35, 13, 5, rot(12, 30.0, (4.0, 1.0, 4.0, 40))), memory(3, 12, 20, 4.0), 1.3, -0.6),
    differential(6, 3, 8, 12, 0.5, 0.1, 0, rot(4, 20.0), dense(36)),
    chunked(4, 4, 12, 28, 0.4, 33, moe(3, 3, 20, 0.8)),
])

# widths no tensor-core product takes; one kv head for all, every key seen, no cap and no turn; one of three experts
CFG_B = config(53, 35, 1e-6, 1.0, [
    chunked(5, 1, 10, 6, 0.5, 0, moe(3, 1, 20, 1.0)),
    pair(windowed(3, 3, 10, 0.45, 0, 0, None), memory(2, 9, 13, 15.0), 1.0, 1.0, dense(30)),
    differential(3, 1, 7, 9, 0.5, 0.8, 0, None, moe(4, 2, 12, 2.5)),
])

# sizes all tensor-core kernels take; a chunk longer than a page, a window of one page with kept tokens beyond half of one
CFG_C = config(160, 128, 1e-5, 0.6, [
    pair(windowed(8, 4, 48, 0.2, 64, 34, rot(32, 5000.0, (8.0, 1.0, 4.0, 512))), memory(4, 64, 32, 8.0), 0.9, 0.7, moe(8, 3, 64, 1.2)),
    chunked(8, 2, 32, 48, 0.25, 80, dense(192)),
    differential(8, 4, 16, 32, 0.35, 0.5, 12.0, rot(16, 1000.0), moe(6, 2, 64, 1.5)),
    differential(2, 1, 64, 112, 0.15, 0.2, 20.0, rot(64, 1e4), None),
    pair(windowed(4, 1, 16, 0.3, 24, 0, rot(16, 100.0)), memory(2, 48, 96, 15.0), 0.5, 1.4, dense(128)),
])

# the smallest masks: chunks of three, a window of two with one kept token
CFG_D = config(61, 48, 1e-5, 0.5, [
    chunked(4, 2, 16, 8, 0.4, 3, None),
    pair(windowed(8, 2, 16, 0.4, 2, 1, rot(16, 1e4)), memory(1, 16, 16, 2.0), 1.0, 0.8, dense(40)),
])

CONFIGS = {"A": CFG_A, "B": CFG_B, "C": CFG_C, "D": CFG_D}
SEEDS = {"A": 29, "B": 24, "C": 25, "D": 27}          # weights whose routing choices are seldom close


def make_tensors(cfg, seed):
    """name -> float32 tensor, for every tensor the architecture declares."""
    from mdma_b200.config import load_config
    from mdma_b200.engine.model import expected_tensors
    arch, typed = load_config(cfg)
    g = torch.Generator().manual_seed(seed)
    rn = lambda *shape: torch.randn(tuple(shape), generator=g)
    out = {}
    for name, ts in expected_tensors(arch.describe(typed)).items():
        shape, last = tuple(ts.shape), name.split(".")[-1]
        if name == "embed":
            t = rn(*shape)
        elif name == "head":
            t = rn(*shape) * (1.6 / shape[1] ** 0.5)
        elif last in ("norm1", "norm"):
            t = 1.0 + 0.3 * rn(*shape)
        elif last == "sink":
            t = 1.5 * rn(*shape) + 1.0
        elif last in ("lq1", "lk1", "lq2", "lk2"):
            t = rn(*shape) * (0.8 / shape[0] ** 0.5)
        elif name.endswith("i.b"):
            t = rn(*shape)
        elif name.endswith("f.b"):
            t = 1.5 * rn(*shape) + 2.0                         # memories from a few tokens to a few hundred
        elif last == "correction":
            t = torch.randperm(shape[0], generator=g).float() * 0.3 + 0.05 * rn(*shape)       # choices lie apart
        elif last == "router":
            t = rn(*shape) * (1.0 / shape[1] ** 0.5)
        elif last in ("g", "i", "f"):
            t = rn(*shape) * (1.5 / shape[1] ** 0.5)
        elif len(shape) == 2:
            t = rn(*shape) * (1.3 / shape[1] ** 0.5)
        else:
            raise AssertionError(f"no recipe for {name} {shape}")
        out[name] = t.to(torch.float32)
    return out


def make_model(cfg, seed, dtype=torch.float32, root=None):
    """Write a folder (config.json + model.safetensors in `dtype`); returns (dir, tensors as stored, in float64)."""
    from mdma_b200.weights import write_safetensors
    d = tempfile.mkdtemp(prefix="salipel_tiny_", dir=root)
    with open(os.path.join(d, "config.json"), "w") as f:
        json.dump(cfg, f)
    tensors = {n: t.to(dtype) for n, t in make_tensors(cfg, seed).items()}
    write_safetensors(os.path.join(d, "model.safetensors"), tensors)
    return d, {n: t.double() for n, t in tensors.items()}
