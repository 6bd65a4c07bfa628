"""The Salipel architecture against its plain statement (tests/plain_salipel.py): every mechanism alone through its
kernels, then whole models through the engine's step function, the cache manager, the scheduler and the generation
loop.  Configurations and weights are made here (tests/salipel_tiny.py)."""
import json
import os

import numpy as np
import pytest
import torch

import plain_salipel as ps
from salipel_tiny import CONFIGS, SEEDS, chunked, config, dense, differential, make_model, make_tensors, memory, moe, pair, rot, windowed

# float32: absolute, against the float64 statement.  bfloat16: the largest error as a share of the deviation of the
# reference logits, and a row's root-mean-square error as a share of the row's own deviation.  A head whose result is small
# is divided by its size, so that single rows turn the rounding of their inputs into much of the logits: `ref_of` measures
# how far each row of the statement itself moves when its weights are moved by NOISE (relative), and a row may be off by
# three times that in bfloat16, by 1/250 of that in float32.
TOL_F32 = 5e-5
TOL_BF16, TOL_ROW_BF16 = 0.10, 0.04
NOISE, F32_OF_NOISE = 4e-3, 4e-3
CLOSE_CALL = 0.006       # a bfloat16 row behind a routing choice closer than this may take another expert


def ids_of(cfg, n, seed):
    g = torch.Generator().manual_seed(seed)
    return torch.randint(0, cfg["vocab"], (n,), generator=g).tolist()


def close(got, ref, dtype, what="", calm=None, moves=None):
    """Logits [rows, vocab] against the statement's.  `calm` [rows] of bool: rows that no close routing choice precedes;
    the others are only asked to be finite in bfloat16.  `moves` [rows]: how far the row itself moves (see above)."""
    got, ref = np.atleast_2d(np.asarray(got, dtype=np.float64)), np.atleast_2d(np.asarray(ref, dtype=np.float64))
    assert got.shape == ref.shape, (what, got.shape, ref.shape)
    assert np.isfinite(got).all(), f"{what}: logits that are not finite"
    err = np.abs(got - ref)
    moves = np.zeros(len(ref)) if moves is None else np.asarray(moves)
    if dtype == "float32":
        bad = err.max(axis=-1) >= np.maximum(TOL_F32, F32_OF_NOISE * moves)
        assert not bad.any(), f"{what}: rows {np.nonzero(bad)[0].tolist()} are off by {err.max(axis=-1)[bad]} (they move by {moves[bad]})"
        return
    share = err.max(axis=-1) / max(float(ref.std()), 0.25)
    own = np.maximum(ref.std(axis=-1), 1e-3)
    rel = np.sqrt((err ** 2).mean(axis=-1)) / own
    bad = (share >= np.maximum(TOL_BF16, 9.0 * moves / max(float(ref.std()), 0.25))) | (rel >= np.maximum(TOL_ROW_BF16, 3.0 * moves / own))
    if calm is not None:
        bad &= np.asarray(calm, dtype=bool)
    assert not bad.any(), f"{what}: rows {np.nonzero(bad)[0].tolist()} are off (share {share[bad]}, row error {rel[bad]}, they move by {(moves / own)[bad]})"


# =====================================================================================================
# Without a device.

def test_config_is_read_and_checked(capsys):
    from mdma_b200.config import ConfigError, SalipelConfig
    cfg = CONFIGS["A"]
    c = SalipelConfig.from_dict(cfg)
    assert (c.vocab, c.width, len(c.layers), c.residual_mult) == (97, 60, 5, 0.37)
    a, d, p = (c.layers[i].mixer for i in range(3))
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.chunk) == (6, 2, 24, 16, 19)
    assert (d.diff, d.softcap, d.rot.dims, d.rot.base, d.rot.scaling) == (0.35, 3.0, 8, 100.0, None)
    assert (p.left.window, p.left.keep_first, p.left.rot.scaling.original_max_position_embeddings) == (13, 5, 40)
    assert (p.right.dim, p.right.vdim, p.right.gate_cap, p.left_scale, p.right_scale) == (12, 20, 4.0, 1.3, -0.6)
    assert c.layers[2].mlp is None and (c.layers[1].mlp.top, c.layers[1].mlp.scale) == (2, 1.7)
    b = SalipelConfig.from_dict(CONFIGS["B"])
    assert b.layers[0].mixer.chunk == 0 and b.layers[1].mixer.left.window == 0 and b.layers[2].mixer.rot is None
    assert "leaves alone" not in capsys.readouterr().err
    SalipelConfig.from_dict(dict(cfg, note="x"))
    assert "leaves alone" in capsys.readouterr().err

    def refuse(change):
        bad = json.loads(json.dumps(cfg))
        change(bad)
        with pytest.raises(ConfigError):
            SalipelConfig.from_dict(bad)
    refuse(lambda r: r.pop("norm"))
    refuse(lambda r: r.update(residual_mult=0))
    refuse(lambda r: r["layers"][0].update(type="retention"))
    refuse(lambda r: r["layers"][0]["mixer"].update(kv_heads=4))
    refuse(lambda r: r["layers"][0]["mixer"]["mask"].update(size=0))
    refuse(lambda r: r["layers"][1]["mixer"].pop("diff"))
    refuse(lambda r: r["layers"][1]["mixer"]["rot"].update(dims=14))
    refuse(lambda r: r["layers"][1]["mixer"].update(softcap=-1.0))
    refuse(lambda r: r["layers"][1]["mlp"]["router"].update(top=6))
    refuse(lambda r: r["layers"][2]["mixer"]["left"].update(vdim=24))
    refuse(lambda r: r["layers"][2]["mixer"]["left"]["rot"]["scaling"].update(high=1.0))
    refuse(lambda r: r["layers"][2]["mixer"].pop("right"))
    refuse(lambda r: r["layers"][2]["mixer"]["right"].update(gate_cap=0))
    refuse(lambda r: r["layers"][0].update(mlp={"kind": "sparse"}))


def test_tensors_needs_and_the_unit_of_the_stream():
    from mdma_b200.config import load_config
    from mdma_b200.engine.model import DecoderModel
    arch, typed = load_config(CONFIGS["A"])
    spec = arch.describe(typed)
    model = DecoderModel(spec)
    names = {n: tuple(t.shape) for n, t in model.expected_tensors().items()}
    assert names["l1.mix.q"] == (4 * 2 * 12, 60) and names["l1.mix.k"] == (2 * 2 * 12, 60) and names["l1.mix.v"] == (2 * 20, 60)
    assert names["l1.mix.g"] == (80, 60) and names["l1.mix.lq2"] == (12,) and names["l0.mix.sink"] == (6,)
    assert names["l2.mix.left.k"] == (40, 60) and "l2.mix.left.v" not in names and names["l2.mix.right.f.b"] == (3,)
    assert names["l1.mlp.e4.up"] == (28, 60) and "l1.mlp.e0.gate" not in names and names["l4.mlp.correction"] == (3,)
    assert not any(n.startswith("l2.mlp") or ".norm2" in n for n in names)
    k0, k1, k2 = model.kv_needs()[:3]
    assert (k0.chunk, k0.window, k0.v_dim) == (19, 0, 16)
    assert (k1.n_kv_heads, k1.n_v_heads, k1.head_dim, k1.v_dim, k1.bounded) == (4, 2, 12, 20, False)
    assert (k2.window, k2.keep_first, k2.v_dim) == (13, 5, 0)
    assert [n is not None for n in model.state_needs()] == [False, False, True, False, False]
    # the stream is kept divided by the multiplier: rows over it, norms with eps over its square
    assert spec.stream_unit == 0.37 and spec.embedding.params["scale"] == 1.0 / 0.37
    assert abs(spec.final_norm.params["eps"] - 1e-5 / 0.37 ** 2) < 1e-12


def test_plan_without_a_device(tmp_path):
    from mdma_b200.engine.step import plan_only
    for key in CONFIGS:
        d, _ = make_model(CONFIGS[key], 2, root=str(tmp_path))
        for dtype in ("float32", "bfloat16"):
            p = plan_only(d, dtype=dtype, max_batch=3, max_context=128)
            assert p["total_bytes"] > p["weights_bytes"] > 0 and p["slots"] == 3


def test_the_benchmark_configuration_is_a_valid_model():
    import bench
    from mdma_b200.config import load_config
    from mdma_b200.engine.model import DecoderModel
    from mdma_b200.ops_tensor import attention_general_supported
    arch, typed = load_config(bench.salipel_config(2048, 4, 32000))
    model = DecoderModel(arch.describe(typed))
    assert {l.type for l in typed.layers} == {"attention", "attention_2", "parallel"}
    for l in typed.layers:
        m = l.mixer.left if l.type == "parallel" else l.mixer
        assert attention_general_supported(m.heads, m.kv_heads, m.dim, getattr(m, "vdim", m.dim))
    assert len(model.expected_tensors()) > 80


def test_chunks_give_their_pages_back():
    """A group with chunks holds the pages of the current chunk only; portions may start anywhere."""
    from mdma_b200.cache import KVNeed, SequenceCache
    for chunk in (3, 4, 6, 11):
        need = KVNeed(2, 8, chunk=chunk, n_v_heads=1, v_dim=12)
        c = SequenceCache([need], [None], max_tokens=96, max_slots=2, max_context=96, dtype=torch.float32, device="cpu", page_size=4)
        g = c.groups[0]
        assert g.k.shape[3:] == (2, 8) and g.v.shape[3:] == (1, 12)
        s = c.acquire()
        length = 0
        for n in (21, 1, 1, 7, 2, 1, 1, 1, 1, 30, 1):
            c.extend({s: n})
            first = length // chunk * chunk                     # the first new token's chunk must be there whole
            assert set(range(first // 4, (length + n - 1) // 4 + 1)) <= set(g.seq_pages[s])
            c.commit({s: n})
            length += n
            live = set(range(length // chunk * chunk // 4, (length - 1) // 4 + 1))
            assert set(g.seq_pages[s]) == live, (chunk, length)
            c.check()
        c.release(s)
        assert g.pages.free_count == g.n_pages


def test_the_plain_statement_notices_each_mechanism():
    """With one mechanism of the statement changed, some logit moves by many times the tolerance: a test that passes with
    the engine doing the same wrong thing is not possible without being noticed here."""
    cfg = CONFIGS["A"]
    W = {n: t.double() for n, t in make_tensors(cfg, 23).items()}
    ids = ids_of(cfg, 50, 3)
    ref = ps.forward(cfg, W, ids)

    def moved(cfg2=cfg, W2=W):
        return float((ps.forward(cfg2, W2, ids) - ref).abs().max())

    def change(layer, side=None, **mixer):
        out = json.loads(json.dumps(cfg))
        m = out["layers"][layer]["mixer"]
        (m[side] if side else m).update(mixer)
        return out
    floor = 200 * TOL_F32
    assert moved(change(0, mask={"size": 20})) > floor and moved(change(0, mask=None)) > floor
    assert moved(change(2, "left", mask={"size": 14, "keep_first": 5})) > floor
    assert moved(change(2, "left", mask={"size": 13, "keep_first": 4})) > floor
    assert moved(change(2, "left", mask={"size": 13, "keep_first": 6})) > floor
    assert moved(change(1, softcap=None)) > floor and moved(change(1, diff=0.36)) > floor
    assert moved(change(1, rot={"dims": 8, "base": 110.0})) > floor
    assert moved(change(2, "left", rot={"dims": 12, "base": 30.0})) > floor            # the stretching of slow pairs
    assert moved(change(2, "left", rot=rot(12, 30.0, (4.0, 1.0, 3.0, 40)))) > floor
    assert moved(change(2, "right", gate_cap=4.5)) > floor
    assert moved(change(2, right_scale=-0.5)) > floor and moved(dict(cfg, residual_mult=0.36)) > floor
    other = json.loads(json.dumps(cfg))
    other["layers"][1]["mlp"]["router"]["scale"] = 1.5
    assert moved(other) > floor
    for name in W:
        if ".mlp.e" in name or name in ("l4.mlp.correction",):      # (all of three experts are chosen there)
            continue
        assert moved(cfg, {**W, name: W[name].roll(1, 0)}) > floor, name              # its rows in another order
    for name in ("l0.mix.sink", "l1.mlp.correction", "l2.mix.right.i.b"):
        assert moved(cfg, {**W, name: torch.zeros_like(W[name]) if "sink" not in name else W[name] - 30.0}) > floor, name


# =====================================================================================================
# Kernels alone (GPU).

def _dev(t, dtype=torch.float32):
    return t.to(device="cuda", dtype=dtype).contiguous()


def _i32(a):
    return torch.as_tensor(np.asarray(a, dtype=np.int32), device="cuda")


class _Step:
    """The step metadata the kernels' entry points read, for a call outside an engine."""

    def __init__(self, lengths, pos0, slots):
        self.n_seqs, self.n_tokens = len(lengths), sum(lengths)
        self.max_new, self.max_len = max(lengths), max(p + n for p, n in zip(pos0, lengths))
        self.seq_start = _i32(np.concatenate([[0], np.cumsum(lengths)]))
        self.seq_pos0, self.seq_slot = _i32(pos0), _i32(slots)
        self.tok_seq = _i32(np.concatenate([np.full(n, s) for s, n in enumerate(lengths)]))
        self.tok_pos = _i32(np.concatenate([np.arange(p, p + n) for p, n in zip(pos0, lengths)]))
        self.most_seqs = None


# heads, kv heads, dim, vdim, maps, window, keep, chunk, cap, penalty, sink
ATTENTION_SIZES = [
    (6, 2, 24, 16, 1, 19, 3, 0, 0.0, False, False), (8, 4, 48, 48, 1, 64, 34, 0, 0.0, False, True), (5, 1, 10, 6, 1, 0, 0, 0, 0.0, True, True),
    (8, 2, 32, 48, 1, 0, 0, 80, 0.0, True, True), (8, 8, 112, 64, 1, 0, 0, 37, 0.0, True, True), (4, 2, 16, 128, 2, 0, 0, 0, 9.0, False, False),
    (16, 4, 64, 112, 2, 0, 0, 0, 30.0, False, False), (6, 3, 12, 20, 2, 0, 0, 0, 8.0, False, False), (2, 1, 128, 128, 2, 0, 0, 0, 0.0, False, False),
    (8, 2, 16, 16, 1, 2, 1, 0, 0.0, False, False), (4, 4, 64, 64, 1, 40, 70, 0, 12.0, False, False), (12, 1, 80, 32, 1, 0, 0, 1, 0.0, True, False),
    (32, 2, 128, 16, 1, 50, 65, 0, 20.0, True, True), (4, 2, 32, 64, 2, 30, 5, 0, 10.0, True, True), (3, 3, 200, 256, 1, 33, 2, 0, 0.0, False, False),
]


def _reference(sets, H, maps, scale, sees, cap, slopes, sinks):
    """[T, H, maps, V] of every sequence."""
    out = []
    for q, k, v in sets:
        out.append(torch.stack([ps.attend(q[:, :, m], k[:, :, m], v, scale, sees(len(q)), cap or None, slopes, sinks) for m in range(maps)], 2))
    return out


@pytest.mark.gpu
@pytest.mark.parametrize("kernel", ["plain32", "plain16", "tc", "mma", "step", "step16"])
@pytest.mark.parametrize("H,G,D,V,maps,window,keep,chunk,cap,penalty,sink", ATTENTION_SIZES)
def test_attention_masks_maps_pages_and_batches(kernel, H, G, D, V, maps, window, keep, chunk, cap, penalty, sink):
    """Unequal sequences with shuffled pages (rows nobody owns hold NaN, and so do keys of pages a mask lets go); prompts from
    the start and portions on a cached prefix.  At every row one key stands out: just inside a window or a chunk, just
    outside, the last kept token or the one after it; a mask one token off moves the row by far more than the tolerance."""
    from mdma_b200 import ops, ops_tensor
    half = kernel != "plain32"
    on_tensor = not kernel.startswith("plain")
    if on_tensor and not ops_tensor.attention_general_supported(H, G, D, V):
        pytest.skip("the tensor-core kernels do not take these sizes")
    dtype = torch.bfloat16 if half else torch.float32
    page = {"tc": 64, "step": 32}.get(kernel, 16)
    gen = torch.Generator().manual_seed(11)
    rn = lambda *s: torch.randn(s, generator=gen, dtype=torch.float64)
    r = (lambda t: t.bfloat16().double()) if half else (lambda t: t.float().double())
    scale = D ** -0.5
    slopes = ps.slopes_of(H) * 0.25 if penalty else None
    sinks = (1.0 + rn(H)).float().double() if sink else None
    lengths = [150, 33, 1, 97]
    sets = []
    for T in lengths:
        q, k, v = 0.3 * rn(T, H, maps, D), rn(T, G, maps, D), rn(T, G, V)
        k = k / k.norm(dim=-1, keepdim=True)
        for i in range(T):                              # the key that stands out for row i: by turns
            if chunk:
                at = i // chunk * chunk
                edges = [at, at - 1, i, i - 1]
            elif window:
                edges = [i - window + 1, i - window, keep - 1, keep]
            else:
                edges = [0, i // 2, i, i - 31]
            j = edges[i % 4]
            if 0 <= j <= i:
                q[i] = q[i] + (1.75 / scale) * k[j].repeat_interleave(H // G, 0)
        sets.append((r(q), r(k), r(v)))

    def sees_of(window, keep, chunk):
        return (lambda T: ps.chunk_sees(T, chunk) if chunk else ps.window_sees(T, window, keep) if window else ps.causal(T))
    refs = _reference(sets, H, maps, scale, sees_of(window, keep, chunk), cap, slopes, sinks)
    tol = lambda want: dict(rtol=3e-5, atol=3e-5) if not half else dict(rtol=1.5e-2, atol=1.5e-2 * float(want.abs().max().clamp(min=1.0)))
    others = [(window + 1, keep, 0), (window - 1, keep, 0), (window, keep + 1, 0)] + ([(window, keep - 1, 0)] if keep else []) if window else \
             [(0, 0, chunk + 1), (0, 0, chunk - 1)] if chunk > 1 else []
    for other in others:                                # a token more or less would show
        if max(other) > 0:
            moved = float((_reference(sets[:1], H, maps, scale, sees_of(*other), cap, slopes, sinks)[0] - refs[0]).abs().max())
            assert moved > 3 * tol(refs[0])["atol"], (other, moved)
    pages_per = -(-160 // page)
    perm = torch.randperm(4 * pages_per + 3, generator=gen)[:4 * pages_per].reshape(4, pages_per)
    kc = torch.full((4 * pages_per + 3, page, G * maps, D), float("nan"), dtype=dtype, device="cuda")
    vc = torch.full((4 * pages_per + 3, page, G, V), float("nan"), dtype=dtype, device="cuda")
    slots = [3, 1, 0, 2]

    class View:
        pass
    view = View()
    view.k, view.v, view.page_size, view.max_pages = kc, vc, page, pages_per
    view.page_table = _i32(perm.numpy())
    lam, norm_scale, eps, out_scale = 0.3, 0.7, 1e-5, 1.25

    def fill(first_of):
        """Keys and values of every position that is still owned when a step starts at first_of[s]; NaN elsewhere."""
        kc.fill_(float("nan"))
        vc.fill_(float("nan"))
        for s, (q, k, v) in enumerate(sets):
            p0 = first_of[s]
            first = p0 // chunk * chunk if chunk else max(0, p0 + 1 - window) if window else 0
            for t in range(lengths[s]):
                if t >= first or t < keep:
                    p = int(perm[slots[s], t // page])
                    kc[p, t % page], vc[p, t % page] = k[t].reshape(G * maps, D).to(dtype).cuda(), v[t].to(dtype).cuda()

    def check(new, pos0, which):
        fill([pos0[which.index(s)] if s in which else 0 for s in range(4)])
        ctx = _Step(new, pos0, [slots[s] for s in which])
        pitch = -(-H * maps * D // 8) * 8 + 8
        rows = torch.full((ctx.n_tokens, pitch), float("nan"), dtype=dtype, device="cuda")
        rows[:, :H * maps * D] = torch.cat([sets[s][0][p:p + n].reshape(n, -1) for s, n, p in zip(which, new, pos0)]).to(dtype).cuda()
        gate = rn(ctx.n_tokens, H * V + 5).to(dtype)
        g_dev = gate.cuda()[:, 5:]
        want_rows = torch.cat([refs[s][p:p + n] for s, n, p in zip(which, new, pos0)])
        want = want_rows[:, :, 0]
        if maps == 2:
            want = ps.rms_unit(want_rows[:, :, 0] - lam * want_rows[:, :, 1], eps) * norm_scale
        want = want.reshape(ctx.n_tokens, -1) * torch.sigmoid(gate[:, 5:].double()) * out_scale
        finish = dict(gate=g_dev, out_scale=out_scale, **(dict(maps=2, lam=lam, norm_scale=norm_scale, eps=eps) if maps == 2 else {}))
        out = torch.full((ctx.n_tokens, H * V), float("nan"), dtype=dtype, device="cuda")
        maps_out = torch.full((ctx.n_tokens, H * maps * V), float("nan"), device="cuda")
        d_slopes = None if slopes is None else _dev(slopes)
        d_sinks = None if sinks is None else _dev(sinks)
        log2 = lambda t: None if t is None else _dev(t * 1.4426950408889634)
        if not on_tensor:
            target = maps_out if maps == 2 else out
            ops.attention_distance(rows, kc, vc, ctx, view.page_table, pages_per, page, d_slopes, None, target, H, G, D, V, window, scale,
                                   sinks=d_sinks, keep_first=keep, chunk=chunk, softcap=cap, maps=maps)
            torch.testing.assert_close(target.double().cpu().reshape(want_rows.shape), want_rows, **tol(want_rows))
            ops.attention_finish(out, ctx.n_tokens, H, V, rows=target, **finish)
            torch.testing.assert_close(out.double().cpu(), want, **tol(want))
            return
        for splits in ((None,) if kernel == "tc" else (1, 3, 7)):
            out.fill_(float("nan"))
            maps_out.fill_(float("nan"))
            partial = ops_tensor.attention_general(
                ctx, rows, view, H, G, D, V, scale, out=out if maps == 1 else None, out_f32=maps_out if maps == 2 else None, maps=maps,
                window=window, keep_first=keep, chunk=chunk, softcap=cap, sink_log2=log2(sinks), slope_log2=log2(slopes), splits=splits,
                impl="tc" if kernel == "tc" else "mma")
            assert (partial is None) == (splits in (None, 1))
            if partial is not None:
                ops.attention_finish(out, ctx.n_tokens, H, V, partial=partial, sink_log2=log2(sinks), **finish)
            else:
                ops.attention_finish(out, ctx.n_tokens, H, V, rows=maps_out if maps == 2 else out, **finish)
            torch.testing.assert_close(out.double().cpu(), want, **tol(want))
            ops_tensor.check_status(out.device)
    if kernel.startswith("step"):
        for back in (1, 2, 3, 4, 60):
            which = [s for s in range(4) if lengths[s] >= back]
            check([1] * len(which), [lengths[s] - back for s in which], which)
        return
    for new, pos0, which in (([150, 33, 1, 97], [0, 0, 0, 0], [0, 1, 2, 3]), ([50, 2, 47], [100, 31, 50], [0, 1, 3]), ([3], [147], [0])):
        check(new, pos0, which)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,GV,D,V,dims,norm,v_norm,same", [
    (4, 2, 2, 24, 16, 8, True, False, False), (8, 4, 2, 12, 20, 12, True, False, False), (6, 2, 2, 32, 32, 24, True, False, True),
    (0, 3, 3, 10, 7, 0, False, True, False), (5, 1, 1, 128, 256, 64, True, True, False)])
def test_heads_are_normed_turned_and_cached(dtype, H, G, GV, D, V, dims, norm, v_norm, same):
    """Queries and keys normed, weighted and turned (slow pairs stretched), values of another number or normed or the keys'
    projections; rows whole, or as partial sums with columns behind the heads."""
    from mdma_b200 import ops
    from mdma_b200.config.llama import RopeScaling
    from mdma_b200.parts.rotary import inverse_frequencies
    gen = torch.Generator().manual_seed(5)
    n, page, tail = 9, 4, 37
    k_col = H * D
    v_col = k_col if same else k_col + G * D
    width = (k_col + G * D if same else v_col + GV * V) + tail
    row = torch.randn(n, width, generator=gen, dtype=torch.float64).to(dtype).double()
    q_w, k_w = (1 + 0.3 * torch.randn(D, generator=gen)), (1 + 0.3 * torch.randn(D, generator=gen))
    pos = [3, 4, 5, 6, 7, 30, 31, 32, 33]
    turn = rot(dims, 20.0, (4.0, 1.0, 4.0, 60)) if dims else None
    table = _dev(inverse_frequencies(dims, 20.0, RopeScaling("llama3", 4.0, 1.0, 4.0, 60))) if dims else None
    if dims:
        torch.testing.assert_close(table.double().cpu(), ps.frequencies(turn), rtol=1e-6, atol=0)

    def at(x):                                        # the statement turns positions 0..T-1: place each row at its own
        full = torch.zeros(40, *x.shape[1:], dtype=torch.float64)
        full[pos] = x
        return ps.rotate(full, turn)[pos]
    head = lambda c, m, d: row[:, c:c + m * d].reshape(n, m, d)
    unit = (lambda x, w: ps.rms_unit(x, 1e-5) * w.to(dtype).double()) if norm else (lambda x, w: x)
    q, k = at(unit(head(0, H, D), q_w)), at(unit(head(k_col, G, D), k_w))
    v = head(v_col, GV, V)
    v = ps.rms_unit(v, 1e-5) if v_norm else v
    page_table = _i32([[5, 0, 9, 1, 2, 3, 4, 6, 7, 8], [11, 12, 13, 14, 15, 16, 17, 18, 19, 20]])
    seq, slot = _i32([0] * 5 + [1] * 4), _i32([1, 0])
    for splits in ((0, 3) if H else (0,)):
        kc = torch.full((21, page, G, D), float("nan"), dtype=dtype, device="cuda")
        vc = torch.full((21, page, GV, V), float("nan"), dtype=dtype, device="cuda")
        part = torch.randn(3, n, width, generator=gen)
        part[2] = (row - part[0].double() - part[1].double()).float()
        whole = part.double().sum(0)
        proj = _dev(torch.full((n, width + 3), float("nan")) if splits else torch.nn.functional.pad(row, (0, 3)), dtype)[:, :width]
        ops.qk_norm_rotate(proj, k_col, v_col, seq, _i32(pos), slot, table, 1.0, _dev(q_w, dtype), _dev(k_w, dtype), norm, 1e-5, kc, vc,
                           page_table, 10, page, n, H, G, D, V, dims, False, True, n_v_heads=GV, v_norm=v_norm,
                           partial=_dev(part) if splits else None, splits=splits, split_stride=n * width, row_width=width,
                           tail_col=width - tail)
        tol = dict(rtol=1e-2, atol=1e-2) if dtype == torch.bfloat16 else dict(rtol=2e-5, atol=2e-5)
        torch.testing.assert_close(proj[:, :H * D].double().cpu().reshape(n, H, D), q, **tol)
        torch.testing.assert_close(proj[:, width - tail:].double().cpu(), whole[:, width - tail:], **tol)
        for i, p in enumerate(pos):
            at_page = int(page_table[[1, 0][int(seq[i])], p // page])
            torch.testing.assert_close(kc[at_page, p % page].double().cpu(), k[i], **tol)
            torch.testing.assert_close(vc[at_page, p % page].double().cpu(), v[i], **tol)
        assert int(torch.isfinite(kc.float()).all(-1).all(-1).sum()) == n and int(torch.isfinite(vc.float()).all(-1).all(-1).sum()) == n


MEMORY_SIZES = [(3, 12, 20, 4.0), (2, 9, 13, 15.0), (4, 64, 32, 8.0), (2, 48, 96, 15.0), (1, 16, 16, 2.0), (2, 128, 128, 15.0), (1, 256, 200, 6.0), (1, 160, 256, 15.0)]


@pytest.mark.gpu
@pytest.mark.parametrize("H,D,V,cap", MEMORY_SIZES)
@pytest.mark.parametrize("walk", ["rows", "chunks", "runs", "tokens"])
@pytest.mark.parametrize("mood", ["even", "forgetful", "closed"])
def test_matrix_memory_walks(walk, H, D, V, cap, mood):
    """Unequal sequences in two steps each (the second starts from state, at no chunk's edge), against the statement's
    recurrence: row by row, a chunk of rows at a time, runs side by side, and single tokens from the projection to the gated
    norm.  `forgetful`: forget gates near nothing; `closed`: input gates near nothing for the first rows, so that the sum
    of keys stays below its floor.  Slots are taken out of order; a slot of nobody's holds NaN and is left alone."""
    from mdma_b200 import ops
    if walk == "tokens" and not ops.matrix_memory_token_fits(D, V):
        pytest.skip("the single-token kernel takes value heads of multiples of four")
    gen = torch.Generator().manual_seed(7)
    rn = lambda *s: torch.randn(s, generator=gen, dtype=torch.float64)
    bf = lambda t: t.bfloat16().double()
    cuts = {"tokens": [[1, 1, 1]] * 7, "runs": [[300, 1, 140], [270, 257, 2]]}.get(walk, [[37, 1, 16], [19, 30, 2]])
    slots, n_slots = [2, 0, 3], 4
    total = [sum(c[s] for c in cuts) for s in range(3)]
    width = H * (2 * D + 2 * V + 2)
    k_col, v_col, g_col = H * D, 2 * H * D, 2 * H * D + H * V
    i_col = g_col + H * V
    f_col = i_col + H
    i_b, f_b, norm = bf(rn(H)), bf(1.5 * rn(H) + (2.0 if mood != "forgetful" else -6.0)), bf(1 + 0.3 * rn(H * V))
    rows, refs, gated = [], [], []
    for T in total:
        x = rn(T, width)
        x[:, i_col:f_col] *= 2.0
        if mood == "closed":
            x[:5, i_col:f_col] -= 4.0 * cap
        x = x.float().double()
        li = cap * torch.tanh((x[:, i_col:f_col] + i_b) / cap)
        lf = ps.log_sigmoid(cap * torch.tanh((x[:, f_col:] + f_b) / cap))
        o = ps.matrix_memory_steps(x[:, :k_col].reshape(T, H, D) * D ** -0.5, x[:, k_col:v_col].reshape(T, H, D),
                                   x[:, v_col:g_col].reshape(T, H, V), li, lf)
        rows.append(x)
        refs.append(o.reshape(T, H * V))
        gated.append(ps.rms_unit(o, 1e-5).reshape(T, H * V) * norm * torch.sigmoid(x[:, g_col:i_col]) * -0.6)
    floats = ops.matrix_memory_state_floats(H, D, V)
    state = torch.full((n_slots, floats + 4), float("nan"), device="cuda")[:, :floats]
    for s in slots:
        state[s] = 0.0
    cols = (0, k_col, v_col, i_col, f_col)
    b_i, b_f = _dev(i_b, torch.bfloat16), _dev(f_b, torch.bfloat16)
    at = [0, 0, 0]
    for cut in cuts:
        ctx = _Step(cut, at, slots)
        n = ctx.n_tokens
        proj = torch.full((n, -(-width // 4) * 4), float("nan"), device="cuda")[:, :width]
        proj.copy_(torch.cat([rows[s][at[s]:at[s] + cut[s]] for s in range(3)]))
        if walk == "tokens":
            out = torch.zeros(n, H * V, dtype=torch.bfloat16, device="cuda")
            first = 0.25 * proj                                                   # the projection as two partial sums
            partial = torch.stack([first, proj - first]).contiguous()
            split = at[0] % 2 == 1
            src = torch.full_like(proj, float("nan")) if split else proj
            ops.matrix_memory_token(src, cols, g_col, b_i, b_f, cap, D ** -0.5, _dev(norm, torch.bfloat16), ctx, state, out, H, D, V, 1e-5,
                                    -0.6, partial if split else None, 2, n * width)
            want = torch.cat([gated[s][at[s]:at[s] + 1] for s in range(3)])
            torch.testing.assert_close(out.double().cpu(), want, rtol=1e-2, atol=2e-3)
        else:
            out = torch.full((n, H * V), float("nan"), device="cuda")
            run_rows, most = (128, -(-max(cut) // 128)) if walk == "runs" else (0, 1)
            scratch = torch.full((3 * most * floats + 16,), float("nan"), device="cuda") if run_rows else None
            ops.matrix_memory(proj, cols, b_i, b_f, cap, D ** -0.5, ctx, state, out, H, D, V, walk != "rows", run_rows, most,
                              scratch[:-16] if run_rows else None)
            want = torch.cat([refs[s][at[s]:at[s] + cut[s]] for s in range(3)])
            # a row whose n . q nearly cancels is divided by its floor or by little: errors are judged against the row
            err = (out.double().cpu() - want).abs().reshape(n, H, V).amax(-1)
            size = want.abs().reshape(n, H, V).amax(-1)
            assert float((err / (size + 1e-2)).max()) < (3e-4 if walk != "rows" else 1e-4)
            assert float((err / (size + 1e-2)).median()) < 1e-6
            assert scratch is None or torch.isnan(scratch[-16:]).all()
        at = [a + c for a, c in zip(at, cut)]
    assert torch.isnan(state[1]).all()
    # the state itself: S e^m and n e^m of the statement
    assert torch.isfinite(state[slots]).all()


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("experts,top,W,F,scale", [(5, 2, 60, 28, 1.7), (3, 1, 35, 20, 1.0), (4, 4, 35, 12, 2.5), (16, 3, 128, 64, 0.8)])
@pytest.mark.parametrize("tokens", [7, 150])
def test_experts_without_a_gate(tokens, dtype, experts, top, W, F, scale):
    """Softmax scores, choice by corrected scores, weights that add up to a constant; squared-ReLU experts, token by token,
    expert by expert, and with a product per expert."""
    from mdma_b200 import ops
    from mdma_b200.parts.base import Runtime
    from mdma_b200.parts.routed_mlp import RoutedMLP
    from mdma_b200.spec import PartSpec
    part = RoutedMLP(PartSpec("routed_mlp", dict(hidden_size=W, intermediate_size=F, experts=experts, top=top, gated=False,
                                                 activation="relu_squared", weight_scale=scale)))
    gen = torch.Generator().manual_seed(19)
    tensors = {}
    for name, ts in part.tensor_specs().items():
        t = torch.randn(ts.shape, generator=gen)
        tensors[name] = (t * 0.1 if name == "correction" else t * (1.2 / ts.shape[-1] ** 0.5)).to(dtype)
    h = torch.randn(tokens, W, generator=gen).to(dtype)
    w = {"m." + n: t.double() for n, t in tensors.items()}
    calls = []
    want = ps.feed_forward(h.double(), w, "m.", {"kind": "moe", "router": {"experts": experts, "top": top, "scale": scale}}, calls)
    part.bind({n: t.cuda() for n, t in tensors.items()}, Runtime(dtype, torch.device("cuda"), gemm="tensor" if dtype == torch.bfloat16 else "simt"))

    class Ctx:
        n_tokens, decode_only = tokens, False
        bufs = {}

        def buf(self, name, cols, dt=None):
            kind = dt or dtype
            return self.bufs.setdefault(name, torch.zeros(tokens, cols, dtype=kind, device="cuda"))
    ways = ["as chosen"] + (["expert by expert"] if dtype == torch.bfloat16 and tokens >= 33 else [])
    for way in ways:
        part.by_products = part.by_products and way == "as chosen"
        x = torch.ones(tokens, W, device="cuda")
        part.forward(Ctx(), h.cuda(), x)
        got = x.double().cpu() - 1.0
        sure = calls[0] > (1e-3 if dtype == torch.bfloat16 else 1e-6)              # (h is exact: only the router's sums round)
        tol = dict(rtol=2e-2, atol=2e-2 * float(want.abs().max())) if dtype == torch.bfloat16 else dict(rtol=1e-4, atol=2e-5)
        torch.testing.assert_close(got[sure], want[sure], **tol)
    assert ops is not None


@pytest.mark.gpu
@pytest.mark.parametrize("H,V,gdtype,odtype", [(3, 28, torch.float32, torch.float32), (4, 5, torch.float32, torch.bfloat16)])
def test_gated_norm_with_a_weight_per_number(H, V, gdtype, odtype):
    from mdma_b200 import ops
    gen = torch.Generator().manual_seed(3)
    n = 19
    o, w = torch.randn(n, H * V, generator=gen), torch.randn(H * V, generator=gen)
    gate = torch.randn(n, H * V + 3, generator=gen).to(gdtype)
    out = torch.full((n, H * V), float("nan"), dtype=odtype, device="cuda")
    ops.gated_head_rmsnorm(_dev(o), gate.cuda()[:, 3:], _dev(w), out, n, H, V, 1e-5, scale=-0.7)
    want = ps.rms_unit(o.double().reshape(n, H, V), 1e-5).reshape(n, -1) * w.double() * torch.sigmoid(gate[:, 3:].double()) * -0.7
    tol = 1e-5 if odtype == torch.float32 else 1e-2
    torch.testing.assert_close(out.double().cpu(), want, rtol=tol, atol=tol)


# =====================================================================================================
# Whole models through the engine (GPU).

_models: dict = {}


def model_of(key, dtype, drawn=None, seed=None):
    """(folder, config, float64 tensors as the engine holds them) of configuration `key`."""
    k = (key, dtype)
    if k not in _models:
        store = torch.float32 if dtype == "float32" else torch.bfloat16
        cfg = drawn or CONFIGS[key]
        d, W = make_model(cfg, seed if seed is not None else SEEDS[key], store)
        _models[k] = (d, cfg, W)
    return _models[k]


_refs: dict = {}


def ref_of(key, dtype, ids):
    """(the statement's logits, whether no close routing choice lies at or before a row, how far the row moves)."""
    k = (key, dtype, tuple(ids))
    if k not in _refs:
        _, cfg, W = model_of(key, dtype)
        calls = []
        logits = ps.forward(cfg, W, ids, closeness=calls).numpy()
        gap = torch.stack(calls).min(0).values.numpy() if calls else np.full(len(ids), 9.0)
        gen = torch.Generator().manual_seed(1)
        moves = np.zeros(len(ids))
        for _ in range(2):
            other = {n: t * (1.0 + NOISE * torch.randn(t.shape, generator=gen, dtype=torch.float64)) for n, t in W.items()}
            moves = np.maximum(moves, np.sqrt(((ps.forward(cfg, other, ids).numpy() - logits) ** 2).mean(-1)))
        _refs[k] = (logits, np.minimum.accumulate(gap) > CLOSE_CALL, moves)
    return _refs[k]


def check(got, pairs, dtype, what):
    """`pairs`: per row (reference of `ref_of`, position)."""
    close(got, np.stack([r[0][p] for r, p in pairs]), dtype, what, [r[1][p] for r, p in pairs], [r[2][p] for r, p in pairs])


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("key", ["A", "B", "C", "D"])
def test_every_layer_against_the_plain_statement(key, dtype):
    """The residual stream after every layer, then the logits; one short prompt, the first tokens among the rows."""
    from mdma_b200.engine import Engine, StepEntry
    d, cfg, W = model_of(key, dtype)
    ids = ids_of(cfg, 45, 4)
    _, trace = ps.forward(cfg, W, ids, return_layers=True)
    ref = ref_of(key, dtype, ids)
    rows = np.nonzero(ref[1])[0] if dtype == "bfloat16" else np.arange(len(ids))
    assert len(rows) > 10
    eng = Engine(d, dtype=dtype, max_batch=2, max_context=64, logit_rows=64, page_size=16)
    got = []
    eng.model.on_layer = lambda n, x: got.append(x.detach().double().cpu())
    s = eng.acquire()
    logits = eng.step([StepEntry(s, ids, list(range(len(ids))))]).cpu().numpy()
    assert len(got) == len(trace) == len(cfg["layers"])
    tol = 1e-4 if dtype == "float32" else 0.05
    for n, (a, b) in enumerate(zip(got, trace)):
        err = float((a - b)[rows].abs().max())
        assert err < tol * max(1.0, float(b.abs().max())), f"after layer {n}: {err}"
    check(logits, [(ref, p) for p in range(len(ids))], dtype, "logits")


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("key", ["A", "B", "C", "D"])
def test_batches_portions_decoding_and_reuse(key, dtype):
    """Unequal prompts in one step; the same prompts cut in portions down to one and two tokens on a cached prefix;
    token-by-token decoding; sequences that end early while others go on; slots and pages freed and taken again (rows
    nobody owns hold NaN throughout).  In float32 every way of cutting gives the same logits to within a few units of
    the last place."""
    from mdma_b200.engine import Engine, StepEntry
    d, cfg, W = model_of(key, dtype)
    lengths = [90, 1, 33, 2, 17]
    seqs = [ids_of(cfg, n, 20 + i) for i, n in enumerate(lengths)]
    refs = [ref_of(key, dtype, s) for s in seqs]
    eng = Engine(d, dtype=dtype, max_batch=5, max_context=96, logit_rows=160, page_size=16)

    def run(plan):
        """plan: per sequence, the sizes of its portions.  All sequences advance together, one portion a step."""
        slots = [eng.acquire() for _ in seqs]
        rows = [[] for _ in seqs]
        at = [0] * len(seqs)
        for step in range(max(len(p) for p in plan)):
            live = [i for i in range(len(seqs)) if step < len(plan[i])]
            eng.cache.poison_unused()
            out = eng.step([StepEntry(slots[i], seqs[i][at[i]:at[i] + plan[i][step]], list(range(plan[i][step])))
                            for i in live]).cpu().numpy()
            o = 0
            for i in live:
                n = plan[i][step]
                rows[i].append(out[o:o + n].copy())
                o += n
                at[i] += n
                if at[i] == len(seqs[i]):
                    eng.release(slots[i])           # ends early; its slot and its pages go back
        eng.cache.check()
        return [np.concatenate(r) for r in rows]

    whole = run([[n] for n in lengths])
    alone = []
    for i, s in enumerate(seqs):                    # each alone, in a slot that the batch used
        slot = eng.acquire()
        alone.append(eng.step([StepEntry(slot, s, list(range(len(s))))]).cpu().numpy().copy())
        eng.release(slot)
    pieces = run([[2, 1, 30, 37, 1, 2, 16, 1], [1], [16, 1, 15, 1], [1, 1], [3, 14]])
    pairs = run([[2] * 45, [1], [2] * 16 + [1], [2], [2] * 8 + [1]])
    decoded = run([[25] + [1] * 65, [1], [1] * 33, [2], [16, 1]])
    for name, other in (("whole prompts", whole), ("alone", alone), ("portions", pieces), ("two at a time", pairs), ("decoded", decoded)):
        for i, (got, ref) in enumerate(zip(other, refs)):
            check(got, [(ref, p) for p in range(lengths[i])], dtype, f"{name}, sequence {i}")
            if dtype == "float32":
                assert np.abs(got - whole[i]).max() <= 6e-6, f"{name}, sequence {i}: differs from the whole prompt"


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("key", ["A", "C"])
def test_passes_smaller_than_a_step_and_long_decoding(key, dtype):
    """A step run as passes of 19 tokens (cuts inside sequences), then 150 tokens decoded one by one across many page and
    chunk borders and out of the window, beside a batch mate that ends on the way and whose slot another request takes."""
    from mdma_b200.engine import Engine, StepEntry
    d, cfg, W = model_of(key, dtype)
    long_ids, mate, late = ids_of(cfg, 190, 31), ids_of(cfg, 60, 32), ids_of(cfg, 25, 33)
    r_long, r_mate, r_late = (ref_of(key, dtype, s) for s in (long_ids, mate, late))
    eng = Engine(d, dtype=dtype, max_batch=2, max_context=192, logit_rows=64, page_size=16, chunk_tokens=19)
    a, b = eng.acquire(), eng.acquire()
    out = eng.step([StepEntry(a, long_ids[:40], [0, 39, 18, 19]), StepEntry(b, mate[:41], [40, 13])]).cpu().numpy()
    assert eng.forward_passes > 4
    check(out, [(r_long, 0), (r_long, 39), (r_long, 18), (r_long, 19), (r_mate, 40), (r_mate, 13)], dtype, "passes")
    pb = 41
    for p in range(40, 190):
        entries, pairs = [StepEntry(a, [long_ids[p]], [0])], [(r_long, p)]
        if pb < len(mate):
            entries.append(StepEntry(b, [mate[pb]], [0]))
            pairs.append((r_mate, pb))
            pb += 1
        elif pb == len(mate):                       # the mate is done: its slot goes to a late request
            eng.release(b)
            b = eng.acquire()
            entries.append(StepEntry(b, late, [len(late) - 1]))
            pairs.append((r_late, len(late) - 1))
            pb += 1
        eng.cache.poison_unused()
        check(eng.step(entries).cpu().numpy(), pairs, dtype, f"decoded position {p}")
    eng.cache.check()
    eng.check_status()


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("key", ["A", "B", "C"])
def test_long_prompts_in_uneven_portions(key, dtype):
    """Prompts of several hundred tokens in one batch, cut at places that are no page's, window's or chunk's edge, then
    decoded: the kernels for many rows, their chunks and runs, on filled caches and states."""
    from mdma_b200.engine import Engine, StepEntry
    d, cfg, W = model_of(key, dtype)
    seqs = [ids_of(cfg, 620, 71), ids_of(cfg, 301, 72), ids_of(cfg, 17, 73)]
    refs = [ref_of(key, dtype, s) for s in seqs]
    eng = Engine(d, dtype=dtype, max_batch=3, max_context=640, logit_rows=1024)
    slots = [eng.acquire() for _ in seqs]
    at = [0, 0, 0]
    for cut in ((331, 296, 9), (2, 1, 7), (279, 0, 0), (1, 1, 1), (3, 0, 0), (4, 3, 0)):
        eng.cache.poison_unused()
        live = [i for i in range(3) if cut[i]]
        out = eng.step([StepEntry(slots[i], seqs[i][at[i]:at[i] + cut[i]], list(range(cut[i]))) for i in live]).cpu().numpy()
        check(out, [(refs[i], at[i] + j) for i in live for j in range(cut[i])], dtype, f"portion {cut}")
        at = [a + c for a, c in zip(at, cut)]
    assert at == [len(s) for s in seqs]
    eng.check_status()


@pytest.mark.gpu
def test_a_token_far_back_moves_the_end_and_the_engine_follows():
    """One early token of a prompt of 330 is changed: the last logits move, in the plain statement and in the engine
    alike, in portions that cut across pages."""
    from mdma_b200.engine import Engine, StepEntry
    d, cfg, W = model_of("B", "float32")
    ids = ids_of(cfg, 330, 61)
    other = list(ids)
    other[5] = (other[5] + 11) % cfg["vocab"]
    ra, rb = ref_of("B", "float32", ids), ref_of("B", "float32", other)
    assert np.abs(ra[0][-1] - rb[0][-1]).max() > 20 * TOL_F32
    eng = Engine(d, dtype="float32", max_batch=2, max_context=384, logit_rows=16, page_size=16)
    s, t = eng.acquire(), eng.acquire()
    eng.step([StepEntry(s, ids[:300], []), StepEntry(t, other[:280], [])])
    out = eng.step([StepEntry(s, ids[300:], [29]), StepEntry(t, other[280:], [49])]).cpu().numpy()
    check(out, [(ra, 329), (rb, 329)], "float32", "the prompts")


@pytest.mark.gpu
@pytest.mark.parametrize("key", ["A", "C"])
def test_greedy_generation_through_the_scheduler(key):
    """`Engine.generate`: batches, the decode session's replayed graphs, argmax.  float32 tokens equal the plain
    statement's greedy continuation; replayed and step-by-step runs give the same tokens in both dtypes."""
    from mdma_b200.engine import Engine
    d, cfg, W = model_of(key, "float32")
    prompts = [ids_of(cfg, n, 40 + n) for n in (9, 30, 3)]
    want = []
    for p in prompts:
        ids = list(p)
        for _ in range(12):
            ids.append(int(ps.forward(cfg, W, ids)[-1].argmax()))
        want.append(ids[len(p):])
    eng = Engine(d, dtype="float32", max_batch=2, max_context=64)            # three requests, two slots: two batches
    assert eng.decode_session().graph_safe
    for graphs in (True, False):
        outs = eng.generate(prompts, max_tokens=12, use_graphs=graphs)
        assert [o.tokens for o in outs] == want, graphs
    d16, _, _ = model_of(key, "bfloat16")
    eng = Engine(d16, dtype="bfloat16", max_batch=3, max_context=64)
    a = eng.generate(prompts, max_tokens=12, use_graphs=True)
    b = eng.generate(prompts, max_tokens=12, use_graphs=False)
    assert [o.tokens for o in a] == [o.tokens for o in b]
    sampled = eng.generate(prompts, max_tokens=8, temperature=0.9, top_p=0.9, seed=3)
    assert all(len(o.tokens) == 8 for o in sampled)
    assert eng.held_bytes()["total_bytes"] == eng.memory_plan()["total_bytes"]


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_replay_and_the_command_line(dtype, tmp_path):
    """`bin/trace_run` on a folder of this architecture: a prompt in a step, two requests decoded together, one ends,
    its slot is taken by a new request; `mdma plan` and `mdma run` take the folder too."""
    import subprocess
    d, cfg, W = model_of("A", dtype)
    a, b, c = ids_of(cfg, 40, 81), ids_of(cfg, 9, 82), ids_of(cfg, 12, 83)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:30], "want": [0, 29]}, {"id": "b", "tokens": b[:5], "want": [4]}], "end": []}]
    for j in range(4):
        steps.append({"step": 1 + j, "entries": [{"id": "a", "tokens": [a[30 + j]], "want": [0]}, {"id": "b", "tokens": [b[5 + j]], "want": [0]}],
                      "end": ["b"] if j == 3 else []})
    steps.append({"step": 5, "entries": [{"id": "c", "tokens": c, "want": [11]}], "end": ["c"]})
    steps.append({"step": 6, "entries": [{"id": "a", "tokens": a[34:], "want": [5]}], "end": ["a"]})
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    out = tmp_path / "out"
    res = subprocess.run([os.path.join(root, "bin", "trace_run"), "--model", d, "--dtype", dtype, "--out", str(out), "--max-tokens", "128"],
                         input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, timeout=600)
    assert res.returncode == 0, res.stderr[-2000:]
    assert [l for l in res.stdout.splitlines() if l.startswith("done")] == [f"done {i}" for i in range(7)]
    ra, rb, rc = (ref_of("A", dtype, s) for s in (a, b, c))
    read = lambda i: np.fromfile(out / f"{i}.f32", dtype="<f4").reshape(-1, cfg["vocab"])
    check(read(0), [(ra, 0), (ra, 29), (rb, 4)], dtype, "step 0")
    for j in range(4):
        check(read(1 + j), [(ra, 30 + j), (rb, 5 + j)], dtype, f"step {1 + j}")
    check(read(5), [(rc, 11)], dtype, "step 5")
    check(read(6), [(ra, 39)], dtype, "step 6")
    if dtype == "float32":
        from mdma_b200.cli import main
        assert main(["run", d, " ".join(map(str, a[:5])), "--max-tokens", "4", "--dtype", "float32", "--max-context", "64"]) == 0
        assert main(["plan", d, "--ctx", "64"]) == 0
        assert main(["run", os.path.join(d, "config.json"), "3 1 4", "--random-weights", "7", "--max-tokens", "3", "--max-context", "32"]) == 0


def random_config(seed):
    """A configuration drawn from a seed: layer kinds in any order, head counts and sizes of many values, some multiples of
    8 or 16 and some not, windows and chunks from one token to beyond the prompt."""
    rng = np.random.default_rng(3000 + seed)
    pick = lambda xs: xs[int(rng.integers(len(xs)))]
    width = pick([35, 48, 64, 72, 96, 128])

    def mlp():
        kind = pick(["none", "dense", "moe", "moe"])
        if kind == "none":
            return None
        if kind == "dense":
            return dense(pick([24, 40, 64]))
        n = pick([2, 3, 5, 8])
        return moe(n, int(rng.integers(1, n + 1)), pick([12, 24, 32]), float(rng.uniform(0.5, 2.5)))

    def turn(D, scaled=False):
        dims = pick([0, D // 4 * 2 or 2, D // 2 * 2, 2])
        return rot(dims, pick([1e4, 50.0, 7.0]), pick([None, (4.0, 1.0, 4.0, 100), (2.5, 0.5, 3.0, 30)]) if scaled else None) if dims else None
    layers = []
    for _ in range(int(rng.integers(2, 6))):
        kind = pick(["chunked", "differential", "pair"])
        G = pick([1, 2, 3, 4])
        H = G * pick([1, 1, 2, 4])
        D, V = pick([8, 16, 32, 48, 10, 80]), pick([6, 8, 16, 24, 64, 112])
        scale = float(rng.uniform(0.8, 1.6)) * D ** -0.5
        if kind == "chunked":
            layers.append(chunked(H, G, D, V, scale, pick([0, 1, 5, 16, 40, 64, 100, 500]), mlp()))
        elif kind == "differential":
            layers.append(differential(H, G, D, V, scale, float(rng.uniform(0.0, 0.8)), pick([0, 2.5, 20.0]), turn(D), mlp()))
        else:
            left = windowed(H, G, D, scale, pick([0, 1, 5, 16, 40, 64, 500]), pick([0, 1, 4, 17, 70]), turn(D, True))
            right = memory(pick([1, 2, 3, 4]), pick([8, 9, 16, 48, 64]), pick([4, 6, 24, 40, 96]), pick([2.0, 8.0, 15.0]))
            layers.append(pair(left, right, float(rng.uniform(0.5, 1.5)), float(rng.uniform(-1.0, 1.5)), mlp()))
    return config(int(rng.integers(40, 200)), width, pick([1e-5, 1e-6]), pick([1.0, 0.5, 0.3, 1.4]), layers)


@pytest.mark.gpu
@pytest.mark.parametrize("seed", range(int(os.environ.get("SALIPEL_DRAWN_CONFIGS", "12"))))
def test_random_configurations(seed):
    """Drawn configurations in both engines: a batch of unequal prompts, portions on a cached prefix, decoding."""
    from mdma_b200.engine import Engine, StepEntry
    drawn = random_config(seed)
    for dtype in ("float32", "bfloat16"):
        key = f"drawn{seed}"
        d, cfg, W = model_of(key, dtype, drawn, seed)
        seqs = [ids_of(cfg, n, 90 + i) for i, n in enumerate((75, 12, 300))]
        refs = [ref_of(key, dtype, s) for s in seqs]
        eng = Engine(d, dtype=dtype, max_batch=3, max_context=320, logit_rows=512)
        slots = [eng.acquire() for _ in seqs]
        eng.cache.poison_unused()
        first = [60, 12, 280]
        out = eng.step([StepEntry(slots[i], seqs[i][:first[i]], list(range(first[i]))) for i in range(3)]).cpu().numpy()
        check(out, [(refs[i], p) for i in range(3) for p in range(first[i])], dtype, f"seed {seed} {dtype}: prompts")
        eng.release(slots[1])
        eng.cache.poison_unused()
        out = eng.step([StepEntry(slots[0], seqs[0][60:67], [6]), StepEntry(slots[2], seqs[2][280:282], [0, 1])]).cpu().numpy()
        check(out, [(refs[0], 66), (refs[2], 280), (refs[2], 281)], dtype, f"seed {seed} {dtype}: portions")
        for j in range(8):
            eng.cache.poison_unused()
            out = eng.step([StepEntry(slots[0], [seqs[0][67 + j]], [0]), StepEntry(slots[2], [seqs[2][282 + j]], [0])]).cpu().numpy()
            check(out, [(refs[0], 67 + j), (refs[2], 282 + j)], dtype, f"seed {seed} {dtype}: decoded {j}")
        eng.cache.check()
        eng.check_status()
