"""The Degavik architecture against its plain statement (tests/plain_degavik.py): every mechanism alone through its
kernels, then whole models through the engine's step function, the cache manager, the scheduler and the generation
loop.  Configurations and weights are made here (tests/degavik_tiny.py)."""
import json
import os

import numpy as np
import pytest
import torch

import plain_degavik as pd
from degavik_tiny import CONFIGS, attention, config, delta, dense, make_model, make_tensors, moe, retention, with_ranks

# float32: absolute, against the float64 statement.  bfloat16: the largest error as a share of the deviation of the
# reference logits, and a row's root-mean-square error as a share of the row's own deviation.  A head or a sublayer whose
# result is small is divided by its size, so that single rows turn the rounding of their inputs into a tenth of the
# logits: `ref_of` measures how far each row of the statement itself moves when its weights are moved by NOISE (relative),
# and a row may be off by three times that in bfloat16, by 1/250 of that in float32.
TOL_F32 = 5e-5
TOL_BF16, TOL_ROW_BF16 = 0.10, 0.04
NOISE, F32_OF_NOISE = 4e-3, 4e-3
CLOSE_CALL = 0.06        # a bfloat16 row behind a routing choice closer than this may take another expert


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
    from mdma_b200.config import ConfigError, DegavikConfig
    cfg, ranks = CONFIGS["A"]
    c = DegavikConfig.from_dict(with_ranks(cfg, ranks))
    assert (c.vocab, c.width, len(c.layers)) == (97, 60, 6)
    a = c.layers[1].mixer
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.window, a.keep_first, a.softcap, a.rot_dims) == (6, 2, 24, 16, 19, 3, 6.0, 8)
    d = c.layers[0].mixer
    assert (d.kv_heads, d.conv, d.decay_rank, d.gate_rank) == (2, 3, 11, 7)
    assert [l.weights_of for l in c.layers] == [None, None, None, 0, 2, 1]
    assert c.layers[2].mlp is None and c.layers[1].mlp.shared_ff == 36
    b = DegavikConfig.from_dict(CONFIGS["B"][0])
    assert b.layers[1].mixer.window == 0 and b.layers[1].mixer.rot_dims == 0 and b.layers[1].mixer.softcap == 0.0
    assert "leaves alone" not in capsys.readouterr().err
    chain = json.loads(json.dumps(cfg))
    chain["layers"][5] = dict(chain["layers"][3], weights_of=3)                # a layer whose source has a source
    assert DegavikConfig.from_dict(chain).layers[5].weights_of == 0

    def refuse(change):
        bad = json.loads(json.dumps(cfg))
        change(bad)
        with pytest.raises(ConfigError):
            DegavikConfig.from_dict(bad)
    refuse(lambda r: r.pop("norm"))
    refuse(lambda r: r["layers"][0].update(type="mamba"))
    refuse(lambda r: r["layers"][0]["mixer"].update(kv_heads=3))
    refuse(lambda r: r["layers"][1]["mixer"]["rot"].update(dims=26))
    refuse(lambda r: r["layers"][1]["mlp"]["router"].update(top=6))
    refuse(lambda r: r["layers"][2]["mixer"].update(decay=[0.5]))
    refuse(lambda r: r["layers"][3].update(weights_of=3))
    refuse(lambda r: r["layers"][3].update(weights_of=9))
    refuse(lambda r: r["layers"][3]["mixer"].update(dim=8))                    # not what the tensors' layer says
    refuse(lambda r: r["layers"][0].update(mlp={"kind": "sparse"}))


def test_sizes_come_from_the_tensors_shapes(tmp_path):
    """The low-rank sizes stand in no config.json: a folder's headers give them, for layers with other layers' tensors too."""
    from mdma_b200.config import load_config
    from mdma_b200.engine.model import expected_tensors
    from mdma_b200.weights import check_entries, open_model_files
    cfg, ranks = CONFIGS["C"]
    d, _ = make_model(cfg, ranks, 1, root=str(tmp_path))
    arch, typed = load_config(d)
    assert [(l.mixer.decay_rank, l.mixer.gate_rank) for l in typed.layers if l.type == "channel_delta"] == [(16, 24), (24, 8), (16, 24)]
    entries = {}
    for f in open_model_files(d):
        entries.update(f.entries)
    check_entries(entries, expected_tensors(arch.describe(typed)))
    os.remove(os.path.join(d, "model.safetensors"))
    _, typed = load_config(d)                                                   # no tensors: a head's size
    assert typed.layers[1].mixer.decay_rank == 64


def test_layers_with_other_layers_tensors_are_runs_of_those_layers():
    from mdma_b200.config import load_config
    from mdma_b200.engine.model import DecoderModel
    arch, typed = load_config(with_ranks(*CONFIGS["A"]))
    spec = arch.describe(typed)
    assert [e.layer for e in spec.schedule] == [0, 1, 2, 0, 2, 1] and all(e.cache is None for e in spec.schedule)
    model = DecoderModel(spec)
    names = set(model.expected_tensors())
    assert "l1.mix.talk" in names and "l0.mix.q.conv" in names and not any(n.startswith(("l3.", "l4.", "l5.")) for n in names)
    assert [n is not None for n in model.kv_needs()] == [False, True, False, False, False, True]
    assert [n is not None for n in model.state_needs()] == [True, False, True, True, True, False]


def test_plan_without_a_device(tmp_path):
    from mdma_b200.engine.step import plan_only
    for key in CONFIGS:
        d, _ = make_model(*CONFIGS[key], 2, root=str(tmp_path))
        for dtype in ("float32", "bfloat16"):
            p = plan_only(d, dtype=dtype, max_batch=3, max_context=128)
            assert p["total_bytes"] > p["weights_bytes"] > 0 and p["slots"] == 3


def test_the_benchmark_configuration_is_a_valid_model():
    import bench
    from mdma_b200.config import load_config
    from mdma_b200.engine.model import DecoderModel
    from mdma_b200.ops_tensor import mixed_weights_supported
    arch, typed = load_config(bench.degavik_config(2048, 4, 32000))
    model = DecoderModel(arch.describe(typed))
    assert {l.type for l in typed.layers} == {"channel_delta", "attention", "retention"}
    assert mixed_weights_supported(16, 4, 128, 128) and len(model.expected_tensors()) > 100


def test_the_plain_statement_notices_each_mechanism():
    """With one mechanism of the statement changed, some logit moves by many times the tolerance: a test that passes with
    the engine doing the same wrong thing is not possible without being noticed here."""
    cfg, ranks = CONFIGS["A"]
    W = {n: t.double() for n, t in make_tensors(cfg, ranks, 23).items()}
    ids = ids_of(cfg, 40, 3)
    ref = pd.forward(cfg, W, ids)

    def moved(cfg2=cfg, W2=W):
        return float((pd.forward(cfg2, W2, ids) - ref).abs().max())

    def change(layer, **mixer):
        out = json.loads(json.dumps(cfg))
        for key, v in mixer.items():
            out["layers"][layer]["mixer"][key] = v
        return out
    floor = 200 * TOL_F32
    assert moved(change(1, mask={"size": 20, "keep_first": 3})) > floor        # the window's edge
    assert moved(change(1, mask={"size": 19, "keep_first": 2})) > floor        # the kept tokens' edge
    assert moved(change(1, softcap=None)) > floor
    assert moved(change(1, rot={"dims": 8, "base": 110.0})) > floor
    assert moved(change(2, decay=[0.6, 0.93, 0.99])) > floor
    assert moved(change(2, rot=None)) > floor
    for name in W:
        if not name.startswith(("l0.", "l1.", "l2.")) or ".mlp.e" in name:
            continue
        assert moved(cfg, {**W, name: W[name].roll(1, 0)}) > floor, name        # its rows in another order
    layers = json.loads(json.dumps(cfg))["layers"]
    layers[3]["weights_of"] = 3
    own = {n.replace("l0.", "l3."): t * 1.1 for n, t in W.items() if n.startswith("l0.")}
    assert moved(dict(cfg, layers=layers), {**W, **own}) > floor                # a layer with tensors of its own


def test_kept_first_tokens_keep_their_pages():
    """A windowed group with kept tokens gives pages back in the middle of a sequence, never those of the first tokens."""
    from mdma_b200.cache import KVNeed, SequenceCache
    for keep, pages in ((0, 0), (1, 1), (4, 1), (5, 2)):
        c = SequenceCache([KVNeed(1, 8, window=6, keep_first=keep)], [None], max_tokens=64, max_slots=2, max_context=64,
                          dtype=torch.float32, device="cpu", page_size=4)
        s, t = c.acquire(), c.acquire()
        for slot, n in ((s, 21), (t, 3)):
            c.extend({slot: n})
            c.commit({slot: n})
        g = c.groups[0]
        for length in range(21, 40):
            held = set(g.seq_pages[s])
            live = set(range(max(0, length + 1 - 6) // 4, (length - 1) // 4 + 1))
            assert held == live | set(range(pages)), (keep, length, held)
            c.check()
            c.extend({s: 1})
            c.commit({s: 1})
        c.release(s)
        c.release(t)
        c.check()
        assert g.pages.free_count == g.n_pages


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


DELTA_SIZES = [(3, 3, 32, 32, 4, 24, 24, 0.0), (4, 2, 12, 20, 3, 11, 7, 0.0), (2, 2, 9, 13, 1, 5, 13, 0.0), (2, 2, 96, 40, 2, 16, 8, 0.0),
               (2, 1, 160, 64, 7, 8, 16, 0.0), (3, 3, 48, 96, 5, 20, 12, 0.0), (2, 2, 128, 128, 4, 128, 64, 0.0), (2, 2, 64, 48, 4, 16, 16, 4.0)]


@pytest.mark.gpu
@pytest.mark.parametrize("H,G,D,V,taps,ra,rg,strong", DELTA_SIZES)
@pytest.mark.parametrize("walk", ["rows", "chunks", "tokens"])
def test_delta_rule_walks(walk, H, G, D, V, taps, ra, rg, strong):
    """Unequal sequences in two steps each (the second starts from kept inputs and state, at no chunk's edge), against the
    statement's recurrence: row by row, a chunk of rows at a time, and single tokens from the projection to the gated
    norm.  `strong`: decays that take a channel to nothing within a token.  Slots are taken out of order."""
    from mdma_b200 import ops
    if walk == "chunks" and (D % 4 or V % 4):
        pytest.skip("the chunk kernels take heads of multiples of four")
    if walk == "tokens" and not ops.delta_token_fits(H, G, D, V, ra, rg, taps):
        pytest.skip("the single-token kernel does not take these sizes")
    gen = torch.Generator().manual_seed(5)
    rn = lambda *s: torch.randn(s, generator=gen, dtype=torch.float64)
    bf = lambda t: t.bfloat16().double()
    ch = 2 * G * D + H * V
    conv_at = -(-H * D * V // 4) * 4
    conv = bf(0.6 * rn(ch, taps))
    a_log, dt, norm = bf(1.5 * rn(H) - 1), bf(rn(H * D) - 1.5 + strong), bf(1 + 0.3 * rn(V))
    a2, g2 = bf(rn(H * D, ra) * ra ** -0.5), bf(rn(H * V, rg) * rg ** -0.5)
    first, then = ([37, 1, 16], [19, 30, 2]) if walk != "tokens" else ([1, 1, 1], [1, 1, 1])
    cuts = [first, then] if walk != "tokens" else [[1, 1, 1]] * 7
    slots, n_slots = [2, 0, 3], 4
    total = [sum(c[s] for c in cuts) for s in range(3)]
    rows = [rn(t, ch + H + ra + rg).float().double() for t in total]
    refs, gated = [], []
    for x in rows:
        T = x.shape[0]
        y = pd.silu(pd.short_conv(x[:, :ch], conv))
        q = pd.unit_vector(y[:, :G * D].reshape(T, G, D)) * D ** -0.5
        k = pd.unit_vector(y[:, G * D:2 * G * D].reshape(T, G, D))
        rep = H // G
        step = pd.softplus(x[:, ch + H:ch + H + ra] @ a2.T + dt).reshape(T, H, D)
        g = torch.exp(-torch.exp(a_log)[None, :, None] * step)
        o = pd.delta_steps(q.repeat_interleave(rep, 1), k.repeat_interleave(rep, 1), y[:, 2 * G * D:].reshape(T, H, V), g,
                           torch.sigmoid(x[:, ch:ch + H]))
        refs.append(o.reshape(T, H * V))
        gated.append((pd.rms_unit(o, 1e-5) * norm).reshape(T, H * V) * torch.sigmoid(x[:, ch + H + ra:] @ g2.T))
    state = torch.full((n_slots, conv_at + (taps - 1) * ch + 4), float("nan"), device="cuda")[:, :conv_at + (taps - 1) * ch]
    for s in slots:
        state[s] = 0.0
    kept = state[:, conv_at:] if taps > 1 else None
    c_conv, c_a, c_dt = _dev(conv, torch.bfloat16), _dev(a_log, torch.bfloat16), _dev(dt, torch.bfloat16)
    at = [0, 0, 0]
    for cut in cuts:
        ctx = _Step(cut, at, slots)
        n = ctx.n_tokens
        x = torch.cat([rows[s][at[s]:at[s] + cut[s]] for s in range(3)])
        proj = _dev(x)
        want = torch.cat([refs[s][at[s]:at[s] + cut[s]] for s in range(3)])
        if walk == "tokens":
            out = torch.zeros(n, H * V, dtype=torch.bfloat16, device="cuda")
            half = 0.25 * proj                                                   # the projection as two partial sums
            partial = torch.stack([half, proj - half]).contiguous()
            split = at[0] % 2 == 1
            src = torch.full_like(proj, float("nan")) if split else proj
            ops.delta_token(src, _dev(a2, torch.bfloat16), _dev(g2, torch.bfloat16), c_conv, taps, c_a, c_dt, _dev(norm, torch.bfloat16),
                            ctx, state, conv_at, out, H, D, V, 1e-6, D ** -0.5, 1e-5, partial if split else None, 2, n * proj.shape[1])
            want = torch.cat([gated[s][at[s]:at[s] + 1] for s in range(3)])
            torch.testing.assert_close(out.double().cpu(), want, rtol=1e-2, atol=2e-3)
        else:
            raw = _dev(x[:, ch + H:ch + H + ra] @ a2.T)
            out = torch.zeros(n, H * V, device="cuda")
            if walk == "rows":
                e = lambda c: torch.empty(n, c, device="cuda")
                q, k, v, lg, beta = e(G * D), e(G * D), e(H * V), e(H * D), e(H)
                ops.delta_prepare(proj, raw, c_conv, taps, c_a, c_dt, ctx, kept, q, k, v, lg, beta, H, G, D, V, 1e-6, D ** -0.5)
                ops.delta_scan(q, k, v, lg, beta, ctx, state[:, :H * D * V], out, H, G, D, V)
            else:
                floats = (n // 16 + 4) * ops.delta_chunk_floats(H, D, V)
                scratch = torch.full((floats + 64,), float("nan"), device="cuda")
                ops.delta_chunks(proj, raw, c_conv, taps, c_a, c_dt, kept, scratch[:floats], ctx, state[:, :H * D * V], out, H, G, D, V,
                                 1e-6, D ** -0.5)
                assert torch.isnan(scratch[floats:]).all()
            ops.delta_conv_keep(proj, taps, ch, ctx, kept)
            torch.testing.assert_close(out.double().cpu(), want, rtol=2e-5, atol=4e-6)
        at = [a + c for a, c in zip(at, cut)]
    assert torch.isnan(state[1]).all()                                           # a slot of nobody's is left alone
    if taps > 1:
        for s in range(3):                                                       # the kept inputs: the last rows, zeros before
            have = torch.cat([torch.zeros(taps - 1, ch, dtype=torch.float64), rows[s][:, :ch]])[-(taps - 1):]
            torch.testing.assert_close(kept[slots[s]].reshape(taps - 1, ch).double().cpu(), have, rtol=1e-6, atol=1e-6)


def _plain_mixed(q, k, v, mix, factor, cap, window, keep):
    """q [T, H, D], k [T, G, D], v [T, G, V] -> [T, H * V]: the statement's softmax, visibility and mixing."""
    T, H, _ = q.shape
    rep = H // k.shape[1]
    s = torch.einsum("ihd,jhd->hij", q, k.repeat_interleave(rep, 1)) * factor[:, None, None]
    if cap:
        s = cap * torch.tanh(s / cap)
    see = pd.visible(T, {"size": window, "keep_first": keep} if window else None)
    p = torch.einsum("hg,gij->hij", mix, torch.softmax(s.masked_fill(~see, -float("inf")), -1))
    return torch.einsum("hij,jhd->ihd", p, v.repeat_interleave(rep, 1)).reshape(T, -1)


ATTENTION_SIZES = [(6, 2, 24, 16, 19, 3, 6.0), (8, 4, 32, 48, 64, 18, 12.0), (5, 1, 10, 6, 0, 0, 0.0), (8, 2, 16, 8, 2, 1, 3.0),
                   (16, 4, 64, 128, 48, 0, 30.0), (24, 2, 16, 16, 33, 5, 4.0), (4, 4, 48, 96, 0, 0, 8.0), (12, 12, 128, 128, 70, 2, 0.0),
                   (3, 3, 256, 16, 40, 70, 5.0), (32, 8, 128, 32, 100, 1, 20.0)]


@pytest.mark.gpu
@pytest.mark.parametrize("kernel", ["plain32", "plain16", "rows", "step"])
@pytest.mark.parametrize("H,G,D,V,window,keep,cap", ATTENTION_SIZES)
def test_attention_with_mixed_weights_edges_pages_and_batches(kernel, H, G, D, V, window, keep, cap):
    """Unequal sequences with shuffled pages (rows nobody owns hold NaN); prompts from the start and portions on a cached
    prefix.  At every row one key stands out: the first one inside the window, or the last one before it (whose weight must
    be nothing), or the last kept token, or the one after it: a window or a kept range one token off moves the row by far
    more than the tolerance."""
    from mdma_b200 import ops, ops_tensor
    half = kernel != "plain32"
    if kernel in ("rows", "step") and not ops_tensor.mixed_weights_supported(H, G, D, V):
        pytest.skip("the tensor-core kernels do not take these sizes")
    if kernel == "step" and not ops_tensor.mixed_weights_step_fits(H, G, D, V):
        pytest.skip("the single-token kernel does not take these sizes")
    dtype = torch.bfloat16 if half else torch.float32
    gen = torch.Generator().manual_seed(11)
    rn = lambda *s: torch.randn(s, generator=gen, dtype=torch.float64)
    r = (lambda t: t.bfloat16().double()) if half else (lambda t: t.float().double())
    mix, factor = r(torch.eye(H, dtype=torch.float64) + 0.5 * rn(H, H)), (0.7 + 0.5 * torch.rand(H, generator=gen, dtype=torch.float64)).float().double() * D ** -0.5
    page, lengths, pages_per = 16, [150, 33, 1, 97], 10
    sets = []
    for T in lengths:
        q, k, v = 0.3 * rn(T, H, D), rn(T, G, D), rn(T, G, V)
        k = k / k.norm(dim=-1, keepdim=True)
        for i in range(T):                              # the key that stands out for row i: by turns
            edges = ([i - window + 1, i - window, keep - 1, keep] if window else [0, i // 2, i, i - 31])
            j = edges[i % 4]
            if 0 <= j <= i:
                q[i] = q[i] + (14.0 / D ** -0.5 / 8) * k[j].repeat_interleave(H // G, 0)
        sets.append((r(q), r(k), r(v)))
    refs = [_plain_mixed(q, k, v, mix, factor, cap, window, keep) for q, k, v in sets]
    if window:                                          # a token more or less would show
        for w2, k2 in ((window + 1, keep), (window - 1 or 3, keep), (window, keep + 1)) + (((window, keep - 1),) if keep else ()):
            moved = float((_plain_mixed(*sets[0], mix, factor, cap, w2, k2) - refs[0]).abs().max())
            assert moved > 3 * (1e-2 * float(refs[0].abs().max().clamp(min=1.0)) if half else 3e-5), (w2, k2, moved)
    perm = torch.randperm(4 * pages_per + 3, generator=gen)[:4 * pages_per].reshape(4, pages_per)
    kc = torch.full((4 * pages_per + 3, page, G, D), float("nan"), dtype=dtype, device="cuda")
    vc = torch.full((4 * pages_per + 3, page, G, V), float("nan"), dtype=dtype, device="cuda")
    slots = [3, 1, 0, 2]

    class View:
        pass
    view = View()
    view.k, view.v, view.page_size, view.max_pages = kc, vc, page, pages_per
    view.page_table = _i32(perm.numpy())
    for s, (q, k, v) in enumerate(sets):
        for t in range(lengths[s]):
            p = int(perm[slots[s], t // page])
            kc[p, t % page], vc[p, t % page] = k[t].to(dtype).cuda(), v[t].to(dtype).cuda()

    def call(new, pos0, which):
        ctx = _Step(new, pos0, [slots[s] for s in which])
        pitch = -(-H * D // 8) * 8 + 8
        rows = torch.full((ctx.n_tokens, pitch), float("nan"), dtype=dtype, device="cuda")
        rows[:, :H * D] = torch.cat([sets[s][0][p:p + n].reshape(n, -1) for s, n, p in zip(which, new, pos0)]).to(dtype).cuda()
        out = torch.full((ctx.n_tokens, H * V), float("nan"), dtype=dtype, device="cuda")
        m, f = _dev(mix), _dev(factor)
        if kernel.startswith("plain"):
            ops.mixed_weights_attention(rows, kc, vc, m, f, cap, ctx, view.page_table, pages_per, page, out, H, G, D, V, window, keep)
        elif kernel == "rows":
            scratch = torch.full((41 * H * G * V,), float("nan"), device="cuda")             # slabs of 41 tokens
            ops_tensor.mixed_weights_attention(ctx, rows, view, m, f, cap, out, scratch, H, G, D, V, window, keep)
        else:
            for splits in (1, 3, 40):
                out.fill_(float("nan"))
                scratch = torch.full((ctx.n_seqs * splits * H * (G * V + 2),), float("nan"), device="cuda")
                ops_tensor.mixed_weights_attention(ctx, rows, view, m, f, cap, out, scratch, H, G, D, V, window, keep, step=splits)
                compare(out, new, pos0, which)
        return out

    def compare(out, new, pos0, which):
        want = torch.cat([refs[s][p:p + n] for s, n, p in zip(which, new, pos0)])
        tol = dict(rtol=3e-5, atol=3e-5) if not half else dict(rtol=1e-2, atol=1e-2 * float(want.abs().max().clamp(min=1.0)))
        torch.testing.assert_close(out.double().cpu(), want, **tol)
    if kernel == "step":
        for back in (1, 2, 3, 4, 60):
            which = [s for s in range(4) if lengths[s] >= back]
            call([1] * len(which), [lengths[s] - back for s in which], which)
        return
    for new, pos0, which in (([150, 33, 1, 97], [0, 0, 0, 0], [0, 1, 2, 3]), ([50, 2, 47], [100, 31, 50], [0, 1, 3]), ([3], [147], [0])):
        compare(call(new, pos0, which), new, pos0, which)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,D,V,dims,layout,decay", [(3, 20, 28, 20, "split_half", (0.6, 0.93, 0.995)), (2, 10, 6, 4, "split_half", (1.0, 0.8)),
                                                     (2, 64, 64, 0, "split_half", (0.9, 0.99)), (2, 64, 32, 64, "split_half", (0.97, 0.9995)),
                                                     (1, 128, 48, 96, "interleaved", (0.99,)), (4, 16, 16, 16, "interleaved", (0.5, 0.9, 0.99, 1.0))])
@pytest.mark.parametrize("walk", ["rows", "chunks", "runs", "single"])
def test_retention_walks(walk, dtype, H, D, V, dims, layout, decay):
    """Linear attention without SiLU on turned q and k: two steps of unequal sequences from positions that go on, against
    the statement's recurrence, for every walk of the kernel."""
    from mdma_b200 import ops
    from mdma_b200.parts.rotary import inverse_frequencies
    gen = torch.Generator().manual_seed(13)
    rn = lambda *s: torch.randn(s, generator=gen, dtype=torch.float64)
    cuts = {"single": [[1, 1]] * 6, "runs": [[300, 70], [280, 259]]}.get(walk, [[45, 3], [20, 33]])
    total = [sum(c[s] for c in cuts) for s in range(2)]
    width = H * (2 * D + V)
    rows = [rn(t, width).to(dtype).double() for t in total]
    k_scale, base = D ** -0.5, 50.0
    refs = []
    for x in rows:
        T, pos = x.shape[0], torch.arange(x.shape[0])
        rot = {"dims": dims, "base": base}
        q = pd.rotate(x[:, :H * D].reshape(T, H, D), pos, rot, layout)
        k = pd.rotate(x[:, H * D:2 * H * D].reshape(T, H, D), pos, rot, layout) * k_scale
        v = x[:, 2 * H * D:].reshape(T, H, V)
        S, o = torch.zeros(H, D, V, dtype=torch.float64), torch.empty(T, H, V, dtype=torch.float64)
        dk = torch.tensor(decay, dtype=torch.float64)[:, None, None]
        for t in range(T):
            S = dk * S + k[t][:, :, None] * v[t][:, None, :]
            o[t] = torch.einsum("hdc,hd->hc", S, q[t])
        refs.append(o.reshape(T, H * V))
    table = _dev(inverse_frequencies(dims, base)) if dims else None
    state = torch.zeros(4, H * D * V, device="cuda")
    at, slots = [0, 0], [3, 1]
    for cut in cuts:
        ctx = _Step(cut, at, slots)
        proj = _dev(torch.cat([rows[s][at[s]:at[s] + cut[s]] for s in range(2)]), dtype)
        out = torch.full((ctx.n_tokens, H * V), float("nan"), device="cuda")
        run_rows, most = (128, -(-max(cut) // 128)) if walk == "runs" else (0, 1)
        scratch = torch.full((2 * most * H * D * V,), float("nan"), device="cuda") if run_rows else None
        ops.linear_attention(proj, 0, H * D, 2 * H * D, _dev(torch.tensor(decay)), ctx.seq_start, ctx.seq_slot, state, out, 2, H, D, V,
                             walk in ("chunks", "runs"), run_rows, most, scratch, single=walk == "single", silu=False, k_scale=k_scale,
                             inv_freq=table, rotary_dim=dims, interleaved=layout == "interleaved", tok_pos=ctx.tok_pos)
        want = torch.cat([refs[s][at[s]:at[s] + cut[s]] for s in range(2)])
        torch.testing.assert_close(out.double().cpu(), want, rtol=5e-5, atol=5e-5 * float(want.abs().max()))
        at = [a + c for a, c in zip(at, cut)]


@pytest.mark.gpu
@pytest.mark.parametrize("gate_act", ["sigmoid", "silu"])
@pytest.mark.parametrize("gdtype,odtype", [(torch.float32, torch.float32), (torch.bfloat16, torch.bfloat16)])
@pytest.mark.parametrize("H,V,weighted", [(3, 28, True), (1, 5, False), (16, 128, True), (7, 40, False)])
def test_gated_norm_per_head(H, V, weighted, gdtype, odtype, gate_act):
    from mdma_b200 import ops
    gen = torch.Generator().manual_seed(3)
    n = 19
    o, w = torch.randn(n, H * V, generator=gen), torch.randn(V, generator=gen)
    gate = torch.randn(n, H * V + 3, generator=gen).to(gdtype)
    out = torch.full((n, H * V), float("nan"), dtype=odtype, device="cuda")
    ops.gated_head_rmsnorm(_dev(o), gate.cuda()[:, 3:], _dev(w) if weighted else None, out, n, H, V, 1e-5, gate_act)
    g = gate[:, 3:].double()
    want = pd.rms_unit(o.double().reshape(n, H, V), 1e-5) * (w.double() if weighted else 1.0)
    want = want.reshape(n, H * V) * (pd.silu(g) if gate_act == "silu" else torch.sigmoid(g))
    tol = 1e-5 if odtype == torch.float32 else 1e-2
    torch.testing.assert_close(out.double().cpu(), want, rtol=tol, atol=tol)


@pytest.mark.gpu
@pytest.mark.parametrize("width", [35, 60, 128, 2048, 5120, 9000])
@pytest.mark.parametrize("splits,stored", [(0, True), (3, True), (5, False)])
@pytest.mark.parametrize("copy", [None, torch.bfloat16, torch.float32])
def test_norm_on_a_result_added_with_a_copy_of_the_stream(width, splits, stored, copy):
    """x += norm(y) * w, y whole or as partial sums (alone, or on top of what y holds), and the new x in another dtype."""
    from mdma_b200 import ops
    gen = torch.Generator().manual_seed(7)
    n = 6
    x, y, w = (torch.randn(*s, generator=gen) for s in ((n, width), (n, width), (width,)))
    part = torch.randn(max(splits, 1), n, width, generator=gen)
    only = stored and splits > 0
    full = (torch.zeros_like(y) if only else y).double() + (part.double().sum(0) if splits else 0.0)
    want = x.double() + pd.rms_unit(full, 1e-5) * w.double()
    xd, yd = _dev(x), _dev(torch.full_like(y, float("nan")) if only else y)
    out = None if copy is None else torch.full((n, width), float("nan"), dtype=copy, device="cuda")
    pt = _dev(part) if splits else None
    ops.rmsnorm_add(xd, yd, _dev(w), 1e-5, n, pt, splits, n * width, only, out)
    torch.testing.assert_close(xd.double().cpu(), want, rtol=1e-5, atol=1e-5)
    if out is not None:
        assert torch.equal(out, xd.to(copy))
    rounded = torch.empty(n, width, dtype=torch.bfloat16, device="cuda")
    ops.copy_rows(xd, rounded, n)
    assert torch.equal(rounded, xd.bfloat16())


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("experts,top,W", [(5, 2, 60), (3, 1, 35), (4, 4, 35), (64, 6, 128)])
def test_router_with_a_bias_on_its_logits(dtype, experts, top, W):
    """Choice and weights both follow the biased logits."""
    from mdma_b200 import ops
    gen = torch.Generator().manual_seed(19)
    h, router = torch.randn(33, W, generator=gen).to(dtype), (torch.randn(experts, W, generator=gen) * W ** -0.5).to(dtype)
    bias = (torch.randn(experts, generator=gen) * 4).to(dtype)
    chosen, weights = torch.zeros(33, top, dtype=torch.int32, device="cuda"), torch.zeros(33, top, device="cuda")
    ops.route(_dev(h, dtype), _dev(router, dtype), None, None, 33, top, 1, 1, chosen, weights, None, logit_bias=_dev(bias, dtype))
    z = h.double() @ router.double().T + bias.double()
    best = torch.sort(z, -1, descending=True)
    want = torch.zeros(33, experts, dtype=torch.float64).scatter(1, best.indices[:, :top], torch.softmax(best.values[:, :top], -1))
    got = torch.zeros(33, experts, dtype=torch.float64).scatter(1, chosen.long().cpu(), weights.double().cpu())
    torch.testing.assert_close(got, want, rtol=1e-4, atol=1e-5)


# =====================================================================================================
# Whole models through the engine (GPU).

_models: dict = {}


def model_of(key, dtype, drawn=None, seed=None):
    """(folder, config, float64 tensors as the engine holds them) of configuration `key`."""
    k = (key, dtype)
    if k not in _models:
        store = torch.float32 if dtype == "float32" else torch.bfloat16
        cfg, ranks = drawn or CONFIGS[key]
        d, W = make_model(cfg, ranks, seed if seed is not None else 23 + ord(key[0]), store)
        _models[k] = (d, cfg, W)
    return _models[k]


_refs: dict = {}


def ref_of(key, dtype, ids):
    """(the statement's logits, whether no close routing choice lies at or before a row, how far the row moves)."""
    k = (key, dtype, tuple(ids))
    if k not in _refs:
        _, cfg, W = model_of(key, dtype)
        calls = []
        logits = pd.forward(cfg, W, ids, closeness=calls).numpy()
        gap = torch.stack(calls).min(0).values.numpy() if calls else np.full(len(ids), 9.0)
        gen = torch.Generator().manual_seed(1)
        moves = np.zeros(len(ids))
        for _ in range(2):
            other = {n: t * (1.0 + NOISE * torch.randn(t.shape, generator=gen, dtype=torch.float64)) for n, t in W.items()}
            moves = np.maximum(moves, np.sqrt(((pd.forward(cfg, other, ids).numpy() - logits) ** 2).mean(-1)))
        _refs[k] = (logits, np.minimum.accumulate(gap) > CLOSE_CALL, moves)
    return _refs[k]


def check(got, pairs, dtype, what):
    """`pairs`: per row (reference of `ref_of`, position)."""
    close(got, np.stack([r[0][p] for r, p in pairs]), dtype, what, [r[1][p] for r, p in pairs], [r[2][p] for r, p in pairs])


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("key", ["A", "B", "C", "D"])
def test_every_layer_against_the_plain_statement(key, dtype):
    """The residual stream after every layer run, then the logits; one short prompt, the first tokens among the rows."""
    from mdma_b200.engine import Engine, StepEntry
    d, cfg, W = model_of(key, dtype)
    ids = ids_of(cfg, 29, 4)
    _, trace = pd.forward(cfg, W, ids, return_layers=True)
    ref = ref_of(key, dtype, ids)
    rows = np.nonzero(ref[1])[0] if dtype == "bfloat16" else np.arange(len(ids))
    eng = Engine(d, dtype=dtype, max_batch=2, max_context=64, logit_rows=64, page_size=16)
    got = []
    eng.model.on_layer = lambda n, x: got.append(x.detach().double().cpu())
    s = eng.acquire()
    logits = eng.step([StepEntry(s, ids, list(range(len(ids))))]).cpu().numpy()
    assert len(got) == len(trace) == len(cfg["layers"])
    tol = 1e-4 if dtype == "float32" else 0.05
    for n, (a, b) in enumerate(zip(got, trace)):
        err = float((a - b)[rows].abs().max()) if len(rows) else 0.0
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
    decoded = run([[25] + [1] * 65, [1], [1] * 33, [2], [16, 1]])
    for name, other in (("whole prompts", whole), ("alone", alone), ("portions", pieces), ("decoded", decoded)):
        for i, (got, ref) in enumerate(zip(other, refs)):
            check(got, [(ref, p) for p in range(lengths[i])], dtype, f"{name}, sequence {i}")
            if dtype == "float32":
                assert np.abs(got - whole[i]).max() <= 6e-6, f"{name}, sequence {i}: differs from the whole prompt"


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("key", ["A", "C"])
def test_passes_smaller_than_a_step_and_long_decoding(key, dtype):
    """A step run as passes of 19 tokens (cuts inside sequences), then 150 tokens decoded one by one across many page
    borders and out of the window, beside a batch mate that ends on the way and whose slot another request takes."""
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
            ids.append(int(pd.forward(cfg, W, ids)[-1].argmax()))
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
    """A configuration drawn from a seed: layer kinds in any order, layers with other layers' tensors, head counts and
    sizes of many values, some multiples of 8 or 16 and some not, windows from one token to beyond the prompt."""
    rng = np.random.default_rng(2000 + seed)
    pick = lambda xs: xs[int(rng.integers(len(xs)))]
    width = pick([35, 48, 64, 72, 96, 128])

    def mlp():
        kind = pick(["none", "dense", "moe", "moe"])
        if kind == "none":
            return None
        if kind == "dense":
            return dense(pick([24, 40, 64]))
        n = pick([2, 3, 5, 8])
        return moe(n, int(rng.integers(1, n + 1)), pick([12, 24, 32]), pick([None, 20, 32]))

    def turn(D):
        return pick([None, (D // 2 // 2 * 2 or 2, 1e4), (D, 50.0), (2, 7.0)])
    layers = []
    for i in range(int(rng.integers(2, 7))):
        if i and rng.random() < 0.25:
            j = int(rng.integers(i))
            layers.append({"weights_of": layers[j].get("weights_of", j)})
            continue
        kind = pick(["delta", "attention", "retention"])
        G = pick([1, 2, 3, 4])
        H = G * pick([1, 1, 2, 4])
        if kind == "delta":
            layers.append(delta(H, pick([G, H]), pick([8, 12, 9, 32, 48, 64]), pick([4, 8, 20, 32, 96]), pick([1, 2, 3, 4, 6]), mlp(),
                                ranks=(pick([5, 8, 16, 24]), pick([7, 8, 32]))))
        elif kind == "attention":
            D = pick([8, 16, 32, 48, 10])
            window = pick([0, 1, 5, 16, 40, 500])
            layers.append(attention(H, G, D, pick([6, 8, 16, 24, 64]), float(rng.uniform(0.15, 0.4)), pick([0, 2.5, 20.0]), window,
                                    pick([0, 1, 4, 17]), turn(D), mlp()))
        else:
            D = pick([8, 10, 32, 64])
            layers.append(retention(H, D, pick([4, 6, 24, 64]), [float(rng.uniform(0.5, 1.0)) ** pick([1, 0.01]) for _ in range(H)], turn(D), mlp()))
    return config(int(rng.integers(40, 200)), width, pick([1e-5, 1e-6]), layers)


@pytest.mark.gpu
@pytest.mark.parametrize("seed", range(int(os.environ.get("DEGAVIK_DRAWN_CONFIGS", "14"))))
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
