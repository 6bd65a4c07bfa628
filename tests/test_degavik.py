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
# reference logits, and a row's root-mean-square error as a share of the row's own deviation.
TOL_F32 = 5e-5
TOL_BF16, TOL_ROW_BF16 = 0.12, 0.04
CLOSE_CALL = 0.15        # a bfloat16 row behind a routing choice closer than this may take another expert


def ids_of(cfg, n, seed):
    g = torch.Generator().manual_seed(seed)
    return torch.randint(0, cfg["vocab"], (n,), generator=g).tolist()


def close(got, ref, dtype, what="", calm=None):
    """Logits [rows, vocab] against the statement's.  `calm` [rows] of bool: rows that no close routing choice precedes;
    the others are only asked to be finite in bfloat16."""
    got, ref = np.atleast_2d(np.asarray(got, dtype=np.float64)), np.atleast_2d(np.asarray(ref, dtype=np.float64))
    assert got.shape == ref.shape, (what, got.shape, ref.shape)
    assert np.isfinite(got).all(), f"{what}: logits that are not finite"
    err = np.abs(got - ref)
    if dtype == "float32":
        assert err.max() < TOL_F32, f"{what}: {err.max()}"
        return
    share = err.max(axis=-1) / max(float(ref.std()), 0.25)
    rel = np.sqrt((err ** 2).mean(axis=-1)) / np.maximum(ref.std(axis=-1), 1e-3)
    bad = (share >= TOL_BF16) | (rel >= TOL_ROW_BF16)
    if calm is not None:
        bad &= np.asarray(calm, dtype=bool)
    assert not bad.any(), f"{what}: rows {np.nonzero(bad)[0].tolist()} are off (share {share[bad]}, row error {rel[bad]})"


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
