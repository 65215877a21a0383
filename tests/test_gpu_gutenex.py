"""GPU: layer-described stacks with norms on the sublayers' inputs (lightning attention, the channel-wise delta rule, differential
attention, looped layers) against the plain implementation in gutenex_plain.py, on small configurations with random weights.  Limits
are those of test_gpu_nuzopel.py: a floor plus a multiple of what a disturbance of the size of the rounding does to a row."""
import importlib
import json
import os
import struct
import subprocess
import sys

import numpy as np
import pytest

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import gutenex_plain as plain  # noqa: E402
from test_gpu_nuzopel import DTYPES, FLOOR, Case as BaseCase, check_greedy, on_stream  # noqa: E402

import __graft_entry__ as entry  # noqa: E402

pytestmark = pytest.mark.gpu


@pytest.fixture(scope="module")
def models(ops):
    entry.load_package()
    return importlib.import_module(entry.PKG_NAME + ".models")


@pytest.fixture(scope="module")
def batching(ops):
    return importlib.import_module(entry.PKG_NAME + ".batching")


@pytest.fixture(scope="module")
def wts():
    entry.load_package()
    return importlib.import_module(entry.PKG_NAME + ".weights")


class Case(BaseCase):
    plain_model = plain.PlainModel

    def residual_unit(self, residual):
        return float(np.std(residual))


# ---- configurations and random weights -----------------------------------------------------------------------------------
def entry_of(kind, mixer, ff):
    return dict(type=kind, mixer=mixer, mlp=None if ff is None else dict(kind="dense", ff=ff))


def lightning(heads, dim, vdim, decay=None, ff=None):
    decay = decay if decay is not None else [float(1.0 - 0.6 ** (1 + 2 * h)) for h in range(heads)]
    return entry_of("lightning", dict(heads=heads, dim=dim, vdim=vdim, decay=list(decay)), ff)


def delta(heads, kv_heads, dim, vdim, conv=3, a_rank=7, g_rank=12, ff=None):
    return dict(entry_of("channel_delta", dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, conv=conv), ff), ranks=(a_rank, g_rank))


def diff(heads, kv_heads, dim, vdim, rot, size, keep, lam=0.4, ff=None, base=3000.0, sharp=1.0):
    return entry_of("attention", dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, rot=dict(base=base, dims=rot), mask=dict(size=size, keep_first=keep),
                                      scale=sharp / float(np.sqrt(dim)), diff=lam), ff)


def make(layers, width=80, vocab=97, seed=0, eps=1e-5, softcap=7.0, loop=None):
    layers = json.loads(json.dumps(layers))
    ranks = [L.pop("ranks", None) for L in layers]
    cfg = dict(architecture="Gutenex", layers=layers, width=width, vocab=vocab, norm=dict(eps=eps), logit_softcap=softcap)
    if loop:
        cfg["loop"] = dict(zip(("start", "stop", "times"), loop))
    rng = np.random.default_rng(seed)
    t = {}

    def mat(name, rows, cols, gain=1.0):
        t[name] = rng.standard_normal((rows, cols)).astype(np.float32) * (gain / np.sqrt(cols))

    def vec(name, n, lo=0.5, hi=1.5):
        t[name] = rng.uniform(lo, hi, n).astype(np.float32)
    t["embed"] = rng.standard_normal((vocab, width)).astype(np.float32)
    mat("head", vocab, width, 3.0)
    vec("final.norm", width)
    for i, L in enumerate(layers):
        m, p = L["mixer"], f"l{i}."
        H, D, V = m["heads"], m["dim"], m["vdim"]
        vec(p + "norm1", width)
        mat(p + "mix.o", width, H * V)
        if L["type"] == "lightning":
            for n, r in (("q", H * D), ("k", H * D), ("v", H * V), ("g", H * V)):
                mat(p + "mix." + n, r, width, 1.5)
            vec(p + "mix.norm", H * V)
        elif L["type"] == "channel_delta":
            G = m["kv_heads"]
            for n, r in (("q", G * D), ("k", G * D), ("v", H * V)):
                mat(p + "mix." + n, r, width, 1.5)
                t[p + f"mix.{n}.conv"] = rng.standard_normal((r, m["conv"])).astype(np.float32)
            mat(p + "mix.b", H, width)
            a, g = ranks[i]
            mat(p + "mix.a1", a, width); mat(p + "mix.a2", H * D, a, 2.0); mat(p + "mix.g1", g, width); mat(p + "mix.g2", H * V, g, 2.0)
            vec(p + "mix.A_log", H, -4.0, 1.0); vec(p + "mix.dt_bias", H * D, -4.0, 0.5); vec(p + "mix.norm", V)
        else:
            G = m["kv_heads"]
            mat(p + "mix.q", H * 2 * D, width); mat(p + "mix.k", G * 2 * D, width); mat(p + "mix.v", G * V, width)
            vec(p + "mix.q.norm", D); vec(p + "mix.k.norm", D)
            for n in ("lq1", "lk1", "lq2", "lk2"):
                t[p + "mix." + n] = rng.standard_normal(D).astype(np.float32) * (0.6 / D ** 0.5)
        if L["mlp"] is not None:
            ff = L["mlp"]["ff"]
            vec(p + "norm2", width)
            mat(p + "mlp.gate", ff, width); mat(p + "mlp.up", ff, width); mat(p + "mlp.down", width, ff)
    return cfg, t


LIGHTNING_SIZES = [(2, 64, 64), (3, 128, 128), (3, 40, 72), (1, 96, 160), (4, 16, 8), (5, 24, 132), (2, 130, 20), (1, 300, 36), (1, 64, 256), (1, 1, 3)]
# heads, kv_heads, dim, vdim, conv taps, inner sizes of the gates
DELTA_SIZES = [(2, 2, 128, 128, 4, 32, 24), (4, 2, 64, 64, 3, 7, 12), (3, 1, 40, 72, 2, 5, 9), (2, 2, 96, 160, 4, 16, 16), (4, 4, 16, 8, 5, 8, 3), (1, 1, 24, 132, 1, 1, 2),
               (2, 1, 130, 20, 4, 6, 6), (1, 1, 300, 36, 3, 4, 4), (6, 2, 32, 32, 4, 64, 40), (1, 1, 64, 256, 7, 10, 10)]
# heads, kv_heads, dim, vdim, rotated, window, kept
DIFF_SIZES = [(4, 2, 64, 128, 64, 70, 5), (16, 2, 64, 128, 16, 130, 64), (3, 1, 40, 56, 12, 17, 1), (2, 2, 128, 128, 128, 90, 70), (1, 1, 16, 8, 2, 1, 3), (8, 8, 32, 64, 32, 64, 0),
              (2, 1, 8, 72, 4, 65, 66), (2, 2, 144, 136, 32, 33, 130), (12, 1, 24, 24, 6, 1000, 4), (2, 1, 64, 256, 32, 40, 20), (1, 1, 4, 3, 4, 200, 200), (9, 3, 56, 100, 28, 3, 2)]


def sequence(c, torch, toks, want, many_cuts, what):
    with on_stream(torch):
        c.stack.begin_batching()
        for cuts in many_cuts:
            row = c.stack.open()
            c.judge(c.run(torch, row, toks, cuts), want, f"{what} cuts {cuts}")
            c.stack.retire(row)


# ---- each mechanism alone: a one-layer model without feed-forward -----------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("size", LIGHTNING_SIZES)
def test_lightning_layer(cuda, models, wts, size, dtype):
    c = Case(models, wts, *make([lightning(*size)], seed=11), dtype)
    toks = c.tokens(300)
    sequence(c, cuda, toks, c.expect(toks), ([300], [1], [130, 2, 100], [17]), size)


@pytest.mark.parametrize("dtype", DTYPES)
def test_lightning_decays(cuda, models, wts, dtype):
    """Heads that keep everything, next to everything, little and nothing."""
    c = Case(models, wts, *make([lightning(5, 48, 56, decay=[1.0, 0.9999, 0.7, 1e-3, 0.0])], seed=4), dtype)
    toks = c.tokens(280)
    sequence(c, cuda, toks, c.expect(toks), ([280], [1], [129, 2, 31]), "decays")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("size", DELTA_SIZES)
def test_channel_delta_layer(cuda, models, wts, size, dtype):
    c = Case(models, wts, *make([delta(*size)], seed=12), dtype)
    toks = c.tokens(300)
    sequence(c, cuda, toks, c.expect(toks), ([300], [1], [130, 2, 100], [17], [2], [64, 3, 1, 1, 61]), size)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("a_log,dt", [(2.5, 3.0), (-9.0, -6.0), (0.0, -2.0)])
def test_channel_delta_decay_extremes(cuda, models, wts, a_log, dt, dtype):
    """Channels that forget at once (their decays multiply to zero inside a chunk), hardly at all, and both side by side."""
    cfg, t = make([delta(2, 2, 48, 64, 4, 8, 8)], seed=5)
    t["l0.mix.A_log"][:] = a_log
    t["l0.mix.dt_bias"][:] = dt
    t["l0.mix.dt_bias"][::3] = -12.0
    c = Case(models, wts, cfg, t, dtype)
    toks = c.tokens(200, 3)
    sequence(c, cuda, toks, c.expect(toks), ([200], [1], [65, 2, 63]), "decays")


@pytest.mark.parametrize("dtype", DTYPES)
def test_channel_delta_repeated_key(cuda, models, wts, dtype):
    """One token over and over writes the same key: the rule replaces its value instead of adding to it."""
    cfg, t = make([delta(2, 1, 64, 64, 1, 8, 8)], seed=6)
    t["l0.mix.b"] *= 4.0
    t["l0.mix.A_log"][:] = -6.0
    c = Case(models, wts, cfg, t, dtype)
    toks = np.repeat(c.tokens(30, 2), 8)
    sequence(c, cuda, toks, c.expect(toks), ([240], [1], [100, 64, 2]), "repeated key")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("size", DIFF_SIZES)
def test_diff_layer(cuda, models, wts, size, dtype):
    c = Case(models, wts, *make([diff(*size, sharp=2.0)], seed=13), dtype)
    toks = c.tokens(330)
    sequence(c, cuda, toks, c.expect(toks), ([330], [1], [63, 2, 3, 130], [50]), size)


@pytest.mark.parametrize("dtype", DTYPES)
def test_diff_constants(cuda, models, wts, dtype):
    """Lambda far from its constant, negative, and no constant at all."""
    for lam, gain in ((0.0, 1.0), (0.8, 3.0), (0.2, -2.0)):
        cfg, t = make([diff(4, 2, 48, 40, 24, 50, 3, lam=lam)], seed=9)
        t["l0.mix.lk1"] *= gain
        c = Case(models, wts, cfg, t, dtype)
        toks = c.tokens(90)
        sequence(c, cuda, toks, c.expect(toks), ([90], [1]), f"lambda {lam}")


@pytest.mark.parametrize("dtype", DTYPES)
def test_feed_forward_head_and_softcap(cuda, models, wts, dtype):
    for ff, width, cap in ((200, 72, 2.0), (33, 50, 30.0), (256, 2304, 8.0)):
        c = Case(models, wts, *make([lightning(1, 8, 8, ff=ff)], width=width, softcap=cap, seed=7), dtype)
        toks = c.tokens(40)
        sequence(c, cuda, toks, c.expect(toks), ([40], [1]), f"ff {ff} width {width}")


# ---- loops ------------------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("loop", [(0, 3, 2), (1, 2, 3), (2, 4, 2), (0, 1, 4), (3, 4, 1), None])
def test_loops(cuda, models, wts, loop, dtype):
    """Every pass has a cache and states of its own; the embedding output is added ahead of each but the first."""
    layers = [diff(2, 1, 24, 32, 8, 30, 4, ff=40), lightning(2, 16, 24), delta(2, 1, 16, 24), diff(2, 2, 16, 16, 16, 9, 2)]
    c = Case(models, wts, *make(layers, seed=14, loop=loop), dtype)
    toks = c.tokens(100)
    sequence(c, cuda, toks, c.expect(toks), ([100], [1], [33, 2, 40]), f"loop {loop}")


def test_layer_runs_one_by_one(cuda, models, wts):
    """The residual stream behind every layer run of a looped model."""
    layers = [diff(2, 1, 24, 32, 8, 30, 4, ff=40), lightning(2, 16, 24), delta(2, 1, 16, 24, ff=24)]
    c = Case(models, wts, *make(layers, seed=15, loop=(1, 3, 3)), "float32")
    toks, trace = c.tokens(70), []
    c.plain.forward(c.plain.start(), toks, trace)
    assert len(trace) == 7
    with on_stream(cuda):
        c.stack.begin_batching()
        for n in range(1, 8):
            c.stack.stop_after(n)
            row = c.stack.open()
            got = c.run(cuda, row, toks, [70])[1]
            c.stack.retire(row)
            assert np.abs(got - trace[n - 1]).max() < 2e-4 * np.std(trace[n - 1]), f"behind run {n}"
        c.stack.stop_after(-1)


# ---- the edges of a window and of the kept positions, with one key that stands out ------------------------------------------------
def standout_case(size, seed=3):
    """One attention layer in which a query of token 1 scores far above everything else on a key of token 0, in map 1."""
    heads, kv, dim, vdim, rot, window, keep = size
    cfg, t = make([diff(*size, lam=0.1)], seed=seed, width=96)
    e, eps = t["embed"].astype(np.float64), cfg["norm"]["eps"]
    h0, h1 = (plain.rms_norm(e[i], t["l0.norm1"], eps) for i in (0, 1))
    q = t["l0.mix.q"].reshape(heads, 2, dim, -1)
    k = t["l0.mix.k"].reshape(kv, 2, dim, -1)
    at = rot                                          # a dimension that does not turn
    for g in range(kv):                               # token 0 puts all of its map-1 key there
        k[g, 0] -= np.outer(k[g, 0] @ h0, h0) / (h0 @ h0)
        k[g, 0, at] += np.sqrt(dim) * h0 / (h0 @ h0)
    for h in range(heads):
        q[h, 0] -= np.outer(q[h, 0] @ h1, h1) / (h1 @ h1)
        q[h, 0, at] += np.sqrt(dim) * h1 / (h1 @ h1)
    t["l0.mix.q.norm"][:] = 1.0
    t["l0.mix.k.norm"][:] = 1.0
    cfg["layers"][0]["mixer"]["scale"] = 14.0 / dim   # both are sqrt(dim) long
    return cfg, t


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("window,keep", [(2, 1), (40, 3), (63, 64), (64, 0), (65, 65), (128, 2), (129, 63), (200, 100)])
@pytest.mark.parametrize("size", [(4, 2, 64, 128, 32), (2, 1, 24, 40, 8)])
def test_window_edge(cuda, models, wts, size, window, keep, dtype):
    """A key just inside and just outside the window, behind the kept positions and as the last of them."""
    c = Case(models, wts, *standout_case((*size, window, keep)), dtype)
    mask = c.plain.c["layers"][0]["mixer"]["mask"]
    for key in sorted({keep, keep + 1, keep + 61, 127 + keep} | ({0, keep - 1} if keep else set())):
        n = key + window + 4
        toks = 2 + c.tokens(n, key) % (c.vocab - 2)
        toks[key] = 0
        toks[key + window - 1] = 1          # sees the key in its last place
        toks[key + window] = 1              # only if it is kept
        want = c.expect(toks)
        # an edge that is one off shows in the yardstick itself
        edges = [dict(keep_first=key)] if key == keep - 1 else [dict(size=window + 1), dict(keep_first=keep + 1)][:2 if key == keep else 1] if key >= keep else []
        for off in edges:
            old = dict(mask)
            mask.update(off)
            assert np.sqrt(np.mean((c.expect(toks)[1][key + window] - want[1][key + window]) ** 2)) > 20 * FLOOR[dtype] * np.std(want[1])
            mask.update(old)
        sequence(c, cuda, toks, want, ([n], [1], [max(2, key + window - 1), 2], [key + 1, window - 1 or 1, 1]), f"key {key}")


@pytest.mark.parametrize("dtype", DTYPES)
def test_far_and_kept_keys_across_pages(cuda, models, wts, dtype):
    """A key hundreds of positions back, inside a wide window or among the kept ones, reached in a prompt and in decoding."""
    for window, keep in ((700, 2), (70, 150)):
        c = Case(models, wts, *standout_case((4, 2, 64, 128, 32, window, keep)), dtype)
        for key, at in ((0, 600), (63, 640), (64, 511), (130, 829)):
            toks = 2 + c.tokens(at + 2, key) % (c.vocab - 2)
            toks[key], toks[at] = 0, 1
            sequence(c, cuda, toks, c.expect(toks), ([at + 2], [at - 1, 1], [at, 2]), f"key {key} at {at}")


@pytest.mark.parametrize("dtype", DTYPES)
def test_lightning_remembers_one_token(cuda, models, wts, dtype):
    """One token writes strongly where the others hardly do: its value must come back hundreds of tokens later."""
    cfg, t = make([lightning(2, 64, 64, decay=[0.9995, 0.9999])], seed=8)
    h0 = plain.rms_norm(t["embed"][0].astype(np.float64), t["l0.norm1"], cfg["norm"]["eps"])
    across = h0 * t["l0.norm1"]              # the other tokens have no part in token 0's direction
    t["embed"][1:] -= np.outer(t["embed"][1:] @ across, across) / (across @ across)
    t["l0.mix.k"] = (0.05 * t["l0.mix.k"] + np.outer(np.full(128, 6.0), h0 / (h0 @ h0))).astype(np.float32)
    c = Case(models, wts, cfg, t, dtype)
    toks = 1 + c.tokens(520) % (c.vocab - 1)
    forgotten = c.expect(toks)
    toks[5] = 0
    want = c.expect(toks)
    assert np.sqrt(np.mean((want[1][500] - forgotten[1][500]) ** 2)) > 0.1 * np.std(want[1])
    sequence(c, cuda, toks, want, ([520], [128, 256, 1], [100, 3, 200]), "memory")


@pytest.mark.parametrize("dtype", DTYPES)
def test_channel_delta_remembers_one_token(cuda, models, wts, dtype):
    """One token has a large beta and a value of its own, the others nearly none; half of the channels hardly decay."""
    cfg, t = make([delta(2, 2, 64, 64, 2, 8, 8)], seed=8)
    h0 = plain.rms_norm(t["embed"][0].astype(np.float64), t["l0.norm1"], cfg["norm"]["eps"])
    t["l0.mix.b"] = (0.05 * t["l0.mix.b"] + np.outer(np.full(2, 6.0), h0 / (h0 @ h0))).astype(np.float32)
    t["l0.mix.A_log"][:] = -5.0
    t["l0.mix.dt_bias"][:] = -6.0
    c = Case(models, wts, cfg, t, dtype)
    toks = 1 + c.tokens(520) % (c.vocab - 1)
    forgotten = c.expect(toks)
    toks[405] = 0
    want = c.expect(toks)
    assert np.sqrt(np.mean((want[1][500] - forgotten[1][500]) ** 2)) > 0.02 * np.std(want[1])
    sequence(c, cuda, toks, want, ([520], [128, 278, 1], [100, 3, 200]), "memory")


# ---- whole models ---------------------------------------------------------------------------------------------------------------
def whole_layers():
    return [diff(4, 2, 40, 56, 12, 37, 5, ff=96), lightning(2, 64, 128), delta(4, 2, 64, 128, 4, 16, 24), lightning(3, 24, 40, ff=64),
            diff(6, 2, 64, 128, 64, 64, 70), delta(3, 3, 32, 40, 3, ff=70)]


LOOP = (1, 4, 2)


@pytest.mark.parametrize("dtype", DTYPES)
def test_whole_model_portions(cuda, models, wts, dtype):
    c = Case(models, wts, *make(whole_layers(), seed=21, loop=LOOP), dtype)
    toks = c.tokens(410)
    sequence(c, cuda, toks, c.expect(toks), ([410], [1], [2], [64], [200, 1, 2, 63, 65, 3, 1]), "model")


@pytest.mark.parametrize("dtype", DTYPES)
def test_layers_of_different_sizes_share_the_working_buffers(cuda, models, wts, dtype):
    mixed = [lightning(7, 8, 200, ff=40), diff(5, 1, 40, 72, 8, 50, 3), delta(2, 2, 128, 96, 4, 40, 8), lightning(3, 20, 130), diff(9, 9, 8, 24, 4, 33, 9, ff=90),
             delta(1, 1, 140, 300, 2), lightning(4, 64, 40), delta(5, 5, 24, 60, 4, 3, 30)]
    c = Case(models, wts, *make(mixed, width=72, seed=31), dtype)
    toks = c.tokens(180)
    sequence(c, cuda, toks, c.expect(toks), ([180], [1], [60, 1, 1, 30, 2, 1], [180], [17, 1]), "mixed")


@pytest.mark.parametrize("dtype", DTYPES)
def test_first_tokens_and_single_token(cuda, models, wts, dtype):
    c = Case(models, wts, *make(whole_layers(), seed=22, loop=LOOP), dtype)
    for n in (1, 2, 3, 5):
        toks = c.tokens(n, n)
        sequence(c, cuda, toks, c.expect(toks), ([n], [1]), f"{n} tokens")


@pytest.mark.parametrize("dtype", DTYPES)
def test_slots_and_pages_are_reused_clean(cuda, models, wts, dtype):
    """Few pages: sequences come and go, interleaved, and each gets what it gets alone."""
    c = Case(models, wts, *make(whole_layers(), seed=23, loop=LOOP), dtype, max_seqs=3, max_seq_len=256, num_pages=7)
    seqs = {k: c.tokens(n, 100 + k) for k, n in enumerate((150, 64, 65, 190, 31, 128))}
    want = {k: c.expect(v) for k, v in seqs.items()}
    with on_stream(cuda):
        c.stack.begin_batching()
        rows, got = [], {k: [] for k in seqs}

        def feed(k, n):
            at = sum(len(g[0]) for g in got[k])
            got[k].append(c.run(cuda, rows.index(k), seqs[k][at:at + n], [n]))

        def close(k):
            r = rows.index(k)
            c.stack.retire(r)
            last = rows.pop()
            if r < len(rows):
                rows[r] = last

        for k in (0, 1, 2):
            rows.append(k); c.stack.open()
        feed(0, 100); feed(1, 64); feed(2, 40); feed(0, 1); feed(2, 25); feed(0, 49)
        close(1)
        rows.append(4); c.stack.open()
        feed(4, 31)
        close(0); close(2)
        rows.append(3); c.stack.open()
        feed(3, 189); feed(3, 1)
        close(4); close(3)
        rows.append(5); c.stack.open()
        feed(5, 128)
        for k in seqs:
            c.judge(tuple(np.concatenate(p) for p in zip(*got[k])), want[k], f"sequence {k}")


# ---- batches, the captured step, generation ----------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
def test_generation_through_the_scheduler(cuda, models, wts, batching, dtype):
    """More requests than rows, unequal lengths, the captured step over all rows; each as if alone."""
    c = Case(models, wts, *make(whole_layers(), seed=24, loop=LOOP), dtype, max_seqs=3, max_seq_len=320)
    prompts = [c.tokens(n, 50 + n).tolist() for n in (5, 130, 64, 1, 77, 200)]
    with on_stream(cuda):
        got = batching.generate(c.stack, prompts, 24)
        assert c.stack.device_status() == 0
        for p, g in zip(prompts, got):
            assert len(g) == 24
            check_greedy(c, p, g)
        alone = batching.generate(c.stack, prompts[1:2], 24)[0]
    if dtype == "float32":
        assert alone == got[1]


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding(cuda, models, wts, batching, dtype):
    c = Case(models, wts, *make(whole_layers(), seed=25, loop=LOOP), dtype, max_seqs=2, max_seq_len=500)
    prompt = c.tokens(9).tolist()
    with on_stream(cuda):
        got = batching.generate(c.stack, [prompt, prompt[:4]], 400)
    check_greedy(c, prompt, got[0])
    check_greedy(c, prompt[:4], got[1])


@pytest.mark.parametrize("dtype", DTYPES)
def test_batched_prefill_and_decode(cuda, models, wts, dtype):
    """Plain (not continuous) batches: equal prompts in one pass, the captured step against eager decode."""
    c = Case(models, wts, *make(whole_layers(), seed=26, loop=LOOP), dtype, max_seqs=4, max_seq_len=200, max_pass_rows=300)
    prompts = np.stack([c.tokens(130, k) for k in range(4)])
    with on_stream(cuda):
        t = cuda.tensor(prompts, dtype=cuda.int32, device="cuda")
        toks = [c.stack.forward_batch_prefill(t).clone()]
        for _ in range(4):
            toks.append(c.stack.forward_batch_decode(toks[-1]).clone())
        eager = cuda.stack(toks, 1).cpu().numpy()
        c.stack.reset_cache()
        c.stack.set_tokens(c.stack.forward_batch_prefill(t))
        c.stack.capture_decode(4)
        toks = [c.stack.get_tokens(4).clone()]
        for _ in range(4):
            c.stack.launch_decode(1)
            toks.append(c.stack.get_tokens(4).clone())
        assert (cuda.stack(toks, 1).cpu().numpy() == eager).all()
        assert c.stack.device_status() == 0
    for k in range(4):
        check_greedy(c, prompts[k], eager[k])


def test_trace_and_generate_programs(cuda, models, wts, tmp_path):
    """bin/trace_run and bin/generate on a model folder written here."""
    cfg, t = make(whole_layers(), seed=27, loop=LOOP)
    c = Case(models, wts, cfg, t, "float32")
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    head, blob = {}, b""
    for k, v in c.bits.items():
        head[k] = dict(dtype="BF16", shape=list(v.shape), data_offsets=[len(blob), len(blob) + v.nbytes])
        blob += v.tobytes()
    j = json.dumps(head).encode()
    (tmp_path / "model.safetensors").write_bytes(struct.pack("<Q", len(j)) + j + blob)
    toks = [int(x) for x in c.tokens(70)]
    steps = [dict(step=0, entries=[dict(id="a", tokens=toks[:50], want=[49, 3])], end=[]), dict(step=1, entries=[dict(id="a", tokens=toks[50:51], want=[])], end=[]),
             dict(step=2, entries=[dict(id="a", tokens=toks[51:], want=[0])], end=["a"]), dict(step=3, entries=[dict(id="b", tokens=toks[:2], want=[1])], end=["b"])]
    p = subprocess.run([os.path.join(entry.ROOT, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", "float32", "--out", str(tmp_path),
                        "--max-tokens", "128"], input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, timeout=280)
    assert p.returncode == 0, p.stderr[-2000:]
    want = c.expect(toks)[0]
    for step, places in ((0, [49, 3]), (2, [51]), (3, [1])):
        got = np.fromfile(tmp_path / f"{step}.f32", "<f4").reshape(len(places), -1)
        assert np.abs(got - want[places]).max() < 1e-3 * np.std(want)
    p = subprocess.run([os.path.join(entry.ROOT, "bin", "generate"), "--model", str(tmp_path), "--dtype", "float32", "--max-new-tokens", "6"],
                       input=json.dumps(toks[:20]) + "\n" + json.dumps(toks[:3]) + "\n", capture_output=True, text=True, timeout=280)
    assert p.returncode == 0, p.stderr[-2000:]
    out = [json.loads(x) for x in p.stdout.strip().split("\n")[-2:]]
    check_greedy(c, toks[:20], out[0])
    check_greedy(c, toks[:3], out[1])
