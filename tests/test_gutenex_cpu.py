"""CPU: layer descriptions of looped stacks with norms on the sublayers' inputs, and the plain implementation itself (portions against
whole runs, recurrences against their sums; a mistake planted in it must move its outputs, or it could not show one in the product)."""
import ctypes as C
import importlib
import json
import os
import sys

import numpy as np
import pytest

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import gutenex_plain as plain  # noqa: E402
from test_gpu_gutenex import delta, diff, lightning, make, standout_case  # noqa: E402

import __graft_entry__ as entry  # noqa: E402


@pytest.fixture(scope="module")
def models():
    entry.load_package()
    return importlib.import_module(entry.PKG_NAME + ".models")


def shapes(t):
    return {k: v.shape for k, v in t.items()}


def test_layer_descriptions_take_every_size_from_the_config_and_the_tensors(models, ops):
    cfg, t = make([lightning(3, 24, 40, decay=[0.5, 0.25, 1.0], ff=33), delta(6, 3, 20, 28, conv=5, a_rank=11, g_rank=17), diff(8, 2, 36, 44, 10, 77, 9, lam=0.3, base=123.0, ff=50)])
    a, b, c = models.gutenex_layers(cfg, shapes(t), ops)
    assert (a.mixer, a.heads, a.dim, a.vdim, a.ff, a.act) == (ops.MIXER_LIGHTNING, 3, 24, 40, 33, ops.ACT_SILU) and list(a.decay[:3]) == [0.5, 0.25, 1.0]
    assert (b.mixer, b.heads, b.kv_heads, b.dim, b.vdim, b.conv_taps, b.a_rank, b.g_rank, b.ff) == (ops.MIXER_CHANNEL_DELTA, 6, 3, 20, 28, 5, 11, 17, 0)
    assert (c.mixer, c.heads, c.kv_heads, c.dim, c.vdim, c.rot_dim, c.window, c.keep_first, c.rot_base, c.diff, c.ff) == (ops.MIXER_DIFF, 8, 2, 36, 44, 10, 77, 9, 123.0, 0.3, 50)
    assert c.scale == cfg["layers"][2]["mixer"]["scale"]


@pytest.mark.parametrize("change,match", [(dict(type="conv"), "unknown type"), (dict(mlp=dict(kind="sparse", ff=4)), "unknown feed-forward")])
def test_unknown_parts_of_a_config_are_refused(models, ops, change, match):
    cfg, t = make([lightning(1, 8, 8)])
    cfg["layers"][0].update(change)
    with pytest.raises(ValueError, match=match):
        models.gutenex_layers(cfg, shapes(t), ops)


def test_one_decay_per_head(models, ops):
    cfg, t = make([lightning(2, 8, 8, decay=[0.5, 0.5])])
    cfg["layers"][0]["mixer"]["decay"] = [0.5]
    with pytest.raises(ValueError, match="decays"):
        models.gutenex_layers(cfg, shapes(t), ops)


def test_bad_descriptions_are_rejected_without_a_device(ops):
    h, f = C.c_void_p(), ops.lib().b200attn_stack_create_layers
    cfg = ops.ModelConfig(64, 10, 1, 64, 0, 0, ops.DTYPE_F32, 1e-6, 1.0, 1.0, 5.0, 1, 1, 0, 0, 1)
    for d in (ops.LayerDesc(mixer=ops.MIXER_LIGHTNING, heads=1, dim=8, vdim=8), ops.LayerDesc(mixer=ops.MIXER_CHANNEL_DELTA, heads=3, kv_heads=2, dim=8, vdim=8, conv_taps=4, a_rank=4, g_rank=4),
              ops.LayerDesc(mixer=ops.MIXER_DIFF, heads=2, kv_heads=1, dim=8, vdim=8, rot_dim=10), ops.LayerDesc(mixer=ops.MIXER_DIFF, heads=2, kv_heads=0, dim=8, vdim=8)):
        assert f(C.byref(cfg), C.byref(d), 1, C.byref(h)) == ops.ERR_INVALID


# ---- the yardstick ---------------------------------------------------------------------------------------------------------------
def layers():
    return [diff(3, 1, 20, 16, 8, 13, 2, ff=40, sharp=3.0), lightning(2, 16, 24), delta(2, 1, 12, 16, 3, 5, 6), lightning(2, 8, 8, ff=24)]


def test_layer_runs():
    cfg, _ = make(layers(), loop=(1, 3, 3))
    assert plain.layer_runs(cfg) == [(0, False), (1, False), (2, False), (1, True), (2, False), (1, True), (2, False), (3, False)]
    cfg.pop("loop")
    assert plain.layer_runs(cfg) == [(i, False) for i in range(4)]


@pytest.mark.parametrize("loop", [None, (1, 4, 2)])
def test_plain_portions_equal_the_whole(loop):
    cfg, t = make(layers(), seed=2, loop=loop)
    m = plain.PlainModel(cfg, t)
    toks = np.random.default_rng(3).integers(0, cfg["vocab"], 70)
    whole = m.forward(m.start(), toks)
    for cuts in ([1] * 70, [2] * 35, [13, 1, 30, 26], [69, 1]):
        seq, out, at = m.start(), [], 0
        for n in cuts:
            out.append(m.forward(seq, toks[at:at + n]))
            at += n
        assert np.abs(np.concatenate(out) - whole).max() < 1e-10 * np.abs(whole).max()


def test_plain_constant_decay_against_its_sum():
    rng = np.random.default_rng(4)
    T, H, D, V = 30, 2, 5, 4
    q, k, v, dec = rng.standard_normal((T, H, D)), rng.standard_normal((T, H, D)), rng.standard_normal((T, H, V)), np.array([0.9, 0.3])
    o, _ = plain.decay_recurrence(q, k, v, dec)
    for t in range(T):
        for h in range(H):
            w = dec[h] ** (t - np.arange(t + 1)) * (k[:t + 1, h] @ q[t, h])
            assert np.allclose(o[t, h], w @ v[:t + 1, h], rtol=1e-9, atol=1e-12)


def test_plain_delta_rule_against_its_triangular_form():
    """The writes of a run of tokens solve a unit lower triangular system whose entries carry the decays between two tokens."""
    rng = np.random.default_rng(5)
    T, D, V = 24, 6, 5
    unit = lambda x: x / np.linalg.norm(x, axis=-1, keepdims=True)
    q, k, v = unit(rng.standard_normal((T, 1, D))), unit(rng.standard_normal((T, 1, D))), rng.standard_normal((T, 1, V))
    g, beta = rng.uniform(0.3, 1.0, (T, 1, D)), rng.uniform(0.1, 0.9, (T, 1))
    S0 = rng.standard_normal((1, D, V))
    o, S = plain.channel_delta_recurrence(q, k, v, g, beta, S0)
    G = np.cumsum(np.log(g[:, 0]), 0)
    dot = lambda a, t, s: np.sum(a[t, 0] * k[s, 0] * np.exp(G[t] - G[s]))
    A = np.array([[beta[t, 0] * dot(k, t, s) if s < t else 0.0 for s in range(T)] for t in range(T)])
    rhs = beta * (v[:, 0] - (k[:, 0] * np.exp(G)) @ S0[0])
    U = np.linalg.solve(np.eye(T) + A, rhs)
    M = np.array([[dot(q, t, s) if s <= t else 0.0 for s in range(T)] for t in range(T)])
    assert np.allclose(o[:, 0], (q[:, 0] * np.exp(G)) @ S0[0] + M @ U, rtol=1e-9, atol=1e-11)
    assert np.allclose(S[0], np.exp(G[-1])[:, None] * S0[0] + (k[:, 0] * np.exp(G[-1] - G)).T @ U, rtol=1e-9, atol=1e-11)


def test_visible_positions():
    see = plain.visible(np.arange(12), np.arange(12), 4, 2)
    assert list(np.flatnonzero(see[9])) == [0, 1, 6, 7, 8, 9]
    assert list(np.flatnonzero(see[1])) == [0, 1]
    assert list(np.flatnonzero(plain.visible(np.array([9]), np.arange(12), 4, 0)[0])) == [6, 7, 8, 9]


@pytest.mark.parametrize("mistake", ["window", "keep_first", "rotation_layout", "rotation_base", "lambda", "diff_factor", "one_map", "decay", "kv_group", "lost_state", "lost_conv",
                                     "decay_per_head", "read_before_write", "unit_norm", "embedding_again", "pass_cache", "softcap", "norm_eps_place", "head_norms"])
def test_a_planted_mistake_shows_in_the_yardstick(mistake, monkeypatch):
    base = [diff(4, 2, 20, 16, 8, 13, 2, ff=40, sharp=3.0), lightning(2, 16, 24), delta(4, 2, 12, 16, 3, 5, 6), lightning(2, 8, 8, ff=24)]
    cfg, t = make(base, seed=5, eps=0.05, loop=(1, 3, 2))
    toks = np.random.default_rng(6).integers(0, cfg["vocab"], 60)
    m = plain.PlainModel(cfg, t)
    want = m.forward(m.start(), toks)
    bad = json.loads(json.dumps(cfg))
    mix = [L["mixer"] for L in bad["layers"]]
    if mistake == "window":
        mix[0]["mask"]["size"] += 1
    elif mistake == "keep_first":
        mix[0]["mask"]["keep_first"] -= 1
    elif mistake == "rotation_layout":          # halves instead of neighbours
        monkeypatch.setattr(plain, "rotate_pairs", lambda x, pos, base, dims, f=plain.rotate_pairs: f(x[..., np.r_[0:dims:2, 1:dims:2, dims:x.shape[-1]]], pos, base, dims))
    elif mistake == "rotation_base":
        mix[0]["rot"]["base"] *= 2.0
    elif mistake == "lambda":
        monkeypatch.setattr(plain, "diff_lambda", lambda W, c: c["diff"])
    elif mistake == "diff_factor":
        t = dict(t, **{"l0.mix.o": t["l0.mix.o"] / (1.0 - mix[0]["diff"])})
    elif mistake == "one_map":
        monkeypatch.setattr(plain, "diff_lambda", lambda W, c: 0.0)
    elif mistake == "decay":
        mix[1]["decay"][0] *= 0.97
    elif mistake == "kv_group":
        t = dict(t, **{"l2.mix.k": np.roll(t["l2.mix.k"], 12, 0), "l2.mix.k.conv": np.roll(t["l2.mix.k.conv"], 12, 0)})
    elif mistake == "decay_per_head":
        t = dict(t, **{"l2.mix.dt_bias": np.repeat(t["l2.mix.dt_bias"].reshape(4, 12).mean(1), 12)})
    elif mistake == "read_before_write":
        def late(q, k, v, g, beta, S=None, f=plain.channel_delta_recurrence):
            o, S1 = f(q, k, v, g, beta, S)
            return o - np.einsum("thd,thd->th", q, k)[..., None] * (beta[..., None] * v), S1
        monkeypatch.setattr(plain, "channel_delta_recurrence", late)
    elif mistake == "unit_norm":
        monkeypatch.setattr(plain, "unit", lambda x: x)
    elif mistake == "embedding_again":
        monkeypatch.setattr(plain, "layer_runs", lambda c, f=plain.layer_runs: [(i, False) for i, _ in f(c)])
    elif mistake == "softcap":
        bad["logit_softcap"] = 1e6
    elif mistake == "norm_eps_place":
        monkeypatch.setattr(plain, "rms_norm", lambda x, w, eps: x / (np.sqrt(np.mean(x * x, -1, keepdims=True)) + eps) * w)
    elif mistake == "head_norms":               # every head of a lightning layer normed by itself
        def by_head(h, W, c, eps, S=None, r=plain.exact):
            T, H, V = h.shape[0], c["heads"], c["vdim"]
            q, k, v = (plain.silu(h @ W[n].T).reshape(T, H, -1) for n in "qkv")
            o, S = plain.decay_recurrence(q, k, v, np.asarray(c["decay"]), S)
            return plain.rms_unit(o, eps).reshape(T, H * V) * W["norm"] * plain.sigmoid(h @ W["g"].T) @ W["o"].T, S
        monkeypatch.setattr(plain, "lightning_mixer", by_head)
    m = plain.PlainModel(bad, t)
    if mistake in ("lost_state", "lost_conv", "pass_cache"):
        seq = m.start()
        m.forward(seq, toks[:30])
        if mistake == "lost_state":
            seq["runs"][1] = None
        elif mistake == "lost_conv":
            seq["runs"][2]["v"][:] = 0.0
        else:                                   # the second pass reads the first one's state
            seq["runs"][3] = seq["runs"][1]
        got = np.concatenate([want[:30], m.forward(seq, toks[30:])])
    else:
        got = m.forward(m.start(), toks)
    assert np.abs(got - want).max() > 2e-2 * np.std(want)


def test_standout_key_decides_the_edges():
    cfg, t = standout_case((2, 1, 24, 40, 8, 20, 3))
    m = plain.PlainModel(cfg, t)
    mask = cfg["layers"][0]["mixer"]["mask"]
    toks = 2 + np.random.default_rng(1).integers(0, cfg["vocab"] - 2, 40)
    toks[5], toks[24], toks[25] = 0, 1, 1
    want = []
    m.forward(m.start(), toks, want)
    for change, at in ((dict(size=19), 24), (dict(size=21), 25), (dict(keep_first=6), 25)):
        old = dict(mask)
        mask.update(change)
        got = []
        m.forward(m.start(), toks, got)
        mask.update(old)
        assert np.sqrt(np.mean((got[-1][at] - want[-1][at]) ** 2)) > 0.2
