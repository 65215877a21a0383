"""CPU: the model registry, the reader of model folders, and the plain implementation itself (portions against whole runs;
a mistake planted in it must move its outputs, or it could not show one in the product)."""
import importlib
import json
import os
import struct
import sys

import numpy as np
import pytest

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import nuzopel_plain as plain  # noqa: E402
from test_gpu_nuzopel import latent, make, mlstm, standout_case  # noqa: E402

import __graft_entry__ as entry  # noqa: E402


@pytest.fixture(scope="module")
def models():
    entry.load_package()
    return importlib.import_module(entry.PKG_NAME + ".models")


@pytest.fixture(scope="module")
def weights():
    entry.load_package()
    return importlib.import_module(entry.PKG_NAME + ".weights")


def write_safetensors(path, tensors):
    head, blob = {"__metadata__": {"format": "x"}}, b""
    names = {np.dtype(np.uint16): "BF16", np.dtype(np.float32): "F32", np.dtype(np.int32): "I32"}
    for k, v in tensors.items():
        head[k] = dict(dtype=names[v.dtype], shape=list(v.shape), data_offsets=[len(blob), len(blob) + v.nbytes])
        blob += v.tobytes()
    j = json.dumps(head).encode()
    j += b" " * (-len(j) % 8)
    path.write_bytes(struct.pack("<Q", len(j)) + j + blob)


def test_safetensors_reader(weights, tmp_path):
    rng = np.random.default_rng(0)
    t = dict(a=rng.standard_normal((3, 5)).astype(np.float32), b=weights.bf16_bits(rng.standard_normal((7, 2)).astype(np.float32)),
             c=np.arange(4, dtype=np.int32))
    write_safetensors(tmp_path / "m.safetensors", t)
    got = weights.read_safetensors(str(tmp_path / "m.safetensors"))
    assert set(got) == set(t)
    for k in t:
        assert got[k].dtype == t[k].dtype and (got[k] == t[k]).all()


def test_bf16_conversion_rounds_to_nearest_even(weights):
    import torch
    x = np.concatenate([np.random.default_rng(1).standard_normal(1000).astype(np.float32), np.float32([1.00390625, 1.01171875, 0.0, -0.0, 65280.0])])
    want = torch.from_numpy(x).to(torch.bfloat16)
    got = weights.bf16_bits(x)
    assert (got.view(np.int16) == want.view(torch.int16).numpy()).all()
    assert (weights.bf16_to_f32(got) == want.float().numpy()).all()


def test_registry_knows_both_designs(models):
    assert {"Nuzopel", "Qwen3_5Hybrid"} <= set(models.REGISTRY)
    with pytest.raises(ValueError, match="unknown architecture"):
        models.build_model(dict(architecture="nothing"), models.Limits())


def test_layer_descriptions_take_every_size_from_the_config(models, ops):
    cfg, _ = make([mlstm(3, 24, 40, cap=7.5, ff=33), latent(5, 20, 12, 28, 36, 77, base=123.0), latent(2, 8, 12, 16, 36, 9, ff=50, kv_from=1)])
    a, b, c = models.nuzopel_layers(cfg, ops)
    assert (a.mixer, a.heads, a.dim, a.vdim, a.gate_cap, a.ff) == (ops.MIXER_MLSTM, 3, 24, 40, 7.5, 33)
    assert (b.mixer, b.heads, b.dim, b.rot_dim, b.vdim, b.kv_rank, b.window, b.kv_from, b.rot_base, b.ff) == (ops.MIXER_LATENT, 5, 20, 12, 28, 36, 77, -1, 123.0, 0)
    assert b.scale == cfg["layers"][1]["mixer"]["scale"]
    assert (c.kv_from, c.window, c.ff) == (1, 9, 50)


@pytest.mark.parametrize("change,match", [(dict(type="conv"), "unknown type"), (dict(mlp=dict(kind="sparse", ff=4)), "unknown feed-forward")])
def test_unknown_parts_of_a_config_are_refused(models, ops, change, match):
    cfg, _ = make([mlstm(1, 8, 8)])
    cfg["layers"][0].update(change)
    with pytest.raises(ValueError, match=match):
        models.nuzopel_layers(cfg, ops)


def test_rotation_of_part_of_the_rotated_key_is_refused(models, ops):
    cfg, _ = make([latent(1, 8, 8, 8, 8, 8)])
    cfg["layers"][0]["mixer"]["rot"]["dims"] = 4
    with pytest.raises(ValueError, match="rot.dims"):
        models.nuzopel_layers(cfg, ops)


def test_bad_stack_descriptions_are_rejected_without_a_device(ops):
    import ctypes as C
    h = C.c_void_p()
    f = ops.lib().b200attn_stack_create_layers
    cfg = ops.ModelConfig(64, 10, 1, 64, 0, 0, ops.DTYPE_F32, 1e-6, 1.0, 1.0)
    d = ops.LayerDesc(mixer=ops.MIXER_MLSTM, heads=1, dim=8, vdim=8, gate_cap=1.0, kv_from=-1)
    assert f(None, C.byref(d), 1, C.byref(h)) == ops.ERR_INVALID
    assert f(C.byref(cfg), C.byref(d), 0, C.byref(h)) == ops.ERR_INVALID
    cfg.width = 0
    assert f(C.byref(cfg), C.byref(d), 1, C.byref(h)) == ops.ERR_INVALID
    cfg.width, cfg.dtype = 64, 9
    assert f(C.byref(cfg), C.byref(d), 1, C.byref(h)) == ops.ERR_INVALID
    cfg.dtype, d.heads = ops.DTYPE_F32, 0
    assert f(C.byref(cfg), C.byref(d), 1, C.byref(h)) == ops.ERR_INVALID
    assert ops.lib().b200attn_stack_set_tensor(None, b"embed", None, 0, 1, 1) == ops.ERR_INVALID


# ---- the yardstick ---------------------------------------------------------------------------------------------------------------
def layers():
    return [latent(3, 20, 8, 16, 24, 13, ff=40), mlstm(2, 16, 24), latent(2, 12, 8, 16, 24, 30, kv_from=0), mlstm(2, 8, 8, ff=24)]


def test_plain_portions_equal_the_whole():
    cfg, t = make(layers(), seed=2)
    m = plain.PlainModel(cfg, t)
    toks = np.random.default_rng(3).integers(0, cfg["vocab"], 70)
    whole = m.forward(m.start(), toks)
    for cuts in ([1] * 70, [2] * 35, [13, 1, 30, 26], [69, 1]):
        seq, out, at = m.start(), [], 0
        for n in cuts:
            out.append(m.forward(seq, toks[at:at + n]))
            at += n
        assert np.abs(np.concatenate(out) - whole).max() < 1e-10 * np.abs(whole).max()


def test_plain_recurrence_against_its_sum():
    """The stabilised recurrence is a weighted sum over earlier tokens with the running maximum divided out."""
    rng = np.random.default_rng(4)
    T, H, D, V = 40, 2, 6, 5
    q, k, v = rng.standard_normal((T, H, D)), rng.standard_normal((T, H, D)), rng.standard_normal((T, H, V))
    ig, fg = 3 * rng.standard_normal((T, H)), plain.log_sigmoid(3 * rng.standard_normal((T, H)))
    o, _ = plain.mlstm_recurrence(q, k, v, ig, fg)
    F = np.cumsum(fg, 0)
    for t in range(T):
        for h in range(H):
            w = np.exp(F[t, h] - F[:t + 1, h] + ig[:t + 1, h])
            dots = k[:t + 1, h] @ q[t, h]
            m = max([0.0 + F[t, h]] + [F[t, h] - F[s, h] + ig[s, h] for s in range(t + 1)])
            den = max(abs((w * dots).sum()), 1.0) + 1e-6 * np.exp(m)
            assert np.allclose(o[t, h], (w * dots) @ v[:t + 1, h] / den, rtol=1e-9, atol=1e-12)


@pytest.mark.parametrize("mistake", ["window", "rotation", "q_scale", "gate_cap", "kv_from", "lost_state", "norm_eps_place"])
def test_a_planted_mistake_shows_in_the_yardstick(mistake, monkeypatch):
    cfg, t = make(layers(), seed=5, eps=0.2)
    for x in (1, 3):
        t[f"l{x}.mix.i.b"][0] -= 3.0    # one head with a small state: e^-m bounds its divisor and eps counts, else the norms hide factors
    toks = np.random.default_rng(6).integers(0, cfg["vocab"], 60)
    want = plain.PlainModel(cfg, t)
    want = want.forward(want.start(), toks)
    bad = json.loads(json.dumps(cfg))
    if mistake == "window":
        bad["layers"][0]["mixer"]["mask"]["size"] += 1
    elif mistake == "rotation":
        monkeypatch.setattr(plain, "rotate_half", lambda x, pos, base: x)
    elif mistake == "q_scale":
        for x in (1, 3):
            t[f"l{x}.mix.q"] = t[f"l{x}.mix.q"] * 0.5
    elif mistake == "gate_cap":         # gates that are not capped
        for x in (1, 3):
            bad["layers"][x]["mixer"]["gate_cap"] = 1e6
    elif mistake == "kv_from":
        bad["layers"][2]["mixer"].pop("kv_from")
        t["l2.mix.dkv"], t["l2.mix.dkv.norm"] = t["l0.mix.dkv"], t["l0.mix.dkv.norm"]
    elif mistake == "norm_eps_place":
        monkeypatch.setattr(plain, "rms_unit", lambda x, eps: x / (np.sqrt(np.mean(x * x, -1, keepdims=True)) + eps))
    m = plain.PlainModel(bad, t)
    if mistake == "lost_state":
        seq = m.start()
        m.forward(seq, toks[:30])
        seq["layers"][1] = None
        got = np.concatenate([want[:30], m.forward(seq, toks[30:])])
    else:
        got = m.forward(m.start(), toks)
    assert np.abs(got - want).max() > 2e-2 * np.std(want)


def test_standout_key_decides_the_window_edge():
    cfg, t = standout_case((2, 24, 8, 40, 32, 20))
    m = plain.PlainModel(cfg, t)
    toks = 2 + np.random.default_rng(1).integers(0, cfg["vocab"] - 2, 40)
    toks[5], toks[24], toks[25] = 0, 1, 1
    want = []
    m.forward(m.start(), toks, want)
    for size, at in ((19, 24), (21, 25)):
        cfg["layers"][0]["mixer"]["mask"]["size"] = size
        got = []
        m.forward(m.start(), toks, got)
        assert np.sqrt(np.mean((got[-1][at] - want[-1][at]) ** 2)) > 0.2
