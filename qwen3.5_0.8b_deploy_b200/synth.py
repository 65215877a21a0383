"""Seeded synthetic weights and inputs for the attention hot path.

Every test, fixture and benchmark draws from here so the CPU checker and the GPU path see the
same bits.  The distributions are the ones the workload definitions state: matrices ~ N(0, 0.02),
hidden states ~ N(0, 1), A_log ~ U(0, 2.7), dt_bias ~ N(0, 0.1), q/k norm weights 0 (they enter as
1 + w), DeltaNet norm weight 1.  Generator: numpy Philox, keyed by (seed, stream name).
"""
from __future__ import annotations

import zlib

import numpy as np

HIDDEN = 1024
FA_HEADS, FA_KV_HEADS, FA_HEAD_DIM, FA_ROTARY = 8, 2, 256, 64
ROPE_THETA = 1e7
LA_HEADS, LA_KD, LA_VD, LA_CONV_K = 16, 128, 128, 4
LA_CONV_DIM = LA_HEADS * (2 * LA_KD + LA_VD)          # 6144
FFN_INTER = 3584
VOCAB = 248320
NUM_LAYERS = 24


def is_full_attention_layer(i: int) -> bool:
    """Layers 3, 7, ..., 23 are gated full attention; the other 18 are Gated DeltaNet
    (src/backend/cpu/core/common/language_common.hpp:36-53 in the reference)."""
    return i % 4 == 3


def rng(seed: int, name: str) -> np.random.Generator:
    return np.random.Generator(np.random.Philox(key=[seed, zlib.crc32(name.encode())]))


def normal(seed, name, shape, std=1.0):
    return (rng(seed, name).standard_normal(shape, dtype=np.float32) * np.float32(std)).astype(np.float32)


def fa_weights(seed: int, tag: str = "fa") -> dict:
    """W_q [4096,1024] (per head: 256 q rows then 256 gate rows), W_k/W_v [512,1024],
    q_norm/k_norm [256], W_o [1024,2048]; row-major (out, in)."""
    return dict(
        wq=normal(seed, tag + ".wq", (FA_HEADS * FA_HEAD_DIM * 2, HIDDEN), 0.02),
        wk=normal(seed, tag + ".wk", (FA_KV_HEADS * FA_HEAD_DIM, HIDDEN), 0.02),
        wv=normal(seed, tag + ".wv", (FA_KV_HEADS * FA_HEAD_DIM, HIDDEN), 0.02),
        q_norm=np.zeros(FA_HEAD_DIM, np.float32),
        k_norm=np.zeros(FA_HEAD_DIM, np.float32),
        wo=normal(seed, tag + ".wo", (HIDDEN, FA_HEADS * FA_HEAD_DIM), 0.02),
    )


def la_weights(seed: int, tag: str = "la") -> dict:
    """W_qkv [6144,1024], W_a/W_b [16,1024], W_z [2048,1024], conv [6144,4], A_log/dt_bias [16],
    norm [128], W_out [1024,2048]."""
    return dict(
        w_qkv=normal(seed, tag + ".w_qkv", (LA_CONV_DIM, HIDDEN), 0.02),
        w_a=normal(seed, tag + ".w_a", (LA_HEADS, HIDDEN), 0.02),
        w_b=normal(seed, tag + ".w_b", (LA_HEADS, HIDDEN), 0.02),
        w_z=normal(seed, tag + ".w_z", (LA_HEADS * LA_VD, HIDDEN), 0.02),
        conv_w=normal(seed, tag + ".conv_w", (LA_CONV_DIM, LA_CONV_K), 0.02),
        a_log=rng(seed, tag + ".a_log").uniform(0.0, 2.7, LA_HEADS).astype(np.float32),
        dt_bias=normal(seed, tag + ".dt_bias", (LA_HEADS,), 0.1),
        norm_w=np.ones(LA_VD, np.float32),
        w_out=normal(seed, tag + ".w_out", (HIDDEN, LA_HEADS * LA_VD), 0.02),
    )


def ffn_weights(seed: int, tag: str) -> dict:
    return dict(
        gate=normal(seed, tag + ".gate", (FFN_INTER, HIDDEN), 0.02),
        up=normal(seed, tag + ".up", (FFN_INTER, HIDDEN), 0.02),
        down=normal(seed, tag + ".down", (HIDDEN, FFN_INTER), 0.02),
    )


def hidden_states(seed: int, name: str, rows: int) -> np.ndarray:
    return normal(seed, name, (rows, HIDDEN), 1.0)


def gutenex_tensors(config: dict, ranks: tuple, seed: int, std: float = 0.02) -> dict:
    """Random weights of a Gutenex configuration under the names a model file has: matrices ~ N(0, std), norms 1, short
    convolutions ~ N(0, 0.5), decay gates around e^-0.05 per token; `ranks` are the inner sizes of the decay and output gates."""
    w, vocab = config["width"], config["vocab"]
    out = {"embed": normal(seed, "embed", (vocab, w), std), "head": normal(seed, "head", (vocab, w), std), "final.norm": np.ones(w, np.float32)}
    for i, layer in enumerate(config["layers"]):
        m, p = layer["mixer"], f"l{i}."
        heads, dim, vdim = m["heads"], m["dim"], m["vdim"]
        shapes = {"o": (w, heads * vdim)}
        if layer["type"] == "lightning":
            shapes.update(q=(heads * dim, w), k=(heads * dim, w), v=(heads * vdim, w), g=(heads * vdim, w))
            out[p + "mix.norm"] = np.ones(heads * vdim, np.float32)
        elif layer["type"] == "channel_delta":
            kv, a, g = m["kv_heads"], *ranks
            shapes.update(q=(kv * dim, w), k=(kv * dim, w), v=(heads * vdim, w), b=(heads, w), a1=(a, w), a2=(heads * dim, a), g1=(g, w), g2=(heads * vdim, g))
            for n in "qkv":
                out[p + f"mix.{n}.conv"] = normal(seed, p + n + ".conv", (shapes[n][0], m["conv"]), 0.5)
            out.update({p + "mix.A_log": np.zeros(heads, np.float32), p + "mix.dt_bias": np.full(heads * dim, -3.0, np.float32),
                        p + "mix.norm": np.ones(vdim, np.float32)})
        else:
            kv = m["kv_heads"]
            shapes.update(q=(heads * 2 * dim, w), k=(kv * 2 * dim, w), v=(kv * vdim, w))
            out.update({p + f"mix.{n}.norm": np.ones(dim, np.float32) for n in "qk"})
            out.update({p + "mix." + n: normal(seed, p + n, (dim,), 0.05) for n in ("lq1", "lk1", "lq2", "lk2")})
        for n, shape in shapes.items():
            out[p + "mix." + n] = normal(seed, p + "mix." + n, shape, std)
        out[p + "norm1"] = np.ones(w, np.float32)
        if layer["mlp"] is not None:
            ff = layer["mlp"]["ff"]
            out[p + "norm2"] = np.ones(w, np.float32)
            for n, shape in (("gate", (ff, w)), ("up", (ff, w)), ("down", (w, ff))):
                out[p + "mlp." + n] = normal(seed, p + "mlp." + n, shape, std)
    return out


def nuzopel_tensors(config: dict, seed: int, std: float = 0.02) -> dict:
    """Random weights of a Nuzopel configuration under the names a model file has: matrices ~ N(0, std), norms 1, gate biases
    0 (input) and 3 (forget)."""
    out = {"embed": normal(seed, "embed", (config["vocab"], config["width"]), std), "final.norm": np.ones(config["width"], np.float32)}
    w = config["width"]
    for i, layer in enumerate(config["layers"]):
        m, p = layer["mixer"], f"l{i}."
        heads, dim, vdim = m["heads"], m["dim"], m["vdim"]
        if layer["type"] == "mlstm":
            shapes = {"q": (heads * dim, w), "k": (heads * dim, w), "v": (heads * vdim, w), "g": (heads * vdim, w), "o": (w, heads * vdim), "i": (heads, w),
                      "f": (heads, w)}
            out.update({p + "mix.norm": np.ones(heads * vdim, np.float32), p + "mix.i.b": np.zeros(heads, np.float32),
                        p + "mix.f.b": np.full(heads, 3.0, np.float32)})
        else:
            rot, rank = m["rot_dim"], m["kv_rank"]
            shapes = {"q": (heads * (dim + rot), w), "uk": (heads * dim, rank), "uv": (heads * vdim, rank), "o": (w, heads * vdim)}
            if m.get("kv_from") is None:
                shapes["dkv"] = (rank + rot, w)
                out[p + "mix.dkv.norm"] = np.ones(rank, np.float32)
        for n, shape in shapes.items():
            out[p + "mix." + n] = normal(seed, p + "mix." + n, shape, std)
        out[p + "norm1"] = np.ones(w, np.float32)
        if layer["mlp"] is not None:
            ff = layer["mlp"]["ff"]
            out[p + "norm2"] = np.ones(w, np.float32)
            for n, shape in (("gate", (ff, w)), ("up", (ff, w)), ("down", (w, ff))):
                out[p + "mlp." + n] = normal(seed, p + "mlp." + n, shape, std)
    return out
