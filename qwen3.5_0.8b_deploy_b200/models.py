"""Model registry: config.json's "architecture" selects the entry that turns a configuration into a stack.

An entry is a function (config, limits, shapes) -> stack, where `shapes` names the model's tensors with their shapes; `load_tensors`
gives the stack its weights.  Both kinds of stack share prefill, decode, capture and continuous batching (ops.Stack), so everything above works on either.
"""
from __future__ import annotations

import ctypes
import os
from dataclasses import dataclass

import numpy as np

from . import weights


@dataclass
class Limits:
    """What the serving process wants to hold: sequences, tokens per sequence, cache pages (0 = all sequences at full length),
    tokens per prefill pass (0 = default) and the element type."""
    max_seqs: int = 8
    max_seq_len: int = 4096
    num_pages: int = 0
    max_pass_rows: int = 0
    dtype: str = "bfloat16"


REGISTRY: dict = {}


def register(architecture: str):
    def add(builder):
        REGISTRY[architecture] = builder
        return builder
    return add


def _ops():
    from . import ops
    return ops


# ---- Nuzopel: mLSTM and latent-attention layers, norms on the sublayers' outputs --------------------------------------------
def nuzopel_layers(config: dict, ops) -> list:
    out = []
    for i, layer in enumerate(config["layers"]):
        m, mlp = layer["mixer"], layer["mlp"]
        d = ops.LayerDesc(heads=m["heads"], dim=m["dim"], vdim=m["vdim"], kv_from=-1)
        if layer["type"] == "mlstm":
            d.mixer, d.gate_cap = ops.MIXER_MLSTM, m["gate_cap"]
        elif layer["type"] == "latent_attention":
            if m["rot"]["dims"] != m["rot_dim"]:
                raise ValueError(f"layer {i}: rot.dims {m['rot']['dims']} differs from rot_dim {m['rot_dim']}")
            d.mixer, d.kv_rank, d.rot_dim = ops.MIXER_LATENT, m["kv_rank"], m["rot_dim"]
            d.window, d.rot_base, d.scale = m["mask"]["size"], m["rot"]["base"], m["scale"]
            if m.get("kv_from") is not None:
                d.kv_from = m["kv_from"]
        else:
            raise ValueError(f"layer {i}: unknown type {layer['type']!r}")
        if mlp is not None:
            if mlp["kind"] != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward {mlp['kind']!r}")
            d.ff = mlp["ff"]
        out.append(d)
    return out


@register("Nuzopel")
def build_nuzopel(config: dict, limits: Limits, shapes: dict):
    ops = _ops()
    cfg = ops.ModelConfig(config["width"], config["vocab"], limits.max_seqs, limits.max_seq_len, limits.num_pages, limits.max_pass_rows,
                          {"bfloat16": ops.DTYPE_BF16, "float32": ops.DTYPE_F32}[limits.dtype],
                          config["norm"]["eps"], config["embedding"]["scale"], config["logit_scale"])
    return ops.LayerStack(cfg, nuzopel_layers(config, ops))


# ---- Gutenex: lightning, channel-wise delta rule and differential attention, norms on the sublayers' inputs, looped layers ---
def gutenex_layers(config: dict, shapes: dict, ops) -> list:
    """`shapes`: tensor name -> shape; it alone gives the inner sizes of the low-rank gates."""
    out = []
    for i, layer in enumerate(config["layers"]):
        m, mlp = layer["mixer"], layer["mlp"]
        d = ops.LayerDesc(heads=m["heads"], dim=m["dim"], vdim=m["vdim"], kv_from=-1, act=ops.ACT_SILU)
        if layer["type"] == "lightning":
            if len(m["decay"]) != m["heads"]:
                raise ValueError(f"layer {i}: {len(m['decay'])} decays for {m['heads']} heads")
            d.mixer = ops.MIXER_LIGHTNING
            d.decay = (ctypes.c_double * m["heads"])(*m["decay"])
        elif layer["type"] == "channel_delta":
            d.mixer, d.kv_heads, d.conv_taps = ops.MIXER_CHANNEL_DELTA, m["kv_heads"], m["conv"]
            d.a_rank, d.g_rank = (shapes[f"l{i}.mix.{n}"][0] for n in ("a1", "g1"))
        elif layer["type"] == "attention":
            d.mixer, d.kv_heads, d.scale, d.diff = ops.MIXER_DIFF, m["kv_heads"], m["scale"], m["diff"]
            d.window, d.keep_first = m["mask"].get("size") or 0, m["mask"].get("keep_first") or 0
            d.rot_dim, d.rot_base = m["rot"]["dims"], m["rot"]["base"]
        else:
            raise ValueError(f"layer {i}: unknown type {layer['type']!r}")
        if mlp is not None:
            if mlp["kind"] != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward {mlp['kind']!r}")
            d.ff = mlp["ff"]
        out.append(d)
    return out


@register("Gutenex")
def build_gutenex(config: dict, limits: Limits, shapes: dict):
    ops = _ops()
    loop = config.get("loop") or dict(start=0, stop=0, times=1)
    cfg = ops.ModelConfig(config["width"], config["vocab"], limits.max_seqs, limits.max_seq_len, limits.num_pages, limits.max_pass_rows,
                          {"bfloat16": ops.DTYPE_BF16, "float32": ops.DTYPE_F32}[limits.dtype], config["norm"]["eps"], 1.0, 1.0,
                          config["logit_softcap"], 1, 1, loop["start"], loop["stop"], loop["times"])
    return ops.LayerStack(cfg, gutenex_layers(config, shapes, ops))


# ---- the hybrid stack: Gated DeltaNet and gated full attention ---------------------------------------------------------------
@register("Qwen3_5Hybrid")
def build_hybrid(config: dict, limits: Limits, shapes: dict):
    """Keys: num_layers, intermediate_size, vocab_size, rms_eps, kv_dtype ("fp16" or "int8"), int8_weights."""
    ops = _ops()
    if limits.dtype != "bfloat16":
        raise ValueError("the hybrid stack serves 16-bit weights and activations only")
    return ops.HybridStack(config["num_layers"], config["intermediate_size"], config["vocab_size"], limits.max_seqs, limits.max_seq_len,
                           max(1, (limits.max_pass_rows or limits.max_seq_len) // limits.max_seq_len),
                           ops.KV_INT8 if config.get("kv_dtype") == "int8" else ops.KV_FP16, bool(config.get("int8_weights", False)),
                           config.get("rms_eps", 1e-6))


def load_tensors(stack, tensors: dict) -> None:
    """Gives a stack its weights.  Layer-described stacks take the tensors by their own names; the hybrid stack reads
    "layers.<i>.<input_norm|post_norm>", "layers.<i>.ffn.<gate|up|down>", "layers.<i>.<fa|la>.<name>", "embed", "final_norm"."""
    ops = _ops()

    def f32(a):
        return weights.bf16_to_f32(a) if a.dtype == np.uint16 else np.asarray(a, np.float32)
    if isinstance(stack, ops.LayerStack):
        for name, a in tensors.items():
            stack.set_tensor(name, a)
        return
    for i in range(stack.cfg.num_layers):
        def group(prefix):
            p = f"layers.{i}.{prefix}"
            return {k[len(p):]: f32(v) for k, v in tensors.items() if k.startswith(p)}
        norms = {k: f32(tensors[f"layers.{i}.{k}"]) for k in ("input_norm", "post_norm")}
        stack.set_layer_weights(i, norms, group("ffn."), fa=group("fa.") or None, la=group("la.") or None)
    stack.set_embedding(f32(tensors["embed"]), f32(tensors["final_norm"]))


def build_model(config: dict, limits: Limits, shapes: dict | None = None):
    arch = config.get("architecture")
    if arch not in REGISTRY:
        raise ValueError(f"unknown architecture {arch!r}; known: {sorted(REGISTRY)}")
    return REGISTRY[arch](config, limits, shapes or {})


def load_model(folder: str, limits: Limits):
    """config.json and model.safetensors of `folder` -> a stack ready to run."""
    tensors = weights.read_safetensors(os.path.join(folder, "model.safetensors"))
    stack = build_model(weights.read_config(folder), limits, {k: v.shape for k, v in tensors.items()})
    load_tensors(stack, tensors)
    return stack
