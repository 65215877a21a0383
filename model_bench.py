"""Prefill and decode throughput of layer-described models beside the hybrid stack at equal size (bench.py --workload nuzopel
or gutenex).

Every case runs both stacks with the same width, feed-forward, vocabulary, number of layers, batch and lengths: random weights,
random token ids, one prefill pass over the batch's prompts and captured decode steps behind it, timed with CUDA events after
warm-up.  The kernels that matter are timed by class (prefill kernels with event pairs, decode kernels with in-kernel stamps
inside the captured step) and set against the measured copy bandwidth and sustained GEMM rate."""
from __future__ import annotations

import importlib

import numpy as np

import __graft_entry__ as entry

WINDOW = 1024
# width, ff, vocabulary, layers (every fourth one attention), batch, prompt, generated tokens, hybrid stack beside it
CASES = [dict(name="width 1024, batch 128", width=1024, ff=3584, vocab=32768, layers=8, batch=128, prompt=1024, gen=128, hybrid=True),
         dict(name="width 1024, batch 16", width=1024, ff=3584, vocab=32768, layers=8, batch=16, prompt=1024, gen=128, hybrid=True),
         dict(name="width 1024, batch 4, prompt 4096", width=1024, ff=3584, vocab=32768, layers=8, batch=4, prompt=4096, gen=128, hybrid=True),
         dict(name="width 2048, batch 64", width=2048, ff=5632, vocab=32768, layers=8, batch=64, prompt=1024, gen=128, hybrid=False)]


def nuzopel_config(c: dict) -> dict:
    heads = c["width"] // 64
    mlp = dict(kind="dense", ff=c["ff"])
    layers = []
    for i in range(c["layers"]):
        if i % 4 == 3:
            m = dict(heads=heads, dim=128, rot_dim=64, vdim=128, kv_rank=512, mask=dict(size=WINDOW), rot=dict(base=1e4, dims=64), scale=192 ** -0.5)
            if i > 3:
                m["kv_from"] = 3
            layers.append(dict(type="latent_attention", mixer=m, mlp=mlp))
        else:
            layers.append(dict(type="mlstm", mixer=dict(heads=heads, dim=128, vdim=128, gate_cap=15.0), mlp=mlp))
    return dict(architecture="Nuzopel", width=c["width"], vocab=c["vocab"], layers=layers, norm=dict(eps=1e-6), embedding=dict(scale=1.0), logit_scale=1.0)


def build_nuzopel(pkg, models, c):
    st = models.build_model(nuzopel_config(c), models.Limits(c["batch"], c["prompt"] + c["gen"], 0, c["batch"] * c["prompt"], "bfloat16"))
    models.load_tensors(st, pkg.synth.nuzopel_tensors(nuzopel_config(c), 1234))
    return st


KEEP, GATE_RANKS = 64, (128, 128)


def gutenex_config(c: dict) -> dict:
    """Every fourth layer differential attention, the others channel-wise delta rule, lightning, channel-wise delta rule; every layer
    with a feed-forward, no loop: as many layers, heads and cached values per token as the hybrid stack beside it."""
    heads = c["width"] // 64
    mlp = dict(kind="dense", ff=c["ff"])
    layers = []
    for i in range(c["layers"]):
        if i % 4 == 3:
            layers.append(dict(type="attention", mlp=mlp, mixer=dict(heads=heads, kv_heads=heads // 4, dim=64, vdim=128, scale=64 ** -0.5, diff=0.5,
                                                                     mask=dict(size=WINDOW, keep_first=KEEP), rot=dict(base=1e4, dims=32))))
        elif i % 4 == 1:
            layers.append(dict(type="lightning", mlp=mlp, mixer=dict(heads=heads, dim=128, vdim=128, decay=[1.0 - 2.0 ** (-3 - h % 8) for h in range(heads)])))
        else:
            layers.append(dict(type="channel_delta", mlp=mlp, mixer=dict(heads=heads, kv_heads=heads, dim=128, vdim=128, conv=4)))
    return dict(architecture="Gutenex", width=c["width"], vocab=c["vocab"], layers=layers, norm=dict(eps=1e-6), logit_softcap=30.0)


def build_gutenex(pkg, models, c):
    cfg = gutenex_config(c)
    t = pkg.synth.gutenex_tensors(cfg, GATE_RANKS, 1234)
    st = models.build_model(cfg, models.Limits(c["batch"], c["prompt"] + c["gen"], 0, c["batch"] * c["prompt"], "bfloat16"), {k: v.shape for k, v in t.items()})
    models.load_tensors(st, t)
    return st


BUILDERS = dict(nuzopel=build_nuzopel, gutenex=build_gutenex)


def build_hybrid(pkg, ops, c):
    st = ops.HybridStack(c["layers"], c["ff"], c["vocab"], c["batch"], c["prompt"] + c["gen"],
                         -(-c["batch"] * c["prompt"] // (c["prompt"] + c["gen"])), ops.KV_FP16, False)
    z = np.zeros(1024, np.float32)
    for i in range(c["layers"]):
        ffn = {k: pkg.synth.normal(1, f"L{i}.{k}", (1024, c["ff"]) if k == "down" else (c["ff"], 1024), 0.02) for k in ("gate", "up", "down")}
        fa = pkg.synth.fa_weights(1, f"L{i}.fa") if i % 4 == 3 else None
        st.set_layer_weights(i, dict(input_norm=z, post_norm=z), ffn, fa=fa, la=None if fa else pkg.synth.la_weights(1, f"L{i}.la"))
    st.init_embedding_random(1, 0.02, z)
    return st


def window_pairs(length: int, window: int | None) -> float:
    w = min(window or length, length)
    return w * (w + 1) / 2 + (length - w) * w


def kernel_work(kind: str, c: dict) -> dict:
    """Algorithmic work per launch: (bound, amount) of each kernel class."""
    B, P, ctx = c["batch"], c["prompt"], c["prompt"] + c["gen"] // 2
    if kind == "hybrid":
        chunks = -(-P // 64)
        return dict(la_prefill=("tensor", B * 16 * chunks * (5 * 2 * 64 * 64 * 128 + 3 * 2 * 64 * 128 * 128 + 64 ** 3 / 3)),
                    fa_prefill=("tensor", B * 8 * 2 * 2 * 256 * window_pairs(P, None)),
                    la_decode=("hbm", B * (2 * 16 * 128 * 128 * 4 + 2 * 3 * 6144 * 4 + 8224 * 4 + 2048 * 2)),
                    fa_decode=("hbm", B * (2048.0 * ctx + 8 * 256 * 6)))
    H = c["width"] // 64
    if kind == "gutenex":
        chunks = -(-P // 64)
        return dict(la_prefill=("tensor", B * H * chunks * (2 * 2 * 64 * 64 * 128 + 2 * 2 * 64 * 128 * 128)),
                    delta_prefill=("tensor", B * H * chunks * (5 * 2 * 64 * 64 * 128 + 3 * 2 * 64 * 128 * 128 + 64 ** 3 / 3)),
                    fa_prefill=("tensor", B * H * 2 * 2 * (64 + 128) * window_pairs(P, WINDOW)),
                    la_decode=("hbm", B * H * (2 * 128 * 128 * 4 + 3 * 128 * 4 + 128 * 4)),
                    delta_decode=("hbm", B * H * (2 * (128 * 128 + 3 * 3 * 128) * 4 + (3 * 128 + 1) * 4 + 2 * 128 * 4 + 128 * 2)),
                    fa_decode=("hbm", B * (min(WINDOW, ctx) * (H // 4) * 256 * 2 + (H // 4) * 16 * 128 * 2 + H * 128 * 2)))
    return dict(la_prefill=("tensor", B * H * -(-P // 64) * (2 * 2 * 64 * 64 * 128 + 2 * 2 * 64 * 128 * 128)),     # QK^T, PV, Q S, K^T V in chunks of 64
                fa_prefill=("tensor", B * H * 2 * (192 + 128) * window_pairs(P, WINDOW)),
                la_decode=("hbm", B * (2 * H * (128 * 128 + 128 + 1) * 4 + H * (4 * 128 + 2) * 4 + H * 128 * 2)),
                fa_decode=("hbm", B * (min(WINDOW, ctx) * 576 * 2 + H * (576 + 512) * 2)))


def measure(torch, ops, st, kind: str, c: dict, peaks: dict, steps: int) -> dict:
    B, P, G = c["batch"], c["prompt"], c["gen"]
    s = torch.cuda.current_stream()
    toks = torch.randint(0, c["vocab"], (B, P), dtype=torch.int32, device="cuda")

    def ev():
        return torch.cuda.Event(enable_timing=True)

    st.reset_cache()
    st.forward_batch_decode(st.forward_batch_prefill(toks))
    st.capture_decode(B)
    pre, dec = [], []
    for i in range(3 + steps):
        a, b, d = ev(), ev(), ev()
        st.reset_cache()
        a.record(s)
        st.set_tokens(st.forward_batch_prefill(toks))
        b.record(s)
        st.launch_decode(G)
        d.record(s)
        s.synchronize()
        if i >= 3:
            pre.append(a.elapsed_time(b)); dec.append(b.elapsed_time(d) / G)
    st.reset_cache()
    ops.profile_reset(); ops.profile_enable(True)
    st.set_tokens(st.forward_batch_prefill(toks))
    s.synchronize()
    t = {n: ops.profile_read(n) for n in ("la_prefill", "delta_prefill", "fa_prefill")}
    ops.profile_reset()
    st.capture_decode(B)
    ops.profile_enable(False)
    st.launch_decode(G // 2)
    s.synchronize()
    acc = {n: [0.0, 0] for n in ("la_decode", "delta_decode", "fa_decode")}
    for n in acc:
        ops.profile_read(n)
    for _ in range(8):
        st.launch_decode(1)
        s.synchronize()
        for n in acc:
            ms, k = ops.profile_read(n)
            acc[n][0] += ms; acc[n][1] += k
    t.update(acc)
    st.capture_decode(B)
    ops.profile_reset()
    status = st.device_status()
    assert status == 0, f"device status {status}"
    kernels = {}
    for n, (bound, work) in kernel_work(kind, c).items():
        ms, k = t[n]
        if not k:
            continue
        rate = work / (ms / k * 1e-3)
        peak = peaks["hbm_gbs"] * 1e9 if bound == "hbm" else peaks["tflops_sustained"] * 1e12
        kernels[n] = dict(us=ms / k * 1e3, bound=bound, achieved=rate / (1e9 if bound == "hbm" else 1e12), unit="GB/s" if bound == "hbm" else "TFLOP/s",
                          frac=rate / peak)
    mp, md = float(np.median(pre)), float(np.median(dec))
    return dict(prefill_ms=mp, prefill_tok_s=B * P / mp * 1e3, decode_step_ms=md, decode_tok_s=B / md * 1e3, kernels=kernels)


def run(peaks: dict, steps: int, clocks, model: str = "nuzopel") -> dict:
    import torch
    pkg = entry.load_package()
    ops = entry.load_ops()
    models = importlib.import_module(entry.PKG_NAME + ".models")
    torch.cuda.set_device(0)
    out = []
    clocks.start()
    with torch.cuda.stream(torch.cuda.Stream()):
        for c in CASES:
            row = dict(case=c)
            for kind in ((model, "hybrid") if c["hybrid"] else (model,)):
                st = build_hybrid(pkg, ops, c) if kind == "hybrid" else BUILDERS[kind](pkg, models, c)
                row[kind] = measure(torch, ops, st, kind, c, peaks, steps)
                del st
                torch.cuda.synchronize()
            out.append(row)
    return dict(workload=model, data="synthetic", dtype="bf16 (hybrid: fp16)", peaks=peaks, steps=steps, warmup=3, cases=out, clocks=clocks.stop(),
                l2="a pass's activations and a step's state and weights exceed L2, except the state and latents of the small batches")
