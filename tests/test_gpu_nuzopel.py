"""GPU: layer-described stacks (mLSTM, latent attention) against the plain implementation in nuzopel_plain.py, on small
configurations with random weights.  Errors are judged on the residual stream (the norms on the sublayers' outputs put
every contribution at about 1) and on logits over their standard deviation.  A row's limit is a floor plus a multiple of what a
disturbance of the size of the rounding does to that row in the plain model: some rows are badly conditioned (a head whose
output nearly cancels before its norm)."""
import importlib
import os
import sys

import numpy as np
import pytest

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import nuzopel_plain as plain  # noqa: E402

import __graft_entry__ as entry  # noqa: E402

pytestmark = pytest.mark.gpu
FLOOR = {"float32": 1.5e-5, "bfloat16": 1e-2}
SHARE = {"float32": 2.0 ** -13, "bfloat16": 1.0}                # error over that of bf16 rounding; fp32 sums add to their rounding, bf16 products are summed in fp32


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


# ---- configurations and random weights -----------------------------------------------------------------------------------
def mlstm(heads, dim, vdim, cap=9.0, ff=None):
    return dict(type="mlstm", mixer=dict(heads=heads, dim=dim, vdim=vdim, gate_cap=cap), mlp=None if ff is None else dict(kind="dense", ff=ff))


def latent(heads, dim, rot, vdim, rank, window, ff=None, kv_from=None, base=5000.0, sharp=1.0):
    m = dict(heads=heads, dim=dim, rot_dim=rot, vdim=vdim, kv_rank=rank, mask=dict(size=window), rot=dict(base=base, dims=rot),
             scale=sharp / float(np.sqrt(dim + rot)))
    if kv_from is not None:
        m["kv_from"] = kv_from
    return dict(type="latent_attention", mixer=m, mlp=None if ff is None else dict(kind="dense", ff=ff))


def make(layers, width=80, vocab=97, seed=0, eps=1e-5, embed_scale=3.0, logit_scale=0.7):
    cfg = dict(architecture="Nuzopel", layers=layers, width=width, vocab=vocab, norm=dict(eps=eps), embedding=dict(scale=embed_scale),
               logit_scale=logit_scale)
    rng = np.random.default_rng(seed)
    t = {}

    def mat(name, rows, cols, gain=1.0):
        t[name] = rng.standard_normal((rows, cols)).astype(np.float32) * (gain / np.sqrt(cols))

    def vec(name, n, lo=0.5, hi=1.5):
        t[name] = rng.uniform(lo, hi, n).astype(np.float32)
    t["embed"] = rng.standard_normal((vocab, width)).astype(np.float32) * 0.4
    vec("final.norm", width)
    for i, L in enumerate(layers):
        m, p = L["mixer"], f"l{i}."
        vec(p + "norm1", width)
        if L["type"] == "mlstm":
            H, D, V = m["heads"], m["dim"], m["vdim"]
            mat(p + "mix.q", H * D, width); mat(p + "mix.k", H * D, width); mat(p + "mix.v", H * V, width); mat(p + "mix.g", H * V, width)
            mat(p + "mix.o", width, H * V); vec(p + "mix.norm", H * V)
            mat(p + "mix.i", H, width, 2.0); mat(p + "mix.f", H, width, 2.0)
            vec(p + "mix.i.b", H, -1.0, 1.0); vec(p + "mix.f.b", H, 1.0, 6.0)
            t[p + "mix.k"] += t[p + "mix.q"]      # a token's key agrees with its query: fewer heads whose output nearly cancels before its norm
        else:
            H, D, R, V, K = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
            mat(p + "mix.q", H * (D + R), width); mat(p + "mix.uk", H * D, K); mat(p + "mix.uv", H * V, K); mat(p + "mix.o", width, H * V)
            if "kv_from" not in m:
                mat(p + "mix.dkv", K + R, width); vec(p + "mix.dkv.norm", K)
        if L["mlp"] is not None:
            ff = L["mlp"]["ff"]
            vec(p + "norm2", width)
            mat(p + "mlp.gate", ff, width); mat(p + "mlp.up", ff, width); mat(p + "mlp.down", width, ff)
    return cfg, t


class Case:
    """A model in both implementations; weights rounded to bf16 for both."""
    plain_model = plain.PlainModel

    def __init__(self, models, wts, cfg, tensors, dtype, **limits):
        self.bits = {k: wts.bf16_bits(v) for k, v in tensors.items()}
        self.plain = self.plain_model(cfg, {k: wts.bf16_to_f32(v) for k, v in self.bits.items()})
        args = dict(max_seqs=4, max_seq_len=1024, num_pages=0, max_pass_rows=0, dtype=dtype)
        args.update(limits)
        self.stack = models.build_model(cfg, models.Limits(**args), {k: v.shape for k, v in self.bits.items()})
        models.load_tensors(self.stack, self.bits)
        self.cfg, self.dtype, self.vocab = cfg, dtype, cfg["vocab"]

    def tokens(self, n, seed=1):
        return np.random.default_rng(seed).integers(0, self.vocab, n)

    def residual_unit(self, residual):
        return 1.0                          # norms on the sublayers' outputs

    def expect(self, tokens):
        """Logits, residual stream, and the limits of the two by row."""
        trace = []
        logits = self.plain.forward(self.plain.start(), tokens, trace)
        std = max(float(np.std(logits)), 1e-3)
        worst = np.zeros((2, len(tokens)))
        for seed in range(3):
            rng, tr = np.random.default_rng(seed), []
            lg = self.plain.forward(self.plain.start(), tokens, tr, lambda a: a * (1.0 + 1.2e-3 * rng.standard_normal(a.shape)))
            for k, (d, unit) in enumerate(((lg - logits, std), (tr[-1] - trace[-1], self.residual_unit(trace[-1])))):
                worst[k] = np.maximum(worst[k], np.sqrt(np.mean((d / unit) ** 2, axis=-1)))
        return logits, trace[-1], FLOOR[self.dtype] + 8.0 * SHARE[self.dtype] * worst

    def run(self, torch, row, tokens, cuts):
        """Feeds tokens in the given portion sizes (the last size repeats); returns logits and residual stream of every place."""
        toks = torch.tensor(np.asarray(tokens), dtype=torch.int32, device="cuda")
        out, res, at, k = [], [], 0, 0
        while at < len(tokens):
            n = min(cuts[min(k, len(cuts) - 1)], len(tokens) - at)
            out.append(self.stack.extend(row, toks[at:at + n].contiguous(), range(n)))
            res.append(self.stack.residual(n))
            at, k = at + n, k + 1
        assert self.stack.device_status() == 0
        return torch.cat(out).cpu().numpy(), torch.cat(res).cpu().numpy()

    def judge(self, got, want, what=""):
        for k, (name, unit) in enumerate((("logits", max(float(np.std(want[0])), 1e-3)), ("residual", self.residual_unit(want[1])))):
            assert np.isfinite(got[k]).all(), f"{what}: {name} not finite"
            row = np.sqrt(np.mean(((got[k] - want[k]) / unit) ** 2, axis=-1))
            ratio = row / want[2][k]
            assert ratio.max() <= 1.0, f"{what}: {name} row {ratio.argmax()} is {row[ratio.argmax()]:.2e} off, {ratio.max():.2f} of its limit"
            assert np.median(ratio) <= 0.4, f"{what}: {name} median {np.median(row):.2e}, {np.median(ratio):.2f} of the limits"


def on_stream(torch):
    return torch.cuda.stream(torch.cuda.Stream())


DTYPES = ["float32", "bfloat16"]
MLSTM_SIZES = [(2, 64, 64), (2, 128, 128), (3, 40, 72), (1, 96, 160), (4, 16, 8), (1, 1, 1), (5, 24, 132), (2, 130, 20), (1, 300, 36), (1, 64, 256)]
# heads, dim, rot, vdim, rank, window
LATENT_SIZES = [(2, 64, 64, 64, 128, 70), (4, 128, 64, 128, 512, 130), (3, 40, 24, 56, 48, 17), (1, 16, 2, 8, 20, 1), (18, 32, 16, 24, 64, 64),
                (2, 8, 40, 72, 30, 65), (2, 144, 32, 136, 96, 33), (1, 1, 2, 1, 1, 5), (2, 96, 32, 100, 256, 1000), (1, 64, 64, 192, 64, 40), (2, 64, 32, 64, 64, 0), (33, 16, 16, 16, 300, 150)]


# ---- each mechanism alone: a one-layer model without feed-forward -----------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("size", MLSTM_SIZES)
def test_mlstm_layer(cuda, models, wts, size, dtype):
    if size == (1, 1, 1) and dtype == "bfloat16":
        pytest.skip("a normed head of one value is a sign, which rounding may turn")
    c = Case(models, wts, *make([mlstm(*size)], seed=11), dtype)
    toks = c.tokens(300)
    want = c.expect(toks)
    with on_stream(cuda):
        c.stack.begin_batching()
        for cuts in ([300], [1], [130, 2, 100], [17]):
            row = c.stack.open(300)
            c.judge(c.run(cuda, row, toks, cuts), want, f"{size} cuts {cuts}")
            c.stack.retire(row)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("cap,bias,gain", [(0.5, 0.0, 1.0), (25.0, -20.0, 8.0), (25.0, 18.0, 12.0)])
def test_mlstm_gate_extremes(cuda, models, wts, cap, bias, gain, dtype):
    """Caps that bind, forget gates that nearly close (the running maximum falls far) and input gates far from zero."""
    cfg, t = make([mlstm(2, 48, 56, cap=cap)], seed=5)
    for g in ("i", "f"):
        t[f"l0.mix.{g}"] = t[f"l0.mix.{g}"] * gain
        t[f"l0.mix.{g}.b"] = t[f"l0.mix.{g}.b"] * 0 + bias
    c = Case(models, wts, cfg, t, dtype)
    toks = c.tokens(200, 3)
    want = c.expect(toks)
    with on_stream(cuda):
        c.stack.begin_batching()
        for cuts in ([200], [1]):
            row = c.stack.open(200)
            got = c.run(cuda, row, toks, cuts)
            c.judge(got, want, f"cuts {cuts}")
            c.stack.retire(row)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("size", LATENT_SIZES)
def test_latent_layer(cuda, models, wts, size, dtype):
    c = Case(models, wts, *make([latent(*size, sharp=3.0)], seed=12), dtype)
    toks = c.tokens(330)
    want = c.expect(toks)
    with on_stream(cuda):
        c.stack.begin_batching()
        for cuts in ([330], [1], [63, 2, 3, 130], [50]):
            row = c.stack.open(330)
            c.judge(c.run(cuda, row, toks, cuts), want, f"{size} cuts {cuts}")
            c.stack.retire(row)


@pytest.mark.parametrize("dtype", DTYPES)
def test_feed_forward_and_scales(cuda, models, wts, dtype):
    for ff, width, escale, lscale in ((200, 72, 16.0, 0.25), (33, 50, 1.0, 1.0), (256, 2304, 0.1, 2.5)):
        c = Case(models, wts, *make([mlstm(1, 8, 8, ff=ff)], width=width, embed_scale=escale, logit_scale=lscale, seed=7), dtype)
        toks = c.tokens(40)
        want = c.expect(toks)
        with on_stream(cuda):
            c.stack.begin_batching()
            row = c.stack.open(40)
            c.judge(c.run(cuda, row, toks, [40]), want, f"ff {ff} width {width}")


# ---- the edge of a window, with one key that stands out -------------------------------------------------------------------------
def standout_case(size, seed=3):
    """One latent layer in which a query of token 1 scores far above everything else on a key of token 0."""
    heads, dim, rot, vdim, rank, window = size
    cfg, t = make([latent(*size)], seed=seed)
    x = t["embed"].astype(np.float64) * cfg["embedding"]["scale"]
    y = x[0] @ t["l0.mix.dkv"].T.astype(np.float64)[:, :rank]
    c = plain.rms_norm(y, t["l0.mix.dkv.norm"], cfg["norm"]["eps"])
    q = t["l0.mix.q"].reshape(heads, dim + rot, -1)
    uk = t["l0.mix.uk"].reshape(heads, dim, rank)
    for h in range(heads):
        k = uk[h] @ c
        want = k * (14.0 / (cfg["layers"][0]["mixer"]["scale"] * (k @ k)))      # q of token 1, unrotated part: score 14
        q[h, :dim] = 0.1 * q[h, :dim] + np.outer(want - 0.1 * q[h, :dim] @ x[1], x[1]) / (x[1] @ x[1])
    return cfg, t


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("window", [2, 40, 63, 64, 65, 128, 129, 200])
@pytest.mark.parametrize("size", [(2, 64, 64, 64, 128), (2, 24, 8, 40, 32)])
def test_window_edge(cuda, models, wts, size, window, dtype):
    c = Case(models, wts, *standout_case((*size, window)), dtype)
    for key in (0, 1, 61, 64, 127):
        n = key + window + 4
        toks = 2 + c.tokens(n, key) % (c.vocab - 2)
        toks[key] = 0
        toks[key + window - 1] = 1          # sees the key in its last place
        toks[key + window] = 1              # just does not
        want = c.expect(toks)
        # a window that is one off shows in the yardstick itself
        for off, at in ((-1, key + window - 1), (1, key + window)):
            c.plain.c["layers"][0]["mixer"]["mask"]["size"] = window + off
            if window + off > 0:
                assert np.sqrt(np.mean((c.expect(toks)[1][at] - want[1][at]) ** 2)) > 20 * FLOOR[dtype]
        c.plain.c["layers"][0]["mixer"]["mask"]["size"] = window
        with on_stream(cuda):
            c.stack.begin_batching()
            for cuts in ([n], [1], [max(2, key + window - 1), 2], [key + 1, window - 1 or 1, 1]):
                row = c.stack.open(n)
                c.judge(c.run(cuda, row, toks, cuts), want, f"key {key} cuts {cuts}")
                c.stack.retire(row)


@pytest.mark.parametrize("dtype", DTYPES)
def test_far_key_across_pages(cuda, models, wts, dtype):
    """A key hundreds of positions back, reached in a prompt and in decoding, at page borders and inside pages."""
    c = Case(models, wts, *standout_case((2, 64, 32, 64, 64, 700)), dtype)
    for key, at in ((0, 600), (63, 640), (64, 511), (130, 829)):
        toks = 2 + c.tokens(at + 2, key) % (c.vocab - 2)
        toks[key], toks[at] = 0, 1
        want = c.expect(toks)
        with on_stream(cuda):
            c.stack.begin_batching()
            for cuts in ([at + 2], [at - 1, 1], [at, 2]):
                row = c.stack.open()
                c.judge(c.run(cuda, row, toks, cuts), want, f"key {key} at {at} cuts {cuts}")
                c.stack.retire(row)


@pytest.mark.parametrize("dtype", DTYPES)
def test_mlstm_remembers_one_token(cuda, models, wts, dtype):
    """One token writes strongly and later ones hardly at all: its value must come back hundreds of tokens later."""
    cfg, t = make([mlstm(2, 64, 64, cap=15.0)], seed=8)
    x = t["embed"] * cfg["embedding"]["scale"]
    for g in ("i", "f"):
        t[f"l0.mix.{g}"] *= 0.05
    t["l0.mix.i"] += np.outer(np.ones(2), x[0]).astype(np.float32) * (10.0 / float(x[0] @ x[0]))
    t["l0.mix.i.b"][:] = -3.0
    t["l0.mix.f.b"][:] = 9.0
    c = Case(models, wts, cfg, t, dtype)
    toks = 1 + c.tokens(520) % (c.vocab - 1)
    forgotten = c.expect(toks)
    toks[5] = 0
    want = c.expect(toks)
    assert np.sqrt(np.mean((want[1][500] - forgotten[1][500]) ** 2)) > 0.3
    with on_stream(cuda):
        c.stack.begin_batching()
        for cuts in ([520], [128, 256, 1], [100, 3, 200]):
            row = c.stack.open(520)
            c.judge(c.run(cuda, row, toks, cuts), want, f"cuts {cuts}")
            c.stack.retire(row)


# ---- whole models ---------------------------------------------------------------------------------------------------------------
def whole_layers():
    return [latent(3, 40, 24, 56, 48, 37, ff=96), mlstm(2, 64, 128, ff=None), latent(5, 32, 24, 40, 48, 90, ff=120, kv_from=0, base=5000.0),
            mlstm(3, 24, 40, cap=4.0, ff=64), latent(2, 64, 32, 64, 64, 64, ff=None), latent(4, 48, 32, 32, 64, 20, ff=70, kv_from=4)]


@pytest.mark.parametrize("dtype", DTYPES)
def test_whole_model_portions(cuda, models, wts, dtype):
    c = Case(models, wts, *make(whole_layers(), seed=21), dtype)
    toks = c.tokens(410)
    want = c.expect(toks)
    with on_stream(cuda):
        c.stack.begin_batching()
        for cuts in ([410], [1], [2], [64], [200, 1, 2, 63, 65, 3, 1]):
            row = c.stack.open()
            c.judge(c.run(cuda, row, toks, cuts), want, f"cuts {cuts}")
            c.stack.retire(row)


@pytest.mark.parametrize("dtype", DTYPES)
def test_layers_of_different_sizes_share_the_working_buffers(cuda, models, wts, dtype):
    """Layers whose padded sizes differ leave values where another layer's padding lies, and portions of one token use other
    layouts than longer ones: neither may show."""
    mixed = [mlstm(7, 8, 200, ff=40), latent(5, 40, 8, 72, 40, 50), mlstm(2, 128, 96), mlstm(3, 20, 130), latent(9, 8, 48, 24, 72, 33, ff=90), mlstm(1, 140, 300),
             mlstm(4, 64, 40)]
    c = Case(models, wts, *make(mixed, width=72, seed=31), dtype)
    toks = c.tokens(180)
    want = c.expect(toks)
    with on_stream(cuda):
        c.stack.begin_batching()
        for cuts in ([180], [1], [60, 1, 1, 30, 2, 1], [180], [17, 1]):
            row = c.stack.open()
            c.judge(c.run(cuda, row, toks, cuts), want, f"cuts {cuts}")
            c.stack.retire(row)


@pytest.mark.parametrize("dtype", DTYPES)
def test_first_tokens_and_single_token(cuda, models, wts, dtype):
    c = Case(models, wts, *make(whole_layers(), seed=22), dtype)
    with on_stream(cuda):
        c.stack.begin_batching()
        for n in (1, 2, 3, 5):
            toks = c.tokens(n, n)
            for cuts in ([n], [1]):
                row = c.stack.open()
                c.judge(c.run(cuda, row, toks, cuts), c.expect(toks), f"{n} tokens, cuts {cuts}")
                c.stack.retire(row)


@pytest.mark.parametrize("dtype", DTYPES)
def test_slots_and_pages_are_reused_clean(cuda, models, wts, dtype):
    """Few pages: sequences come and go, interleaved, and each gets what it gets alone."""
    c = Case(models, wts, *make(whole_layers(), seed=23), dtype, max_seqs=3, max_seq_len=256, num_pages=7)
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


def test_pool_exhaustion_is_reported_and_recovers(cuda, models, wts, ops):
    c = Case(models, wts, *make(whole_layers(), seed=23), "bfloat16", max_seqs=3, max_seq_len=256, num_pages=5)
    with on_stream(cuda):
        c.stack.begin_batching()
        row = c.stack.open()
        c.stack.extend(row, cuda.zeros(190, dtype=cuda.int32, device="cuda"))
        row2 = c.stack.open()
        with pytest.raises(ops.B200AttnError) as e:
            c.stack.extend(row2, cuda.zeros(250, dtype=cuda.int32, device="cuda"))
        assert e.value.status == ops.ERR_NOMEM
        c.stack.retire(row)
        toks = c.tokens(100)
        c.judge(c.run(cuda, 0, toks, [100]), c.expect(toks))


# ---- batches, the captured step, generation ----------------------------------------------------------------------------------------
def check_greedy(c, prompt, tokens):
    """Every generated token has the highest logit of the plain model up to rounding."""
    logits, _, limits = c.expect(list(prompt) + list(tokens[:-1]))
    lg = logits[len(prompt) - 1:]
    slack = 6.0 * limits[0][len(prompt) - 1:] * np.std(logits)
    gap = lg.max(-1) - lg[np.arange(len(tokens)), tokens]
    assert (gap <= slack).all(), f"gap {(gap / slack).max():.2f} of the slack at {(gap / slack).argmax()}"


@pytest.mark.parametrize("dtype", DTYPES)
def test_generation_through_the_scheduler(cuda, models, wts, batching, dtype):
    """More requests than rows, unequal lengths, the captured step over all rows; each as if alone."""
    c = Case(models, wts, *make(whole_layers(), seed=24), dtype, max_seqs=3, max_seq_len=320)
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
    c = Case(models, wts, *make(whole_layers(), seed=25), dtype, max_seqs=2, max_seq_len=700)
    prompt = c.tokens(9).tolist()
    with on_stream(cuda):
        got = batching.generate(c.stack, [prompt, prompt[:4]], 600)
    check_greedy(c, prompt, got[0])
    check_greedy(c, prompt[:4], got[1])


@pytest.mark.parametrize("dtype", DTYPES)
def test_batched_prefill_and_decode(cuda, models, wts, dtype):
    """Plain (not continuous) batches: equal prompts in one pass, the captured step against eager decode."""
    c = Case(models, wts, *make(whole_layers(), seed=26), dtype, max_seqs=4, max_seq_len=200, max_pass_rows=300)
    prompts = np.stack([c.tokens(130, k) for k in range(4)])
    with on_stream(cuda):
        t = cuda.tensor(prompts, dtype=cuda.int32, device="cuda")
        first = c.stack.forward_batch_prefill(t)
        toks = [first.clone()]
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
    import json
    import struct
    import subprocess
    cfg, t = make(whole_layers(), seed=27)
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
    assert [x for x in p.stdout.split("\n") if x.startswith("done")] == [f"done {i}" for i in range(4)]
    want = c.expect(toks)[0]
    for step, places in ((0, [49, 3]), (2, [51]), (3, [1])):
        got = np.fromfile(tmp_path / f"{step}.f32", "<f4").reshape(len(places), -1)
        assert np.abs(got - want[places]).max() < 1e-3 * np.std(want)
    assert not (tmp_path / "1.f32").exists()
    p = subprocess.run([os.path.join(entry.ROOT, "bin", "generate"), "--model", str(tmp_path), "--dtype", "float32", "--max-new-tokens", "6"],
                       input=json.dumps(toks[:20]) + "\n" + json.dumps(toks[:3]) + "\n", capture_output=True, text=True, timeout=280)
    assert p.returncode == 0, p.stderr[-2000:]
    out = [json.loads(x) for x in p.stdout.strip().split("\n")[-2:]]
    check_greedy(c, toks[:20], out[0])
    check_greedy(c, toks[:3], out[1])
