"""Fetitar on the GPU against the plain implementation: each new or changed kernel alone, whole prompts, portions, token-by-token
decoding, unequal batches, slots and pages that are used again, keys far away and just inside and outside every window, the first
tokens, mixed values, long decoding over page borders, generation through the entry point, the replay program, the command
line."""
import copy
import json
import os
import random
import subprocess
import sys
from types import SimpleNamespace

import numpy as np
import pytest
import torch

import kernel_refs
import tiny_fetitar as tf
from dotllm_b200.kernels import attention_fast, ops

pytestmark = pytest.mark.gpu
DEV = torch.device("cuda", 0)
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
DTYPES = [torch.float32, torch.bfloat16]
# A row's rms error over the row's rms.  float32: summation order only.  bfloat16: both sides read the same bfloat16 weights; the
# engine rounds activations to bfloat16 between parts.
REL = {torch.float32: 3e-5, torch.bfloat16: 3e-2}


def row_errors(got, want):
    g, w = got.double().cpu().reshape(-1, got.shape[-1]), want.double().cpu().reshape(-1, want.shape[-1])
    return (g - w).pow(2).mean(-1).sqrt() / w.pow(2).mean(-1).sqrt().clamp_min(1e-30)


def rel_err(got, want):
    return float(row_errors(got, want).max())


def assert_rows(got, want, dtype, what=""):
    assert torch.isfinite(got).all(), f"{what}: non-finite logits"
    err = row_errors(got, want)
    assert float(err.max()) <= REL[dtype], f"{what}: row {int(err.argmax())} has an rms error of {float(err.max()):.3e} of its rms > {REL[dtype]:.1e}"


@pytest.fixture(scope="module")
def tmp(tmp_path_factory):
    return tmp_path_factory.mktemp("fetitar")


_loaded = {}


def load_pair(tmp, which, dtype, seed=0, change=None, tag=""):
    from dotllm_b200 import Model
    key = (which, dtype, seed, tag)
    if key not in _loaded:
        folder = tf.make_folder(tmp / tag if tag else tmp, which, seed=seed, dtype=dtype)
        if change is not None:
            tf.rewrite(folder, change)
        cfg, weights = tf.read_folder(folder)
        _loaded[key] = (Model.load(folder, dtype=dtype), cfg, weights, folder)
    return _loaded[key]


def g32(*shape, seed=0, scale=1.0):
    return (torch.randn(*shape, generator=torch.Generator().manual_seed(seed), dtype=torch.float32) * scale).to(DEV)


def i32(values):
    return torch.tensor(list(values), dtype=torch.int32, device=DEV)


def cpu(t):
    return None if t is None else t.cpu()


def close(got, want, dtype, tol32=2e-5, tol16=2e-2):
    scale = float(want.double().abs().max().clamp_min(1e-6))
    err = float((got.double().cpu() - want.double().cpu()).abs().max()) / scale
    assert err <= (tol32 if dtype == torch.float32 else tol16), err


def run_cuts(model, tokens, cuts):
    """Feed ``tokens`` to a fresh sequence in portions of the given sizes, the rest one by one; the logits of every token."""
    from dotllm_b200.engine import StepEntry
    cache = model.new_cache(64 * ((len(tokens) + 63) // 64 + 1))
    cache.fill_free_pages(float("nan"))
    seq = cache.open_sequence()
    outs, at = [], 0
    sizes = list(cuts)
    while at < len(tokens):
        n = min(sizes.pop(0) if sizes else 1, len(tokens) - at)
        outs.append(model.step(cache, [StepEntry(seq, tokens[at:at + n], list(range(n)))]).clone())
        at += n
        if at % 16 == 0:
            cache.fill_free_pages(float("nan"))          # what a window gave back is never read again
    cache.close_sequence(seq)
    cache.check()
    return torch.cat(outs)


# ------------------------------------------------------------------ kernels alone
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,buckets,mul_prev,mul_cur", [(52, 1, 3, 5), (64, 97, 37, 11), (101, 40, -13, 29), (1028, 1000, 2000000011, 2000000089), (4096, 3, 0, 1)])
def test_the_embedding_of_token_pairs_alone(H, buckets, mul_prev, mul_cur, dtype):
    """Unequal prompts, portions and single tokens in slots that are not neighbours; a slot that is used again starts anew."""
    table, pairs = g32(50, H, seed=1).to(dtype), g32(buckets + 1, H, seed=2).to(dtype)
    last = torch.full((6, 1), 33, dtype=torch.int32, device=DEV)       # what an earlier sequence left
    rlast = last.cpu().clone()
    slots, starts = [4, 0, 2], [0, 0, 0]
    gen = random.Random(5)
    for sizes in ([1, 70, 9], [2, 1, 13], [1, 1, 1], [1, 300, 2]):
        tokens = [gen.randrange(50) for _ in range(sum(sizes))]
        step = SimpleNamespace(tokens=i32(tokens), token_seq=i32([b for b in range(3) for _ in range(sizes[b])]),
                               token_pos=i32([starts[b] + i for b in range(3) for i in range(sizes[b])]),
                               cu_new=i32([0] + list(np.cumsum(sizes))), slots=i32(slots))
        rstep = SimpleNamespace(**{k: v.cpu() for k, v in vars(step).items()})
        got = ops.embed_pairs(table, pairs, step, last, mul_prev, mul_cur, 2.5)
        close(got, kernel_refs.embed_pairs(table.cpu(), pairs.cpu(), rstep, rlast, mul_prev, mul_cur, 2.5), torch.float32, 1e-6)
        assert torch.equal(last.cpu(), rlast) and int(last[1]) == 33
        starts = [s + n for s, n in zip(starts, sizes)]
        if sizes[0] == 2:
            starts[0] = 0                                              # slot 4 belongs to a new sequence from here on


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H", [52, 64, 1000, 1030, 2048, 4096, 7000, 8192, 9000])
def test_the_norm_of_a_biased_branch_alone(H, dtype):
    """A branch with and without a bias, an extra addend and a norm of the sum behind it, at widths that take each path."""
    T = 5
    x, y, bias, extra = g32(T, H, seed=1, scale=2.0), g32(T, H + 8, seed=2)[:, :H], g32(H, seed=3), g32(T, H, seed=4)
    dg, gain = g32(H, seed=5), g32(H, seed=6)
    for branch in (y.contiguous(), y.to(torch.bfloat16).contiguous(), y):
        for b, e, n in ((bias, None, True), (None, extra, True), (bias, extra, False)):
            mine = ops.NormedBranch(branch if b is None else ops.Biased(branch, b), dg, 1e-5, e)
            theirs = SimpleNamespace(data=branch.cpu().float() + (0.0 if b is None else b.cpu()), gain=dg.cpu(), eps=1e-5, extra=cpu(e))
            xa, xb = x.clone(), x.cpu().clone()
            got = ops.add_normed_branch(xa, mine, gain if n else None, 1e-6, dtype if n else None)
            want = kernel_refs.add_normed_branch(xb, theirs, gain.cpu() if n else None, 1e-6, dtype if n else None)
            close(xa, xb, torch.float32)
            assert (got is None) == (not n)
            if n:
                close(got, want, dtype)
    rows = y.contiguous()
    close(ops.resolve(ops.Biased(rows.clone(), bias)), rows + bias, torch.float32)
    close(ops.resolve(ops.narrow_rows(ops.Biased(rows.clone(), bias), i32([3, 0]))), (rows + bias)[[3, 0]], torch.float32)
    xa = x.clone()                                                     # and a plain pre-norm stream takes it in too
    got = ops.add_rmsnorm(xa, ops.Biased(rows.clone(), bias), gain, 1e-6, torch.float32)
    close(xa, x + rows + bias, torch.float32), close(got, kernel_refs._rms((x + rows + bias).cpu(), 1e-6) * gain.cpu(), torch.float32)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,d,vd,lay", [(4, 1, 64, 48, 64), (6, 2, 24, 20, 32), (3, 1, 10, 7, 16), (7, 7, 9, 14, 32), (32, 8, 128, 128, 128), (16, 2, 96, 128, 128),
                                          (80, 2, 128, 64, 128), (90, 3, 101, 33, 128), (2, 2, 33, 65, 96), (1, 1, 8, 8, 8)])
def test_rows_ready_for_the_cache_alone(H, G, d, vd, lay, dtype):
    """Biases, norms over whole projections, mixed values and the kernels' layout, each alone and together."""
    T = 6
    width = H * d + G * (d + vd)
    x = g32(T, width + 8, seed=1).to(dtype)[:, :width]
    biases = (g32(H * d, seed=2), g32(G * d, seed=3), g32(G * vd, seed=4))
    gains = (g32(H * d, seed=5), g32(G * d, seed=6))
    mix = torch.tensor([0.3], device=DEV)
    wide = -(-vd // 8) * 8 + 8
    for first in (None, g32(T, G * wide, seed=7).to(dtype)):
        for b, g in ((biases, gains), (None, gains), (biases, None), ((None, biases[1], None), None)):
            for lk, lv in ((lay, lay), (d, vd)):
                if lk < d or lv < vd:
                    continue
                m = None if first is None else mix
                got = ops.qkv_rows(x, H, G, d, vd, lk, lv, biases=b, gains=g, eps=1e-5, first=first, mix=m)
                want = kernel_refs.qkv_rows(x.cpu(), H, G, d, vd, lk, lv, biases=None if b is None else tuple(cpu(t) for t in b),
                                            gains=None if g is None else tuple(cpu(t) for t in g), eps=1e-5, first=cpu(first), mix=cpu(m))
                for a, r in zip(got, want):
                    close(a, r, dtype, tol16=1e-2)
                if lk > d:
                    assert not got[0].reshape(T, H, lk)[..., d:].any() and not got[1].reshape(T, G, lk)[..., d:].any()
                if lv > vd:
                    assert not got[2].reshape(T, G, lv)[..., vd:].any()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows", [1, 8, 10, 13, 40, 128, 200])
@pytest.mark.parametrize("ff,K", [(160, 96), (100, 64), (520, 1032), (30, 72)])
def test_a_gated_product_with_biases_alone(ff, K, rows, dtype):
    """The biases in the epilogues of all three products (a few rows, some, many), behind the library's, and in float32."""
    x, w, bias = g32(rows, K, seed=1).to(dtype), g32(2 * ff, K, seed=2, scale=0.1).to(dtype), g32(2 * ff, seed=3)
    for kind in ("silu", "gelu_tanh"):
        want = kernel_refs.gated_linear(x.cpu(), w.cpu(), kind=kind, bias=bias.cpu())
        close(ops.gated_linear(x, w, kind=kind, bias=bias), want, dtype)
        plain = kernel_refs.gated_linear(x.cpu(), w.cpu(), kind=kind)
        close(ops.gated_linear(x, w, kind=kind), plain, dtype)
        assert float((plain.double() - want.double()).abs().max() / want.double().abs().max()) > 0.1


def _paged(n_seqs, pages, nkv, hd, lens, seed):
    """Random keys and values of sequences of the given lengths in scattered pages, NaN in every slot that holds none."""
    gen = torch.Generator().manual_seed(seed)
    k = torch.full((n_seqs * pages + 2, nkv, 64, hd), float("nan"), dtype=torch.bfloat16)
    v = torch.full((n_seqs * pages + 2, nkv, hd, 64), float("nan"), dtype=torch.bfloat16)
    order = torch.randperm(n_seqs * pages + 2, generator=gen).tolist()
    table = torch.full((n_seqs, pages), -1, dtype=torch.int32)
    for b in range(n_seqs):
        for p in range((lens[b] + 63) // 64):
            page = table[b, p] = order.pop()
            n = min(64, lens[b] - 64 * p)
            k[page, :, :n] = torch.randn(nkv, n, hd, generator=gen).to(torch.bfloat16)
            v[page, :, :, :n] = torch.randn(nkv, hd, n, generator=gen).to(torch.bfloat16)
    return k, v, table


@pytest.mark.parametrize("hd", [32, 64, 96, 128])
@pytest.mark.parametrize("nh,nkv", [(4, 2), (20, 1), (24, 2), (17, 1)])
def test_slopes_gates_and_windows_in_the_tensor_core_kernels(nh, nkv, hd):
    """Decode (with the step's own token written inside and without) and both prompt kernels against the plain attention; without the
    slopes the result is far away, and so it is with a window one token off or with the slopes of the neighbouring head."""
    from dotllm_b200.engine.step import AttentionPlan
    lens = [1, 70, 150, 290]
    B, pages = len(lens), 5
    k, v, table = _paged(B, pages, nkv, hd, lens, seed=hd + nh)
    slopes = torch.tensor([2.0 ** (-8.0 * (h + 1) / nh) for h in range(nh)], device=DEV)
    scale = 4.0 * hd ** -0.5                                           # sharp: single keys decide, so that a window's edge shows
    hook, rhook = ops.ScoreHook(0.0, slopes), ops.ScoreHook(0.0, slopes.cpu())
    for name, starts, news in (("decode", [n - 1 for n in lens], [1] * B), ("prompt", [0, 10, 120, 20], [1, 60, 30, 270])):
        T = sum(news)
        q = g32(T, nh * hd, seed=5).to(torch.bfloat16)
        gate = g32(T, nh + 8, seed=6).to(torch.bfloat16)[:, :nh]
        seq = i32([b for b in range(B) for _ in range(news[b])])
        pos = i32([starts[b] + i for b in range(B) for i in range(news[b])])
        plan = lambda: AttentionPlan(B, max(news), max(lens), name == "decode", i32(starts), i32(news), i32([0] + list(np.cumsum(news))), i32(lens),
                                     list(starts), list(news))
        args = (nh, nkv, hd, scale)
        ref = lambda **kw: kernel_refs.attention(q.cpu(), k, v, seq.cpu(), pos.cpu(), table, *args, **kw)
        for window, h, g in ((65, hook, gate), (64, None, gate), (44, hook, None)) + (((0, hook, None), (1, hook, gate)) if name == "decode" or hd == 64 else ()):
            want = ref(window=window, score_hook=rhook if h is not None else None, gate=cpu(g))
            run = lambda: ops.attention(q, k.to(DEV), v.to(DEV), seq, pos, table.to(DEV), *args, window, plan=plan(), score_hook=h, gate=g, split=True)
            close(run(), want, torch.bfloat16)
            if name == "prompt" and hd in attention_fast.PREFILL_TC_HEAD_DIMS:
                try:
                    attention_fast.PREFILL_TC = False                    # the mma.sync kernel at the same sizes
                    close(run(), want, torch.bfloat16)
                finally:
                    attention_fast.PREFILL_TC = True
            if window == 44 and name == "prompt":
                far = lambda other: float((other.double() - want.double()).abs().max() / want.double().abs().max())
                assert far(ref(window=45, score_hook=rhook)) > 0.05 and far(ref(window=44)) > 0.1
                assert far(ref(window=44, score_hook=ops.ScoreHook(0.0, slopes.cpu().roll(1)))) > 0.1
        if hd == 64:                                                     # a cap and slopes together: the mma.sync and the decode kernel
            close(ops.attention(q, k.to(DEV), v.to(DEV), seq, pos, table.to(DEV), *args, 100, plan=plan(), score_hook=ops.ScoreHook(1.5, slopes), split=True),
                  ref(window=100, score_hook=ops.ScoreHook(1.5, slopes.cpu())), torch.bfloat16)
        if name == "decode":                                             # the new token's key and value come with the call
            kd, vd = k.to(DEV), v.to(DEV)
            fresh_k, fresh_v = g32(B, nkv * hd, seed=7).to(torch.bfloat16), g32(B, nkv * hd, seed=8).to(torch.bfloat16)
            got = ops.rope_cache_attention(q, fresh_k, fresh_v, None, None, 0, seq, pos, table.to(DEV), kd, vd, *args, 65, plan=plan(),
                                           score_hook=hook, gate=gate, split=True)
            kr, vr = k.clone(), v.clone()
            kernel_refs.rope_cache_write(q.cpu().clone(), fresh_k.cpu(), fresh_v.cpu(), None, None, 0, seq.cpu(), pos.cpu(), table, kr, vr, nh, nkv, hd)
            close(got, kernel_refs.attention(q.cpu(), kr, vr, seq.cpu(), pos.cpu(), table, *args, window=65, score_hook=rhook, gate=gate.cpu()), torch.bfloat16)
            assert torch.equal(torch.nan_to_num(kd.cpu().float()), torch.nan_to_num(kr.float())) and \
                torch.equal(torch.nan_to_num(vd.cpu().float()), torch.nan_to_num(vr.float()))


# ------------------------------------------------------------------ the model
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("which", ["A", "B", "C", "D", "E"])
def test_whole_portions_and_decoding(tmp, which, dtype):
    model, cfg, w, _ = load_pair(tmp, which, dtype)
    tokens = tf.random_tokens(150, cfg["vocab"], 7)
    ref = tf.plain_logits(cfg, w, tokens)
    whole = run_cuts(model, tokens, [150])
    assert_rows(whole, ref, dtype, "whole prompt")
    for cuts in ([100, 50], [64, 64, 2, 20], [63, 3, 2, 2, 70], [1, 2, 129, 5], [130], [2]):
        got = run_cuts(model, tokens, cuts)
        assert_rows(got, ref, dtype, f"cuts {cuts}")
        if dtype == torch.float32:
            assert rel_err(got, whole) < 1e-5, cuts


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("which", ["A", "B", "D"])
def test_unequal_batches_slots_and_pages_used_again(tmp, which, dtype):
    from dotllm_b200.engine import StepEntry
    model, cfg, w, _ = load_pair(tmp, which, dtype)
    lens = [1, 70, 23, 131]
    prompts = [tf.random_tokens(n + 12, cfg["vocab"], 20 + n) for n in lens]
    refs = [tf.plain_logits(cfg, w, p) for p in prompts]
    cache = model.new_cache(64 * 8)
    for again in range(2):                                           # the second time every slot and page has been used before
        cache.fill_free_pages(float("nan"))
        seqs = [cache.open_sequence() for _ in prompts]
        order = list(range(len(prompts))) if again == 0 else [2, 0, 3, 1]
        out = model.step(cache, [StepEntry(seqs[i], prompts[i][:lens[i]], [0, lens[i] - 1]) for i in order])
        want = torch.cat([refs[i][[0, lens[i] - 1]] for i in order])
        assert_rows(out, want, dtype, "a batch of unequal prompts")
        live = list(order)
        for t in range(12):
            if t == 5:
                gone = live.pop(1)                                   # a request ends early; its slot and pages go back ...
                cache.close_sequence(seqs[gone])
                cache.fill_free_pages(float("nan"))
            out = model.step(cache, [StepEntry(seqs[i], [prompts[i][lens[i] + t]]) for i in live])
            assert_rows(out, torch.stack([refs[i][lens[i] + t] for i in live]), dtype, f"decoding together, step {t}")
        for i in live:
            cache.close_sequence(seqs[i])
        cache.check()
    assert not cache.live


@pytest.mark.parametrize("dtype", DTYPES)
def test_many_sequences_decode_together_as_each_alone(tmp, dtype):
    """Batches of 12, 40 and 140 rows: the products for some and for many rows, with the biases in their epilogues."""
    from dotllm_b200.engine import StepEntry
    model, cfg, w, _ = load_pair(tmp, "B", dtype)
    base = [tf.random_tokens(n, cfg["vocab"], 200 + n) for n in (3, 17, 66, 40)]
    refs = [tf.plain_logits(cfg, w, p) for p in base]
    for n in (12, 40, 140):
        cache = model.new_cache(64 * (n * 2 + 4))
        seqs = [cache.open_sequence() for _ in range(n)]
        which = [i % 4 for i in range(n)]
        model.step(cache, [StepEntry(s, base[k][:-1], []) for s, k in zip(seqs, which)])
        out = model.step(cache, [StepEntry(s, base[k][-1:]) for s, k in zip(seqs, which)])
        assert_rows(out, torch.stack([refs[k][-1] for k in which]), dtype, f"{n} sequences")


@pytest.mark.parametrize("dtype", DTYPES)
def test_steps_that_mix_portions_and_single_tokens(tmp, dtype):
    """One step with a prompt, a portion of another, and sequences that go on by one token."""
    from dotllm_b200.engine import StepEntry
    model, cfg, w, _ = load_pair(tmp, "A", dtype)
    prompts = [tf.random_tokens(n, cfg["vocab"], 90 + n) for n in (90, 140, 30, 66)]
    refs = [tf.plain_logits(cfg, w, p) for p in prompts]
    cache = model.new_cache(64 * 10)
    cache.fill_free_pages(float("nan"))
    seqs = [cache.open_sequence() for _ in prompts]
    at = [0] * 4
    for sizes in ([0, 70, 5, 0], [40, 1, 2, 64], [2, 64, 1, 1], [1, 1, 1, 1], [47, 4, 21, 0]):
        entries = [(i, n) for i, n in enumerate(sizes) if n]
        out = model.step(cache, [StepEntry(seqs[i], prompts[i][at[i]:at[i] + n], [0, n - 1]) for i, n in entries])
        assert_rows(out, torch.cat([refs[i][[at[i], at[i] + n - 1]] for i, n in entries]), dtype, f"{sizes}")
        for i, n in entries:
            at[i] += n


@pytest.mark.parametrize("dtype", DTYPES)
def test_layers_at_a_real_models_widths(tmp, dtype):
    """Width 1,024, heads of 128 channels, latent rows of 96 + 32 and 64 + 64: the sizes of the tensor-core kernels."""
    model, cfg, w, _ = load_pair(tmp, "wide", dtype)
    tokens = tf.random_tokens(230, cfg["vocab"], 11)
    ref = tf.plain_logits(cfg, w, tokens)
    assert_rows(run_cuts(model, tokens, [200]), ref, dtype, "a prompt of 200 tokens and 30 decoded")
    assert_rows(run_cuts(model, tokens[:200], [130, 70]), ref[:200], dtype, "two portions")


@pytest.mark.parametrize("seed", range(8))
def test_configurations_drawn_at_random(tmp_path, seed):
    """Configurations that nobody chose (`tiny_fetitar.random_config`): a prompt and twenty decoded tokens, then a batch of
    three unequal prompts (one of a single token) decoded together, eager and through captured steps, in both dtypes."""
    from dotllm_b200 import Model
    from dotllm_b200.engine import StepEntry
    rng = random.Random(300 + seed)
    cfg_dict = tf.random_config(rng)
    n = rng.randrange(100, 200)
    lens = [1, rng.randrange(2, 80), rng.randrange(80, 150)]
    for dtype in DTYPES:
        folder = tf.make_folder(tmp_path, f"random{seed}", dtype=dtype, cfg=cfg_dict)
        cfg, w = tf.read_folder(folder)
        model = Model.load(folder, dtype=dtype)
        tokens = tf.random_tokens(n, cfg["vocab"], seed)
        prompts = [tf.random_tokens(L + 8, cfg["vocab"], seed * 7 + L) for L in lens]
        ref, refs = tf.plain_logits(cfg, w, tokens), [tf.plain_logits(cfg, w, p) for p in prompts]
        got = [run_cuts(model, tokens, [n - 20])]
        want = [ref]
        cache = model.new_cache(64 * 12)
        cache.fill_free_pages(float("nan"))
        seqs = [cache.open_sequence() for _ in prompts]
        got.append(model.step(cache, [StepEntry(q, p[:L], [L - 1]) for q, p, L in zip(seqs, prompts, lens)]).clone())
        want.append(torch.stack([r[L - 1] for r, L in zip(refs, lens)]))
        for t in range(8):
            got.append(model.step(cache, [StepEntry(q, [p[L + t]]) for q, p, L in zip(seqs, prompts, lens)], graphs=t >= 4).clone())
            want.append(torch.stack([r[L + t] for r, L in zip(refs, lens)]))
        assert_rows(torch.cat(got), torch.cat(want), dtype, f"{seed}: {cfg_dict}")


def _sharp_sloped(t):
    t["l0.mix.o"] *= 6.0


def _sharp_latent(t):
    t["l0.mix.uq"] *= 2.0
    t["l0.mix.o"] *= 12.0


def _agrees(tmp, which, change, tokens, ref):
    model = load_pair(tmp, which, torch.float32, change=change, tag="sharp")[0]
    n = len(tokens)
    for cuts in ([n], [63, 1, 1, 200], [128, 64, 2], [n - 50], [20]):
        assert rel_err(run_cuts(model, tokens, cuts), ref) < 1e-4, cuts
    bf, cfg, w, _ = load_pair(tmp, which, torch.bfloat16, change=change, tag="sharp")
    ref16 = tf.plain_logits(cfg, w, tokens)
    for cuts in ([n - 20], [100]):
        err = row_errors(run_cuts(bf, tokens, cuts), ref16)
        assert float(err.median()) < 3e-2 and int((err > 0.3).sum()) <= 8, (cuts, float(err.median()), int((err > 0.3).sum()))


def test_slopes_biases_norms_and_window_edges_decide_whole_rows(tmp):
    """One attention layer whose scores are sharpened until single keys decide.  A window one token off either way, no slopes, the next
    head's slopes, slopes that start at one, a missing bias and norms per head must each change rows of the plain result;
    the engine agrees with the design over prompts, portions and decoding."""
    import plain_fetitar as pf
    tokens = tf.random_tokens(400, 120, 5)
    _, cfg, w, _ = load_pair(tmp, "sharp_sloped", torch.float32, change=_sharp_sloped, tag="sharp")
    ref = tf.plain_logits(cfg, w, tokens)
    rms = ref.pow(2).mean(-1).sqrt()
    differs = lambda other: int(((other - ref).pow(2).mean(-1).sqrt() / rms > 1e-2).sum())

    def with_window(n):
        other = copy.deepcopy(cfg)
        other["layers"][0]["mixer"]["mask"]["size"] = n
        return tf.plain_logits(other, w, tokens)
    assert min(differs(with_window(69)), differs(with_window(71))) >= 10 and differs(with_window(400)) >= 100
    saved = pf.distance_slopes, pf.rms
    try:
        for slopes in (lambda H: None, lambda H: saved[0](H)[1:] + saved[0](H)[:1], lambda H: [2.0 ** (-8.0 * h / H) for h in range(H)]):
            pf.distance_slopes = slopes
            assert differs(tf.plain_logits(cfg, w, tokens)) >= 100
        pf.distance_slopes = saved[0]
        pf.rms = lambda x, eps: saved[1](x.reshape(len(x), -1, 16), eps).reshape(x.shape) if x.shape[-1] == 32 else saved[1](x, eps)
        assert differs(tf.plain_logits(cfg, w, tokens)) >= 100           # a norm per key head instead of one over all
    finally:
        pf.distance_slopes, pf.rms = saved
    for name in ("q.b", "k.b", "v.b", "o.b"):
        assert differs(tf.plain_logits(cfg, {**w, f"l0.mix.{name}": 0 * w[f"l0.mix.{name}"]}, tokens)) >= 100, name
    _agrees(tmp, "sharp_sloped", _sharp_sloped, tokens, ref)


def test_far_keys_the_rotation_and_the_gate_decide_whole_rows(tmp):
    """One latent-attention layer sharpened the same way: a window one token off, plain frequencies, cosines without their factor,
    channels paired the other way and no gate must each change rows of the plain result; the engine agrees with the design."""
    import plain_fetitar as pf
    tokens = tf.random_tokens(400, 120, 5)
    _, cfg, w, _ = load_pair(tmp, "sharp_latent", torch.float32, change=_sharp_latent, tag="sharp")
    ref = tf.plain_logits(cfg, w, tokens)
    rms = ref.pow(2).mean(-1).sqrt()
    differs = lambda other: int(((other - ref).pow(2).mean(-1).sqrt() / rms > 1e-2).sum())

    def changed(**mixer):
        other = copy.deepcopy(cfg)
        other["layers"][0]["mixer"].update(mixer)
        return tf.plain_logits(other, w, tokens)
    assert min(differs(changed(mask={"size": n})) for n in (149, 151)) >= 8 and differs(changed(mask={"size": 100})) >= 100
    assert differs(changed(rot={"dims": 8, "base": 100.0})) >= 100
    saved = pf.yarn_frequencies, pf.rotate_halves
    try:
        pf.yarn_frequencies = lambda *a: (saved[0](*a)[0], 1.0)
        assert differs(tf.plain_logits(cfg, w, tokens)) >= 100
        pf.yarn_frequencies = saved[0]

        def neighbours(x, positions, dims, base, scaling=None):
            order = list(range(0, dims, 2)) + list(range(1, dims, 2))
            y = x.copy()
            y[..., :dims] = saved[1](x[..., :dims][..., order], positions, dims, base, scaling)[..., np.argsort(order)]
            return y
        pf.rotate_halves = neighbours
        assert differs(tf.plain_logits(cfg, w, tokens)) >= 100
    finally:
        pf.yarn_frequencies, pf.rotate_halves = saved
    assert differs(tf.plain_logits(cfg, {**w, "l0.mix.g": 0 * w["l0.mix.g"]}, tokens)) >= 100
    _agrees(tmp, "sharp_latent", _sharp_latent, tokens, ref)


def _first_counts(t):
    t["l5.mix.vmix"].fill_(0.9)
    for name in ("l0.mix.v", "l0.mix.v.b"):
        t[name] *= 4.0
    t["l5.mix.o"] *= 4.0


def test_mixed_values_and_pair_rows_show(tmp):
    """Values not mixed, or mixed the wrong way round, a pair table that is read without the token before, and a first token with
    another row than the last are far from the design; the engine is close to it."""
    import plain_fetitar as pf
    model, cfg, w, _ = load_pair(tmp, "A", torch.float32, change=_first_counts, tag="mixed")
    tokens = tf.random_tokens(120, cfg["vocab"], 17)
    ref = tf.plain_logits(cfg, w, tokens)
    rms = ref.pow(2).mean(-1).sqrt()
    off = lambda: (tf.plain_logits(cfg, w, tokens) - ref).pow(2).mean(-1).sqrt() / rms
    saved = pf.mixed_values, pf.bigram_rows
    try:
        for mixed in (lambda v, first, weight: v, lambda v, first, weight: weight * v + (1.0 - weight) * first):
            pf.mixed_values = mixed
            assert int((off() > 1e-2).sum()) >= 100
        pf.mixed_values = saved[0]
        pf.bigram_rows = lambda tokens, buckets, a, b: [(int(t) * b) % buckets for t in tokens]
        assert int((off() > 1e-2).sum()) >= 100
        pf.bigram_rows = lambda tokens, buckets, a, b: [(int(tokens[0]) * b) % buckets] + saved[1](tokens, buckets, a, b)[1:]
        assert float(off()[0]) > 1e-2
    finally:
        pf.mixed_values, pf.bigram_rows = saved
    for cuts in ([120], [1, 2, 3, 64], [50]):
        assert_rows(run_cuts(model, tokens, cuts), ref, torch.float32, f"cuts {cuts}")
    bf, cfg16, w16, _ = load_pair(tmp, "A", torch.bfloat16, change=_first_counts, tag="mixed")
    assert_rows(run_cuts(bf, tokens, [90]), tf.plain_logits(cfg16, w16, tokens), torch.bfloat16, "bfloat16")


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding_over_page_borders(tmp, dtype):
    model, cfg, w, _ = load_pair(tmp, "A", dtype)
    tokens = tf.random_tokens(330, cfg["vocab"], 5)
    ref = tf.plain_logits(cfg, w, tokens)
    assert_rows(run_cuts(model, tokens, [30]), ref, dtype, "300 tokens decoded one by one, over five page borders")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("which", ["A", "B"])
def test_greedy_generation_through_the_entry_point(tmp, which, dtype):
    from dotllm_b200 import InferenceOptions
    model, cfg, w, _ = load_pair(tmp, which, dtype)
    prompts = [tf.random_tokens(n, cfg["vocab"], 60 + n) for n in (1, 9, 40, 70)]
    n_new = 24
    options = InferenceOptions(temperature=0.0, max_tokens=n_new, stop_token_ids=[])
    outs = model.generate(prompts, options)
    again = model.generate(prompts, options)                         # through captured steps now
    for p, o in list(zip(prompts, outs)) + list(zip(prompts, again)):
        assert o.finish_reason.value == "length" and o.generated_token_count == n_new
        ref = tf.plain_logits(cfg, w, p + o.generated_token_ids)
        spread = float(ref.std())
        for i, tok in enumerate(o.generated_token_ids):              # teacher-forced: the plain arg-max, or within rounding of it
            row = ref[len(p) - 1 + i]
            assert int(row.argmax()) == tok or float(row.max() - row[tok]) <= (1e-4 if dtype == torch.float32 else 0.1) * spread, \
                (i, tok, int(row.argmax()))
    alone = model.generate(prompts[2], options)
    if dtype == torch.float32:
        assert [o.generated_token_ids for o in again] == [o.generated_token_ids for o in outs]
        assert alone.generated_token_ids == outs[2].generated_token_ids


def test_steps_replayed_from_graphs(tmp):
    """Prompts and decode steps captured as graphs (exact batch size and the shared widths with idle rows) give the eager steps'
    logits; the trial run before a capture leaves the last tokens as they were."""
    from dotllm_b200.engine import StepEntry
    for dtype in DTYPES:
        model, cfg, w, _ = load_pair(tmp, "A", dtype)
        prompts = [tf.random_tokens(n + 10, cfg["vocab"], 80 + n) for n in (5, 66, 30)]
        refs = [tf.plain_logits(cfg, w, p) for p in prompts]
        for graphs in (True, "lazy"):
            cache = model.new_cache(64 * 12)
            for again in range(3):                                   # the third prompt step of this shape runs from its graph
                seqs = [cache.open_sequence() for _ in prompts]
                out = model.step(cache, [StepEntry(s, p[:-10], [len(p) - 11]) for s, p in zip(seqs, prompts)], graphs=graphs)
                assert_rows(out, torch.stack([r[len(r) - 11] for r in refs]), dtype, f"graphs={graphs} prompt {again}")
                for t in range(10):
                    out = model.step(cache, [StepEntry(s, [p[len(p) - 10 + t]]) for s, p in zip(seqs, prompts)], graphs=graphs)
                    assert_rows(out, torch.stack([r[len(r) - 10 + t] for r in refs]), dtype, f"graphs={graphs} step {t}")
                for s in seqs:
                    cache.close_sequence(s)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_replay_program_on_a_fetitar_folder(tmp_path, dtype):
    tdtype = {"float32": torch.float32, "bfloat16": torch.bfloat16}[dtype]
    folder = tf.make_folder(tmp_path, "A", seed=2, dtype=tdtype)
    cfg, w = tf.read_folder(folder)
    a, b = tf.random_tokens(90, cfg["vocab"], 1), tf.random_tokens(30, cfg["vocab"], 2)
    ra, rb = tf.plain_logits(cfg, w, a), tf.plain_logits(cfg, w, b)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:80], "want": [0, 79]}, {"id": "b", "tokens": b[:20], "want": []}], "end": []}]
    for t in range(10):
        steps.append({"step": t + 1, "entries": [{"id": "a", "tokens": [a[80 + t]], "want": [0]},
                                                 {"id": "b", "tokens": [b[20 + t]], "want": [0] if t % 2 else []}],
                      "end": ["a", "b"] if t == 9 else []})
    out_dir = tmp_path / "out"
    proc = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(folder), "--dtype", dtype, "--out", str(out_dir),
                           "--max-tokens", "256"], input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True,
                          text=True, timeout=600)
    assert proc.returncode == 0, proc.stderr[-2000:]
    assert proc.stdout.split() == [x for s in steps for x in ("done", str(s["step"]))]
    read = lambda n: torch.from_numpy(np.fromfile(out_dir / f"{n}.f32", dtype="<f4").reshape(-1, cfg["vocab"]).copy())
    assert_rows(read(0), ra[[0, 79]], tdtype, "prompt step")
    for t in range(10):
        want = [ra[80 + t]] + ([rb[20 + t]] if t % 2 else [])
        assert_rows(read(t + 1), torch.stack(want), tdtype, f"decode step {t}")


def test_command_line_makes_and_runs_a_fetitar_folder(tmp_path):
    """`random` writes a folder from a configuration file, `run` generates from it: greedy tokens are the plain
    implementation's, a seeded sampled request gives the same tokens twice."""
    cfg_path = tmp_path / "cfg.json"
    cfg_path.write_text(json.dumps(tf.CONFIGS["C"]))
    folder = tmp_path / "model"
    made = subprocess.run([sys.executable, "-m", "dotllm_b200", "random", str(cfg_path), str(folder), "--seed", "3", "--dtype", "float32"],
                          cwd=ROOT, capture_output=True, text=True, timeout=600)
    assert made.returncode == 0, made.stderr[-2000:]
    cfg, w = tf.read_folder(folder)
    prompt = tf.random_tokens(11, cfg["vocab"], 9)
    run = lambda *extra: subprocess.run([sys.executable, "-m", "dotllm_b200", "run", str(folder), "-p", ",".join(map(str, prompt)),
                                         "-n", "6", "--dtype", "float32", "--json", *extra], cwd=ROOT, capture_output=True, text=True,
                                        timeout=600)
    proc = run("-t", "0", "--stop-ids", "")
    assert proc.returncode == 0, proc.stderr[-2000:]
    tokens = json.loads(proc.stdout)["results"][0]["generated_token_ids"]
    ref = tf.plain_logits(cfg, w, prompt + tokens)
    assert tokens == [int(ref[len(prompt) - 1 + i].argmax()) for i in range(6)]
    a, b = run("-t", "0.9", "--top-k", "30", "-s", "5"), run("-t", "0.9", "--top-k", "30", "-s", "5")
    assert a.returncode == 0 and json.loads(a.stdout)["results"][0]["generated_token_ids"] == \
        json.loads(b.stdout)["results"][0]["generated_token_ids"]
