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
@pytest.mark.parametrize("H,buckets,mul_prev,mul_cur", [(52, 1, 3, 5), (64, 97, 31, 7), (101, 40, -13, 29), (1028, 1000, 2000000011, 2000000089), (4096, 3, 0, 1)])
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
        for window, h, g in ((65, hook, gate), (64, None, gate), (40, hook, None)) + (((0, hook, None), (1, hook, gate)) if name == "decode" or hd == 64 else ()):
            want = ref(window=window, score_hook=rhook if h is not None else None, gate=cpu(g))
            run = lambda: ops.attention(q, k.to(DEV), v.to(DEV), seq, pos, table.to(DEV), *args, window, plan=plan(), score_hook=h, gate=g, split=True)
            close(run(), want, torch.bfloat16)
            if name == "prompt" and hd in attention_fast.PREFILL_TC_HEAD_DIMS:
                try:
                    attention_fast.PREFILL_TC = False                    # the mma.sync kernel at the same sizes
                    close(run(), want, torch.bfloat16)
                finally:
                    attention_fast.PREFILL_TC = True
            if window == 40 and name == "prompt":
                far = lambda other: float((other.double() - want.double()).abs().max() / want.double().abs().max())
                assert far(ref(window=41, score_hook=rhook)) > 0.05 and far(ref(window=40)) > 0.1
                assert far(ref(window=40, score_hook=ops.ScoreHook(0.0, slopes.cpu().roll(1)))) > 0.1
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
