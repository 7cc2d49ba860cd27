"""Semanex on the GPU against the plain implementation: each new or changed kernel alone, whole prompts, portions, token-by-token
decoding, unequal batches, slots, states and pages that are used again, far keys, the first tokens, sinks and caps that decide
rows, long decoding over page borders, generation through the entry point, the replay program, the command line."""
import copy
import json
import os
import random
import subprocess
import sys

import numpy as np
import pytest
import torch

import kernel_refs
import tiny_semanex as ts
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
    return tmp_path_factory.mktemp("semanex")


_loaded = {}


def load_pair(tmp, which, dtype, seed=0, change=None, tag=""):
    from dotllm_b200 import Model
    key = (which, dtype, seed, tag)
    if key not in _loaded:
        folder = ts.make_folder(tmp / tag if tag else tmp, which, seed=seed, dtype=dtype)
        if change is not None:
            ts.rewrite(folder, change)
        cfg, weights = ts.read_folder(folder)
        _loaded[key] = (Model.load(folder, dtype=dtype), cfg, weights, folder)
    return _loaded[key]


def g32(*shape, seed=0, scale=1.0):
    return (torch.randn(*shape, generator=torch.Generator().manual_seed(seed), dtype=torch.float32) * scale).to(DEV)


def i32(values):
    return torch.tensor(list(values), dtype=torch.int32, device=DEV)


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
    cache.close_sequence(seq)
    cache.check()
    return torch.cat(outs)


# ------------------------------------------------------------------ kernels alone
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H", [52, 64, 1000, 1028, 4096, 7000, 9000])
def test_the_norm_behind_the_sum_alone(H, dtype):
    T, K = 5, 4
    x, y = g32(T, H, seed=1, scale=2.0), g32(T, H, seed=2)
    taps, slots = g32(K, H, seed=4, scale=0.5), i32([4, 0, 2, 5, 1])
    for gain in (g32(1, seed=3) + 2.0, g32(H, seed=3)):
        for branch in (y, y.to(torch.bfloat16), None):
            write = ops.PostNormed(branch, 2.5, gain, 1e-5) if branch is not None else None
            rwrite = kernel_refs.PostNormed(branch.cpu(), 2.5, gain.cpu(), 1e-5) if branch is not None else None
            xa, xb = x.clone(), x.cpu().clone()
            got, want = ops.post_norm(xa, write, dtype), kernel_refs.post_norm(xb, rwrite, dtype)
            close(got, want, dtype), close(xa, xb, torch.float32)
            xa, xb = x.clone(), x.cpu().clone()                       # the model's last norm on top
            got, want = ops.post_norm(xa, write, dtype, last=(gain, 1e-6)), kernel_refs.post_norm(xb, rwrite, dtype, last=(gain.cpu(), 1e-6))
            close(got, want, dtype), close(xa, xb, torch.float32)
            xa, xb = x.clone(), x.cpu().clone()                       # the next mixer's input convolution on top, twice in a row
            memory = g32(7, (K - 1) * H, seed=5)
            rmem = memory.cpu().clone()
            for _ in range(2):
                got = ops.post_norm(xa, write, dtype, conv=(taps, memory, slots))
                want = kernel_refs.post_norm(xb, rwrite, dtype, conv=(taps.cpu(), rmem, slots.cpu()))
                close(got, want, dtype), close(xa, xb, torch.float32), close(memory, rmem, torch.float32)
    ops.post_norm(x, ops.PostNormed(y, 0.0, g32(1, seed=3), 1e-5))    # without a copy
    idle = torch.full((T,), 7, dtype=torch.int32, device=DEV)         # a slot outside the memory: no convolution, nothing written
    before = memory.clone()
    assert torch.equal(ops.post_norm(x, None, torch.float32, conv=(taps, memory, idle)), x) and torch.equal(memory, before)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("C,K", [(64, 4), (52, 3), (101, 5), (96, 1), (40, 2), (1024, 4), (24, 9), (20, 40), (33, 20)])
def test_causal_convolution_alone(C, K, dtype):
    """Unequal prompts, portions (shorter than the taps and longer than a run) and single tokens, in slots that are not neighbours."""
    taps, bias = g32(K, C, seed=1, scale=0.5), g32(C, seed=2)
    memory = torch.zeros((6, 8 + (K - 1) * C), dtype=torch.float32, device=DEV)
    rmem, view = memory.cpu().clone(), (lambda m: m[:, 8:])             # a slot's history behind something else
    slots = i32([4, 0, 2])
    for n, sizes in enumerate(([1, 70, 9], [2, 1, 130], [1, 1, 1], [3, 2, 1])):
        T = sum(sizes)
        x = g32(T, C + 16, seed=10 + n).to(dtype)[:, :C]
        cu = i32([0] + list(np.cumsum(sizes)))
        kw = dict(bias=bias, activation="silu") if n % 2 == 0 else dict(add_input=True, out_dtype=dtype)
        rkw = {k: v.cpu() if torch.is_tensor(v) else v for k, v in kw.items()}
        got = ops.causal_conv(x, taps, view(memory), cu, slots, max(sizes), **kw)
        want = kernel_refs.causal_conv(x.cpu(), taps.cpu(), view(rmem), cu.cpu(), slots.cpu(), max(sizes), **rkw)
        close(got, want, dtype if n % 2 else torch.float32)
        close(memory, rmem, torch.float32)


@pytest.mark.parametrize("dtype,side", [(torch.float32, 0), (torch.bfloat16, 296), (torch.bfloat16, 0)])
@pytest.mark.parametrize("H,G,N,P", [(4, 2, 40, 48), (2, 1, 16, 8), (3, 1, 256, 40), (2, 2, 128, 128), (3, 3, 1, 5), (6, 1, 19, 7), (8, 2, 128, 64), (2, 1, 64, 24), (2, 2, 200, 10), (1, 1, 400, 9),
                                     (5, 5, 32, 33)])
def test_state_space_scan_alone(monkeypatch, H, G, N, P, dtype, side):
    """Unequal prompts, then portions and single tokens from the states they left, in slots that are not neighbours; the step
    logits span decays from almost one to almost nothing.  bfloat16 prompts go a chunk at a time through the tensor cores where
    the sizes allow - the chunks side by side in three launches, or walked in one - and give the scan's float32 results."""
    monkeypatch.setattr(ops, "SSD_SIDE_BLOCKS", side)
    bias, a_log, skip = g32(H, seed=1), g32(H, seed=2, scale=0.7), g32(H, seed=3)
    memory = torch.zeros((6, H * N * P + 12), dtype=torch.float32, device=DEV)
    rmem = memory.cpu().clone()
    slots = i32([4, 0, 2])
    for n, sizes in enumerate(([1, 37, 70], [5, 1, 2], [1, 1, 1], [230, 64, 65])):
        T = sum(sizes)
        xbc = g32(T, H * P + 2 * G * N + 8, seed=10 + n, scale=0.7).to(dtype)[:, :H * P + 2 * G * N]
        z = g32(T, H + 3, seed=20 + n, scale=3.0).to(dtype)[:, 1:H + 1]
        cu = i32([0] + list(np.cumsum(sizes)))
        got = ops.ssd_scan(xbc, z, bias, a_log, skip, cu, slots, memory, H, G, N, P, max_new=max(sizes))
        want = kernel_refs.ssd_scan(xbc.cpu(), z.cpu(), bias.cpu(), a_log.cpu(), skip.cpu(), cu.cpu(), slots.cpu(), rmem, H, G, N, P)
        close(got, want, torch.float32), close(memory, rmem, torch.float32)


@pytest.mark.parametrize("dtype", DTYPES)
def test_gates_and_the_norm_over_parts_alone(dtype):
    for W, parts, scale in ((96, 1, 1.0), (90, 5, 0.4), (4096, 2, 0.5), (6000, 1, 2.0), (64, 64, 1.0)):
        y, gate, gain = g32(6, W, seed=1, scale=3.0), g32(6, W + 8, seed=2).to(dtype)[:, :W], g32(W, seed=3)
        wide = torch.zeros((6, W + 24), dtype=dtype, device=DEV)
        got = ops.gated_group_norm(y, gate, gain, parts, 1e-6, scale=scale, out=wide[:, 8:8 + W])
        close(got, kernel_refs.gated_group_norm(y.cpu(), gate.cpu(), gain.cpu(), parts, 1e-6, scale=scale), dtype)
        assert not wide[:, :8].any() and not wide[:, 8 + W:].any()
    for heads, width, lay, scale in ((4, 24, 32, 0.7), (3, 5, 5, 1.0), (8, 64, 128, 0.3), (2, 128, 128, 1.0)):
        o, gate = g32(7, heads * lay, seed=4).to(dtype), g32(7, heads * width + 8, seed=5).to(dtype)[:, 8:]
        close(ops.channel_gate(o, gate, heads, width, lay=lay, scale=scale),
              kernel_refs.channel_gate(o.cpu(), gate.cpu(), heads, width, lay=lay, scale=scale), dtype)
        close(ops.channel_gate(o, None, heads, width, lay=lay, scale=scale), kernel_refs.channel_gate(o.cpu(), None, heads, width, lay=lay, scale=scale), dtype)
    x, ga, gb = g32(5, 6 * 24 + 8, seed=6).to(dtype)[:, :6 * 24], g32(24, seed=7), g32(24, seed=8)
    close(ops.head_rmsnorm(x, ga, 4, 24, 1e-6, gb, 2, lay=32), kernel_refs.head_rmsnorm(x.cpu(), ga.cpu(), 4, 24, 1e-6, gb.cpu(), 2, lay=32), dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T", [9, 3, 40, 150])
@pytest.mark.parametrize("H,dim,rot,dims,rq,r,lay", [(4, 20, 8, 8, 28, 40, 64), (4, 24, 8, 8, 1536, 104, 128), (2, 8, 8, 8, 2056, 24, 32), (2, 72, 64, 64, 32, 64, 128), (3, 7, 6, 0, 11, 13, 19), (6, 32, 32, 32, 96, 96, 128), (5, 16, 24, 12, 0, 40, 64)])
def test_latent_rows_and_queries_alone(H, dim, rot, dims, rq, r, lay, T, dtype):
    x = g32(T, rq + r + rot + 8, seed=1).to(dtype)[:, :rq + r + rot]
    pos = i32(([0, 1, 5, 63, 64, 99, 2, 2, 7] * 20)[:T])
    angle = torch.arange(100)[:, None] * 0.37 ** torch.arange(max(1, dims // 2))[None, :]
    tables = (torch.cos(angle).to(DEV).float().contiguous(), torch.sin(angle).to(DEV).float().contiguous()) if dims else None
    rtables = tuple(t.cpu() for t in tables) if dims else None
    qg, kg = (g32(rq, seed=2) if rq else None), g32(r, seed=3)
    cq, rows = ops.latent_rows(x, qg, kg, 1e-6, rot, tables, pos, lay)
    wcq, wrows = kernel_refs.latent_rows(x.cpu(), None if qg is None else qg.cpu(), kg.cpu(), 1e-6, rot, rtables, pos.cpu(), lay)
    close(rows, wrows, dtype)
    assert not rows[:, r + rot:].any() and ((cq is None) if not rq else close(cq, wcq, dtype) is None)
    q, w = g32(T, H * (dim + rot), seed=4).to(dtype), g32(H, r, dim, seed=5, scale=0.3).to(dtype)
    got = ops.latent_queries(q, w, rot, tables, pos, lay)
    close(got, kernel_refs.latent_queries(q.cpu(), w.cpu(), rot, rtables, pos.cpu(), lay), dtype)
    assert not got.view(T, H, lay)[:, :, r + rot:].any()
    wo = g32(H, 12, r, seed=6, scale=0.3).to(dtype)
    gate = g32(T, H * 12 + 8, seed=7).to(dtype)[:, 8:]
    for gt in (gate, None):
        close(ops.latent_values(got, wo, lay, gate=gt), kernel_refs.latent_values(got.cpu(), wo.cpu(), lay, gate=None if gt is None else gt.cpu()), dtype)
    close(ops.linear_per_head(got, wo, x_head=lay), kernel_refs.linear_per_head(got.cpu(), wo.cpu(), x_head=lay), dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows", [3, 40, 200])
def test_exact_gelu_behind_a_product(rows, dtype):
    """In the weight-streaming product's epilogue (few rows), behind the library's (some), in the tcgen05 product's (many)."""
    x, w = g32(rows, 96, seed=1).to(dtype), g32(160, 96, seed=2, scale=0.3).to(dtype)
    close(ops.activated_linear(x, w, "gelu"), torch.nn.functional.gelu(x.double().cpu() @ w.double().cpu().T), dtype)
    z = torch.linspace(-6, 6, 4 * 50, device=DEV).reshape(4, 50).to(dtype)
    close(ops.unary_activation(z, "gelu"), torch.nn.functional.gelu(z.double().cpu()), dtype, 1e-6, 1e-2)


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
@pytest.mark.parametrize("nh,nkv", [(4, 2), (20, 1), (32, 1), (24, 8), (17, 1)])
def test_capped_scores_sinks_and_wide_groups_in_the_tensor_core_kernels(nh, nkv, hd):
    """Decode (scores capped, sinks, more query heads on a key head than a tile has rows, the step's own token written inside) and both
    prompt kernels, against the plain attention; with a cap that bends the scores the uncapped result is far away."""
    from dotllm_b200.engine.step import AttentionPlan
    lens = [1, 70, 200]
    B, pages = len(lens), 4
    k, v, table = _paged(B, pages, nkv, hd, lens, seed=hd + nh)
    sinks = g32(nh, seed=3)
    scale = 2.0 * hd ** -0.5
    hook = ops.ScoreHook(1.5)
    cases = [("decode", [n - 1 for n in lens], [1] * B), ("prompt", [0, 10, 0], [1, 60, 200])]
    for name, starts, news in cases:
        q = g32(sum(news), nh * hd, seed=5).to(torch.bfloat16)
        seq = i32([b for b in range(B) for _ in range(news[b])])
        pos = i32([starts[b] + i for b in range(B) for i in range(news[b])])
        plan = lambda: AttentionPlan(B, max(news), max(lens), name == "decode", i32(starts), i32(news), i32([0] + list(np.cumsum(news))), i32(lens),
                                     list(starts), list(news))
        for h, s in ((hook, None), (None, sinks), (hook, sinks)):
            want = kernel_refs.attention(q.cpu(), k, v, seq.cpu(), pos.cpu(), table, nh, nkv, hd, scale, score_hook=h, sinks=None if s is None else s.cpu())
            got = ops.attention(q, k.to(DEV), v.to(DEV), seq, pos, table.to(DEV), nh, nkv, hd, scale, plan=plan(), score_hook=h, sinks=s, split=True)
            close(got, want, torch.bfloat16)
            if name == "prompt" and hd in attention_fast.PREFILL_TC_HEAD_DIMS:
                try:
                    attention_fast.PREFILL_TC = False                    # the mma.sync kernel at the same sizes
                    close(ops.attention(q, k.to(DEV), v.to(DEV), seq, pos, table.to(DEV), nh, nkv, hd, scale, plan=plan(), score_hook=h, sinks=s, split=True), want,
                          torch.bfloat16)
                finally:
                    attention_fast.PREFILL_TC = True
            if h is not None and s is None:
                plain = kernel_refs.attention(q.cpu(), k, v, seq.cpu(), pos.cpu(), table, nh, nkv, hd, scale)
                assert float((plain.double() - want.double()).abs().max() / want.double().abs().max()) > 0.1
        if name == "decode":                                             # the new token's key and value come with the call
            kd, vd = k.to(DEV), v.to(DEV)
            fresh_k, fresh_v = g32(B, nkv * hd, seed=7).to(torch.bfloat16), g32(B, nkv * hd, seed=8).to(torch.bfloat16)
            got = ops.rope_cache_attention(q, fresh_k, fresh_v, None, None, 0, seq, pos, table.to(DEV), kd, vd, nh, nkv, hd, scale, plan=plan(),
                                           score_hook=hook, sinks=sinks, split=True)
            kr, vr = k.clone(), v.clone()
            kernel_refs.rope_cache_write(q.cpu().clone(), fresh_k.cpu(), fresh_v.cpu(), None, None, 0, seq.cpu(), pos.cpu(), table, kr, vr, nh, nkv, hd)
            want = kernel_refs.attention(q.cpu(), kr, vr, seq.cpu(), pos.cpu(), table, nh, nkv, hd, scale, score_hook=hook, sinks=sinks.cpu())
            close(got, want, torch.bfloat16)
            assert torch.equal(torch.nan_to_num(kd.cpu().float()), torch.nan_to_num(kr.float())) and \
                torch.equal(torch.nan_to_num(vd.cpu().float()), torch.nan_to_num(vr.float()))


# ------------------------------------------------------------------ the model
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("which", ["A", "B", "C", "D", "E"])
def test_whole_portions_and_decoding(tmp, which, dtype):
    model, cfg, w, _ = load_pair(tmp, which, dtype)
    tokens = ts.random_tokens(150, cfg["vocab"], 7)
    ref = ts.plain_logits(cfg, w, tokens)
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
    prompts = [ts.random_tokens(n + 12, cfg["vocab"], 20 + n) for n in lens]
    refs = [ts.plain_logits(cfg, w, p) for p in prompts]
    cache = model.new_cache(64 * 8)
    for round_ in range(2):                                          # the second time every slot, state and page has been used before
        cache.fill_free_pages(float("nan"))
        seqs = [cache.open_sequence() for _ in prompts]
        order = list(range(len(prompts))) if round_ == 0 else [2, 0, 3, 1]
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
def test_steps_that_mix_portions_and_single_tokens(tmp, dtype):
    """One step with a prompt, a portion of another, and sequences that go on by one token."""
    from dotllm_b200.engine import StepEntry
    model, cfg, w, _ = load_pair(tmp, "A", dtype)
    prompts = [ts.random_tokens(n, cfg["vocab"], 90 + n) for n in (90, 140, 30, 66)]
    refs = [ts.plain_logits(cfg, w, p) for p in prompts]
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
    """Width 1,024, heads of 128 channels, a state of 128, latents of 96 + 32 and 64 + 64: the sizes of the tensor-core kernels."""
    model, cfg, w, _ = load_pair(tmp, "wide", dtype)
    tokens = ts.random_tokens(230, cfg["vocab"], 11)
    ref = ts.plain_logits(cfg, w, tokens)
    assert_rows(run_cuts(model, tokens, [200]), ref, dtype, "a prompt of 200 tokens and 30 decoded")
    assert_rows(run_cuts(model, tokens[:200], [130, 70]), ref[:200], dtype, "two portions")


@pytest.mark.parametrize("seed", range(8))
def test_configurations_drawn_at_random(tmp_path, seed):
    """Configurations that nobody chose (`tiny_semanex.random_config`): a prompt and twenty decoded tokens, then a batch of
    three unequal prompts (one of a single token) decoded together, eager and through captured steps, in both dtypes."""
    from dotllm_b200 import Model
    from dotllm_b200.engine import StepEntry
    rng = random.Random(300 + seed)
    cfg_dict = ts.random_config(rng)
    n = rng.randrange(100, 200)
    lens = [1, rng.randrange(2, 80), rng.randrange(80, 150)]
    for dtype in DTYPES:
        folder = ts.make_folder(tmp_path, f"random{seed}", dtype=dtype, cfg=cfg_dict)
        cfg, w = ts.read_folder(folder)
        model = Model.load(folder, dtype=dtype)
        tokens = ts.random_tokens(n, cfg["vocab"], seed)
        prompts = [ts.random_tokens(L + 8, cfg["vocab"], seed * 7 + L) for L in lens]
        ref, refs = ts.plain_logits(cfg, w, tokens), [ts.plain_logits(cfg, w, p) for p in prompts]
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
        err = row_errors(torch.cat(got), torch.cat(want))
        # (a norm over a part whose values nearly vanish magnifies whatever rounding is in front of it: the odd row in bfloat16)
        over = int((err > REL[dtype]).sum())
        assert torch.isfinite(err).all() and float(err.max()) <= (REL[dtype] if dtype == torch.float32 else 0.2) and \
            over <= (0 if dtype == torch.float32 else 2) and float(err.median()) <= REL[dtype] / 3, (seed, dtype, float(err.max()), over, cfg_dict)


def _sharp_latent(t):
    t["l0.mix.uq"] *= 2.0
    t["l0.mix.o"] *= 12.0
    t["l0.mix.sink"] += 12.0


def test_far_keys_the_rotation_and_the_sinks_decide_whole_rows(tmp):
    """One latent-attention layer whose scores are scaled until single keys decide.  Dropping the keys beyond the last hundred, pairing
    the rotated channels the other way and leaving the sinks out must each change many rows of the plain result; the engine
    agrees with the design over prompts, portions and decoding."""
    import plain_semanex as ps
    tokens = ts.random_tokens(400, 120, 5)
    model, cfg, w, _ = load_pair(tmp, "sharp_latent", torch.float32, change=_sharp_latent, tag="sharp")
    ref = ts.plain_logits(cfg, w, tokens)
    rms = ref.pow(2).mean(-1).sqrt()
    differs = lambda other: int(((other - ref).pow(2).mean(-1).sqrt() / rms > 1e-2).sum())
    saved = ps.softmax_attention, ps.rotate_interleaved

    def near_only(q, k, v, scale, softcap=None, sink=None):
        out = saved[0](q, k, v, scale, softcap, sink)
        for i in range(100, len(q)):
            out[i] = saved[0](q[i - 99:i + 1], k[i - 99:i + 1], v[i - 99:i + 1], scale, softcap, sink)[-1]
        return out

    def half_pairs(x, positions, dims, base):
        order = list(range(0, dims, 2)) + list(range(1, dims, 2))
        y = x.copy()
        y[..., :dims] = saved[1](x[..., :dims][..., np.argsort(order)], positions, dims, base)[..., order]
        return y
    try:
        ps.softmax_attention = near_only
        assert differs(ts.plain_logits(cfg, w, tokens)) >= 20
        ps.softmax_attention = lambda q, k, v, scale, softcap=None, sink=None: saved[0](q, k, v, scale, softcap, None)
        without = ts.plain_logits(cfg, w, tokens)
        assert differs(without) >= 20 and int(((without - ref).pow(2).mean(-1).sqrt() / rms > 1e-2)[:12].sum()) >= 4
        ps.softmax_attention = saved[0]
        ps.rotate_interleaved = half_pairs
        assert differs(ts.plain_logits(cfg, w, tokens)) >= 20
    finally:
        ps.softmax_attention, ps.rotate_interleaved = saved
    for cuts in ([400], [63, 1, 1, 200], [128, 64, 2], [350], [20]):
        assert rel_err(run_cuts(model, tokens, cuts), ref) < 1e-4, cuts
    bf = load_pair(tmp, "sharp_latent", torch.bfloat16, change=_sharp_latent, tag="sharp")
    ref16 = ts.plain_logits(bf[1], bf[2], tokens)
    for cuts in ([380], [100]):
        row_err = row_errors(run_cuts(bf[0], tokens, cuts), ref16)
        assert float(row_err.median()) < 3e-2 and int((row_err > 0.3).sum()) <= 8, (cuts, float(row_err.median()), int((row_err > 0.3).sum()))


def _sharp_capped(t):
    t["l0.mix.left.q.norm"] *= 1.0
    t["l0.mix.left.k.norm"] *= 2.0
    t["l0.mix.left.o"] *= 12.0


def test_far_keys_and_the_cap_decide_whole_rows(tmp):
    """One parallel layer whose attention is sharpened the same way: without the far keys, without the cap, with a cap a tenth larger
    and with the norm of queries and keys left out many rows of the plain result change; the engine agrees with the design."""
    import plain_semanex as ps
    tokens = ts.random_tokens(330, 120, 6)
    model, cfg, w, _ = load_pair(tmp, "sharp_capped", torch.float32, change=_sharp_capped, tag="sharp")
    ref = ts.plain_logits(cfg, w, tokens)
    rms = ref.pow(2).mean(-1).sqrt()
    differs = lambda other: int(((other - ref).pow(2).mean(-1).sqrt() / rms > 1e-2).sum())

    def with_cap(cap):
        other = copy.deepcopy(cfg)
        other["layers"][0]["mixer"]["left"]["softcap"] = cap
        return ts.plain_logits(other, w, tokens)

    saved = ps.softmax_attention
    try:
        def near_only(q, k, v, scale, softcap=None, sink=None):
            out = saved(q, k, v, scale, softcap, sink)
            for i in range(100, len(q)):
                out[i] = saved(q[i - 99:i + 1], k[i - 99:i + 1], v[i - 99:i + 1], scale, softcap, sink)[-1]
            return out
        ps.softmax_attention = near_only
        assert differs(ts.plain_logits(cfg, w, tokens)) >= 20
    finally:
        ps.softmax_attention = saved
    assert differs(with_cap(None)) >= 20 and differs(with_cap(22.0)) >= 20
    for cuts in ([330], [63, 1, 1, 200], [128, 64, 2], [290], [20]):
        assert rel_err(run_cuts(model, tokens, cuts), ref) < 1e-4, cuts
    bf = load_pair(tmp, "sharp_capped", torch.bfloat16, change=_sharp_capped, tag="sharp")
    ref16 = ts.plain_logits(bf[1], bf[2], tokens)
    for cuts in ([300], [100]):
        row_err = row_errors(run_cuts(bf[0], tokens, cuts), ref16)
        assert float(row_err.median()) < 3e-2 and int((row_err > 0.3).sum()) <= 8, (cuts, float(row_err.median()), int((row_err > 0.3).sum()))


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding_over_page_borders(tmp, dtype):
    model, cfg, w, _ = load_pair(tmp, "A", dtype)
    tokens = ts.random_tokens(330, cfg["vocab"], 5)
    ref = ts.plain_logits(cfg, w, tokens)
    got = run_cuts(model, tokens, [30])                              # 300 tokens one by one, over five page borders
    assert_rows(got, ref, dtype, "300 decoded tokens")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("which", ["A", "B"])
def test_greedy_generation_through_the_entry_point(tmp, which, dtype):
    from dotllm_b200 import InferenceOptions
    model, cfg, w, _ = load_pair(tmp, which, dtype)
    prompts = [ts.random_tokens(n, cfg["vocab"], 60 + n) for n in (1, 9, 40, 70)]
    n_new = 24
    options = InferenceOptions(temperature=0.0, max_tokens=n_new, stop_token_ids=[])
    outs = model.generate(prompts, options)
    for p, o in zip(prompts, outs):
        assert o.finish_reason.value == "length" and o.generated_token_count == n_new
        ref = ts.plain_logits(cfg, w, p + o.generated_token_ids)
        spread = float(ref.std())
        for i, tok in enumerate(o.generated_token_ids):              # teacher-forced: the plain arg-max, or within rounding of it
            row = ref[len(p) - 1 + i]
            assert int(row.argmax()) == tok or float(row.max() - row[tok]) <= (1e-4 if dtype == torch.float32 else 0.1) * spread, \
                (i, tok, int(row.argmax()))
    again = model.generate(prompts, options)                         # through captured steps now
    alone = model.generate(prompts[2], options)
    if dtype == torch.float32:
        assert [o.generated_token_ids for o in again] == [o.generated_token_ids for o in outs]
        assert alone.generated_token_ids == outs[2].generated_token_ids


def test_decode_steps_replayed_from_graphs(tmp):
    """Steps captured as graphs (exact batch size and the shared widths with idle rows) give the eager steps' logits."""
    from dotllm_b200.engine import StepEntry
    for dtype in DTYPES:
        model, cfg, w, _ = load_pair(tmp, "A", dtype)
        prompts = [ts.random_tokens(n + 10, cfg["vocab"], 80 + n) for n in (5, 66, 30)]
        refs = [ts.plain_logits(cfg, w, p) for p in prompts]
        for graphs in (True, "lazy"):
            cache = model.new_cache(64 * 6)
            seqs = [cache.open_sequence() for _ in prompts]
            model.step(cache, [StepEntry(s, p[:-10], []) for s, p in zip(seqs, prompts)])
            for t in range(10):
                out = model.step(cache, [StepEntry(s, [p[len(p) - 10 + t]]) for s, p in zip(seqs, prompts)], graphs=graphs)
                assert_rows(out, torch.stack([r[len(r) - 10 + t] for r in refs]), dtype, f"graphs={graphs} step {t}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_replay_program_on_a_semanex_folder(tmp_path, dtype):
    tdtype = {"float32": torch.float32, "bfloat16": torch.bfloat16}[dtype]
    folder = ts.make_folder(tmp_path, "D", seed=2, dtype=tdtype)
    cfg, w = ts.read_folder(folder)
    a, b = ts.random_tokens(90, cfg["vocab"], 1), ts.random_tokens(30, cfg["vocab"], 2)
    ra, rb = ts.plain_logits(cfg, w, a), ts.plain_logits(cfg, w, b)
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


def test_command_line_makes_and_runs_a_semanex_folder(tmp_path):
    """`random` writes a folder from a configuration file, `run` generates from it: greedy tokens are the plain
    implementation's, a seeded sampled request gives the same tokens twice."""
    cfg_path = tmp_path / "cfg.json"
    cfg_path.write_text(json.dumps(ts.CONFIGS["C"]))
    folder = tmp_path / "model"
    made = subprocess.run([sys.executable, "-m", "dotllm_b200", "random", str(cfg_path), str(folder), "--seed", "3", "--dtype", "float32"],
                          cwd=ROOT, capture_output=True, text=True, timeout=600)
    assert made.returncode == 0, made.stderr[-2000:]
    cfg, w = ts.read_folder(folder)
    prompt = ts.random_tokens(11, cfg["vocab"], 9)
    run = lambda *extra: subprocess.run([sys.executable, "-m", "dotllm_b200", "run", str(folder), "-p", ",".join(map(str, prompt)),
                                         "-n", "6", "--dtype", "float32", "--json", *extra], cwd=ROOT, capture_output=True, text=True,
                                        timeout=600)
    proc = run("-t", "0", "--stop-ids", "")
    assert proc.returncode == 0, proc.stderr[-2000:]
    tokens = json.loads(proc.stdout)["results"][0]["generated_token_ids"]
    ref = ts.plain_logits(cfg, w, prompt + tokens)
    assert tokens == [int(ref[len(prompt) - 1 + i].argmax()) for i in range(6)]
    a, b = run("-t", "0.9", "--top-k", "30", "-s", "5"), run("-t", "0.9", "--top-k", "30", "-s", "5")
    assert a.returncode == 0 and json.loads(a.stdout)["results"][0]["generated_token_ids"] == \
        json.loads(b.stdout)["results"][0]["generated_token_ids"]
