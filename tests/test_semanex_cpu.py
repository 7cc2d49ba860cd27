"""Semanex without a GPU: configuration, model description, tensor names, cache needs, the plain implementation's own mechanisms,
and the engine's host logic (steps, cache, schedule) with the plain kernel references."""
import copy
import json
import math
import random

import numpy as np
import pytest
import torch

import plain_semanex as ps
import tiny_semanex as ts
from dotllm_b200.config import build_spec, config_from_dict, load_config
from dotllm_b200.engine import StepEntry, run_step
from dotllm_b200.errors import ConfigError
from dotllm_b200.models.decoder import DecoderModel
from dotllm_b200.parts.base import Runtime
from dotllm_b200.weights import load_into

CPU = Runtime(torch.float32, torch.device("cpu"))


def test_configuration_reads_every_key_and_writes_it_back():
    for name, d in ts.CONFIGS.items():
        cfg = config_from_dict(copy.deepcopy(d))
        assert cfg.to_dict() == d, name
        assert type(cfg).__name__ == "SemanexConfig"
    for broken, match in ((lambda c: c.pop("width"), "width"), (lambda c: c.pop("postln_alpha"), "postln_alpha"),
                          (lambda c: c.pop("canon"), "taps"), (lambda c: c["canon"].update(taps=0), "taps"),
                          (lambda c: c["layers"][0].update(type="gla"), "type"),
                          (lambda c: c["layers"][0]["mixer"].pop("left_scale"), "left_scale"),
                          (lambda c: c["layers"][0]["mixer"]["left"].update(kv_heads=4), "kv_heads"),
                          (lambda c: c["layers"][0]["mixer"]["left"].update(softcap=-1.0), "softcap"),
                          (lambda c: c["layers"][0]["mixer"]["right"].update(groups=4), "groups"),
                          (lambda c: c["layers"][0]["mixer"]["right"].update(norm_groups=7), "norm_groups"),
                          (lambda c: c["layers"][0]["mixer"]["right"].pop("state"), "state"),
                          (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=10), "rot"),
                          (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=3), "rot"),
                          (lambda c: c["layers"][1]["mixer"].pop("rot"), "rot"),
                          (lambda c: c["layers"][1]["mixer"].pop("kv_rank"), "kv_rank"),
                          (lambda c: c["layers"][1]["mixer"].update(scale=0.0), "scale"),
                          (lambda c: c["layers"][0]["mlp"].update(kind="moe"), "kind"),
                          (lambda c: c["layers"][0]["mlp"].update(ff=0), "mlp")):
        bad = copy.deepcopy(ts.CONFIGS["A"])
        broken(bad)
        with pytest.raises(ConfigError, match=match):
            config_from_dict(bad)


def test_description_tensor_names_and_cache_needs():
    spec = build_spec(config_from_dict(copy.deepcopy(ts.CONFIGS["A"])))
    model = DecoderModel(spec, CPU)
    expected, optional = model.expected_weights()
    sides = ["left.q", "left.k", "left.v", "left.q.norm", "left.k.norm", "left.g", "left.o", "right.in", "right.conv", "right.conv.b",
             "right.dt_bias", "right.A_log", "right.D", "right.norm", "right.o"]
    latent = ["dq", "dq.norm", "uq", "dkv", "dkv.norm", "uk", "uv", "sink", "g", "o"]
    want = {"embed", "head", "final.norm"}
    for i, (mix, mlp) in enumerate(((sides, True), (latent, True), (sides, False), (latent, False))):
        want |= {f"l{i}.canon1", f"l{i}.norm1"} | {f"l{i}.mix.{n}" for n in mix}
        want |= {f"l{i}.norm2", f"l{i}.mlp.up", f"l{i}.mlp.down"} if mlp else set()
    assert set(expected) == want and not optional
    shape = lambda n: tuple(expected[n].shape)
    assert shape("l0.norm1") == () and shape("final.norm") == () and shape("l0.canon1") == (80, 3)
    assert shape("l0.mix.left.g") == (120, 80) and shape("l0.mix.left.q.norm") == (24,) and shape("l0.mix.left.v") == (40, 80)
    assert shape("l0.mix.right.in") == (2 * 60 + 2 * 2 * 20 + 6, 80) and shape("l0.mix.right.conv") == (60 + 80, 3)
    assert shape("l1.mix.uq") == (4 * 28, 28) and shape("l1.mix.dkv") == (48, 80) and shape("l1.mix.uk") == (80, 40)
    assert shape("l1.mix.g") == (48, 80) and shape("l1.mix.sink") == (4,)
    needs = model.cache_needs()
    assert [n.kind for n in needs[0]] == ["state", "kv", "state"] and [n.kind for n in needs[1]] == ["state", "kv"]
    assert needs[0][0].state_shape == (2 * 80,) and needs[0][2].state_shape == (6 * 20 * 10 + 2 * 140,)
    assert (needs[0][1].key_width(), needs[0][1].value_width()) == (24, 20) and (needs[1][1].key_width(), needs[1][1].value_width()) == (48, 40)
    # bfloat16 rows that fit a tensor-core width are laid out at it: heads of 24 and 20 at 32, a latent row of 48 at 64
    wide = DecoderModel(spec, Runtime(torch.bfloat16, torch.device("cpu"))).cache_needs()
    assert (wide[0][1].key_width(), wide[0][1].value_width()) == (32, 32) and (wide[1][1].key_width(), wide[1][1].value_width()) == (64, 64)
    with pytest.raises(ConfigError, match="share its products"):
        from dotllm_b200.config.spec import PartSpec
        from dotllm_b200.parts.base import make_part
        side = {"kind": "latent_attention", "params": {"n_heads": 1, "key_dim": 8, "value_dim": 8, "q_rank": 8, "kv_rank": 8, "eps": 1e-6}}
        make_part("mixer", PartSpec("summed", {"weights": (1, 1), "left": side, "right": side}), 16, CPU)


# ------------------------------------------------------------------ the plain implementation's own mechanisms
def test_plain_convolution_and_state_space_scan_alone():
    rng = np.random.default_rng(0)
    x, taps = rng.normal(size=(12, 3)), rng.normal(size=(3, 4))
    y = ps.causal_convolution(x, taps)
    assert np.allclose(y[0], taps[:, 3] * x[0]) and np.allclose(y[5], (taps.T * x[2:6]).sum(0))
    # closed form: y_t = sum_{j<=t} exp(-rate sum_{j<i<=t} dt_i) dt_j (C_t . B_j) x_j + D x_t
    T, H, P, G, N = 7, 4, 3, 2, 5
    x, B, C = rng.normal(size=(T, H, P)), rng.normal(size=(T, G, N)), rng.normal(size=(T, G, N))
    dt, rate, D = np.abs(rng.normal(size=(T, H))), np.abs(rng.normal(size=H)), rng.normal(size=H)
    got = ps.state_space_scan(x, B, C, dt, rate, D)
    for t in range(T):
        for h in range(H):
            want = D[h] * x[t, h]
            for j in range(t + 1):
                want = want + math.exp(-rate[h] * dt[j + 1:t + 1, h].sum()) * dt[j, h] * (C[t, h // 2] @ B[j, h // 2]) * x[j, h]
            assert np.allclose(got[t, h], want)


def test_plain_attention_mechanisms_alone():
    rng = np.random.default_rng(1)
    q, k, v = rng.normal(size=(6, 4, 3)), rng.normal(size=(6, 2, 3)), rng.normal(size=(6, 2, 5))
    o = ps.softmax_attention(q, k, v, 0.7)
    assert np.allclose(o[0, :, :], v[0][[0, 0, 1, 1]])                # the first token sees itself alone
    # a sink takes exp(s) of the first token's denominator and gives nothing
    s = q[0, 3] @ k[0, 1] * 0.7
    sink = np.array([0.0, 0.0, 0.0, 1.3])
    assert np.allclose(ps.softmax_attention(q, k, v, 0.7, None, sink)[0, 3], v[0, 1] * math.exp(s) / (math.exp(s) + math.exp(1.3)))
    # a cap far above the scores changes nothing, one of almost nothing makes every visible key equal
    assert np.allclose(ps.softmax_attention(q, k, v, 0.7, 1e7), o) and np.allclose(ps.softmax_attention(q, k, v, 0.7, 1e-9)[4, 0], v[:5, 0].mean(0))
    # expanding keys and values from the latent equals attention in the latent's own basis
    m = {"heads": 2, "dim": 3, "rot_dim": 4, "vdim": 5, "q_rank": 6, "kv_rank": 7, "scale": 0.4, "rot": {"dims": 4, "base": 50.0}}
    w = {n: rng.normal(size=s) for n, s in (("dq", (6, 8)), ("uq", (14, 6)), ("dkv", (11, 8)), ("uk", (6, 7)), ("uv", (10, 7)), ("g", (10, 8)),
                                            ("sink", (2,)), ("dq.norm", (6,)), ("dkv.norm", (7,)))}
    w["o"] = np.eye(10)
    h = rng.normal(size=(9, 8))
    got = ps.latent_attention(m, w, "", h, np.arange(9), 1e-6)
    c = ps.rms((h @ w["dkv"].T)[:, :7], 1e-6) * w["dkv.norm"]
    kr = ps.rotate_interleaved((h @ w["dkv"].T)[:, None, 7:], np.arange(9), 4, 50.0)
    qq = ((ps.rms(h @ w["dq"].T, 1e-6) * w["dq.norm"]) @ w["uq"].T).reshape(9, 2, 7)
    qr = ps.rotate_interleaved(qq[..., 3:], np.arange(9), 4, 50.0)
    ql = np.einsum("thd,hdr->thr", qq[..., :3], w["uk"].reshape(2, 3, 7))
    a = ps.softmax_attention(np.concatenate([ql, qr], -1), np.concatenate([c[:, None], kr], -1), c[:, None], 0.4, None, w["sink"])
    o = np.einsum("thr,hvr->thv", a, w["uv"].reshape(2, 5, 7)).reshape(9, 10)
    assert np.allclose(got, o * ps.sigmoid(h @ w["g"].T))


def test_plain_rotation_against_the_packages_tables_and_exact_gelu():
    from dotllm_b200.parts.rotary import rotary_frequencies
    x = np.random.default_rng(3).normal(size=(5, 3, 12))
    y = ps.rotate_interleaved(x, np.arange(5), 8, 100.0)
    assert np.array_equal(y[..., 8:], x[..., 8:]) and np.array_equal(y[0], x[0])
    assert np.allclose(y[..., 0:8:2] ** 2 + y[..., 1:8:2] ** 2, x[..., 0:8:2] ** 2 + x[..., 1:8:2] ** 2)
    f = rotary_frequencies(8, 100.0)
    assert np.allclose(np.arctan2(y[1, 0, 1:8:2], y[1, 0, 0:8:2]) - np.arctan2(x[1, 0, 1:8:2], x[1, 0, 0:8:2]) - f, 0.0, atol=1e-9) or \
        np.allclose(np.exp(1j * (np.arctan2(y[1, 0, 1:8:2], y[1, 0, 0:8:2]) - np.arctan2(x[1, 0, 1:8:2], x[1, 0, 0:8:2]) - f)), 1.0)
    assert np.array_equal(ps.rotate_interleaved(x, np.arange(5), 0, 100.0), x)
    z = torch.linspace(-4, 4, 33, dtype=torch.float64)
    assert np.allclose(ps.gelu_exact(z.numpy()), torch.nn.functional.gelu(z).numpy())


# ------------------------------------------------------------------ the engine's host logic
def load(tmp_path, which, cfg=None, change=None):
    folder = ts.make_folder(tmp_path, which, cfg=cfg)
    if change is not None:
        ts.rewrite(folder, change)
    cfg, weights = ts.read_folder(folder)
    return load_into(DecoderModel(build_spec(load_config(folder)), CPU), folder), cfg, weights


@pytest.mark.parametrize("which", ["A", "C", "D", "E"])
def test_steps_cuts_and_batches_agree_with_the_plain_implementation(cpu_kernels, tmp_path, which):
    model, cfg, w = load(tmp_path, which)
    a, b = ts.random_tokens(83, cfg["vocab"], 1), ts.random_tokens(21, cfg["vocab"], 2)
    ra, rb = ts.plain_logits(cfg, w, a).float(), ts.plain_logits(cfg, w, b).float()
    near = lambda got, want: torch.allclose(got, want, atol=3e-4 * float(want.abs().max()))
    cache = model.new_cache(64 * 4)
    cache.fill_free_pages(float("nan"))
    sa, sb = cache.open_sequence(), cache.open_sequence()
    out = run_step(model, cache, [StepEntry(sa, a[:66], [0, 1, 65]), StepEntry(sb, b[:5], [4])])
    assert near(out, torch.cat([ra[[0, 1, 65]], rb[[4]]]))
    out = run_step(model, cache, [StepEntry(sa, a[66:68], [0, 1]), StepEntry(sb, b[5:19], [13])])       # portions of 2 and 14
    assert near(out, torch.cat([ra[[66, 67]], rb[[18]]]))
    for t in range(68, 83):
        entries = [StepEntry(sa, [a[t]])] + ([StepEntry(sb, [b[t - 49]])] if t - 49 < 21 else [])
        out = run_step(model, cache, entries)
        assert near(out[0], ra[t])
        if len(entries) == 2:
            assert near(out[1], rb[t - 49])
    cache.close_sequence(sa)
    cache.fill_free_pages(float("nan"))
    sc = cache.open_sequence()                           # takes the slot, the states and the pages that a gave back
    out = run_step(model, cache, [StepEntry(sc, b, None)])
    assert near(out[0], rb[-1])
    cache.check()


def test_configurations_drawn_at_random(cpu_kernels, tmp_path):
    rng = random.Random(12)
    for n in range(3):
        model, cfg, w = load(tmp_path, f"random{n}", cfg=ts.random_config(rng))
        a = ts.random_tokens(70, cfg["vocab"], n)
        ref = ts.plain_logits(cfg, w, a).float()
        cache = model.new_cache(256)
        s = cache.open_sequence()
        out = [run_step(model, cache, [StepEntry(s, a[:61], [60])]), run_step(model, cache, [StepEntry(s, a[61:68], [6])])]
        out += [run_step(model, cache, [StepEntry(s, [t])]) for t in a[68:]]
        assert torch.allclose(torch.cat(out), ref[[60, 67, 68, 69]], atol=3e-4 * float(ref.abs().max())), cfg


def test_a_lost_history_would_show(cpu_kernels, tmp_path):
    """What a sequence carries beside its keys - both convolutions' last inputs and the recurrence's state - is visible in the
    logits behind a cut: wiping it (or half a history) changes the next tokens' rows, and keeping it gives the plain ones."""
    model, cfg, w = load(tmp_path, "A")
    tokens = ts.random_tokens(40, cfg["vocab"], 4)
    ref = ts.plain_logits(cfg, w, tokens).float()
    rms = ref.pow(2).mean(-1).sqrt()

    def run(wipe):
        cache = model.new_cache(256)
        s = cache.open_sequence()
        run_step(model, cache, [StepEntry(s, tokens[:30], [])])
        wipe([g for g in cache.groups if g.kind == "state"])
        out = torch.cat([run_step(model, cache, [StepEntry(s, [t])]) for t in tokens[30:]])
        return (out - ref[30:]).pow(2).mean(-1).sqrt() / rms[30:]

    assert float(run(lambda groups: None).max()) < 1e-4
    for i in range(3):                                   # the input convolutions' history, then each recurrence's memory
        assert float(run(lambda groups: groups[i].state.zero_())[:2].max()) > 1e-2, i

    def swap(groups):                                    # the two rows of the first layer's history in the wrong order
        h = next(g for g in groups if g.need.state_shape == (160,)).state[0, 0].view(2, 80)
        h.copy_(h.flip(0).clone())
    assert float(run(swap)[0]) > 1e-3


def test_trace_replay_of_a_semanex_folder(cpu_kernels, tmp_path):
    import io
    from dotllm_b200.engine.trace import TraceReplayer
    model, cfg, w = load(tmp_path, "C")

    class Wrapped:                                        # what the replayer needs of a Model
        def new_cache(self, n):
            return model.new_cache(n)

        def step(self, cache, entries):
            return run_step(model, cache, entries)

    a = ts.random_tokens(12, cfg["vocab"], 3)
    ref = ts.plain_logits(cfg, w, a).float()
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": a[:9], "want": [0, 8]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": a[9:10], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "x", "tokens": a[10:], "want": [1]}], "end": ["x"]}]
    out = io.StringIO()
    replayer = TraceReplayer(Wrapped(), 128, tmp_path / "out")
    replayer.check_kernels = lambda: None
    replayer.run([json.dumps(s) for s in steps], out)
    assert out.getvalue().split() == ["done", "0", "done", "1", "done", "2"]
    read = lambda n: torch.from_numpy(np.fromfile(tmp_path / "out" / f"{n}.f32", dtype="<f4").reshape(-1, cfg["vocab"]).copy())
    assert not (tmp_path / "out" / "1.f32").exists()
    assert torch.allclose(read(0), ref[[0, 8]], atol=3e-4) and torch.allclose(read(2), ref[[11]], atol=3e-4)
    assert not replayer.sequences and not replayer.cache.live
