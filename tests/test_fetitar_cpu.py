"""Fetitar without a GPU: configuration, model description, tensor names, cache needs, the plain implementation's own mechanisms,
and the engine's host logic (steps, cache, schedule) with the plain kernel references."""
import copy
import json
import math
import random

import numpy as np
import pytest
import torch

import plain_fetitar as pf
import tiny_fetitar as tf
from dotllm_b200.config import build_spec, config_from_dict, load_config
from dotllm_b200.engine import StepEntry, run_step
from dotllm_b200.errors import ConfigError
from dotllm_b200.models.decoder import DecoderModel
from dotllm_b200.parts.base import Runtime
from dotllm_b200.weights import load_into

CPU = Runtime(torch.float32, torch.device("cpu"))


def test_configuration_reads_every_key_and_writes_it_back():
    for name, d in tf.CONFIGS.items():
        cfg = config_from_dict(copy.deepcopy(d))
        assert cfg.to_dict() == d, name
        assert type(cfg).__name__ == "FetitarConfig"
    mixer = lambda i, **kw: (lambda c: c["layers"][i]["mixer"].update(**kw))
    for broken, match in ((lambda c: c.pop("width"), "width"), (lambda c: c.pop("norm"), "norm"),
                          (lambda c: c["layers"][0].update(type="gla"), "type"), (lambda c: c["layers"][0].pop("mixer"), "mixer"),
                          (lambda c: c["layers"][0]["mixer"].pop("scale"), "scale"), (mixer(0, scale=-1.0), "scale"),
                          (mixer(0, kv_heads=4), "kv_heads"), (mixer(0, mask={"size": 0}), "mask"), (mixer(0, mask={"kind": "x"}), "size"),
                          (mixer(0, vdim=24), "vdim"),                   # the mixing layers' values would not fit together
                          (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=10), "rot"),
                          (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=3), "rot"),
                          (lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].pop("fast"), "fast"),
                          (lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].update(factor=0.0), "scaling"),
                          (lambda c: c["layers"][1]["mixer"].pop("rot"), "rot"),
                          (lambda c: c["layers"][1]["mixer"].pop("kv_rank"), "kv_rank"),
                          (lambda c: c["embedding"]["bigram"].update(buckets=0), "bigram"),
                          (lambda c: c["embedding"]["bigram"].pop("mul_cur"), "mul_cur"),
                          (lambda c: c["layers"][0]["mlp"].update(kind="moe"), "kind"),
                          (lambda c: c["layers"][0]["mlp"].update(ff=0), "mlp")):
        bad = copy.deepcopy(tf.CONFIGS["A"])
        broken(bad)
        with pytest.raises(ConfigError, match=match):
            config_from_dict(bad)


def test_description_tensor_names_and_cache_needs():
    spec = build_spec(config_from_dict(copy.deepcopy(tf.CONFIGS["A"])))
    model = DecoderModel(spec, CPU)
    expected, optional = model.expected_weights()
    attention = ["q", "k", "v", "o", "q.b", "k.b", "v.b", "o.b", "q.norm", "k.norm"]
    latent = ["dq", "dq.norm", "uq", "dkv", "dkv.norm", "uk", "uv", "g", "o"]
    mlp = ["gate", "up", "down", "gate.b", "up.b", "down.b"]
    want = {"embed", "bigram", "head", "final.norm"}
    for i, (mix, ff) in enumerate(((attention, True), (latent, True), (attention, False), (attention, True), (latent, False), (attention, False))):
        want |= {f"l{i}.norm1", f"l{i}.norm1b"} | {f"l{i}.mix.{n}" for n in mix}
        want |= {f"l{i}.norm2", f"l{i}.norm2b"} | {f"l{i}.mlp.{n}" for n in mlp} if ff else set()
    assert set(expected) == want | {"l5.mix.vmix"}                       # the one layer that mixes another's values in
    assert optional == {"l0.mix.vmix", "l2.mix.vmix", "l3.mix.vmix"} | {f"l{i}.norm2{b}" for i in (2, 4, 5) for b in ("", "b")}
    shape = lambda n: tuple(expected[n].shape)
    assert shape("bigram") == (98, 80) and shape("l5.mix.vmix") == () and shape("l0.mix.q.norm") == (144,) and shape("l0.mix.k.norm") == (48,)
    assert shape("l0.mix.v") == (40, 80) and shape("l0.mix.o.b") == (80,) and shape("l1.mix.g") == (4, 80) and shape("l1.mix.uq") == (4 * 28, 28)
    assert shape("l0.mlp.gate.b") == (72,) and shape("l0.mlp.down.b") == (80,)
    needs = model.cache_needs()
    assert len(needs) == 7 and [n.kind for n in needs] == ["kv"] * 6 + ["state"]
    assert needs[6].state_shape == (1,) and needs[6].state_dtype == torch.int32
    assert [n.window for n in needs[:6]] == [70, 33, 9, None, None, 100]
    assert (needs[0].key_width(), needs[0].value_width()) == (24, 20) and (needs[1].key_width(), needs[1].value_width()) == (48, 40)
    # bfloat16 rows that fit a tensor-core width are laid out at it: heads of 24 and 20 at 32, a latent row of 48 at 64
    wide = DecoderModel(spec, Runtime(torch.bfloat16, torch.device("cpu"))).cache_needs()
    assert [(n.key_width(), n.value_width()) for n in wide[:6]] == [(32, 32), (64, 64), (32, 32), (32, 32), (64, 64), (64, 64)]
    # the pair table is the one part of the model whose absence leaves the cache without state
    spec = build_spec(config_from_dict(copy.deepcopy(tf.CONFIGS["D"])))
    assert [n.kind for n in DecoderModel(spec, CPU).cache_needs()] == ["kv"] * 3


def test_parts_refuse_what_they_cannot_do():
    from dotllm_b200.config.spec import PartSpec
    from dotllm_b200.parts.base import make_part
    params = {"n_heads": 2, "n_kv_heads": 1, "head_dim": 8, "bias": "all", "qk_norm": {"eps": 1e-6, "over": "projection"}}
    for extra in ({"own_kv": False}, {"values": "keys", "bias": False, "value_mix": {"first": True}}, {"pairing": "interleaved"},
                  {"qk_norm": {"eps": 1e-6}, "value_mix": {"first": True}}):
        with pytest.raises(ConfigError, match="biases ahead of a norm"):
            make_part("mixer", PartSpec("attention", {**params, **extra}), 16, CPU)
    with pytest.raises(ConfigError, match="pairs"):
        make_part("mixer", PartSpec("latent_attention", {"n_heads": 1, "key_dim": 8, "value_dim": 8, "q_rank": 8, "kv_rank": 8, "eps": 1e-6,
                                                         "pairing": "thirds"}), 16, CPU)
    with pytest.raises(ConfigError, match="bucket"):
        make_part("embedding", PartSpec("token_pair_embedding", {"vocab_size": 4, "buckets": 0, "mul_prev": 1, "mul_cur": 1}), 16, CPU)


# ------------------------------------------------------------------ the plain implementation's own mechanisms
def test_plain_pair_rows_alone():
    assert pf.bigram_rows([7, 7, 0, 3], 10, 3, 4) == [10, (21 + 28) % 10, 21 % 10, 12 % 10]
    assert pf.bigram_rows([5, 5], 1, 9, 9) == [1, 0] and pf.bigram_rows([2, 1], 61, -13, 29) == [61, (-26 + 29) % 61]
    w = {"embed": np.arange(8.0).reshape(4, 2), "bigram": np.array([[100.0, 200.0], [300.0, 400.0], [0.5, 0.25]])}
    x = pf.embed({"embedding": {"scale": 3.0, "bigram": {"buckets": 2, "mul_prev": 1, "mul_cur": 0}}}, w, [1, 2, 3])
    assert np.array_equal(x, [[6.5, 9.25], [312.0, 415.0], [118.0, 221.0]])                 # the constant is the token embedding's alone


def test_plain_attention_mechanisms_alone():
    rng = np.random.default_rng(1)
    q, k, v = rng.normal(size=(6, 4, 3)), rng.normal(size=(6, 2, 3)), rng.normal(size=(6, 2, 5))
    o = pf.softmax_attention(q, k, v, 0.7)
    assert np.allclose(o[0], v[0][[0, 0, 1, 1]])                      # the first token sees itself alone
    assert np.allclose(pf.softmax_attention(q, k, v, 0.7, window=1), v[:, [0, 0, 1, 1]])         # and so does everyone in a window of one
    assert np.allclose(pf.softmax_attention(q, k, v, 0.7, window=6), o) and not np.allclose(pf.softmax_attention(q, k, v, 0.7, window=5)[5], o[5])
    assert np.allclose(pf.softmax_attention(q, k, v, 0.7, window=3)[5, 1], pf.softmax_attention(q[3:], k[3:], v[3:], 0.7)[2, 1])
    # two keys of equal score at distances 2 and 0: their weights stand e^(-2 slope) to 1
    same = np.repeat(k[:1], 6, axis=0)
    p = np.exp(-0.3 * np.array([2, 1, 0])) / np.exp(-0.3 * np.array([2, 1, 0])).sum()
    assert np.allclose(pf.softmax_attention(q, same, v, 0.7, None, [0.3] * 4)[2, 0], p @ v[:3, 0])
    assert pf.distance_slopes(4) == [0.25, 0.0625, 0.015625, 0.00390625] and np.allclose(pf.distance_slopes(3)[0], 2 ** (-8 / 3))
    assert np.allclose(pf.mixed_values(v, 2 * v, 0.25), 1.25 * v) and np.array_equal(pf.mixed_values(v, 2 * v, 0.0), v)
    # the norm runs over all heads at once: scaling one head changes the others
    x = rng.normal(size=(1, 8))
    y = x.copy()
    y[0, :4] *= 3.0
    assert not np.allclose(pf.rms(x, 0.0)[0, 4:], pf.rms(y, 0.0)[0, 4:])


def test_plain_latent_attention_equals_attention_in_the_latents_own_basis():
    rng = np.random.default_rng(2)
    m = {"heads": 2, "dim": 3, "rot_dim": 4, "vdim": 5, "q_rank": 6, "kv_rank": 7, "scale": 0.4, "mask": {"size": 5},
         "rot": {"dims": 4, "base": 50.0, "scaling": {"factor": 4.0, "original": 30.0, "fast": 2.0, "slow": 0.5}}}
    w = {n: rng.normal(size=s) for n, s in (("dq", (6, 8)), ("uq", (14, 6)), ("dkv", (11, 8)), ("uk", (6, 7)), ("uv", (10, 7)), ("g", (2, 8)),
                                            ("dq.norm", (6,)), ("dkv.norm", (7,)))}
    w["o"] = np.eye(10)
    h = rng.normal(size=(9, 8))
    got = pf.latent_attention(m, w, "", h, np.arange(9), 1e-6)
    turn = lambda x: pf.rotate_halves(x, np.arange(9), 4, 50.0, m["rot"]["scaling"])
    c = pf.rms((h @ w["dkv"].T)[:, :7], 1e-6) * w["dkv.norm"]
    qq = ((pf.rms(h @ w["dq"].T, 1e-6) * w["dq.norm"]) @ w["uq"].T).reshape(9, 2, 7)
    ql = np.einsum("thd,hdr->thr", qq[..., :3], w["uk"].reshape(2, 3, 7))
    a = pf.softmax_attention(np.concatenate([ql, turn(qq[..., 3:])], -1), np.concatenate([c[:, None], turn((h @ w["dkv"].T)[:, None, 7:])], -1),
                             c[:, None], 0.4, 5)
    a = a * pf.sigmoid(h @ w["g"].T)[..., None]                        # a gate per head may come before the change of basis
    assert np.allclose(got, np.einsum("thr,hvr->thv", a, w["uv"].reshape(2, 5, 7)).reshape(9, 10))


def test_plain_rotation_against_the_packages_tables():
    from dotllm_b200.parts.rotary import rotary_frequencies, rotary_magnitude
    x = np.random.default_rng(3).normal(size=(5, 3, 12))
    y = pf.rotate_halves(x, np.arange(5), 8, 100.0)
    assert np.array_equal(y[..., 8:], x[..., 8:]) and np.array_equal(y[0], x[0])
    assert np.allclose(y[..., :4] ** 2 + y[..., 4:8] ** 2, x[..., :4] ** 2 + x[..., 4:8] ** 2)
    z = lambda t: t[..., :4] + 1j * t[..., 4:8]
    assert np.allclose(z(y[1]) / z(x[1]), np.exp(1j * rotary_frequencies(8, 100.0))[None, :])
    assert np.array_equal(pf.rotate_halves(x, np.arange(5), 0, 100.0), x)
    for dims, base, s in ((8, 100.0, (4.0, 64.0, 8.0, 1.0)), (32, 1e5, (5.0, 3000.0, 24.0, 1.5)), (12, 50.0, (8.0, 100.0, 3.0, 0.5)), (2, 10.0, (2.0, 4.0, 50.0, 40.0))):
        mine = dict(zip(("factor", "original", "fast", "slow"), s))
        theirs = {"rope_type": "yarn", "factor": s[0], "original_max_position_embeddings": s[1], "fast_turns": s[2], "slow_turns": s[3]}
        f, grow = pf.yarn_frequencies(dims, base, mine)
        assert np.allclose(f, rotary_frequencies(dims, base, theirs)) and math.isclose(grow, rotary_magnitude(theirs)), (dims, base)


# ------------------------------------------------------------------ the engine's host logic
def load(tmp_path, which, cfg=None, change=None):
    folder = tf.make_folder(tmp_path, which, cfg=cfg)
    if change is not None:
        tf.rewrite(folder, change)
    cfg, weights = tf.read_folder(folder)
    return load_into(DecoderModel(build_spec(load_config(folder)), CPU), folder), cfg, weights


@pytest.mark.parametrize("which", ["A", "C", "D", "E"])
def test_steps_cuts_and_batches_agree_with_the_plain_implementation(cpu_kernels, tmp_path, which):
    model, cfg, w = load(tmp_path, which)
    a, b = tf.random_tokens(83, cfg["vocab"], 1), tf.random_tokens(21, cfg["vocab"], 2)
    ra, rb = tf.plain_logits(cfg, w, a).float(), tf.plain_logits(cfg, w, b).float()
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
    sc = cache.open_sequence()                           # takes the slot, its last token and the pages that a gave back
    out = run_step(model, cache, [StepEntry(sc, b, None)])
    assert near(out[0], rb[-1])
    cache.check()


def test_configurations_drawn_at_random(cpu_kernels, tmp_path):
    rng = random.Random(12)
    for n in range(3):
        model, cfg, w = load(tmp_path, f"random{n}", cfg=tf.random_config(rng))
        a = tf.random_tokens(70, cfg["vocab"], n)
        ref = tf.plain_logits(cfg, w, a).float()
        cache = model.new_cache(256)
        s = cache.open_sequence()
        out = [run_step(model, cache, [StepEntry(s, a[:61], [60])]), run_step(model, cache, [StepEntry(s, a[61:68], [6])])]
        out += [run_step(model, cache, [StepEntry(s, [t])]) for t in a[68:]]
        assert torch.allclose(torch.cat(out), ref[[60, 67, 68, 69]], atol=3e-4 * float(ref.abs().max())), cfg


def test_a_lost_last_token_would_show(cpu_kernels, tmp_path):
    """The token before a portion is state: the kept one gives the plain rows; a wrong one changes the next token's row."""
    model, cfg, w = load(tmp_path, "A")
    tokens = tf.random_tokens(40, cfg["vocab"], 4)
    ref = tf.plain_logits(cfg, w, tokens).float()
    rms = ref.pow(2).mean(-1).sqrt()

    def run(spoil):
        cache = model.new_cache(256)
        s = cache.open_sequence()
        run_step(model, cache, [StepEntry(s, tokens[:30], [])])
        group = next(g for g in cache.groups if g.kind == "state")
        assert int(group.state[0, s.slot, 0]) == tokens[29]
        spoil(group.state)
        out = torch.cat([run_step(model, cache, [StepEntry(s, [t])]) for t in tokens[30:]])
        return (out - ref[30:]).pow(2).mean(-1).sqrt() / rms[30:]

    assert float(run(lambda state: None).max()) < 1e-4
    assert float(run(lambda state: state.zero_())[0]) > 1e-2 and float(run(lambda state: state.add_(1).remainder_(cfg["vocab"]))[0]) > 1e-2


def test_values_mixed_in_must_come_from_an_earlier_layer(cpu_kernels):
    from dotllm_b200.config.spec import PartSpec
    from dotllm_b200.parts.base import make_part
    params = {"n_heads": 2, "n_kv_heads": 1, "head_dim": 8, "position": None, "value_mix": {"first": False}}
    mixer = make_part("mixer", PartSpec("attention", params), 16, CPU)
    mixer.bind({n: torch.zeros(s.shape) for n, s in mixer.weight_specs().items()})

    class Step:
        carry = {}
    with pytest.raises(ConfigError, match="mixes values"):
        mixer._ready_rows(torch.zeros(3, 32), Step())


def test_trace_replay_of_a_fetitar_folder(cpu_kernels, tmp_path):
    import io
    from dotllm_b200.engine.trace import TraceReplayer
    model, cfg, w = load(tmp_path, "C")

    class Wrapped:                                        # what the replayer needs of a Model
        def new_cache(self, n):
            return model.new_cache(n)

        def step(self, cache, entries):
            return run_step(model, cache, entries)

    a = tf.random_tokens(12, cfg["vocab"], 3)
    ref = tf.plain_logits(cfg, w, a).float()
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": a[:9], "want": [0, 8]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": a[9:10], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "x", "tokens": a[10:], "want": [1]}], "end": ["x"]}]
    out = io.StringIO()
    replayer = TraceReplayer(Wrapped(), 128, tmp_path / "out")
    replayer.check_kernels = lambda: None
    replayer.run([json.dumps(s) for s in steps], out)
    assert out.getvalue().split() == ["done", "0", "done", "1", "done", "2"]
    read = lambda n: torch.from_numpy(np.fromfile(tmp_path / "out" / f"{n}.f32", dtype="<f4").reshape(-1, cfg["vocab"]).copy())
    tol = 3e-4 * float(ref.abs().max())
    assert not (tmp_path / "out" / "1.f32").exists()
    assert torch.allclose(read(0), ref[[0, 8]], atol=tol) and torch.allclose(read(2), ref[[11]], atol=tol)
    assert not replayer.sequences and not replayer.cache.live
