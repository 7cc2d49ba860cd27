"""Small Semanex configurations for the tests, and helpers to make their model folders.

They differ from each other in every size and option: one to seven query heads a key/value head, keys and values of equal,
different and odd widths, latents with and without a width the tensor-core kernels take, rotations of a whole shared key part, of
a part of it and of no channel, capped and uncapped scores, states of one to 33 channels with one to three groups, one to five
taps in both convolutions, one and several norm parts, layers without a feed-forward, an alpha of one.
"""
from __future__ import annotations

import copy
import random

import numpy as np
import torch


def latent(heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, rot, mlp=None):
    """rot: (dims, base)"""
    return {"type": "latent_attention", "mlp": mlp,
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": scale,
                      "rot": {"dims": rot[0], "base": rot[1]}}}


def parallel(left, right, scales, mlp=None):
    """left: (heads, kv_heads, dim, vdim, scale, softcap); right: (heads, vdim, state, groups, conv, norm_groups)"""
    lh, lg, ld, lv, ls, cap = left
    rh, rv, rn, rg, conv, parts = right
    left_d = {"heads": lh, "kv_heads": lg, "dim": ld, "vdim": lv, "scale": ls}
    if cap is not None:
        left_d["softcap"] = cap
    return {"type": "parallel", "mlp": mlp,
            "mixer": {"left": left_d, "right": {"heads": rh, "vdim": rv, "state": rn, "groups": rg, "conv": conv, "norm_groups": parts},
                      "left_scale": scales[0], "right_scale": scales[1]}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def config(width, vocab, eps, alpha, taps, layers, embedding_scale=1.0):
    return {"architecture": "Semanex", "width": width, "vocab": vocab, "norm": {"eps": eps}, "postln_alpha": alpha, "canon": {"taps": taps},
            "embedding": {"scale": embedding_scale}, "layers": layers}


CONFIGS = {
    # different key and value widths under the cap, two groups, three norm parts, a latent that fills no kernel width
    "A": config(80, 200, 1e-6, 2.0, 3,
                [parallel((6, 2, 24, 20, 0.2, 5.0), (6, 10, 20, 2, 3, 3), (0.7, 0.4), dense(72)),
                 latent(4, 20, 8, 12, 28, 40, 0.2, (8, 500.0), dense(100)),
                 parallel((2, 2, 16, 16, 0.3, 8.0), (4, 12, 16, 1, 2, 1), (0.3, 1.2), None),
                 latent(3, 12, 16, 20, 36, 24, 0.3, (16, 20.0), None)],
                embedding_scale=3.0),
    # sizes the tensor-core kernels take: heads of 64 and 128, latents of 48 + 16 and 112 + 16, eight query heads a key head
    "B": config(128, 333, 1e-5, 1.5, 4,
                [latent(4, 32, 16, 32, 64, 48, 0.14, (16, 10000.0), dense(256)),
                 parallel((8, 1, 64, 64, 0.1, 20.0), (4, 64, 128, 2, 4, 2), (0.5, 0.5), dense(192)),
                 latent(8, 64, 16, 64, 96, 112, 0.1, (16, 10000.0), dense(160)),
                 parallel((4, 2, 128, 64, 0.09, 12.0), (8, 32, 64, 4, 4, 1), (0.9, 0.6), dense(128))],
                embedding_scale=8.0),
    # multiples of nothing: odd widths everywhere, one tap, one state channel, an alpha of one, no cap, no rotated channel
    "C": config(52, 101, 1e-5, 1.0, 1,
                [parallel((3, 1, 10, 7, 0.4, None), (3, 5, 1, 3, 1, 5), (1.0, 1.0), dense(30)),
                 latent(3, 7, 6, 5, 11, 13, 0.4, (0, 100.0), dense(24)),
                 parallel((7, 7, 9, 14, 0.3, 2.0), (1, 9, 33, 1, 5, 1), (0.2, 1.5), dense(20))],
                embedding_scale=1.0),
    # a rotation of a part of the shared key part, five taps, more query heads on the latent than a tile has rows
    "D": config(96, 160, 1e-5, 3.0, 5,
                [latent(20, 8, 24, 6, 40, 40, 0.25, (12, 50.0), dense(40)),
                 parallel((4, 4, 32, 96, 0.2, 3.0), (2, 24, 40, 1, 4, 2), (0.6, 0.8), dense(64)),
                 latent(34, 6, 8, 4, 20, 24, 0.3, (8, 1000.0), dense(48))],
                embedding_scale=5.0),
    # a latent row wider than any tensor-core width, a state of 256 channels, a single layer type in a row
    "E": config(72, 90, 1e-6, 2.5, 2,
                [latent(2, 24, 40, 24, 24, 130, 0.1, (40, 300.0), None),
                 latent(2, 16, 8, 16, 16, 24, 0.2, (8, 300.0), dense(48)),
                 parallel((4, 1, 40, 40, 0.2, 30.0), (2, 16, 256, 2, 3, 1), (1.1, 0.3), dense(56))],
                embedding_scale=2.0),
}

# One layer alone whose scores are sharp: far keys decide.
SHARP_LATENT = config(64, 120, 1e-5, 1.0, 2, [latent(4, 16, 8, 16, 32, 32, 3.0, (8, 100.0))], embedding_scale=4.0)
SHARP_CAPPED = config(64, 120, 1e-5, 1.0, 2, [parallel((4, 2, 16, 16, 4.0, 20.0), (2, 8, 8, 1, 2, 1), (1.0, 0.1))], embedding_scale=4.0)
# Layers at the widths of a real model's layers.
WIDE = config(1024, 1000, 1e-5, 3.0, 4,
              [latent(8, 96, 32, 128, 512, 96, 128 ** -0.5, (32, 10000.0), dense(2048)),
               parallel((8, 2, 128, 128, 128 ** -0.5, 30.0), (16, 64, 128, 2, 4, 2), (0.7, 0.5), dense(2048)),
               latent(32, 64, 64, 64, 256, 64, 128 ** -0.5, (64, 10000.0), dense(1024))],
              embedding_scale=1.0)
CONFIGS.update(wide=WIDE, sharp_latent=SHARP_LATENT, sharp_capped=SHARP_CAPPED)


def random_config(rng):
    """A configuration drawn from ``rng`` (a random.Random): two to five layers of both kinds with sizes that are and are not
    multiples of 8, 16 or 64."""
    layers = []
    for _ in range(rng.randrange(2, 6)):
        mlp = None if rng.random() < 0.2 else dense(rng.choice([24, 64, 100, 136, 30, 256]))
        if rng.random() < 0.5:
            rot_dim = rng.choice([2, 8, 16, 32, 40])
            dims = rng.choice([rot_dim, rot_dim, rot_dim // 2 - (rot_dim // 2) % 2, 0])
            layers.append(latent(rng.choice([1, 2, 3, 6, 8, 16, 17, 24]), rng.choice([8, 16, 24, 32, 13]), rot_dim, rng.choice([8, 16, 24, 40, 11]),
                                 rng.choice([16, 24, 48, 64, 31]), rng.choice([16, 24, 32, 56, 64, 88, 96, 120, 29]), rng.choice([0.1, 0.2, 0.35]),
                                 (dims, rng.choice([100.0, 10000.0, 1e6])), mlp))
        else:
            kv, g = rng.choice([1, 1, 2, 3]), rng.choice([1, 2, 3])
            dim, heads, vd = rng.choice([8, 16, 24, 32, 40, 64, 96, 128]), g * rng.choice([1, 2, 3]), rng.choice([8, 12, 16, 32, 64, 7])
            parts = rng.choice([p for p in range(1, 7) if (heads * vd) % p == 0])
            layers.append(parallel((kv * rng.choice([1, 2, 4, 5]), kv, dim, rng.choice([dim, dim, 16, 40, 128]), rng.choice([0.1, 0.3, dim ** -0.5]),
                                    rng.choice([None, 2.0, 10.0, 50.0])),
                                   (heads, vd, rng.choice([4, 8, 16, 32, 48, 64, 128, 19]), g, rng.randrange(1, 6), parts),
                                   (rng.choice([0.3, 0.8, 1.0]), rng.choice([0.3, 0.5, 1.0])), mlp))
    return config(rng.choice([64, 96, 128, 160, 192, 100, 72, 50]), rng.randrange(100, 600), rng.choice([1e-5, 1e-6]), rng.choice([1.0, 2.0, 3.0, 1.7]),
                  rng.randrange(1, 6), layers, rng.choice([1.0, 4.0, 9.5]))


def make_folder(tmp_path, which, seed=0, dtype=torch.float32, cfg=None):
    """Write a model folder with the package's random-weights mode; returns its path."""
    from dotllm_b200.config import config_from_dict
    from dotllm_b200.weights import write_random_model
    cfg_dict = copy.deepcopy(cfg or CONFIGS[which])
    folder = tmp_path / f"semanex_{which}_{seed}_{str(dtype).split('.')[-1]}"
    write_random_model(folder, config_from_dict(cfg_dict), seed, dtype=dtype)
    return folder


def read_folder(folder):
    """(config dict, weights as float64 arrays) as the plain implementation takes them."""
    import plain_llama
    cfg, weights = plain_llama.read_model_folder(folder)
    return cfg, {name: t.double().numpy() for name, t in weights.items()}


def plain_logits(cfg, w, tokens):
    """The plain implementation's logits as a float64 tensor [T, vocab]."""
    import plain_semanex
    return torch.from_numpy(np.ascontiguousarray(plain_semanex.forward(cfg, w, tokens)[0]))


def random_tokens(n, vocab, seed):
    rng = random.Random(seed)
    return [rng.randrange(vocab) for _ in range(n)]


def rewrite(folder, change):
    """Read the folder's tensors, let ``change(tensors)`` edit the dict in place, write them back."""
    from dotllm_b200.weights.safetensors_io import SafetensorsFile, save_safetensors
    path = folder / "model.safetensors"
    with SafetensorsFile(path) as f:
        tensors = {n: f.tensor(n).clone() for n in f.names()}
    change(tensors)
    save_safetensors(path, tensors, metadata={"format": "pt"})
    return folder
