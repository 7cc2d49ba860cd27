"""Small Fetitar configurations for the tests, and helpers to make their model folders.

They differ from each other in every size and option: one to seven query heads a key/value head, keys and values of equal,
different and odd widths, latent rows with and without a width the tensor-core kernels take, one to 34 heads on a latent, rotations
of a whole shared key part, of a part of it and of no channel, with YaRN frequencies and without, windows of one token, of less than,
exactly and more than a page, and none, attention layers that mix values (first, in the middle, last) and that do not, layers
without a feed-forward, pair tables of one bucket and of many, negative and large multipliers, and no pair table.
"""
from __future__ import annotations

import copy
import random

import numpy as np
import torch


def latent(heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, rot, window=None, mlp=None):
    """rot: (dims, base) or (dims, base, (factor, original, fast, slow))"""
    mixer = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": scale,
             "rot": {"dims": rot[0], "base": rot[1]}}
    if len(rot) > 2:
        mixer["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), rot[2]))
    if window:
        mixer["mask"] = {"size": window}
    return {"type": "latent_attention", "mlp": mlp, "mixer": mixer}


def sloped(heads, kv_heads, dim, vdim, scale, window=None, v_mix=True, mlp=None):
    mixer = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "v_mix": v_mix}
    if window:
        mixer["mask"] = {"size": window}
    return {"type": "attention", "mlp": mlp, "mixer": mixer}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def config(width, vocab, eps, layers, embedding_scale=1.0, bigram=(97, 5, 3)):
    """bigram: (buckets, mul_prev, mul_cur) or None"""
    embedding = {"scale": embedding_scale}
    if bigram:
        embedding["bigram"] = dict(zip(("buckets", "mul_prev", "mul_cur"), bigram))
    return {"architecture": "Fetitar", "width": width, "vocab": vocab, "norm": {"eps": eps}, "embedding": embedding, "layers": layers}


CONFIGS = {
    # an attention layer first and last, one in the middle that does not mix, windows below and above a page
    "A": config(80, 200, 1e-6,
                [sloped(6, 2, 24, 20, 0.2, 70, True, dense(72)),
                 latent(4, 20, 8, 12, 28, 40, 0.2, (8, 500.0, (4.0, 64.0, 8.0, 1.0)), 33, dense(100)),
                 sloped(4, 4, 16, 16, 0.3, 9, False, None),
                 sloped(3, 1, 24, 28, 0.25, None, False, dense(40)),
                 latent(3, 12, 16, 20, 36, 24, 0.3, (16, 20.0), None, None),
                 sloped(2, 2, 40, 20, 0.2, 100, True, None)],
                embedding_scale=3.0),
    # sizes the tensor-core kernels take: heads of 64 and 128, latent rows of 48 + 16 and 112 + 16, eight query heads a key head
    "B": config(128, 333, 1e-5,
                [latent(4, 32, 16, 32, 64, 48, 0.14, (16, 10000.0, (16.0, 512.0, 16.0, 2.0)), 50, dense(256)),
                 sloped(8, 1, 64, 64, 0.12, 129, True, dense(192)),
                 latent(8, 64, 16, 64, 96, 112, 0.1, (16, 10000.0, (2.0, 128.0, 4.0, 1.0)), 64, dense(160)),
                 sloped(4, 1, 128, 64, 0.09, 65, True, dense(128)),
                 sloped(16, 1, 96, 64, 0.1, 128, True, dense(64))],
                embedding_scale=8.0, bigram=(500, 1234567, 89)),
    # multiples of nothing: odd widths everywhere, a window of one token, no rotated channel, one bucket
    "C": config(52, 101, 1e-5,
                [sloped(3, 1, 10, 7, 0.4, 1, True, dense(30)),
                 latent(3, 7, 6, 5, 11, 13, 0.4, (0, 100.0), 2, dense(24)),
                 sloped(7, 1, 9, 7, 0.3, 31, True, dense(20))],
                bigram=(1, 7, 11)),
    # a rotation of a part of the shared key part, more query heads on a key head than a tile has rows, no pair table
    "D": config(96, 160, 1e-5,
                [latent(20, 8, 24, 6, 40, 40, 0.25, (12, 50.0, (8.0, 100.0, 3.0, 0.5)), 90, dense(40)),
                 sloped(20, 1, 32, 8, 0.2, 127, False, dense(64)),
                 latent(34, 6, 8, 4, 20, 24, 0.3, (8, 1000.0), None, dense(48))],
                embedding_scale=5.0, bigram=None),
    # a latent row wider than any tensor-core width, heads wider than any, a single layer type in a row, multipliers of both signs
    "E": config(72, 90, 1e-6,
                [latent(2, 24, 40, 24, 24, 130, 0.1, (40, 300.0, (3.0, 50.0, 2.0, 1.0)), 42, None),
                 latent(2, 16, 8, 16, 16, 24, 0.2, (8, 300.0), 63, dense(48)),
                 sloped(2, 1, 136, 40, 0.09, 80, True, dense(56)),
                 sloped(2, 1, 8, 40, 0.3, 20, True, dense(56))],
                embedding_scale=2.0, bigram=(61, -13, 29)),
}

# One layer alone whose scores are sharp: single keys decide.
SHARP_SLOPED = config(64, 120, 1e-5, [sloped(8, 2, 16, 16, 3.0, 70, True)], embedding_scale=4.0, bigram=None)
SHARP_LATENT = config(64, 120, 1e-5, [latent(4, 16, 8, 16, 32, 32, 3.0, (8, 100.0, (8.0, 64.0, 4.0, 1.0)), 150)], embedding_scale=4.0, bigram=None)
# Layers at the widths of a real model's layers.
WIDE = config(1024, 1000, 1e-5,
              [latent(8, 96, 32, 128, 512, 96, 128 ** -0.5, (32, 10000.0, (6.0, 4096.0, 24.0, 1.0)), 100, dense(2048)),
               sloped(8, 2, 128, 128, 128 ** -0.5, 150, True, dense(2048)),
               latent(32, 64, 64, 64, 256, 64, 128 ** -0.5, (64, 10000.0), 77, dense(1024)),
               sloped(16, 2, 64, 128, 64 ** -0.5, 64, True, dense(1024))],
              embedding_scale=1.0, bigram=(5000, 331, 17))
CONFIGS.update(wide=WIDE, sharp_sloped=SHARP_SLOPED, sharp_latent=SHARP_LATENT)


def random_config(rng):
    """A configuration drawn from ``rng`` (a random.Random): two to five layers of both kinds with sizes that are and are not
    multiples of 8, 16 or 64."""
    layers = []
    g, vd = rng.choice([1, 1, 2, 3]), rng.choice([8, 16, 24, 32, 48, 64, 7])          # the mixing layers' common sizes
    window = lambda: rng.choice([None, 1, 5, 16, 33, 63, 64, 65, 100, 128, 150])
    for _ in range(rng.randrange(2, 6)):
        mlp = None if rng.random() < 0.2 else dense(rng.choice([24, 64, 100, 136, 30, 256]))
        if rng.random() < 0.5:
            rot_dim = rng.choice([2, 8, 16, 32, 40])
            dims = rng.choice([rot_dim, rot_dim, rot_dim // 2 - (rot_dim // 2) % 2, 0])
            rot = (dims, rng.choice([100.0, 10000.0, 1e6]))
            if dims and rng.random() < 0.7:
                rot += ((rng.choice([2.0, 8.0, 32.0]), rng.choice([32.0, 100.0, 4096.0]), rng.choice([4.0, 32.0]), rng.choice([0.5, 1.0])),)
            layers.append(latent(rng.choice([1, 2, 3, 6, 8, 16, 17, 24]), rng.choice([8, 16, 24, 32, 13]), rot_dim, rng.choice([8, 16, 24, 40, 11]),
                                 rng.choice([16, 24, 48, 64, 31]), rng.choice([16, 24, 32, 56, 64, 88, 96, 120, 29]), rng.choice([0.1, 0.2, 0.35]),
                                 rot, window(), mlp))
        else:
            mixes = rng.random() < 0.7
            kv, v = (g, vd) if mixes else (rng.choice([1, 2, 5]), rng.choice([8, 20, 64, 128]))
            dim = rng.choice([8, 16, 24, 32, 40, 64, 96, 128])
            layers.append(sloped(kv * rng.choice([1, 2, 4, 5]), kv, dim, v, rng.choice([0.1, 0.3, dim ** -0.5]), window(), mixes, mlp))
    bigram = None if rng.random() < 0.2 else (rng.choice([1, 2, 64, 1000]), rng.randrange(0, 100000), rng.randrange(0, 100000))
    return config(rng.choice([64, 96, 128, 160, 192, 100, 72, 50]), rng.randrange(100, 600), rng.choice([1e-5, 1e-6]), layers,
                  rng.choice([1.0, 4.0, 9.5]), bigram)


def make_folder(tmp_path, which, seed=0, dtype=torch.float32, cfg=None):
    """Write a model folder with the package's random-weights mode; returns its path."""
    from dotllm_b200.config import config_from_dict
    from dotllm_b200.weights import write_random_model
    cfg_dict = copy.deepcopy(cfg or CONFIGS[which])
    folder = tmp_path / f"fetitar_{which}_{seed}_{str(dtype).split('.')[-1]}"
    write_random_model(folder, config_from_dict(cfg_dict), seed, dtype=dtype)
    return folder


def read_folder(folder):
    """(config dict, weights as float64 arrays) as the plain implementation takes them."""
    import plain_llama
    cfg, weights = plain_llama.read_model_folder(folder)
    return cfg, {name: t.double().numpy() for name, t in weights.items()}


def plain_logits(cfg, w, tokens):
    """The plain implementation's logits as a float64 tensor [T, vocab]."""
    import plain_fetitar
    return torch.from_numpy(np.ascontiguousarray(plain_fetitar.forward(cfg, w, tokens)[0]))


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
