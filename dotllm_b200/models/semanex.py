"""The Semanex decoder as a model description.

Token embedding times a constant; post-norm layers, x = norm(a x + sublayer(x)), every norm an RMS norm with a single number as its
gain; what a mixer reads is the stream plus a short causal convolution of it; per layer one of two mixers - latent attention with
a rotated key part shared by the heads, a learned sink and a gate per channel, or a weighted sum of softmax attention (an RMS norm
per query and key head, capped scores, no positions, a gate per channel) and a state-space recurrence - and a dense feed-forward
without a gate (exact gelu), or none; a last norm and a head of its own.
Tensor names: ``embed``, ``l<i>.canon1``, ``l<i>.norm1``, ``l<i>.norm2``, ``l<i>.mix.*`` (a sum's sides under ``left.`` and ``right.``),
``l<i>.mlp.*``, ``final.norm``, ``head``.
"""
from __future__ import annotations

from ..config.registry import register_architecture
from ..config.semanex import SemanexConfig
from ..config.spec import LayerPart, LayerSpec, ModelSpec, PartSpec, ScheduleEntry


def _norm(cfg, name, alpha=1.0):
    return PartSpec("post_rmsnorm", {"eps": cfg.eps, "alpha": alpha, "gain": "scalar", "tensor": ""}, name)


def _latent(cfg, m):
    rotation = {"rotary_dim": m.rot.dims, "theta": m.rot.base, "max_positions": cfg.positions(), "scaling": None}
    return {"n_heads": m.heads, "key_dim": m.dim, "rot_dim": m.rot_dim, "value_dim": m.vdim, "q_rank": m.q_rank, "kv_rank": m.kv_rank,
            "eps": cfg.eps, "scale": m.scale, "window": None, "sink": True, "gate": "channel_sigmoid",
            "position": {"kind": "rotary", "params": rotation} if m.rot.dims else None,
            "tensors": {"q_down": "dq", "q_norm": "dq.norm", "q_up": "uq", "kv_down": "dkv", "kv_norm": "dkv.norm", "k_up": "uk",
                        "v_up": "uv", "out": "o", "gate": "g", "sink": "sink"}}


def _mixer(cfg, layer, prefix):
    m = layer.mixer
    if layer.type == "latent_attention":
        return PartSpec("latent_attention", _latent(cfg, m), prefix)
    a, r = m.left, m.right
    left = {"n_heads": a.heads, "n_kv_heads": a.kv_heads, "head_dim": a.dim, "value_dim": a.vdim, "scale": a.scale, "window": None,
            "position": None, "qk_norm": {"eps": cfg.eps}, "gate": "channel_sigmoid", "score": {"softcap": a.softcap or 0.0},
            "tensors": {"q": "q", "k": "k", "v": "v", "o": "o", "q_norm": "q.norm", "k_norm": "k.norm", "gate": "g"}}
    right = {"n_heads": r.heads, "value_dim": r.vdim, "state": r.state, "groups": r.groups, "taps": r.conv, "norm_parts": r.norm_groups,
             "eps": cfg.eps}
    return PartSpec("summed", {"weights": (m.left_scale, m.right_scale), "left": {"kind": "attention", "params": left, "prefix": "left."},
                               "right": {"kind": "state_space", "params": right, "prefix": "right."}}, prefix)


def build_semanex_spec(cfg: SemanexConfig) -> ModelSpec:
    layers = []
    for i, layer in enumerate(cfg.layers):
        p = f"l{i}."
        parts = [LayerPart("mixer_input", "mixer_input", PartSpec("causal_convolution", {"taps": cfg.taps, "tensor": "canon1"}, p)),
                 LayerPart("mixer", "mixer", _mixer(cfg, layer, p + "mix.")),
                 LayerPart("mixer_norm", "norm", _norm(cfg, p + "norm1", cfg.alpha))]
        if layer.ff:
            parts += [LayerPart("feed_forward", "feed_forward",
                                PartSpec("plain_mlp", {"intermediate_size": layer.ff, "activation": "gelu", "tensors": ("up", "down")},
                                         p + "mlp.")),
                      LayerPart("feed_forward_norm", "norm", _norm(cfg, p + "norm2", cfg.alpha))]
        layers.append(LayerSpec("post_norm", tuple(parts)))
    return ModelSpec(
        architecture=cfg.architecture,
        hidden_size=cfg.width,
        vocab_size=cfg.vocab,
        max_positions=cfg.positions(),
        embedding=PartSpec("token_embedding", {"vocab_size": cfg.vocab, "tensor": "embed", "init_std": 1.0,
                                               "scale": cfg.embedding_scale}, ""),
        layers=tuple(layers),
        schedule=tuple(ScheduleEntry(i) for i in range(len(layers))),
        final_norm=_norm(cfg, "final.norm"),
        head=PartSpec("linear_head", {"vocab_size": cfg.vocab, "tensor": ""}, "head"),
        stop_token_ids=tuple(cfg.eos_token_id),
        bos_token_id=cfg.bos_token_id)


register_architecture("Semanex", SemanexConfig, build_semanex_spec, model_types=("semanex",))
