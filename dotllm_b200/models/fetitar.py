"""The Fetitar decoder as a model description.

Token embedding times a constant plus a row for the pair of a token and the one before it; layers with a norm before and behind
each sublayer, every gain kept around zero; per layer one of two mixers - softmax attention over a window (biases on all four
projections, one RMS norm over all query and one over all key channels, no rotation but a penalty per distance with a slope per
head, values mixed with the first such layer's) or latent attention over a window (a rotated key part shared by the heads under
YaRN frequencies, a gate per head) - and a dense gated feed-forward with biases (silu), or none; a last norm and a head of its own.
Tensor names: ``embed``, ``bigram``, ``l<i>.norm1``, ``l<i>.norm1b``, ``l<i>.norm2``, ``l<i>.norm2b``, ``l<i>.mix.*``, ``l<i>.mlp.*``
(a bias is its matrix's name with ``.b`` behind it), ``final.norm``, ``head``.
"""
from __future__ import annotations

from ..config.fetitar import FetitarConfig
from ..config.registry import register_architecture
from ..config.spec import LayerPart, LayerSpec, ModelSpec, PartSpec, ScheduleEntry


def distance_slopes(heads):
    """The penalty per token of distance of every head: 2^(-8 (h + 1) / heads)."""
    return [2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)]


def _norm(cfg, name):
    return PartSpec("rmsnorm", {"eps": cfg.eps, "offset": 1.0, "tensor": ""}, name)


def _rotation(rot, positions):
    scaling = None
    if rot.scaling:
        scaling = {"rope_type": "yarn", "factor": rot.scaling.factor, "original_max_position_embeddings": rot.scaling.original,
                   "fast_turns": rot.scaling.fast, "slow_turns": rot.scaling.slow}
    return {"kind": "rotary", "params": {"rotary_dim": rot.dims, "theta": rot.base, "max_positions": positions, "scaling": scaling}}


def _mixer(cfg, i, prefix):
    m = cfg.layers[i].mixer
    if cfg.layers[i].type == "latent_attention":
        return PartSpec("latent_attention",
                        {"n_heads": m.heads, "key_dim": m.dim, "rot_dim": m.rot_dim, "value_dim": m.vdim, "q_rank": m.q_rank,
                         "kv_rank": m.kv_rank, "eps": cfg.eps, "scale": m.scale, "window": m.window, "gate": "head_sigmoid", "pairing": "half",
                         "position": _rotation(m.rot, cfg.positions()) if m.rot.dims else None,
                         "tensors": {"q_down": "dq", "q_norm": "dq.norm", "q_up": "uq", "kv_down": "dkv", "kv_norm": "dkv.norm", "k_up": "uk",
                                     "v_up": "uv", "out": "o", "gate": "g"}}, prefix)
    params = {"n_heads": m.heads, "n_kv_heads": m.kv_heads, "head_dim": m.dim, "value_dim": m.vdim, "scale": m.scale, "window": m.window,
              "position": None, "bias": "all", "qk_norm": {"eps": cfg.eps, "over": "projection"},
              "score": {"slopes": distance_slopes(m.heads)},
              "tensors": {"q": "q", "k": "k", "v": "v", "o": "o", "q_bias": "q.b", "k_bias": "k.b", "v_bias": "v.b", "o_bias": "o.b",
                          "q_norm": "q.norm", "k_norm": "k.norm", "mix": "vmix"}}
    if m.v_mix:
        first = next(j for j, layer in enumerate(cfg.layers) if layer.type == "attention" and layer.mixer.v_mix)
        params["value_mix"] = {"first": i == first}
    return PartSpec("attention", params, prefix)


def build_fetitar_spec(cfg: FetitarConfig) -> ModelSpec:
    layers, unused = [], []
    for i, layer in enumerate(cfg.layers):
        p = f"l{i}."
        parts = [LayerPart("mixer_norm", "norm", _norm(cfg, p + "norm1")),
                 LayerPart("mixer", "mixer", _mixer(cfg, i, p + "mix.")),
                 LayerPart("mixer_post_norm", "norm", _norm(cfg, p + "norm1b"))]
        if layer.type == "attention" and not layer.mixer.v_mix:
            unused.append(p + "mix.vmix")
        if layer.ff:
            parts += [LayerPart("feed_forward_norm", "norm", _norm(cfg, p + "norm2")),
                      LayerPart("feed_forward", "feed_forward",
                                PartSpec("gated_mlp", {"intermediate_size": layer.ff, "activation": "silu", "bias": ".b",
                                                       "tensors": ("gate", "up", "down")}, p + "mlp.")),
                      LayerPart("feed_forward_post_norm", "norm", _norm(cfg, p + "norm2b"))]
        else:                                                  # a checkpoint may still carry the absent sublayer's norms
            unused += [p + "norm2", p + "norm2b"]
        layers.append(LayerSpec("sandwich_norm", tuple(parts)))
    tables = {"vocab_size": cfg.vocab, "tensor": "embed", "init_std": 1.0, "scale": cfg.embedding_scale}
    if cfg.bigram:
        embedding = PartSpec("token_pair_embedding", {**tables, "pair_tensor": "bigram", "buckets": cfg.bigram.buckets,
                                                      "mul_prev": cfg.bigram.mul_prev, "mul_cur": cfg.bigram.mul_cur}, "")
    else:
        embedding = PartSpec("token_embedding", tables, "")
    return ModelSpec(
        architecture=cfg.architecture,
        hidden_size=cfg.width,
        vocab_size=cfg.vocab,
        max_positions=cfg.positions(),
        embedding=embedding,
        layers=tuple(layers),
        schedule=tuple(ScheduleEntry(i) for i in range(len(layers))),
        final_norm=_norm(cfg, "final.norm"),
        head=PartSpec("linear_head", {"vocab_size": cfg.vocab, "tensor": ""}, "head"),
        stop_token_ids=tuple(cfg.eos_token_id),
        bos_token_id=cfg.bos_token_id,
        optional_weights=tuple(unused))


register_architecture("Fetitar", FetitarConfig, build_fetitar_spec, model_types=("fetitar",))
