"""Attention whose keys and values are expanded from one small latent per token, and only the latent is cached.

    cq = rms(Wdq x) * gq,   q_h = Wuq_h cq                      (queries through a latent of their own)
    c  = rms(Wdkv x) * gc                                        (the cached latent, width r)
    k_h = Wuk_h c,  v_h = Wuv_h c,   score = (q_h . k_h) * scale, softmax over the visible keys, out = Wo concat(o_h)

With ``q_rank`` None the queries come straight from one projection, q_h = Wq_h x (tensor ``q``), and the design has no query
latent.  No position enters the scores.  Since k_h and v_h are linear in c, the expansion moves to the query side:
q_h . (Wuk_h c) = (Wuk_h^T q_h) . c and sum_j p_j Wuv_h c_j = Wuv_h (sum_j p_j c_j).  What runs over the cache
is therefore attention of H query heads of width r against ONE shared key/value head, the latent itself:
the paged cache of the layer holds c (as keys and, transposed, as values) and the library's own
attention kernels (prefill on tcgen05, decode over pages, windows, page recycling) serve it unchanged.
The two per-head changes of basis are batched products around the attention.

A part of the keys may carry positions (``rot_dim`` R, ``position``): the queries then hold R more channels per head, one more
projection of x gives R channels that all heads share as keys, and both are rotated (channel 2i with 2i + 1, or, with ``pairing``
"half", channel i with i + half the rotated ones: then those rows of the two projections are interleaved once, when the weights are
bound, and the same kernels serve; scores do not change when queries and keys are permuted alike):

    score = (q_h . k_h + rot(q'_h) . rot(k')) * scale

The cached row is [c | rot(k')] (width r + R), the query against it [Wuk_h^T q_h | rot(q'_h)].  Options that go with it, each a
parameter: a learned sink per head in the softmax's denominator (``sink``), a gate per output channel (``gate``
"channel_sigmoid") and a gate per head ("head_sigmoid": o_h times sigmoid of one logit; being one factor per head it is applied to
the attention's output in the latent's basis, where the attention kernel writes it).  In this form every projection of x - query latent, key/value latent with the shared key part, gate - is a row of
one stacked matrix.  In a bfloat16 run whose r + R fits a width of the tensor-core attention kernels the row is laid out at that
width, zeros behind it, and serves as key and value alike: the value's channels beyond r are read by nobody.
"""
from __future__ import annotations

import math

import torch

from ..config.spec import PartSpec
from ..errors import ConfigError
from ..kernels import ops
from .attention import BRANCH_DTYPE, AttentionMixer
from .base import CacheNeed, Mixer, WeightSpec, make_part, pad_rows, register_mixer


class LatentAttentionMixer(Mixer):
    """params: ``n_heads``, ``key_dim``, ``value_dim`` (per head), ``q_rank`` (None: queries without a latent), ``kv_rank`` (the latents),
    ``eps`` (of the latents' norms), optional ``scale`` (default key_dim^-1/2), ``window`` (None: every
    earlier key; w: a query sees itself and the w - 1 tokens before it), ``tensors`` (local names); optional ``rot_dim`` with
    ``position`` ({"kind": "rotary", "params"}), ``sink`` (True: tensor ``sink`` [n_heads]), ``gate`` (None, "channel_sigmoid":
    tensor ``gate`` [n_heads * value_dim, H], or "head_sigmoid": [n_heads, H]) and ``pairing`` ("interleaved" or "half")."""

    NAMES = {"q_down": "q_a_proj.weight", "q_norm": "q_a_norm.weight", "q_up": "q_b_proj.weight",
             "kv_down": "kv_a_proj.weight", "kv_norm": "kv_a_norm.weight", "k_up": "k_b_proj.weight",
             "v_up": "v_b_proj.weight", "out": "o_proj.weight", "q": "q_proj.weight", "gate": "g_proj.weight", "sink": "sinks"}
    GATES = (None, "channel_sigmoid", "head_sigmoid")

    def __init__(self, params, hidden_size, runtime):
        super().__init__(params, hidden_size, runtime)
        self.n_heads = int(params["n_heads"])
        self.key_dim = int(params["key_dim"])
        self.value_dim = int(params["value_dim"])
        self.q_rank = int(params["q_rank"]) if params.get("q_rank") is not None else None
        self.kv_rank = int(params["kv_rank"])
        self.eps = float(params["eps"])
        if min(self.n_heads, self.key_dim, self.value_dim, self.q_rank if self.q_rank is not None else 1, self.kv_rank) <= 0:
            raise ConfigError("latent attention: heads and sizes must be positive")
        scale = params.get("scale")
        self.scale = float(scale) if scale is not None else 1.0 / math.sqrt(self.key_dim)
        window = params.get("window")
        self.window = int(window) if window else None
        if self.window is not None and self.window < 1:
            raise ConfigError("latent attention: a window holds at least the token itself")
        self.names = dict(self.NAMES, **(params.get("tensors") or {}))
        self.rot_dim = int(params.get("rot_dim") or 0)
        self.sink = bool(params.get("sink", False))
        self.gate = params.get("gate")
        self.gate_width = {None: 0, "channel_sigmoid": self.n_heads * self.value_dim, "head_sigmoid": self.n_heads}.get(self.gate, 0)
        self.pairing = str(params.get("pairing", "interleaved"))
        if self.pairing not in ("half", "interleaved"):
            raise ConfigError(f"latent attention: rotation pairs are 'half' or 'interleaved', not {self.pairing!r}")
        if self.gate not in self.GATES or self.rot_dim < 0:
            raise ConfigError(f"latent attention: unknown gate {self.gate!r} or a negative rotated width")
        position = params.get("position")
        self.position = make_part("position_encoding", PartSpec(position["kind"], position.get("params", {})), hidden_size, runtime) \
            if position else None
        self.tables = None
        if self.position is not None:
            fused = self.position.fused_rotary()
            if fused is None or int(fused[2]) > self.rot_dim:
                raise ConfigError("latent attention: positions are a rotation of at most the shared key part's channels")
            self.tables = (fused[0], fused[1]) if fused[2] else None
        self.stacked = bool(self.rot_dim or self.sink or self.gate)
        # what the cache keeps of a token, and the width of the attention's keys and values
        self.row = self.kv_rank + self.rot_dim
        self.key_width, self.value_width = self.row, self.kv_rank
        if self.stacked and runtime.dtype == torch.bfloat16:
            fits = [w for w in AttentionMixer.TENSOR_CORE_WIDTHS if w >= self.row]
            if fits:
                self.key_width = self.value_width = fits[0]
        self.w_in = self.w_gate = self.sinks = None
        self.w_dq = self.w_dkv = self.q_gain = self.kv_gain = self.w_uq = self.w_uk_t = self.w_uv = self.w_o = None

    def weight_specs(self):
        h, n, H = self.hidden_size, self.names, self.n_heads
        if self.q_rank is None:
            queries = {n["q"]: WeightSpec((H * (self.key_dim + self.rot_dim), h))}
        else:
            queries = {n["q_down"]: WeightSpec((self.q_rank, h)),
                       n["q_norm"]: WeightSpec((self.q_rank,), "precise", ("one_plus_uniform", 0.1)),
                       n["q_up"]: WeightSpec((H * (self.key_dim + self.rot_dim), self.q_rank), init=("normal", 0.1))}
        if self.sink:
            queries[n["sink"]] = WeightSpec((H,), "precise", ("normal", 1.0))
        if self.gate:
            queries[n["gate"]] = WeightSpec((self.gate_width, h), init=("normal", 0.1))
        return {**queries,
                n["kv_down"]: WeightSpec((self.row, h)),
                n["kv_norm"]: WeightSpec((self.kv_rank,), "precise", ("one_plus_uniform", 0.1)),
                n["k_up"]: WeightSpec((H * self.key_dim, self.kv_rank), init=("normal", 0.1)),
                n["v_up"]: WeightSpec((H * self.value_dim, self.kv_rank), init=("normal", 0.1)),
                n["out"]: WeightSpec((h, H * self.value_dim))}

    def _interleaved(self, rows, head, heads):
        """``rows`` [heads * head, n] whose heads end in the rotated part: its pairs (i, i + r/2) brought side by side."""
        dims = 2 * self.tables[0].shape[1] if self.tables is not None else 0
        if self.pairing == "interleaved" or not dims:
            return rows
        at = head - self.rot_dim
        order = list(range(at)) + [at + i + half for i in range(dims // 2) for half in (0, dims // 2)] + list(range(at + dims, head))
        return rows.view(heads, head, -1)[:, torch.tensor(order, device=rows.device)].reshape(rows.shape)

    def bind(self, tensors):
        n, H = self.names, self.n_heads
        if self.q_rank is None:
            self.w_uq = self._interleaved(tensors[n["q"]], self.key_dim + self.rot_dim, H).contiguous()
        else:
            self.w_dq = tensors[n["q_down"]].contiguous()
            self.q_gain = tensors[n["q_norm"]].contiguous()
            self.w_uq = self._interleaved(tensors[n["q_up"]], self.key_dim + self.rot_dim, H).contiguous()
        self.w_dkv = self._interleaved(tensors[n["kv_down"]], self.row, 1).contiguous()
        self.kv_gain = tensors[n["kv_norm"]].contiguous()
        # [H, r, d]: the transposed key expansion of every head, applied to its query
        self.w_uk_t = tensors[n["k_up"]].view(H, self.key_dim, self.kv_rank).transpose(1, 2).contiguous()
        self.w_uv = tensors[n["v_up"]].view(H, self.value_dim, self.kv_rank).contiguous()
        self.w_o = tensors[n["out"]].contiguous()
        self.sinks = tensors[n["sink"]].contiguous() if self.sink else None
        if self.stacked:
            rows = [m for m in (self.w_dq, self.w_dkv) if m is not None]
            self.gate_at = -(-sum(m.shape[0] for m in rows) // 8) * 8             # the gate's columns start 16-byte aligned
            self.w_in = pad_rows([pad_rows(rows, 8)] + ([tensors[n["gate"]]] if self.gate else []))
            self.w_dq = self.w_dkv = None

    def weight_bytes(self):
        mats = (self.w_in, self.w_dq, self.w_dkv, self.w_uq, self.w_uk_t, self.w_uv, self.w_o)
        return sum(m.numel() for m in mats if m is not None) * self.w_o.element_size()

    def cache_need(self):
        # one shared head whose keys and values are both the latent
        return CacheNeed("kv", n_kv_heads=1, head_dim=self.key_width, window=self.window,
                         v_dim=self.value_width if self.value_width != self.key_width else None)

    def _forward_stacked(self, x, step, cache_view):
        """One product of x, both latents' norms with the rotated key part in one kernel, the queries changed to the latent's basis,
        attention over the cached rows (a gate per head in it), back to the values' basis, a gate per channel, the output product."""
        x = ops.resolve(x)
        H, r, rq = self.n_heads, self.kv_rank, self.q_rank or 0
        proj = ops.linear(x, self.w_in, resident=True)
        cq, rows = ops.latent_rows(proj[:, :rq + self.row], self.q_gain if self.q_rank is not None else None, self.kv_gain, self.eps,
                                   self.rot_dim, self.tables, step.token_pos, self.key_width)
        q = ops.linear(cq if cq is not None else x, self.w_uq, resident=True)
        q = ops.latent_queries(q, self.w_uk_t, self.rot_dim, self.tables, step.token_pos, self.key_width)
        keys, values = (rows, rows[:, :self.value_width]) if cache_view.writes else (None, None)
        g = proj[:, self.gate_at:self.gate_at + self.gate_width] if self.gate else None
        per_head = self.gate == "head_sigmoid"
        a = ops.rope_cache_attention(q, keys, values, None, None, 0, step.token_seq, step.token_pos, cache_view.block_table,
                                     cache_view.k, cache_view.v, H, 1, self.key_width, self.scale, int(self.window or 0),
                                     plan=step.attention_plan, value_dim=self.value_width, gate=g if per_head else None,
                                     sinks=self.sinks, split=True)
        o = ops.latent_values(a, self.w_uv, self.value_width, gate=None if per_head else g)       # [T, H*dv]
        return ops.linear(o, self.w_o, out_dtype=BRANCH_DTYPE, resident=True, lazy=True)

    def forward(self, x, step, cache_view):
        if self.stacked:
            return self._forward_stacked(x, step, cache_view)
        dtype = self.runtime.dtype
        if self.q_rank is None:
            cq = x
        else:
            cq = ops.add_rmsnorm(ops.linear(x, self.w_dq, out_dtype=torch.float32, resident=True), None, self.q_gain,
                                 self.eps, dtype)
        q = ops.linear_per_head(ops.linear(cq, self.w_uq, resident=True), self.w_uk_t)            # [T, H*r]
        if cache_view.writes:
            c = ops.add_rmsnorm(ops.linear(x, self.w_dkv, out_dtype=torch.float32, resident=True), None, self.kv_gain,
                                self.eps, dtype)
        else:                                   # reads another execution's latents
            c = None
        a = ops.rope_cache_attention(q, c, c, None, None, 0, step.token_seq, step.token_pos, cache_view.block_table,
                                     cache_view.k, cache_view.v, self.n_heads, 1, self.kv_rank, self.scale,
                                     int(self.window or 0), plan=step.attention_plan)
        o = ops.linear_per_head(a, self.w_uv)                                                      # [T, H*dv]
        return ops.linear(o, self.w_o, out_dtype=BRANCH_DTYPE, resident=True, lazy=True)


register_mixer("latent_attention", LatentAttentionMixer)
