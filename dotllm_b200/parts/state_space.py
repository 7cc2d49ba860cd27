"""A state-space mixer with one decay per head and token (Mamba-2): a recurrence whose state is a matrix per head.

    [z | x | B | C | dt] = W_in h                                        (inner, inner, G N, G N, heads; inner = heads * P)
    x, B, C <- silu(conv(x, B, C) + b)                                    (a short causal convolution per channel)
    dt <- softplus(dt + dt_bias)
    S_t = exp(-exp(A_h) dt) S_(t-1) + dt B x^T,   y = S_t^T C + D_h x      (S: [N, P] per head; heads share B and C in G groups)
    out = W_o (rms over equal parts of (y * silu(z)) * gain)               (the gate comes before the norm)

What a sequence carries - every head's state and the convolution's last K - 1 inputs - is the layer execution's fixed-size
cache entry, one float32 vector per slot, zero when a sequence opens.  The convolution leaves x, B and C in the run dtype (its sums
are float32); steps, decays, the recurrence and everything up to the gate are float32 in either run dtype.  The kernels walk a sequence's new tokens in order from that entry, so prompts, parts of
prompts and decoded tokens are one code path.
"""
from __future__ import annotations

import torch

from ..errors import ConfigError
from ..kernels import ops
from .attention import BRANCH_DTYPE
from .base import CacheNeed, Mixer, WeightSpec, pad_rows, register_mixer


class StateSpaceMixer(Mixer):
    """params: ``n_heads``, ``value_dim`` (P), ``state`` (N), ``groups`` (G), ``taps`` (K), ``norm_parts``, ``eps``; optional
    ``tensors``: local names of in, conv, conv_bias, dt_bias, rate, skip, norm, out."""

    NAMES = {"in": "in", "conv": "conv", "conv_bias": "conv.b", "dt_bias": "dt_bias", "rate": "A_log", "skip": "D", "norm": "norm",
             "out": "o"}
    MAX_STATE, MAX_TAPS = 512, 64        # SS_MAX_STATE in csrc/ssd.cu, CC_MAX_TAPS in csrc/causal_conv.cu
    stacks = True

    def __init__(self, params, hidden_size, runtime):
        super().__init__(params, hidden_size, runtime)
        self.n_heads, self.value_dim = int(params["n_heads"]), int(params["value_dim"])
        self.state, self.groups = int(params["state"]), int(params["groups"])
        self.taps, self.norm_parts, self.eps = int(params["taps"]), int(params["norm_parts"]), float(params["eps"])
        if min(self.n_heads, self.value_dim, self.state, self.groups, self.taps, self.norm_parts) <= 0:
            raise ConfigError("state-space mixer: heads, sizes, groups, taps and parts must be positive")
        self.inner = self.n_heads * self.value_dim
        if self.n_heads % self.groups or self.inner % self.norm_parts:
            raise ConfigError(f"state-space mixer: {self.n_heads} heads in {self.groups} groups, {self.inner} channels in "
                              f"{self.norm_parts} parts do not come out even")
        if self.state > self.MAX_STATE or self.taps > self.MAX_TAPS:
            raise ConfigError(f"state-space mixer: the kernels take up to {self.MAX_STATE} state channels and convolutions of up to "
                              f"{self.MAX_TAPS} taps, not {self.state} and {self.taps}")
        self.names = dict(self.NAMES, **(params.get("tensors") or {}))
        self.channels = self.inner + 2 * self.groups * self.state             # what passes the convolution
        self.state_size = self.n_heads * self.state * self.value_dim
        self.out_width = self.inner
        self.w_in = self.conv = self.conv_bias = self.dt_bias = self.rate = self.skip = self.norm_gain = self.w_o = None

    def weight_specs(self):
        h, n, H = self.hidden_size, self.names, self.n_heads
        return {n["in"]: WeightSpec((self.inner + self.channels + H, h), init=("normal", 0.1)),
                n["conv"]: WeightSpec((self.channels, self.taps), "precise", ("normal", 0.5)),
                n["conv_bias"]: WeightSpec((self.channels,), "precise", ("normal", 0.1)),
                n["dt_bias"]: WeightSpec((H,), "precise", ("normal", 1.0)),
                n["rate"]: WeightSpec((H,), "precise", ("normal", 0.5)),
                n["skip"]: WeightSpec((H,), "precise", ("normal", 0.5)),
                n["norm"]: WeightSpec((self.inner,), "precise", ("one_plus_uniform", 0.1)),
                n["out"]: WeightSpec((h, self.inner))}

    def bind(self, tensors):
        n = self.names
        # rows in the order xBC, z, dt: the convolution's columns start the product's row, 16-byte aligned whatever the head count
        w = tensors[n["in"]]
        self.w_in = pad_rows([w[self.inner:self.inner + self.channels], w[:self.inner], w[self.inner + self.channels:]])
        self.conv = tensors[n["conv"]].t().contiguous()                       # [K, channels]
        self.conv_bias = tensors[n["conv_bias"]].contiguous()
        self.dt_bias, self.rate, self.skip = (tensors[n[k]].contiguous() for k in ("dt_bias", "rate", "skip"))
        self.norm_gain = tensors[n["norm"]].contiguous()
        self.w_o = tensors[n["out"]].contiguous()

    def weight_bytes(self):
        return (self.w_in.numel() + self.w_o.numel()) * self.w_in.element_size()

    def cache_need(self):
        # per slot: the heads' states, then the convolution's last K - 1 inputs
        return CacheNeed("state", state_shape=(self.state_size + (self.taps - 1) * self.channels,), state_dtype=torch.float32)

    def heads(self, proj, step, cache_view, scale=1.0, out=None):
        C, W, memory = self.channels, self.inner, cache_view.state
        z, dt = proj[:, C:C + W], proj[:, C + W:C + W + self.n_heads]
        xbc = ops.causal_conv(proj[:, :C], self.conv, memory[:, self.state_size:], step.cu_new, cache_view.slots,
                              step.attention_plan.max_new, bias=self.conv_bias, activation="silu", out_dtype=self.runtime.dtype)
        y = ops.ssd_scan(xbc, dt, self.dt_bias, self.rate, self.skip, step.cu_new, cache_view.slots, memory, self.n_heads, self.groups,
                         self.state, self.value_dim, max_new=step.attention_plan.max_new)
        return ops.gated_group_norm(y, z, self.norm_gain, self.norm_parts, self.eps, scale=scale, out=out)

    def forward(self, x, step, cache_view):
        y = self.heads(ops.linear(x, self.w_in, resident=True), step, cache_view)
        return ops.linear(y, self.w_o, out_dtype=BRANCH_DTYPE, resident=True, lazy=True)


register_mixer("state_space", StateSpaceMixer)
