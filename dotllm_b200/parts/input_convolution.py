"""What a mixer reads, mixed with its own past first: h_t = x_t + sum_j w_j x_(t-K+1+j), a short causal convolution over time per
channel, zeros before the sequence's start.

The last K - 1 inputs are part of a sequence's state (float32, one vector per slot).  In a step of one token per sequence the
convolution rides the kernel that settles the stream (``ops.post_norm``); other steps run ``ops.causal_conv`` behind it.
"""
from __future__ import annotations

import torch

from ..errors import ConfigError
from ..kernels import ops
from .base import CacheNeed, MixerInput, WeightSpec, register_mixer_input


class InputConvolution(MixerInput):
    """params: ``taps`` (K); optional ``tensor``: the local name of the weights [H, K] (default "weight"; the last column meets the
    current token)."""

    MAX_TAPS = 64                # CC_MAX_TAPS in csrc/causal_conv.cu

    def __init__(self, params, hidden_size, runtime):
        super().__init__(params, hidden_size, runtime)
        self.taps = int(params["taps"])
        if not 0 < self.taps <= self.MAX_TAPS:
            raise ConfigError(f"input convolution: {self.taps} taps; the kernel takes 1 to {self.MAX_TAPS}")
        self.tensor_name = str(params.get("tensor", "weight"))
        self.weight = None

    def weight_specs(self):
        return {self.tensor_name: WeightSpec((self.hidden_size, self.taps), "precise", ("normal", 0.3))}

    def bind(self, tensors):
        self.weight = tensors[self.tensor_name].t().contiguous()           # [K, H]: a thread's channels lie side by side

    def weight_bytes(self):
        return self.weight.numel() * self.weight.element_size()

    def cache_need(self):
        return CacheNeed("state", state_shape=(max(1, (self.taps - 1) * self.hidden_size),), state_dtype=torch.float32)

    def read(self, stream, pending, step, cache_view):
        plan = step.attention_plan
        if plan.all_single:
            return ops.post_norm(stream, pending, self.runtime.dtype, conv=(self.weight, cache_view.state, cache_view.slots))
        if pending is not None:
            ops.post_norm(stream, pending)
        return ops.causal_conv(stream, self.weight, cache_view.state, step.cu_new, cache_view.slots, plan.max_new, add_input=True,
                               out_dtype=self.runtime.dtype)


register_mixer_input("causal_convolution", InputConvolution)
