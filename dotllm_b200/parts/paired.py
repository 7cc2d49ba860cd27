"""Two mixers side by side that read the same input: each output is RMS-normalised over the model width with a gain of
its own, and the result is a weighted sum of the two (half and half: their mean).

    y = w_l * rms(left(x)) * gain_l + w_r * rms(right(x)) * gain_r

Either mixer is any registered mixer (softmax attention under a window beside a recurrence, say) with its own tensors under
its own prefix, and keeps what it keeps: the layer's cache need is the pair of theirs, and the layer's view of the cache a
pair of views.  The two norms and the sum are one kernel in float32.
"""
from __future__ import annotations

import torch

from ..config.spec import PartSpec
from ..errors import ConfigError
from ..kernels import ops
from .attention import BRANCH_DTYPE
from .base import Mixer, WeightSpec, make_part, pad_rows, register_mixer


class PairedMixer(Mixer):
    """params: ``left`` and ``right`` ({"kind", "params", "prefix"}: a mixer each, the prefix local to this part), ``eps``,
    optional ``weights`` (default (0.5, 0.5)) and ``tensors``: local names of the gains ``left_norm``, ``right_norm``."""

    NAMES = {"left_norm": "left.out", "right_norm": "right.out"}

    def __init__(self, params, hidden_size, runtime):
        super().__init__(params, hidden_size, runtime)
        self.eps = float(params["eps"])
        self.weights = tuple(float(w) for w in params.get("weights", (0.5, 0.5)))
        if len(self.weights) != 2:
            raise ConfigError("paired mixer: one weight per side")
        self.names = dict(self.NAMES, **(params.get("tensors") or {}))
        self.sides = []
        for side in ("left", "right"):
            d = params[side]
            self.sides.append((str(d.get("prefix", side + ".")),
                               make_part("mixer", PartSpec(d["kind"], d.get("params", {})), hidden_size, runtime)))
        self.graph_safe = all(getattr(m, "graph_safe", True) for _, m in self.sides)
        self.gains = None

    def weight_specs(self):
        specs = {}
        for prefix, mixer in self.sides:
            for local, spec in mixer.weight_specs().items():
                specs[prefix + local] = spec
        for key in ("left_norm", "right_norm"):
            specs[self.names[key]] = WeightSpec((self.hidden_size,), "precise", ("one_plus_uniform", 0.1))
        return specs

    def optional_names(self):
        return {prefix + local for prefix, mixer in self.sides for local in mixer.optional_names()}

    def bind(self, tensors):
        for prefix, mixer in self.sides:
            mixer.bind({local: tensors[prefix + local] for local in mixer.weight_specs()})
        self.gains = tuple(tensors[self.names[key]].contiguous() for key in ("left_norm", "right_norm"))

    def weight_bytes(self):
        return sum(m.weight_bytes() for _, m in self.sides)

    def cache_need(self):
        return tuple(m.cache_need() for _, m in self.sides)

    def forward(self, x, step, cache_view):
        x = ops.resolve(x)                         # a plain tensor: two mixers read it
        left, right = (ops.resolve(m.forward(x, step, view)) for (_, m), view in zip(self.sides, cache_view))
        return ops.pair_norm_sum(left, right, self.gains[0], self.gains[1], self.eps, self.weights[0], self.weights[1])


class SummedMixer(Mixer):
    """A weighted sum of mixers side by side without norms: y = w_l left(x) + w_r right(x).  Both sides ``stack`` (``Mixer.heads``), so
    their projections are one product of the shared input, each side scales what it hands to its output matrix by its weight (in
    float32, where it writes it), and one product with the two output matrices side by side is the sum.

    params: ``left`` and ``right`` ({"kind", "params", "prefix"}), ``weights`` (one per side)."""

    def __init__(self, params, hidden_size, runtime):
        super().__init__(params, hidden_size, runtime)
        self.weights = tuple(float(w) for w in params["weights"])
        if len(self.weights) != 2:
            raise ConfigError("summed mixer: one weight per side")
        self.sides = []
        for side in ("left", "right"):
            d = params[side]
            mixer = make_part("mixer", PartSpec(d["kind"], d.get("params", {})), hidden_size, runtime)
            if not mixer.stacks:
                raise ConfigError(f"summed mixer: a mixer of kind {d['kind']!r} does not share its products")
            mixer.compact = True
            self.sides.append((str(d.get("prefix", side + ".")), mixer))
        self.graph_safe = all(getattr(m, "graph_safe", True) for _, m in self.sides)
        self.w_in = self.w_o = None
        self.at = ()                       # where each side's columns start: (in the stacked projection, in the stacked heads)

    def weight_specs(self):
        return {prefix + local: spec for prefix, mixer in self.sides for local, spec in mixer.weight_specs().items()}

    def optional_names(self):
        return {prefix + local for prefix, mixer in self.sides for local in mixer.optional_names()}

    def bind(self, tensors):
        for prefix, mixer in self.sides:
            mixer.bind({local: tensors[prefix + local] for local in mixer.weight_specs()})
        left, right = (m for _, m in self.sides)
        self.at = ((0, 0), (left.w_in.shape[0], left.out_width))
        self.w_in = pad_rows([left.w_in, right.w_in])
        outs = [left.w_o, right.w_o]
        pad = -(left.out_width + right.out_width) % 8                   # the products like whole eights of columns
        if pad:
            outs.append(torch.zeros((self.hidden_size, pad), dtype=left.w_o.dtype, device=left.w_o.device))
        self.w_o = torch.cat(outs, dim=1).contiguous()
        self.widths = tuple((m.w_in.shape[0], m.out_width) for _, m in self.sides)
        self.padded = bool(pad)
        left.w_in = right.w_in = left.w_o = right.w_o = None            # the stacked ones serve

    def weight_bytes(self):
        return (self.w_in.numel() + self.w_o.numel()) * self.w_in.element_size()

    def cache_need(self):
        return tuple(m.cache_need() for _, m in self.sides)

    def forward(self, x, step, cache_view):
        x = ops.resolve(x)
        proj = ops.linear(x, self.w_in, resident=True)
        make = torch.zeros if self.padded else torch.empty
        y = make((x.shape[0], self.w_o.shape[1]), dtype=self.runtime.dtype, device=x.device)
        for (_, mixer), weight, (p0, y0), (pn, yn), view in zip(self.sides, self.weights, self.at, self.widths, cache_view):
            mixer.heads(proj[:, p0:p0 + pn], step, view, scale=weight, out=y[:, y0:y0 + yn])
        return ops.linear(y, self.w_o, out_dtype=BRANCH_DTYPE, resident=True, lazy=True)


register_mixer("paired", PairedMixer)
register_mixer("summed", SummedMixer)
