"""Mixers side by side: all read the same input, and the result is the sum of their outputs, each
times a constant.  Each keeps a cache of its own kind (``RunEntry.cache`` names one for each).  Their
first products are ONE product (mixers with ``shares_input_product``), and their outputs are added up
by the kernel that ends the sublayer where the block lets them (``TermSum``)."""
from __future__ import annotations

import torch

from .. import ops
from .base import Mixer, TermSum, make_part, register_mixer
from .plan import PartSpec


class ParallelMixers(Mixer):
    defers_terms = True

    def __init__(self, mixers: tuple[PartSpec, ...], scales: tuple[float, ...]):
        self.mixers = [make_part("mixer", m) for m in mixers]
        self.scales = [float(s) for s in scales]
        if len(self.mixers) != len(self.scales) or len(self.mixers) != 2:
            raise ValueError("two mixers run side by side, each with a scale")
        if not all(m.shares_input_product for m in self.mixers):
            raise ValueError("mixers side by side start with one product of their input each")

    def tensor_specs(self):
        return [s for m in self.mixers for s in m.tensor_specs()]

    def load(self, tensors, dtype, device):
        rows = [m.input_matrix(tensors) for m in self.mixers]
        self.first = ops.Linear(torch.cat(rows, dim=0), None, out_dtype=torch.float32)
        self.widths = [r.shape[0] for r in rows]
        for m in self.mixers:
            m.load(tensors, dtype, device, own_product=False)

    def cache_spec(self):
        return tuple(m.cache_spec() for m in self.mixers)

    def forward(self, x, ctx, cache, defer_terms: bool = False):
        parts = torch.split(self.first(x), self.widths, dim=1)
        out = TermSum([(m.from_projection(p, ctx, c), s, None)
                       for m, p, c, s in zip(self.mixers, parts, cache, self.scales)])
        return out if defer_terms else out.materialize()


register_mixer("parallel", ParallelMixers)
