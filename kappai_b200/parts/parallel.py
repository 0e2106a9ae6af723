"""Several mixers side by side on the same input: ``parallel``.

Every mixer reads the layer's normed input and adds its output into the residual (a mixer that is weighed in the sum has a
parameter of its own for that, ``out_scale``).  Mixers that offer their first product (``input_product`` -> weight and
bias, ``forward_projected`` on its rows) have it run as one product with the others' (and where all of them do, the whole
offers that product in turn); what the mixers keep is a
:class:`~kappai_b200.cache.spec.CompositeSpec` in their order.

Params: mixers (a dict name -> ``mixer`` PartSpec; a mixer's tensors are known here as ``<name>.<its local name>``, its own
prefix and renaming applied first).
"""
from __future__ import annotations

from typing import Dict

import torch

from ..cache.spec import CompositeSpec
from ..config.schema import ConfigError, PartSpec
from ..ops.linear import linear
from .base import Part, WeightSpec, make_part, register_part


class ParallelMixers(Part):
    category = "mixer"

    def __init__(self, params, env):
        super().__init__(params, env)
        specs = self._p("mixers")
        if not isinstance(specs, dict) or not specs:
            raise ConfigError("parallel: mixers must name at least one mixer")
        self.specs = {n: PartSpec(**s) if isinstance(s, dict) else s for n, s in specs.items()}
        self.mixers = {n: make_part("mixer", s, env) for n, s in self.specs.items()}
        self.inner_parts = tuple(self.mixers.values())
        self.graph_safe = all(m.graph_safe for m in self.inner_parts)
        self.joined = [n for n, m in self.mixers.items() if hasattr(m, "input_product")]
        if len(self.joined) < 2:
            self.joined = []

    def _names(self, n: str) -> Dict[str, str]:
        s = self.specs[n]
        return {local: f"{n}.{s.prefix}{s.rename.get(local, local)}" for local in self.mixers[n].weight_specs()}

    def weight_specs(self) -> Dict[str, WeightSpec]:
        out = {}
        for n, m in self.mixers.items():
            names = self._names(n)
            out.update({names[local]: ws for local, ws in m.weight_specs().items()})
        return out

    def bind(self, w):
        for n, m in self.mixers.items():
            m.bind({local: w[name] for local, name in self._names(n).items() if name in w})
        self.w_in = self.b_in = None
        self.cols = {}
        if self.joined:
            products = [self.mixers[n].input_product() for n in self.joined]
            at = 0
            for n, (wt, _) in zip(self.joined, products):
                self.cols[n] = (at, at + wt.shape[0])
                at += wt.shape[0]
            if any(b is not None for _, b in products):
                self.b_in = torch.cat([b if b is not None else torch.zeros(wt.shape[0], dtype=torch.float32, device=wt.device)
                                       for wt, b in products]).contiguous()
            self.w_in = torch.cat([wt for wt, _ in products], 0).contiguous()
            for n in self.joined:
                self.mixers[n].drop_input_product()

    def input_product(self):
        """The joined product, or None where some mixer runs a product of its own."""
        return (self.w_in, self.b_in) if len(self.joined) == len(self.mixers) else None

    def drop_input_product(self):
        self.w_in = self.b_in = None

    def cache_spec(self):
        return CompositeSpec(tuple(m.cache_spec() for m in self.mixers.values()))

    def forward(self, h, residual, ctx, cache):
        """``cache``: a :class:`~kappai_b200.cache.storage.CompositeView`, one view a mixer."""
        self._run(h, linear(h, self.w_in, self.b_in) if self.joined else None, residual, ctx, cache)

    def forward_projected(self, p, residual, ctx, cache):
        self._run(None, p, residual, ctx, cache)

    def _run(self, h, p, residual, ctx, cache):
        for (n, m), view in zip(self.mixers.items(), cache.parts):
            if n in self.cols:
                a, b = self.cols[n]
                m.forward_projected(p[:, a:b], residual, ctx, view)
            else:
                m.forward(h, residual, ctx, view)


register_part("mixer", "parallel", ParallelMixers)
