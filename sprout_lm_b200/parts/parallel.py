"""Several mixers side by side: all read the same normed input h, and the layer's mixer output is the weighted sum
``sum_i scales[i] * mixer_i(h)``, times ``out_scale``.

Each sub-mixer is a registered mixer of its own, built from its ``PartSpec`` with the prefix ``prefix + names[i]`` and with
its weight as the constructor parameter ``out_scale`` (every mixer that can stand here folds that factor into its own last
step before the output projection, so the sum costs no kernel).  With ``norms`` (two tensor names, a pair of mixers) each
mixer's output is first divided by its root mean square over the model's width (``norm_eps``) and multiplied by a weight of
that width; the scales must then be equal, and one kernel norms both outputs and adds them.

At most one sub-mixer may keep keys and values per token (the layer has one cache slot).  The sub-mixers' per-request states
stand side by side in the layer's one state entry; each gets the views of its own.
"""
from __future__ import annotations

import torch

from .. import kernels
from ..config.specs import PartSpec
from .base import Part, StateView, TensorDecl, build_part, register_part


@register_part("mixer", "parallel_mixers")
class ParallelMixers(Part):
    def __init__(self, prefix: str, mixers, scales, names, out_scale: float = 1.0, norms=None, norm_eps: float = 0.0,
                 hidden_size: int | None = None):
        mixers, scales, names = tuple(mixers), tuple(float(s) for s in scales), tuple(names)
        if not mixers or len(mixers) != len(scales) or len(mixers) != len(names):
            raise ValueError("parallel_mixers: one scale and one name per mixer, at least one mixer")
        self.scales = tuple(s * float(out_scale) for s in scales)
        self.norm_names = None
        if norms is not None:
            if len(norms) != 2 or len(mixers) != 2 or scales[0] != scales[1] or norm_eps <= 0 or not hidden_size:
                raise ValueError("parallel_mixers: output norms are for a pair of mixers of equal scale; they need eps and the width")
            self.norm_names, self.norm_eps, self.hidden_size = tuple(prefix + n for n in norms), float(norm_eps), int(hidden_size)
        factors = (1.0,) * len(mixers) if norms is not None else self.scales
        self.mixers = [build_part("mixer", PartSpec(spec.kind, {**spec.params, "out_scale": factor * spec.params.get("out_scale", 1.0)}),
                                  prefix + name)
                       for spec, factor, name in zip(mixers, factors, names)]
        self.cached = [i for i, m in enumerate(self.mixers) if m.cache_spec() is not None]
        if len(self.cached) > 1:
            raise ValueError("parallel_mixers: at most one mixer with keys and values per token")
        # where each mixer's state tensors stand among the layer's: (first, count), count None for a mixer with a single one
        self.state_places, at = {}, 0
        for i, m in enumerate(self.mixers):
            spec = m.state_spec()
            if spec is None:
                continue
            count = len(spec) if isinstance(spec, (tuple, list)) else None
            self.state_places[i] = (at, count)
            at += 1 if count is None else count
        self.gains = None

    def cache_spec(self):
        return self.mixers[self.cached[0]].cache_spec() if self.cached else None

    def state_spec(self):
        if len(self.state_places) == 1:
            return self.mixers[next(iter(self.state_places))].state_spec()
        specs = []
        for i in self.state_places:
            spec = self.mixers[i].state_spec()
            specs += list(spec) if isinstance(spec, (tuple, list)) else [spec]
        return tuple(specs) or None

    def _state_of(self, index: int, state):
        if state is None or index not in self.state_places:
            return None
        if len(self.state_places) == 1:
            return state
        first, count = self.state_places[index]
        return state.part(first) if count is None else StateView(tuple(state.buffer[first:first + count]), state.slots)

    def decode_plan(self, requests: int, max_keys: int, planned_context: int, page_tokens: int):
        return tuple(m.decode_plan(requests, max_keys, planned_context, page_tokens) for m in self.mixers)

    def tensor_decls(self):
        decls = [decl for m in self.mixers for decl in m.tensor_decls()]
        return decls + [TensorDecl(name, (self.hidden_size,), "gain") for name in self.norm_names or ()]

    def load(self, source):
        for m in self.mixers:
            m.load(source)
        if self.norm_names is not None:
            self.gains = [source.vector(name) for name in self.norm_names]

    def forward(self, h, x, ctx, cache, state):
        targets = [x] * len(self.mixers)
        if self.norm_names is not None:
            both = torch.zeros((2, *x.shape), dtype=torch.float32, device=x.device)
            targets = [both[0], both[1]]
        for i, m in enumerate(self.mixers):
            m.forward(h, targets[i], ctx, cache if i in self.cached else None, self._state_of(i, state))
        if self.norm_names is not None:
            kernels.rms_pair_add(both[0], both[1], self.gains[0], self.gains[1], x, self.norm_eps, self.scales[0])
