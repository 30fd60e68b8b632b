"""Several mixers side by side: one input, one sum.

    y = sum over the members m of  m(h)

params: ``members`` (PartSpecs of the mixer family whose parts offer the split form, see ``gla.py``; a member's weight in
the sum is its own ``out_factor``).  The members' projections are one stacked product, their output projections one
product over the concatenated rows; in between each member runs its own kernels on its columns.  The members ask the cache
manager for what they need themselves (at most one paged cache and one unnamed state among them).
"""
from __future__ import annotations

import torch

from .gla import SplitMixer
from .spec import BuildEnv, PartSpec, part_factory, register_part


class SideBySide(SplitMixer):
    def __init__(self, spec: PartSpec, env: BuildEnv):
        self.members = [part_factory("mixer", m.kind)(m, env) for m in spec.params["members"]]
        for m in self.members:
            if not hasattr(m, "core"):
                raise ValueError(f"side by side: {type(m).__name__} does not offer the split form of a mixer")
        self.dtype = env.dtype
        self.out_dim = sum(m.out_dim for m in self.members)

    def tensor_specs(self):
        return [s for m in self.members for s in m.tensor_specs()]

    @property
    def graph_safe(self):
        return all(getattr(m, "graph_safe", True) for m in self.members)

    def bind(self, tensors):
        for m in self.members:
            m.bind(tensors)
        self.w_in = torch.cat([m.w_in for m in self.members], dim=0).contiguous()
        self.w_out = torch.cat([m.w_out for m in self.members], dim=1).contiguous()
        row = col = 0
        for m in self.members:                  # the members keep views of the joined matrices, not copies of their own
            m.w_in, row = self.w_in[row:row + m.w_in.shape[0]], row + m.w_in.shape[0]
            m.w_out, col = self.w_out[:, col:col + m.out_dim], col + m.out_dim

    def cache_need(self):
        out = []
        for m in self.members:
            need = m.cache_need()
            out += list(need) if isinstance(need, (list, tuple)) else [need]
        return out

    def core(self, proj, ctx, cache, y):
        row = col = 0
        for m in self.members:
            m.core(proj[:, row:row + m.w_in.shape[0]], ctx, cache, y[:, col:col + m.out_dim])
            row, col = row + m.w_in.shape[0], col + m.out_dim


register_part("mixer", "side_by_side", SideBySide)
