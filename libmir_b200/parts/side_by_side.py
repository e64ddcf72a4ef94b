"""Several mixers side by side: all read the same input, and the result is a constant times the sum of their outputs,
each first RMS-normed over the model width with a plain weight of its own,
    out = scale * sum_b rmsnorm(branch_b(x)) * w_b.
Each branch writes its output into a 32-bit buffer (Mixer.forward with overwrite=True); one kernel norms the buffers
and adds the sum into the residual.  With a factor per branch instead of the norms (spec.scales),
    out = sum_b scale_b * branch_b(x),
an arrangement that follows with a kernel over the sum takes the buffers and factors as they are (`results`).  A branch may be any registered mixer: it gets its own part of the schedule
entry's cache (the pages if it asked for pages, its own run of the fixed-size states).
"""

from __future__ import annotations

import torch

from .. import kernels
from ..config.spec import ParamSpec, bundle_requirements, split_requirement
from ..registry import build_part
from .base import Mixer


class SideBySide(Mixer):
    def __init__(self, spec, env):
        super().__init__(spec, env)
        if not 1 <= len(spec.branches) <= 4:
            raise ValueError("one to four branches")
        self.names = [name for name, _ in spec.branches]
        self.branches = [build_part(branch, env) for _, branch in spec.branches]
        self.normed = not spec.scales
        if not self.normed and len(spec.scales) != len(spec.branches):
            raise ValueError("one factor per branch")
        self.out_weights = [None] * len(self.branches)
        # which part of the entry's cache each branch sees: (pages?, first state, states)
        self.cache_parts, cursor = [], 0
        for branch in self.branches:
            pages, states = split_requirement(branch.cache_requirement())
            self.cache_parts.append((pages is not None, cursor, len(states)))
            cursor += len(states)

    @property
    def graph_safe(self):
        return all(branch.graph_safe for branch in self.branches)

    @property
    def takes_normed_residual(self):
        return all(branch.takes_normed_residual for branch in self.branches)

    @property
    def portion_multiple(self):
        import math
        return math.lcm(*[max(1, int(branch.portion_multiple)) for branch in self.branches])

    def cache_requirement(self):
        return bundle_requirements([branch.cache_requirement() for branch in self.branches])

    def parameters(self):
        table = {}
        for name, branch in zip(self.names, self.branches):
            for local, param in branch.parameters().items():
                table[f"{name}.{local}"] = param
            if self.normed:
                table[f"{name}.{self.spec.out_tensor}"] = ParamSpec((self.spec.hidden_size,), init="ones", store="float32")
        return table

    def bind(self, tensors):
        for index, (name, branch) in enumerate(zip(self.names, self.branches)):
            prefix = name + "."
            mine = {local[len(prefix):]: tensor for local, tensor in tensors.items() if local.startswith(prefix)}
            if self.normed:
                self.out_weights[index] = mine.pop(self.spec.out_tensor).contiguous()
            branch.bind(mine)

    def weight_bytes(self):
        return sum(branch.weight_bytes() for branch in self.branches) + \
            sum(w.numel() * 4 for w in self.out_weights if w is not None)

    def outputs(self, ctx, cache, x, shape) -> list:
        outputs = []
        for branch, (pages, first, count) in zip(self.branches, self.cache_parts):
            out = ctx.alloc(shape, torch.float32)
            branch.forward(ctx, cache.part(pages, first, count) if cache is not None else None, x, out, overwrite=True)
            outputs.append(out)
        return outputs

    def results(self, ctx, cache, x, shape):
        if self.normed:
            return super().results(ctx, cache, x, shape)
        return list(zip(self.outputs(ctx, cache, x, shape), self.spec.scales))

    def forward(self, ctx, cache, x, residual, overwrite=False):
        outputs = self.outputs(ctx, cache, x, tuple(residual.shape))
        if not self.normed:
            kernels.scaled_sum(outputs, self.spec.scales, residual, accumulate=not overwrite)
            ctx.residual_stats = None
            return
        if overwrite:
            residual.zero_()
        kernels.add_normed_branches(outputs, self.out_weights, residual, self.spec.eps, self.spec.scale)
        ctx.residual_stats = None
