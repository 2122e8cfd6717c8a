"""Mixers side by side on one input: ``sum_i scale_i * branch_i(h)`` (``ParallelMixerSpec``).

The branches' input products are one product (their matrices stacked), and so are their output products (their matrices
side by side, the branches' results in one row): a branch only fills its columns of that row, times its scale, in
between (``BranchMixer.mix``). The paged cache and the state that the schedule entry binds belong to the branch that asks
for them.
"""

from __future__ import annotations

import torch

from matricxon_b200.ops.linear import EPILOGUE_F32, EPILOGUE_RESIDUAL, linear
from matricxon_b200.parts.base import BranchMixer, Mixer, build_part, part_class, register_part


@register_part("mixer", "parallel")
class ParallelMixer(Mixer):
    def __init__(self, spec, runtime, prefix):
        super().__init__(spec, runtime, prefix)
        self.branches = []
        for sub, scale, name in spec.branches:
            if not issubclass(part_class("mixer", sub.kind), BranchMixer):
                raise ValueError(f"mixer {sub.kind!r} cannot stand beside others (it is no BranchMixer)")
            self.branches.append((build_part("mixer", sub, runtime, prefix + name), float(scale)))
        self.cache_request(spec)
        self.state_request(spec)
        self.capturable = all(branch.capturable for branch, _ in self.branches)

    @classmethod
    def weight_specs(cls, spec, prefix):
        return [item for sub, _, name in spec.branches
                for item in part_class("mixer", sub.kind).weight_specs(sub, prefix + name)]

    @staticmethod
    def _only(requests, what):
        requests = [request for request in requests if request is not None]
        if len(requests) > 1:
            raise ValueError(f"two branches of a parallel mixer ask for {what}")
        return requests[0] if requests else None

    @classmethod
    def cache_request(cls, spec):
        return cls._only([part_class("mixer", sub.kind).cache_request(sub) for sub, _, _ in spec.branches], "paged cache")

    @classmethod
    def state_request(cls, spec):
        return cls._only([part_class("mixer", sub.kind).state_request(sub) for sub, _, _ in spec.branches], "state")

    def load(self, fetch):
        for branch, _ in self.branches:
            branch.load(fetch)
        parts = [branch for branch, _ in self.branches]
        for branch in parts:
            # every branch's columns of the input product start on a 16-byte boundary
            short = -branch.input_weight.shape[0] % 8
            if short:
                branch.input_weight = torch.nn.functional.pad(branch.input_weight, (0, 0, 0, short))
        self.input_rows = [branch.input_weight.shape[0] for branch in parts]
        self.output_columns = [branch.output_weight.shape[1] for branch in parts]
        self.input_weight = torch.cat([branch.input_weight for branch in parts])
        self.output_weight = torch.cat([branch.output_weight for branch in parts], dim=1).contiguous()
        for branch in parts:                       # held once, in the stacked matrices
            branch.input_weight = branch.output_weight = None

    def forward(self, h, residual, ctx, binding):
        rt = self.runtime
        proj = linear(h, self.input_weight, None, EPILOGUE_F32, backend=rt.gemm_backend)
        mixed = torch.empty((h.shape[0], self.output_weight.shape[1]), dtype=rt.dtype, device=h.device)
        row = column = 0
        for (branch, scale), rows, columns in zip(self.branches, self.input_rows, self.output_columns):
            branch.mix(proj[:, row:row + rows], ctx, binding, mixed[:, column:column + columns], scale)
            row, column = row + rows, column + columns
        if residual is None:
            return linear(mixed, self.output_weight, None, EPILOGUE_F32, backend=rt.gemm_backend)
        return linear(mixed, self.output_weight, None, EPILOGUE_RESIDUAL, residual=residual, out=residual,
                      backend=rt.gemm_backend, defer_sum=getattr(ctx, "sums_may_pend", False))
