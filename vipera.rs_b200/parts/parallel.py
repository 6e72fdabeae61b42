"""Mixers side by side: every branch reads the same input, and the layer's mixer output is the
sum of the branches' outputs, each times a constant.

A branch is any registered mixer that takes ``out_scale`` among its parameters (it multiplies
its own output, so the sum forms where the branches add into the stream they are handed).  The
tensors of branch ``name`` live under ``<prefix>.<name>``; what the branches keep between steps
is bundled under their names.

With ``out_norm_eps`` each branch's output is divided by its root mean square over the stream's width
and multiplied by a weight per channel (``<prefix>.<name>.<out_norm_name>.weight``) before the constant
and the sum.  The branches then leave rows, and the mixer leaves branches for the stream's next reader,
which norms them as it adds them (``leaves_branches``).
"""
from __future__ import annotations

import torch

from ..config.registry import MIXERS
from ..config.spec import PartSpec
from ..errors import InvalidArgumentError, UnsupportedError
from ..kernels import ops
from ..weights import TensorSpec
from .base import CacheBundle, Mixer


class ParallelMixers(Mixer):
    """params: ``branches``, a sequence of (name, PartSpec of a mixer, scale); optionally ``out_norm_eps``
    with ``hidden_size`` and ``out_norm_name`` (default ``out``).  With norms there are at most two branches, of
    mixers that leave rows."""

    @staticmethod
    def _branches(params):
        for name, part, scale in params["branches"]:
            if params.get("out_norm_eps") is not None:
                # a constant in front of the norm would cancel: it multiplies the norm's weight
                yield name, MIXERS.find(part.kind), {**part.params, "rows_name": f"parallel.{name}"}
                continue
            yield name, MIXERS.find(part.kind), {**part.params, "out_scale": float(scale) * float(part.params.get("out_scale", 1.0))}

    @classmethod
    def schema(cls, params, prefix):
        schema = {}
        for name, kind, branch_params in cls._branches(params):
            schema.update(kind.schema(branch_params, f"{prefix}.{name}"))
            if params.get("out_norm_eps") is not None:
                schema[cls._norm_tensor(params, prefix, name)] = TensorSpec((int(params["hidden_size"]),), init="norm", store="float32")
        return schema

    @staticmethod
    def _norm_tensor(params, prefix, name):
        return f"{prefix}.{name}.{params.get('out_norm_name', 'out')}.weight"

    def __init__(self, params, prefix, tensors, dtype, device):
        super().__init__(params, prefix, tensors, dtype, device)
        self.branches = [(name, kind(branch_params, f"{prefix}.{name}", tensors, dtype, device))
                         for name, kind, branch_params in self._branches(params)]
        self.out_norm_eps = params.get("out_norm_eps")
        self.leaves_branches = self.out_norm_eps is not None
        if self.leaves_branches:
            if len(self.branches) > 2 or not all(getattr(branch, "leaves_rows", False) for _, branch in self.branches):
                raise UnsupportedError(f"{prefix}: norms behind mixers side by side take two mixers at most, which leave rows")
            if len({name for name, _ in self.branches}) != len(self.branches):
                raise InvalidArgumentError(f"{prefix}: two branches of one name")
            self.scales = [(tensors[self._norm_tensor(params, prefix, name)].to(device=device, dtype=torch.float32)
                            * float(scale)).contiguous() for name, _, scale in params["branches"]]
        self.graph_safe = all(getattr(branch, "graph_safe", True) for _, branch in self.branches)

    def kernel_families(self):
        names = ()
        for _, branch in self.branches:
            names += tuple(branch.kernel_families())
        if self.leaves_branches:
            names += ("rowwise",)
        return tuple(dict.fromkeys(names))

    def prepare(self, max_positions: int) -> None:
        for _, branch in self.branches:
            prepare = getattr(branch, "prepare", None)
            if prepare is not None:
                prepare(max_positions)

    @classmethod
    def cache_request_for(cls, params):
        return CacheBundle.of(**{name: kind.cache_request_for(branch_params)
                                 for name, kind, branch_params in cls._branches(params)})

    @classmethod
    def workspace_bytes(cls, params, tokens, element_bytes):
        return sum(kind.workspace_bytes(branch_params, tokens, element_bytes)
                   for _, kind, branch_params in cls._branches(params))

    def forward(self, ctx, h, residual, cache, writes_cache):
        cache = cache or {}
        if not self.leaves_branches:
            for name, branch in self.branches:
                branch.forward(ctx, h, residual, cache.get(name), writes_cache)
            return None
        branches = []
        for (name, branch), scale in zip(self.branches, self.scales):
            rows, parts = branch.forward(ctx, h, None, cache.get(name), writes_cache)
            branches.append((rows, parts, scale, float(self.out_norm_eps)))
        if residual is None:
            return branches
        ops.join_norms(residual, branches)
        return None


MIXERS.register("parallel", ParallelMixers)
