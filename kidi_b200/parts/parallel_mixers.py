"""Two mixers side by side as one mixer: both read the same input and the mixer's result is a weighted sum of the two.

`combine` = "normed" (the default): each result is first divided by its root mean square over the model width and
multiplied by a weight of its own,

    y = share_left * left(h) / rms(left(h)) * w_left + share_right * right(h) / rms(right(h)) * w_right

with norms and sum in 32-bit and the result handed on in 32-bit. `combine` = "plain": y = share_left * left(h) +
share_right * right(h). Both children then run on projections that this part holds: one product makes the input
projections of both, each child works on its columns of the result and leaves what would enter its output projection,
times its share (32-bit, before it is rounded), in its columns of one matrix, and one product with the two output
projections side by side forms the sum in its 32-bit accumulators. Such a child has `joint_input()`, `joint_output()`,
`out_width`, `activated_columns`, `release_projections()` and `mix(projected, ctx, views, owns_cache, out)`, and takes
the parameter `out_scale`.

Each child keeps what it needs of the cache; the requests of the left child come first.

Parameters (`spec.params`): hidden_size, eps, left and right (the `PartSpec`s of two mixers), combine, left_norm_name and
right_norm_name (the norm weights' tensor names under this part's prefix), share_left and share_right (default 0.5).
"""
from __future__ import annotations

import dataclasses
from typing import List, Optional

import torch

from ..errors import invalid_argument, unsupported
from ..kernels import ops
from . import registry as part_registry
from .base import Part, plain_rows
from .linear import Linear
from .registry import register_part
from .spec import ParamSpec, PartSpec


def with_param(spec: PartSpec, **params) -> PartSpec:
    return dataclasses.replace(spec, params={**spec.params, **params})


@register_part("mixer", "parallel_mixers")
class ParallelMixers(Part):
    def __init__(self, spec, env):
        super().__init__(spec, env)
        self.hidden = int(spec.param("hidden_size"))
        self.share_left = float(spec.param("share_left", 0.5))
        self.share_right = float(spec.param("share_right", 0.5))
        if spec.param("combine", "normed") not in ("normed", "plain"):
            raise invalid_argument("parallel mixers combine their results 'normed' or 'plain'")
        self.normed = spec.param("combine", "normed") == "normed"
        self.eps = float(spec.param("eps")) if self.normed else 0.0
        left, right = spec.param("left"), spec.param("right")
        if not self.normed:
            left, right = with_param(left, out_scale=self.share_left), with_param(right, out_scale=self.share_right)
        self.left = part_registry.build_part("mixer", left, env)
        self.right = part_registry.build_part("mixer", right, env)
        self.left_norm_name = spec.param("left_norm_name", "left.out")
        self.right_norm_name = spec.param("right_norm_name", "right.out")
        if self.hidden <= 0:
            raise invalid_argument("invalid width of parallel mixers")
        if not self.normed and not all(hasattr(child, "joint_input") for child in (self.left, self.right)):
            raise unsupported("mixers whose results are added as they are must be able to share their projections")
        self._split = len(self.left.cache_requests())
        self.left_norm = self.right_norm = None
        self.projection: Optional[Linear] = None
        self.out: Optional[Linear] = None

    def children(self):
        return (self.left, self.right)

    def parameter_specs(self) -> List[ParamSpec]:
        if not self.normed:
            return []
        return [ParamSpec(self.left_norm_name, (self.hidden,), init=("one_plus_normal", 0.1)),
                ParamSpec(self.right_norm_name, (self.hidden,), init=("one_plus_normal", 0.1))]

    def bind(self, tensors) -> None:
        self.left_norm = tensors[self.left_norm_name].float().contiguous()
        self.right_norm = tensors[self.right_norm_name].float().contiguous()

    def bound(self) -> None:
        if self.normed:
            return

        def joined(matrices, dim):
            if matrices[0].dtype != matrices[1].dtype:
                matrices = [matrix.float() for matrix in matrices]
            return torch.cat(matrices, dim=dim).contiguous()

        inputs = [self.left.joint_input(), self.right.joint_input()]
        self._left_columns = inputs[0].shape[0]
        outputs = [self.left.joint_output(), self.right.joint_output()]
        # the columns of what enters the output projection: left, right, zeros up to a multiple of 8
        self._out_used = self.left.out_width + self.right.out_width
        padding = -self._out_used % 8
        if padding:
            outputs[1] = torch.cat([outputs[1], torch.zeros((self.hidden, padding), dtype=outputs[1].dtype,
                                                            device=outputs[1].device)], dim=1)
        self.projection, self.out = Linear(joined(inputs, 0)), Linear(joined(outputs, 1))
        # SiLU columns of the joint projection: one range, of the child that has one
        self._activated = None
        for child, begin in ((self.left, 0), (self.right, self._left_columns)):
            if child.activated_columns is not None:
                if self._activated is not None:
                    raise unsupported("two mixers with activated columns do not share their projections")
                self._activated = (begin + child.activated_columns[0], begin + child.activated_columns[1])
        self.left.release_projections()
        self.right.release_projections()

    def cache_requests(self) -> list:
        return list(self.left.cache_requests()) + list(self.right.cache_requests())

    def forward(self, x, ctx, views, owns_cache: bool, sink=None) -> Optional[torch.Tensor]:
        x = plain_rows(x)
        left_views, right_views = views[:self._split], views[self._split:]
        if self.normed:
            left = self.left.forward(x, ctx, left_views, owns_cache)
            right = self.right.forward(x, ctx, right_views, owns_cache)
            return ops.normed_pair_sum(left, right, self.left_norm, self.right_norm, self.eps, self.share_left,
                                       self.share_right, out_dtype=torch.float32)
        projected = self.projection.forward(x, silu_columns=self._activated)
        make = torch.empty if self.out.in_features == self._out_used else torch.zeros
        mixed = make((x.shape[0], self.out.in_features), dtype=projected.dtype, device=projected.device)
        middle = self.left.out_width
        joined = ctx.beside(lambda: self.right.mix(projected[:, self._left_columns:], ctx, right_views, owns_cache,
                                                   out=mixed[:, middle:self._out_used]))
        self.left.mix(projected[:, :self._left_columns], ctx, left_views, owns_cache, out=mixed[:, :middle])
        joined()
        return self.out.forward(mixed)
