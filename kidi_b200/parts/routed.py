"""A feed-forward of many small gated experts, of which each token uses a few.

    z = W_router h                       router logits, 32-bit
    s = sigmoid(z)                       scores; the `top` experts with the largest scores are taken
    w = s of the chosen experts          (divided by their sum when `renormalise` is set)
    y = sum over the chosen experts of expert_e(w_e h)           `weight_on` = "input"
      or sum of w_e expert_e(h)                                   `weight_on` = "output"
    expert(x) = W_down (silu(W_gate x) * (W_up x))

Parameters (`spec.params`): hidden_size, expert_size, experts, top, score ("sigmoid"), renormalise (false),
weight_on ("input"), router_name ("router"), expert_name ("e{index}."), gate_name, up_name, down_name. A file
holds each expert's three matrices under `<prefix><expert_name><gate|up|down>`; they are bound as two stacked
tensors, [experts, 2 * expert_size, hidden] (gate rows, then up rows) and [experts, hidden, expert_size].

Variants, all parameters: router_bias_name (a tensor [experts] added to the logits; a softmax score that is
renormalised with renormalise_eps 0 is then the softmax over the chosen logits alone, bias included); score "softmax" (s = softmax(z) over all experts); renormalise_eps (added to the sum
that the chosen scores are divided by); groups and keep_groups: the experts form `groups` equal runs of
neighbours, a group's score is its largest, and only experts of the `keep_groups` best groups can be chosen;
expert_form "plain": an expert has no gate, expert(x) = W_down gelu(W_up x) with the exact (erf) gelu, and the
first stacked tensor is [experts, expert_size, hidden]; shared_size and shared_name ("shared."): one more expert
of the same form and that width, under `<prefix><shared_name><gate|up|down>`, that every token passes and whose
result is added with weight 1.

And: correction_name (a tensor [experts] that is added to the scores where experts and groups are chosen, and not to the
weights); group_score "largest" (the default) or "two_largest" (a group's score is the sum of its two largest);
weight_scale (the weights are multiplied by it, after the renormalisation; default 1); activation "silu" (the default) or
"bounded_swish" (a gated expert's form in `gated_mlp`, with limit, alpha and up_shift, and shared_limit for the shared
expert); shared_gate_name (a tensor [1, hidden] under the shared expert's prefix: its result is multiplied by
sigmoid(W_sg h), one number a token, computed beside the router's logits in 32-bit).

Steps of few rows, steps inside a captured decode graph, and every step of the 32-bit engine read the
chosen experts' weights through the choice on the device. Prompts of the bfloat16 engine group the (row,
choice) pairs by expert on the device, gather the rows and run them through two products over groups of this
package's tcgen05 kernel (a gated expert's SiLU gate in the first one's epilogue): no host round trip either.
Where the widths are no multiples of 8, or the experts so many that the groups' padding would more than
triple the rows, the pairs are sorted by expert on the host instead; every expert's rows, up to twice the mean count,
are then padded to one count and run through two batched products of the vendor library, and what an expert has
beyond that (or everything, for odd widths) through the ordinary products, with one activation kernel for all of them.
"""
from __future__ import annotations

import os
from typing import List, Optional

import numpy as np
import torch

from ..errors import invalid_argument, unsupported
from ..kernels import ops, routed, skinny, tcgen05
from .base import Part, plain_rows
from .linear import Linear
from .registry import register_part
from .spec import ParamSpec

# Up to this many (row, choice) pairs a step reads the experts through the choice; above, a bfloat16 prompt
# sorts them by expert.
SLOT_PATH_MAX = 128
# Prompts group the pairs on the device and take the products over groups (0: sorted on the host, batched products).
GROUPED = os.environ.get("KIDI_B200_GROUPED_EXPERTS", "1") == "1"


@register_part("feed_forward", "routed_experts")
class RoutedExperts(Part):
    def __init__(self, spec, env):
        super().__init__(spec, env)
        self.hidden = int(spec.param("hidden_size"))
        self.inter = int(spec.param("expert_size"))
        self.experts = int(spec.param("experts"))
        self.top = int(spec.param("top"))
        self.renormalise = bool(spec.param("renormalise", False))
        self.weight_on_input = spec.param("weight_on", "input") == "input"
        if spec.param("weight_on", "input") not in ("input", "output"):
            raise invalid_argument("routed experts weigh an expert's input or its output")
        self.score = spec.param("score", "sigmoid")
        if self.score not in ("sigmoid", "softmax"):
            raise unsupported(f"router score '{self.score}' is not built (sigmoid and softmax are)")
        self.renormalise_eps = float(spec.param("renormalise_eps", 0.0))
        self.groups = int(spec.param("groups", 1))
        self.keep_groups = int(spec.param("keep_groups", self.groups))
        self.gated = spec.param("expert_form", "gated") == "gated"
        if spec.param("expert_form", "gated") not in ("gated", "plain"):
            raise invalid_argument("an expert is 'gated' (SiLU gate times up) or 'plain' (gelu of up)")
        shared = spec.param("shared_size", None)
        self.shared_size = int(shared) if shared is not None else None
        self.shared_name = spec.param("shared_name", "shared.")
        self.correction_name = spec.param("correction_name", None)
        self.correction: Optional[torch.Tensor] = None
        self.two_largest = spec.param("group_score", "largest") == "two_largest"
        if spec.param("group_score", "largest") not in ("largest", "two_largest"):
            raise invalid_argument("a group of experts is ranked by its largest score or the sum of its two largest")
        self.weight_scale = float(spec.param("weight_scale", 1.0))
        self.shared_gate_name = spec.param("shared_gate_name", None) if self.shared_size is not None else None
        self.shared_gate: Optional[torch.Tensor] = None
        activation = spec.param("activation", "silu")
        if activation not in ("silu", "bounded_swish") or (activation != "silu" and not self.gated):
            raise unsupported(f"expert activation '{activation}' is not built (gated experts: silu and bounded_swish)")
        self.shape = self.shared_shape = None
        if activation == "bounded_swish":
            limits = [float(spec.param("limit"))] + ([float(spec.param("shared_limit", spec.param("limit")))]
                                                     if self.shared_size is not None else [])
            if not all(limit > 0 for limit in limits):
                raise invalid_argument("the bound of a bounded gate must be positive")
            shapes = [ops.GateShape(1, limit, float(spec.param("alpha", 1.702)), float(spec.param("up_shift", 1.0)))
                      for limit in limits]
            self.shape, self.shared_shape = shapes[0], shapes[-1]
        if min(self.hidden, self.inter, self.experts, self.top) <= 0 or self.top > self.experts:
            raise invalid_argument("invalid routed feed-forward dimensions")
        if self.experts > 1024 or self.top > 32:
            raise unsupported("the router takes up to 1,024 experts and 32 choices a token")
        if self.groups < 1 or self.experts % self.groups or not 1 <= self.keep_groups <= self.groups \
                or self.keep_groups * (self.experts // self.groups) < self.top:
            raise invalid_argument("the experts split into equal groups, and the kept groups hold at least `top` experts")
        if self.shared_size is not None and self.shared_size <= 0:
            raise invalid_argument("a shared expert has a positive width")
        self.router_name = spec.param("router_name", "router")
        self.router_bias_name = spec.param("router_bias_name", None)
        self.router_bias: Optional[torch.Tensor] = None
        self.expert_name = spec.param("expert_name", "e{index}.")
        self.gate_name, self.up_name, self.down_name = (spec.param(key + "_name", key) for key in ("gate", "up", "down"))
        self.router: Optional[torch.Tensor] = None
        self.gate_up: Optional[torch.Tensor] = None
        self.down: Optional[torch.Tensor] = None

    def parameter_specs(self) -> List[ParamSpec]:
        names = [self.expert_name.format(index=index) for index in range(self.experts)]
        first, down = [], []
        for name in names:
            if self.gated:
                first.append((name + self.gate_name, (self.inter, self.hidden)))
            first.append((name + self.up_name, (self.inter, self.hidden)))
            down.append((name + self.down_name, (self.hidden, self.inter)))
        per = (2 if self.gated else 1) * self.inter
        specs = [ParamSpec(self.router_name, (self.experts, self.hidden)),
                 *([ParamSpec(self.router_bias_name, (self.experts,), init=("normal", 0.1))]
                   if self.router_bias_name is not None else []),
                 *([ParamSpec(self.correction_name, (self.experts,), init=("normal", 0.1))]
                   if self.correction_name is not None else []),
                 ParamSpec("experts.gate_up", (self.experts * per, self.hidden), sources=tuple(first)),
                 ParamSpec("experts.down", (self.experts * self.hidden, self.inter), sources=tuple(down))]
        if self.shared_size is not None:
            name = self.shared_name
            if self.gated:
                specs.append(ParamSpec(name + "gate_up", (2 * self.shared_size, self.hidden), sources=(
                    (name + self.gate_name, (self.shared_size, self.hidden)),
                    (name + self.up_name, (self.shared_size, self.hidden)))))
            else:
                specs.append(ParamSpec(name + self.up_name, (self.shared_size, self.hidden)))
            specs.append(ParamSpec(name + self.down_name, (self.hidden, self.shared_size)))
            if self.shared_gate_name is not None:
                specs.append(ParamSpec(name + self.shared_gate_name, (1, self.hidden)))
        return specs

    def bind(self, tensors) -> None:
        per = (2 if self.gated else 1) * self.inter
        self.router = tensors[self.router_name]
        if self.router_bias_name is not None:
            self.router_bias = tensors[self.router_bias_name].float().contiguous()
        if self.correction_name is not None:
            self.correction = tensors[self.correction_name].float().contiguous()
        if self.shared_gate_name is not None:       # (the row joins the router's product: in the router's type)
            row = tensors[self.shared_name + self.shared_gate_name]
            if row.dtype != self.router.dtype:
                row, self.router = row.float(), self.router.float()
            self.shared_gate = row.contiguous()
        self.gate_up = tensors["experts.gate_up"].view(self.experts, per, self.hidden)
        self.down = tensors["experts.down"].view(self.experts, self.hidden, self.inter)
        self._gate_up = [Linear(self.gate_up[index]) for index in range(self.experts)]
        self._down = [Linear(self.down[index]) for index in range(self.experts)]
        self._shared = None
        if self.shared_size is not None:
            name = self.shared_name
            self._shared = (Linear(tensors[name + ("gate_up" if self.gated else self.up_name)]),
                            Linear(tensors[name + self.down_name]))

    def _activate(self, first: torch.Tensor, shape=None) -> torch.Tensor:
        """The experts' activation on the first product's result (in place where it can be)."""
        if shape is not None:
            return ops.bounded_gate(first, shape.limit, shape.alpha, shape.shift)
        return ops.silu_gate(first) if self.gated else ops.gelu(first, out=first)

    def forward(self, x, ctx) -> torch.Tensor:
        x = plain_rows(x)
        # The shared expert runs beside the routed ones; its result joins their sum in the kernel that forms it (32-bit).
        beside = getattr(ctx, "beside", None)
        shared = lambda: None
        if self._shared is not None:
            shared = beside(lambda: self._forward_shared(x)) if beside is not None else lambda: self._forward_shared(x)
        return self._forward_routed(x, ctx, shared)

    def _forward_shared(self, x) -> torch.Tensor:
        up, down = self._shared
        if skinny.fits(x, up.weight) and up.bias is None:            # few rows: the activation in the epilogue
            mid = skinny.gemm_silu_gate(x, up.weight, shape=self.shared_shape) if self.gated else skinny.gemm(x, up.weight, x.dtype, activation="gelu")
        else:
            mid = self._activate(up.forward(x), self.shared_shape)
        return down.forward(mid)

    def _forward_routed(self, x, ctx, shared=lambda: None) -> torch.Tensor:
        """`shared()`: the shared expert's result (or None), asked for where the routed sum is formed."""
        rows = x.shape[0]
        share = torch.empty(rows, dtype=torch.float32, device=x.device) if self.shared_gate is not None else None
        chosen, weight = routed.route(x, self.router, self.top, self.renormalise, self.score, self.groups,
                                      self.keep_groups, self.renormalise_eps, self.router_bias, correction=self.correction,
                                      two_largest=self.two_largest, weight_scale=self.weight_scale,
                                      share_row=self.shared_gate, share=share)
        slots = rows * self.top
        if x.dtype == torch.float32 or self.gate_up.dtype == torch.float32 or ctx.plan.is_decode \
                or slots <= SLOT_PATH_MAX:
            return routed.expert_slots(x, self.gate_up, self.down, chosen, weight, self.weight_on_input, self.gated, shared,
                                       shape=self.shape, share=share)
        if GROUPED and self.hidden % 8 == 0 and self.inter % 8 == 0 \
                and 0 < routed.group_rows(slots, self.experts) <= 4 * slots:
            source, place, tiles = routed.group_slots(chosen, self.experts)
            gathered = routed.gather_slots(x, source, weight, self.top, self.weight_on_input)
            mid = tcgen05.gemm_grouped(gathered, self.gate_up, tiles, self.gated, shape=self.shape)
            if not self.gated:
                mid = self._activate(mid)
            result = tcgen05.gemm_grouped(mid, self.down, tiles, False)
            return routed.combine_slots(result, place, weight, rows, self.top, self.weight_on_input, shared(), share)
        # Many rows: (row, choice) pairs in the order of their experts (a stable sort, so a row's place among
        # its expert's rows follows its place in the step), one host round trip for the counts.
        picked = chosen.reshape(-1).cpu().numpy()
        ops.host_waited()
        order = np.argsort(picked, kind="stable").astype(np.int32)
        counts = np.bincount(picked, minlength=self.experts)
        # Every expert's first `cap` rows stand in one padded batch [experts, cap] (two batched products of the
        # vendor library for all experts); the rows that an expert has beyond `cap` follow the batch, expert by
        # expert, and run through the ordinary products. `cap` is the largest count, but at most twice the mean, so
        # that the padding stays below the rows themselves however uneven the choice is. Widths that are no
        # multiples of 8 take the ordinary products only (cap 0).
        cap = 0
        if self.hidden % 8 == 0 and self.inter % 8 == 0:
            cap = int(-(-min(int(counts.max()), -(-2 * slots // self.experts)) // 8) * 8)
        begins = np.concatenate([[0], np.cumsum(counts)[:-1]])
        experts_sorted = picked[order]
        within = np.arange(slots) - begins[experts_sorted]
        over = within >= cap
        extra = np.maximum(counts - cap, 0)
        extra_begins = self.experts * cap + np.concatenate([[0], np.cumsum(extra)[:-1]])
        at = np.where(over, extra_begins[experts_sorted] + within - cap, experts_sorted * cap + within).astype(np.int32)
        total = self.experts * cap + int(extra.sum())
        source = np.full(total, -1, dtype=np.int32)
        source[at] = order
        place = np.empty(slots, dtype=np.int32)
        place[order] = at
        tables = torch.from_numpy(np.concatenate([source, place])).to(x.device)
        gathered = routed.gather_slots(x, tables[:total], weight, self.top, self.weight_on_input)
        first = torch.empty((total, self.gate_up.shape[1]), dtype=x.dtype, device=x.device)
        result = torch.empty((total, self.hidden), dtype=x.dtype, device=x.device)
        batch = self.experts * cap
        spans = [(index, int(begin), int(begin + count)) for index, (begin, count) in enumerate(zip(extra_begins, extra))
                 if count]
        if cap:
            torch.bmm(gathered[:batch].view(self.experts, cap, self.hidden), self.gate_up.transpose(1, 2),
                      out=first[:batch].view(self.experts, cap, first.shape[1]))
            ops.note("library_bmm")
        for index, begin, end in spans:
            self._gate_up[index].forward(gathered[begin:end], out=first[begin:end])
        mid = self._activate(first, self.shape)      # one activation kernel for the rows of all experts
        if cap:
            torch.bmm(mid[:batch].view(self.experts, cap, self.inter), self.down.transpose(1, 2),
                      out=result[:batch].view(self.experts, cap, self.hidden))
            ops.note("library_bmm")
        for index, begin, end in spans:
            self._down[index].forward(mid[begin:end], out=result[begin:end])
        return routed.combine_slots(result, tables[total:], weight, rows, self.top, self.weight_on_input, shared(), share)
