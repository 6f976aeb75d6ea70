"""Linear attention with one fixed decay per head ("lightning attention") as a mixer.

With h the mixer's input, H heads, d the width of a query or key head and e the width of a value head:

    q = silu(W_q h),  k = silu(W_k h)  [H, d],    v = silu(W_v h)  [H, e]
    S_t = decay_h S_(t-1) + k_t v_t^T,            o_t = S_t^T q_t           (nothing else is scaled)
    y = W_o (o / rms(o) * w * sigmoid(W_g h))     the root mean square over all heads' entries together, w [H e]

What a sequence keeps is S, [H, d, e], in 32-bit floats, as fixed-size state per cache slot that starts at zero. State,
decay, read-out and norm are 32-bit.

Variants, all parameters: activation ("silu", the default, or None: q, k and v as projected); position (name of a rotary
encoding in `env.positions`: q and k are rotated) and key_scale (k is multiplied by it, after the rotation; default 1), both
in 32-bit on the way into the recurrence; norm_scope "head" with norm_weight false (each head is divided by its own root mean
square and there is no weight: the tensor `norm` is absent) and gate_activation "silu": "retention",

    y = W_o (o_h / rms(o_h) * silu(W_g h))

Parameters (`spec.params`): hidden_size, num_heads, dim, vdim, decay (one number per head), eps, out_scale (a factor on
what enters W_o, default 1), and the tensor names under the prefix: q, k, v, g, o, norm. The part can also run on
projections that another part holds (`joint_input`, `mix`, `joint_output`; see `parallel_mixers`).
"""
from __future__ import annotations

from typing import List, Optional

import torch

from ..cache.sequence_cache import StateRequest
from ..errors import invalid_argument, unsupported
from ..kernels import linear_attention as kernels
from .base import Part, plain_rows
from .linear import Linear
from .registry import register_part
from .spec import ParamSpec

NAMES = {"q": "q", "k": "k", "v": "v", "g": "g", "o": "o", "norm": "norm"}


@register_part("mixer", "lightning_attention")
class LightningAttention(Part):
    accepts_row_scaled = True     # x may lack its norm's factor: the projection applies it (without an activation)
    takes_sink = True             # the output product may add its result to the residual stream itself

    def __init__(self, spec, env):
        super().__init__(spec, env)
        self.hidden = int(spec.param("hidden_size"))
        self.heads = int(spec.param("num_heads"))
        self.dim = int(spec.param("dim"))
        self.vdim = int(spec.param("vdim"))
        self.eps = float(spec.param("eps"))
        self.out_scale = float(spec.param("out_scale", 1.0))
        decay = [float(value) for value in spec.param("decay")]
        if min(self.hidden, self.heads, self.dim, self.vdim) <= 0:
            raise invalid_argument("invalid linear-attention dimensions")
        if len(decay) != self.heads:
            raise invalid_argument("linear attention needs one decay per head")
        if self.dim > kernels.MAX_DIM:
            raise unsupported(f"a state of {self.dim} rows a head exceeds {kernels.MAX_DIM}, the most the kernel takes")
        self.decay = torch.tensor(decay, dtype=torch.float32, device=env.device)
        self.qk_width, self.out_width = self.heads * self.dim, self.heads * self.vdim
        self.width = 2 * self.qk_width + 2 * self.out_width                     # [q | k | v | g]
        activation = spec.param("activation", "silu")
        if activation not in ("silu", None):
            raise unsupported(f"linear attention activation '{activation}' is not built (silu is)")
        self.activated_columns = (0, 2 * self.qk_width + self.out_width) if activation else None        # what passes SiLU
        name = spec.param("position", None)
        self.position = env.positions[name] if name is not None else None
        if self.position is not None and self.position.head_dim != self.dim:
            raise invalid_argument("the rotary encoding was built for another head width")
        self.key_scale = float(spec.param("key_scale", 1.0))
        self.by_head = spec.param("norm_scope", "row") == "head"
        self.norm_weight = bool(spec.param("norm_weight", True))
        self.gate_silu = spec.param("gate_activation", "sigmoid") == "silu"
        if spec.param("norm_scope", "row") not in ("row", "head") or spec.param("gate_activation", "sigmoid") not in ("sigmoid", "silu"):
            raise invalid_argument("linear attention norms rows or heads and gates by a sigmoid or SiLU")
        if self.by_head == self.norm_weight:
            raise unsupported("linear attention with a norm per head has no weight, with a norm per row it has one")
        if not self.by_head and (self.position is not None or self.key_scale != 1.0 or self.gate_silu):
            raise unsupported("linear attention with rotated or scaled keys or a SiLU gate has a norm per head")
        if self.by_head and self.out_scale != 1.0:
            raise unsupported("linear attention with a norm per head has no factor on its result")
        self.names = {key: spec.param(key + "_name", default) for key, default in NAMES.items()}
        self.projection: Optional[Linear] = None
        self.out: Optional[Linear] = None
        self.norm: Optional[torch.Tensor] = None

    def parameter_specs(self) -> List[ParamSpec]:
        n, hidden = self.names, self.hidden
        return [
            ParamSpec("qkvg", (self.width, hidden), sources=(
                (n["q"], (self.qk_width, hidden)), (n["k"], (self.qk_width, hidden)), (n["v"], (self.out_width, hidden)),
                (n["g"], (self.out_width, hidden)))),
            *([ParamSpec(n["norm"], (self.out_width,), init=("one_plus_normal", 0.1))] if self.norm_weight else []),
            ParamSpec(n["o"], (hidden, self.out_width)),
        ]

    def bind(self, tensors) -> None:
        fused = tensors["qkvg"]
        if self.width % 8:                 # rows of the product's result start on 16-byte boundaries
            pad = torch.zeros((-self.width % 8, self.hidden), dtype=fused.dtype, device=fused.device)
            fused = torch.cat([fused, pad], dim=0).contiguous()
        self.projection, self.out = Linear(fused), Linear(tensors[self.names["o"]])
        if self.norm_weight:
            self.norm = tensors[self.names["norm"]].float().contiguous()

    def cache_requests(self) -> list:
        return [StateRequest((self.heads, self.dim, self.vdim), torch.float32)]

    # --- projections that another part holds
    def joint_input(self) -> torch.Tensor:
        """The fused input projection [rows, hidden], rows a multiple of 8."""
        return self.projection.weight

    def joint_output(self) -> torch.Tensor:
        """The output projection [hidden, out_width]."""
        return self.out.weight

    def release_projections(self) -> None:
        self.projection = self.out = None

    def forward(self, x, ctx, views, owns_cache: bool, sink=None) -> Optional[torch.Tensor]:
        if self.activated_columns is not None:
            projected = self.projection.forward(plain_rows(x), silu_columns=self.activated_columns)
        else:
            projected = self.projection.forward(x)
        return self.out.forward(self.mix(projected, ctx, views, owns_cache), sink=sink)

    def mix(self, projected: torch.Tensor, ctx, views, owns_cache: bool, out: Optional[torch.Tensor] = None) -> torch.Tensor:
        """What enters the output projection, [rows, out_width] (into `out`, if given), from the projected rows, whose
        q, k and v columns have passed their activation."""
        if not owns_cache:
            raise invalid_argument("a linear-attention layer keeps a state of its own")
        qk, v = self.qk_width, self.out_width
        if self.by_head:
            if out is None:
                out = torch.empty((projected.shape[0], v), dtype=projected.dtype, device=projected.device)
            turn = self.position
            return kernels.retention(
                projected[:, :qk], projected[:, qk:2 * qk], projected[:, 2 * qk:2 * qk + v],
                projected[:, 2 * qk + v:2 * qk + 2 * v], self.decay, views[0], out, heads=self.heads, dim=self.dim,
                vdim=self.vdim, tables=ctx.tables, seqs=ctx.plan.n_seqs, one_token=ctx.plan.is_decode,
                longest=ctx.plan.max_new, cos=turn.cos if turn is not None else None,
                sin=turn.sin if turn is not None else None, rotary_dim=turn.rotary_dim if turn is not None else 0,
                key_scale=self.key_scale, eps=self.eps, silu=self.gate_silu)
        read = kernels.linear_attention(projected[:, :qk], projected[:, qk:2 * qk], projected[:, 2 * qk:2 * qk + v],
                                        self.decay, views[0], heads=self.heads, dim=self.dim, vdim=self.vdim,
                                        tables=ctx.tables, seqs=ctx.plan.n_seqs, one_token=ctx.plan.is_decode,
                                        longest=ctx.plan.max_new)
        if out is None:
            out = torch.empty((projected.shape[0], v), dtype=projected.dtype, device=projected.device)
        return kernels.normed_gate(read, self.norm, projected[:, 2 * qk + v:2 * qk + 2 * v], self.eps, self.out_scale, out)
