"""What every part is: a thing built from a `PartSpec` that declares its tensors,
receives them, and runs on the rows of a step.

Interfaces by role (each is registered with `register_part(role, kind)`):

* norm:          `forward(stream) -> normed`     stream: ResidualStream; applies the pending residual add
* position:      built once per model under a name; mixers look it up in `env.positions`;
                 `on_embeddings(stream, ctx)` may change the embeddings (default: nothing)
* mixer:         `cache_requests() -> [KVRequest | StateRequest]`
                 `forward(x, ctx, views, owns_cache) -> y`   x, y: [rows, hidden] in the engine dtype
* feed_forward:  `forward(x, ctx) -> y`
                 (both optionally: class attribute `accepts_row_scaled = True`: x may be a `RowScaled`;
                 `takes_sink = True`: `forward(..., sink=ResidualSink)` may return None after adding y
                 to the residual stream itself)
                 (both of which another part may run on projections it holds itself: see `parallel_mixers`)
* arrangement:   `__init__(spec, env, parts)`; `forward(stream, ctx, views, owns_cache)`
* token_input:   `forward(stream, ctx, mix=None)`: adds something computed from the rows' token ids to the stream
                 (after taking the pending delta); `mix`, a stream_mix part, may be applied in the same kernel
* stream_mix:    `begin(stream, ctx)` before a layer, `forward(stream, ctx)` after it: replaces the stream by a
                 function of the copies of it that earlier layers left (`ResidualStream.kept`)
* shared:        built once per model under a name (`ModelSpec.shared`); parts look it up in `env.shared`
* embedding:     `forward(tokens, ctx) -> float32 [rows, hidden]`
* head:          `forward(x, ctx) -> float32 [rows, vocab]`

No part knows which model it is in: sizes and constants arrive in `spec.params`, tensor
names under `spec.prefix`.
"""
from __future__ import annotations

import dataclasses
from typing import Dict, List, Optional, Sequence, Tuple

import torch

from .spec import ParamSpec, PartSpec


@dataclasses.dataclass
class BuildEnv:
    """What parts are built against."""

    dtype: torch.dtype                 # element type of activations, cache and (bfloat16-stored) weights
    device: torch.device
    max_positions: int
    positions: Dict[str, object] = dataclasses.field(default_factory=dict)
    shared: Dict[str, object] = dataclasses.field(default_factory=dict)   # `ModelSpec.shared`, by name


class Part:
    role = "part"
    kind = "part"

    def __init__(self, spec: PartSpec, env: BuildEnv):
        self.spec = spec
        self.env = env
        self.prefix = spec.prefix

    # --- tensors
    def parameter_specs(self) -> List[ParamSpec]:
        """The tensors this part owns, named relative to its prefix."""
        return []

    def ignored_tensors(self) -> Sequence[str]:
        """Regular expressions, relative to the part's prefix, of tensors a checkpoint may
        carry for this part without the part using them (the reference's IGNORE mapping,
        src/kidi/checkpoint/weights.h:20-24)."""
        return ()

    def children(self) -> Sequence["Part"]:
        return ()

    def bind(self, tensors: Dict[str, torch.Tensor]) -> None:
        """Receives {relative name: tensor} for the tensors of `parameter_specs`."""
        for name, tensor in tensors.items():
            setattr(self, "_" + name.replace(".", "_"), tensor)

    def bound(self) -> None:
        """Called once the part and all its children have received their tensors."""

    # --- cache
    def cache_requests(self) -> list:
        return []

    # --- captured steps
    def launch_signature(self, rows: int, longest: int) -> tuple:
        """What a captured decode step of `rows` sequences of at most `longest` tokens would
        freeze of this part's launch choices (grid shapes that depend on the sequence length,
        say). Two steps with equal signatures can replay one captured graph. Default: the
        signatures of the part's children."""
        return tuple(child.launch_signature(rows, longest) for child in self.children())


def all_parameters(part: Part) -> List[Tuple[str, ParamSpec]]:
    """(prefix, spec) of the part and of its children, depth first."""
    found = [(part.prefix, spec) for spec in part.parameter_specs()]
    for child in part.children():
        found.extend(all_parameters(child))
    return found


def bind_all(part: Part, bound: Dict[str, torch.Tensor]) -> None:
    own = {spec.name: bound[part.prefix + spec.name] for spec in part.parameter_specs()}
    if own:
        part.bind(own)
    for child in part.children():
        bind_all(child, bound)
    part.bound()


class RowScaled:
    """Normalised rows kept in two pieces, so that no kernel of its own has to normalise them:
    `values` [rows, width] (bfloat16: the residual times the norm's weight, not yet divided by
    the row's root mean square) and `parts` [rows, count] (float32: parts of each row's sum of
    squares). Row r of the normalised matrix is values[r] / sqrt(sum(parts[r]) / width + eps).
    A product of such rows with a weight matrix applies the factor to its result
    (`Linear.forward`); `plain()` makes an ordinary matrix for any other consumer. Only parts
    that set `accepts_row_scaled` are ever handed one."""

    def __init__(self, values: torch.Tensor, parts: torch.Tensor, width: int, eps: float):
        self.values, self.parts, self.width, self.eps = values, parts, int(width), float(eps)

    @property
    def shape(self):
        return self.values.shape

    @property
    def dtype(self):
        return self.values.dtype

    @property
    def factors(self):
        return (self.parts, self.width, self.eps)

    def plain(self) -> torch.Tensor:
        from ..kernels import ops
        return ops.apply_row_factors(self.values, self.parts, self.width, self.eps)


def plain_rows(x) -> torch.Tensor:
    """x as an ordinary matrix, whatever it was handed as."""
    return x.plain() if isinstance(x, RowScaled) else x


class ResidualSink:
    """An offer to the product that ends a mixer or a feed-forward: instead of returning its
    result (which the arrangement would add to the residual stream, and the next norm would
    read again), it may add the result to the stream itself and leave the rows for `norm`
    prepared (`ResidualStream.prepared`). A product that cannot do so ignores the offer and
    returns its result as ever. `norm` is the part that reads the stream next and takes such
    rows (`norm.prepared_weight()` is its weight vector)."""

    def __init__(self, stream: "ResidualStream", norm: "Part"):
        self.stream, self.norm = stream, norm


class ResidualStream:
    """The residual stream of a step: `hidden` (float32 [rows, hidden size]) and a
    pending delta that the next norm adds while it normalises, so that the sum is
    formed in 32-bit and the rows are read once. A product that took a `ResidualSink` has
    added its result already and left `prepared` = (norm, values, parts) for that norm."""

    def __init__(self, hidden: torch.Tensor):
        self.hidden = hidden
        self.pending: Optional[torch.Tensor] = None
        self.pending_norm = None      # a norm (with `apply_delta()`) that the pending delta passes before it is added
        self.prepared = None
        # Copies of the stream that a part keeps for later layers (role "stream_mix"): [n, rows, hidden]
        # float32, and how many of them are filled. `hidden` is then a view of one of them.
        self.kept: Optional[torch.Tensor] = None
        self.kept_count = 0
        # A stream that layers keep as several lanes (float32 [count, rows, hidden]; see the `hyper_connections`
        # arrangement): once set, the lanes are the stream, `hidden` is no longer kept up to date, and a norm reads a
        # weighted sum of the lanes (their plain sum, for the norm before the head).
        self.lanes: Optional[torch.Tensor] = None
        # An update of the lanes that the next norm applies in its own kernel, as it applies a pending delta:
        # (mix [lanes, lanes], write [lanes], y [rows, hidden]): lane'_t = sum_s mix[s, t] lane_s + write[t] y.
        self.lane_update: Optional[tuple] = None

    def add(self, delta: Optional[torch.Tensor], normed_by=None) -> None:
        """`delta` None: the part that made it has added it through a sink already. `normed_by`: a norm part
        with `apply_delta()` (a layer norm without bias, an RMS norm) that the delta passes before it is added; what
        reads the stream next does both in its kernel when it can (`take_pending_normed`)."""
        if delta is None:
            return
        if self.pending is not None:
            raise RuntimeError("a residual delta is pending already; a norm must take it first")
        self.pending = delta
        self.pending_norm = normed_by
        self.prepared = None          # rows prepared before this delta are no longer the stream's

    def lane_target(self) -> torch.Tensor:
        """The lanes as memory that an update may write: while one matrix still stands for every lane (a view with a
        lane stride of 0), the lanes get memory of their own here and the view stays what the update reads."""
        if self.lanes.stride(0) == 0:
            return torch.empty(self.lanes.shape, dtype=torch.float32, device=self.lanes.device)
        return self.lanes

    def apply_lane_update(self) -> None:
        """Applies a waiting update of the lanes in a kernel of its own (for a reader that cannot do it itself)."""
        if self.lane_update is not None:
            from ..kernels import ops
            mix, write, y = self.lane_update
            target = self.lane_target()
            ops.lanes_mix(self.lanes, target, mix, write, y)
            self.lanes, self.lane_update = target, None

    def take_pending(self) -> Optional[torch.Tensor]:
        """The delta that the caller must add. A delta that still has to pass a norm of its own is normalised
        and added here (a kernel of its own), so a caller that knows nothing of such deltas gets None."""
        delta, norm = self.take_pending_normed()
        if norm is None:
            return delta
        norm.apply_delta(self.hidden, delta)
        return None

    def read(self, dtype: torch.dtype) -> torch.Tensor:
        """The stream itself, with its pending delta added, in `dtype` (for sublayers that read no norm of it)."""
        from ..kernels import ops
        self.prepared = None
        delta, norm = self.take_pending_normed()
        copy = dtype if dtype != torch.float32 else None
        if delta is not None and norm is not None:
            if hasattr(norm, "delta_parts"):
                weight, groups, eps = norm.delta_parts()
                made = ops.add_parts_norm(self.hidden, delta, copy, delta_weight=weight, delta_groups=groups, delta_eps=eps)
            else:
                norm.apply_delta(self.hidden, delta)
                made = ops.add_parts_norm(self.hidden, None, copy) if copy is not None else None
        else:
            made = ops.add_parts_norm(self.hidden, delta, copy) if delta is not None or copy is not None else None
        return self.hidden if copy is None else made

    def take_pending_normed(self):
        """(delta, norm): the pending delta and the norm it has to pass first (None: none)."""
        delta, norm = self.pending, self.pending_norm
        self.pending = self.pending_norm = None
        return delta, norm

    def take_prepared(self, norm) -> Optional[tuple]:
        """(values, parts) if the stream's rows were prepared for `norm`, once."""
        prepared, self.prepared = self.prepared, None
        if prepared is not None and prepared[0] is norm and self.pending is None:
            return prepared[1], prepared[2]
        return None
