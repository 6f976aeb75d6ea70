"""Python face of the routed-experts kernels (csrc/routed.cu), compiled when a model with such a
feed-forward first runs."""
from __future__ import annotations

import ctypes
from typing import Optional

import torch

from ..csrc.build import load_library
from ..errors import invalid_argument
from . import ops
from .ops import _check, c_float, c_int, c_void_p, dtype_code

_library = None


def library():
    global _library
    if _library is None:
        lib = load_library("routed")
        lib.kidi_route.argtypes = [c_void_p, c_int, c_void_p, c_int, c_void_p, c_void_p, c_int, c_int, c_int, c_int, c_int,
                                   c_int, c_int, c_int, c_float, c_void_p, c_void_p, c_int, c_float, c_void_p, c_void_p,
                                   c_void_p]
        lib.kidi_expert_slots.argtypes = [c_void_p, c_int, c_void_p, c_void_p, c_int, c_void_p, c_void_p, c_void_p,
                                          c_void_p, c_int, c_int, c_int, c_int, c_int, c_int, c_void_p, c_int, c_void_p,
                                          c_void_p, c_void_p]
        lib.kidi_gather_slots.argtypes = [c_void_p, c_int, c_void_p, c_void_p, c_void_p, c_int, c_int, c_int, c_int,
                                          c_void_p]
        lib.kidi_combine_slots.argtypes = [c_void_p, c_int, c_void_p, c_void_p, c_void_p, c_int, c_int, c_int, c_int,
                                           c_void_p, c_void_p, c_void_p]
        lib.kidi_group_slots.argtypes = [c_void_p, c_void_p, c_void_p, c_void_p, c_int, c_int, c_void_p]
        lib.kidi_group_slots_rows.argtypes = [c_int, c_int]
        for name in ("kidi_group_slots", "kidi_group_slots_rows", "kidi_route", "kidi_expert_slots", "kidi_gather_slots", "kidi_combine_slots"):
            getattr(lib, name).restype = c_int
        _library = lib
    return _library


def _check_addend(addend, like: torch.Tensor, rows: int, hidden: int) -> None:
    if addend is not None and (addend.shape != (rows, hidden) or addend.dtype != like.dtype or not addend.is_contiguous()
                               or not addend.is_cuda):
        raise invalid_argument("the addend has the result's shape and type")


def route(x: torch.Tensor, router: torch.Tensor, top: int, renormalise: bool, score: str = "sigmoid", groups: int = 1,
          keep: int = 1, renormalise_eps: float = 0.0, bias: Optional[torch.Tensor] = None,
          correction: Optional[torch.Tensor] = None, two_largest: bool = False, weight_scale: float = 1.0,
          share_row: Optional[torch.Tensor] = None, share: Optional[torch.Tensor] = None):
    """(chosen int32 [rows, top], weight float32 [rows, top]) for rows x [rows, hidden] and a router
    [experts, hidden]: logits in 32-bit, scores (a sigmoid of each logit, or with `score` "softmax" a softmax over
    all experts), the `top` largest (ties: the lower index), their scores as weights (with `renormalise` divided by
    their sum plus `renormalise_eps`). With `groups` > 1 the experts form that many equal runs of neighbours and
    only experts of the `keep` groups with the largest best score can be chosen. `bias` (float32 [experts]) is added
    to the logits. `correction` (float32 [experts]) is added to the scores that choose experts and groups, not to the
    weights; `two_largest`: a group's score is the sum of its two largest; the weights are multiplied by `weight_scale`.
    `share` (float32 [rows], with `share_row` [1, hidden] in the router's type) takes sigmoid(share_row . x)."""
    ops._need_cuda(x, router, bias, correction, share_row, share)
    ops._float_vector(bias, router.shape[0], "the router's bias")
    ops._float_vector(correction, router.shape[0], "the router's correction")
    if share is not None:
        ops._float_vector(share, x.shape[0], "the shared expert's part")
        if share_row is None or share_row.numel() != x.shape[1] or share_row.dtype != router.dtype or not share_row.is_contiguous():
            raise invalid_argument("the shared expert's gate is a row of the router's type")
    if x.dim() != 2 or not x.is_contiguous() or router.dim() != 2 or not router.is_contiguous() \
            or router.shape[1] != x.shape[1]:
        raise invalid_argument("the router takes contiguous rows and a contiguous [experts, hidden] matrix")
    rows, hidden = x.shape
    chosen = torch.empty((rows, top), dtype=torch.int32, device=x.device)
    weight = torch.empty((rows, top), dtype=torch.float32, device=x.device)
    _check(library().kidi_route(x.data_ptr(), dtype_code(x.dtype), router.data_ptr(), dtype_code(router.dtype),
                                chosen.data_ptr(), weight.data_ptr(), rows, hidden, router.shape[0], top,
                                1 if renormalise else 0, 1 if score == "softmax" else 0, int(groups), int(keep),
                                float(renormalise_eps), bias.data_ptr() if bias is not None else 0,
                                correction.data_ptr() if correction is not None else 0, 1 if two_largest else 0,
                                float(weight_scale), share_row.data_ptr() if share is not None else 0,
                                share.data_ptr() if share is not None else 0, ops._stream()),
           "route")
    return chosen, weight


def expert_slots(x: torch.Tensor, gate_up: torch.Tensor, down: torch.Tensor, chosen: torch.Tensor,
                 weight: torch.Tensor, weight_on_input: bool, gated: bool = True,
                 addend=None, shape: Optional[ops.GateShape] = None, share: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Every row through its chosen experts, the experts' weights read through the choice: x [rows, hidden],
    gate_up [experts, 2 * inter, hidden] (without a gate: the up rows only, [experts, inter, hidden], and the
    exact gelu as activation), down [experts, hidden, inter] -> [rows, hidden]. `addend` [rows, hidden], if given, is
    added to the result (in 32-bit, before it is rounded); it may be a function that returns it (or None), which is
    called between the two kernels; `share` (float32 [rows]): the addend's rows are multiplied by it. `shape`: another
    activation of gated experts than SiLU."""
    ops._need_cuda(x, gate_up, down, chosen, weight)
    rows, hidden = x.shape
    experts, first_rows, _ = gate_up.shape
    inter, top = first_rows // (2 if gated else 1), chosen.shape[1]
    if (not x.is_contiguous() or gate_up.shape != (experts, (2 if gated else 1) * inter, hidden) or down.shape != (experts, hidden, inter)
            or not gate_up.is_contiguous() or not down.is_contiguous() or gate_up.dtype != down.dtype):
        raise invalid_argument("expert_slots: the experts' weights do not fit the rows")
    later = addend if callable(addend) else None
    if later is None:
        _check_addend(addend, x, rows, hidden)
    mid = torch.empty((rows * top, inter), dtype=x.dtype, device=x.device)
    out = torch.empty((rows, hidden), dtype=x.dtype, device=x.device)

    def launch(parts: int, what: str, launches: int) -> None:
        _check(library().kidi_expert_slots(
            x.data_ptr(), dtype_code(x.dtype), gate_up.data_ptr(), down.data_ptr(), dtype_code(gate_up.dtype),
            chosen.data_ptr(), weight.data_ptr(), mid.data_ptr(), out.data_ptr(), rows, top, hidden, inter,
            1 if weight_on_input else 0, 1 if gated else 0, addend.data_ptr() if addend is not None else 0, parts,
            ctypes.byref(shape) if shape is not None else None, share.data_ptr() if share is not None else 0,
            ops._stream()), what, launches)

    if later is None:
        launch(3, "expert_slots", 2)
        return out
    addend = None
    launch(1, "expert_slots[gate and up]", 1)
    addend = later()
    _check_addend(addend, x, rows, hidden)
    launch(2, "expert_slots", 1)
    return out


def group_rows(slots: int, experts: int) -> int:
    """Rows that any choice of `slots` (row, choice) pairs among `experts` experts fits in when every expert's run begins
    on a tile of 128 rows (-1: too many)."""
    return library().kidi_group_slots_rows(int(slots), int(experts))


def group_slots(chosen: torch.Tensor, experts: int):
    """Groups the (row, choice) pairs of `chosen` (int32, slot = row * top + choice) by expert on the device: (source,
    place, expert_of_tile), int32: the slot of every grouped row (-1: padding), the row of every slot, the expert of every
    tile of 128 rows (-1: not used). The order within an expert is not fixed."""
    ops._need_cuda(chosen)
    if chosen.dtype != torch.int32 or not chosen.is_contiguous():
        raise invalid_argument("group_slots takes the router's choices")
    slots = chosen.numel()
    rows = group_rows(slots, experts)
    if rows < 0:
        raise invalid_argument("group_slots: too many slots")
    source = torch.empty(rows, dtype=torch.int32, device=chosen.device)
    place = torch.empty(slots, dtype=torch.int32, device=chosen.device)
    tiles = torch.empty(rows // 128, dtype=torch.int32, device=chosen.device)
    _check(library().kidi_group_slots(chosen.data_ptr(), source.data_ptr(), place.data_ptr(), tiles.data_ptr(), slots,
                                      int(experts), ops._stream()), "group_slots")
    return source, place, tiles


def gather_slots(x: torch.Tensor, order: torch.Tensor, weight: torch.Tensor, top: int, weight_on_input: bool) -> torch.Tensor:
    """Row i of the result is x[order[i] // top] (times weight[order[i]] when the weight is on the input); zeros
    where order[i] is negative."""
    slots, hidden = order.shape[0], x.shape[1]
    out = torch.empty((slots, hidden), dtype=x.dtype, device=x.device)
    _check(library().kidi_gather_slots(x.data_ptr(), dtype_code(x.dtype), order.data_ptr(), weight.data_ptr(),
                                       out.data_ptr(), slots, top, hidden, 1 if weight_on_input else 0, ops._stream()),
           "gather_slots")
    return out


def combine_slots(y: torch.Tensor, place: torch.Tensor, weight: torch.Tensor, rows: int, top: int,
                  weight_on_input: bool, addend: Optional[torch.Tensor] = None,
                  share: Optional[torch.Tensor] = None) -> torch.Tensor:
    """out[r] = sum over k of y[place[r * top + k]] (times weight[r, k] when the weight is on the output), plus
    addend[r] if given (times share[r], float32, if given)."""
    hidden = y.shape[1]
    _check_addend(addend, y, rows, hidden)
    out = torch.empty((rows, hidden), dtype=y.dtype, device=y.device)
    _check(library().kidi_combine_slots(y.data_ptr(), dtype_code(y.dtype), place.data_ptr(), weight.data_ptr(),
                                        out.data_ptr(), rows, top, hidden, 1 if weight_on_input else 0,
                                        addend.data_ptr() if addend is not None else 0,
                                        share.data_ptr() if share is not None else 0, ops._stream()),
           "combine_slots")
    return out
