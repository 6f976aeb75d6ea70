"""Python faces of the kernels of linear attention with one fixed decay per head (csrc/linear_attention.cu), compiled
when a model with such a layer first runs."""
from __future__ import annotations

import ctypes
import os
from typing import Dict, Optional

import torch

from ..csrc.build import load_library
from ..errors import invalid_argument
from . import ops, scalar_recurrence
from .ops import _check, c_float, c_int, c_longlong, c_void_p, dtype_code
from .scalar_recurrence import MAX_DIM, _float_tensor, _rows_view


class LinearStepArgs(ctypes.Structure):
    _fields_ = [("q", c_void_p), ("ldq", c_longlong), ("k", c_void_p), ("ldk", c_longlong), ("v", c_void_p),
                ("ldv", c_longlong), ("decay", c_void_p), ("state", c_void_p), ("out", c_void_p), ("row_seq", c_void_p),
                ("seq_slot", c_void_p), ("seq_row0", c_void_p), ("seqs", c_int), ("heads", c_int), ("dim", c_int),
                ("vdim", c_int), ("cos_table", c_void_p), ("sin_table", c_void_p), ("row_pos", c_void_p),
                ("rotary_dim", c_int), ("key_scale", c_float), ("gate", c_void_p), ("ldg", c_longlong),
                ("finished", c_void_p), ("ldf", c_longlong), ("eps", c_float), ("gate_silu", c_int)]

    def __init__(self, *values, **named):
        named.setdefault("key_scale", 1.0)
        super().__init__(*values, **named)


class LinearChunksArgs(ctypes.Structure):
    _fields_ = [("q", c_void_p), ("ldq", c_longlong), ("k", c_void_p), ("ldk", c_longlong), ("v", c_void_p),
                ("ldv", c_longlong), ("decay", c_void_p), ("state", c_void_p), ("out", c_void_p), ("sums", c_void_p),
                ("before", c_void_p), ("row_seq", c_void_p), ("seq_slot", c_void_p), ("seq_row0", c_void_p),
                ("seq_len", c_void_p), ("seqs", c_int), ("heads", c_int), ("head0", c_int), ("group", c_int),
                ("max_chunks", c_int), ("cos_table", c_void_p), ("sin_table", c_void_p), ("row_pos", c_void_p),
                ("rotary_dim", c_int), ("key_scale", c_float), ("gate", c_void_p), ("ldg", c_longlong),
                ("finished", c_void_p), ("ldf", c_longlong), ("eps", c_float), ("gate_silu", c_int)]


# The chunked form on the tensor cores: steps whose longest sequence brings at least this many tokens (0: never).
MIN_CHUNKED_TOKENS = int(os.environ.get("KIDI_B200_LINEAR_CHUNKS", "32"))
CHUNK = 64                              # tokens of a chunk (csrc/linear_chunks.cu)
SCRATCH_FLOATS = 48 * 1024 * 1024       # the heads of a step are taken in groups that need at most this much scratch memory

_library = None
_chunk_libraries: Dict[tuple, ctypes.CDLL] = {}


def chunk_library_request(dim: int, vdim: int, wide: bool = False):
    """(name, sources, definitions) of the chunked kernels for one pair of head widths (`wide`: with rotated and scaled,
    hence 32-bit, queries and keys and a finish head by head)."""
    defines = {"KIDI_LINEAR_DIM": dim, "KIDI_LINEAR_VDIM": vdim, **({"KIDI_LINEAR_WIDE": 1} if wide else {})}
    return f"linear_chunks_d{dim}_v{vdim}" + ("_wide" if wide else ""), ("linear_chunks.cu",), defines


def chunk_library(dim: int, vdim: int, wide: bool = False) -> ctypes.CDLL:
    lib = _chunk_libraries.get((dim, vdim, wide))
    if lib is None:
        lib = load_library(*chunk_library_request(dim, vdim, wide))
        lib.kidi_linear_chunks.argtypes = [c_void_p, c_void_p]
        lib.kidi_linear_chunks.restype = c_int
        lib.kidi_linear_chunks_scratch.argtypes = [c_int, c_int, c_int]
        lib.kidi_linear_chunks_scratch.restype = c_longlong
        _chunk_libraries[(dim, vdim, wide)] = lib
    return lib


def chunks_fit(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, dim: int, vdim: int, longest: int) -> bool:
    """Whether a step takes the chunked kernels: bfloat16 rows on 16-byte boundaries, head widths that are multiples of
    16, and a sequence of enough tokens."""
    return (0 < MIN_CHUNKED_TOKENS <= longest and q.dtype == torch.bfloat16 and dim % 16 == 0 and vdim % 16 == 0
            and dim <= 256 and vdim <= 256
            and all(x.stride(0) % 8 == 0 and x.data_ptr() % 16 == 0 for x in (q, k, v)))


def wide_chunks_fit(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, dim: int, vdim: int, longest: int) -> bool:
    """The same for the form with 32-bit queries and keys, of which a block keeps three parts in shared memory."""
    parts = 3 * CHUNK * (dim + 8)
    first, second = max(parts, 3 * CHUNK * (CHUNK + 8)), max(2 * 3 * 16 * (vdim + 8), parts, CHUNK * (vdim + 8))
    return chunks_fit(q, k, v, dim, vdim, longest) and 2 * (first + second) + 4 * (CHUNK + 4 + 4 * CHUNK) <= 227 * 1024


def library():
    global _library
    if _library is None:
        lib = load_library("linear_attention")
        lib.kidi_linear_step.argtypes = [c_void_p, c_int, c_void_p]
        lib.kidi_normed_gate.argtypes = [c_void_p, c_void_p, c_void_p, c_longlong, c_int, c_void_p, c_longlong, c_int, c_int,
                                         c_float, c_float, c_void_p]
        lib.kidi_silu_columns.argtypes = [c_void_p, c_longlong, c_int, c_int, c_int, c_int, c_void_p]
        lib.kidi_rotate_heads.argtypes = [c_void_p, c_longlong, c_void_p, c_longlong, c_void_p, c_longlong, c_int, c_void_p,
                                          c_void_p, c_void_p, c_void_p, c_int, c_float, c_int, c_int, c_int, c_int, c_void_p]
        lib.kidi_head_norm_gate.argtypes = [c_void_p, c_void_p, c_void_p, c_longlong, c_int, c_void_p, c_longlong, c_int, c_int,
                                            c_int, c_float, c_float, c_int, c_void_p]
        for name in ("kidi_linear_step", "kidi_normed_gate", "kidi_silu_columns", "kidi_rotate_heads", "kidi_head_norm_gate"):
            getattr(lib, name).restype = c_int
        _library = lib
    return _library


def linear_attention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, decay: torch.Tensor, state: torch.Tensor, *,
                     heads: int, dim: int, vdim: int, tables, seqs: int, one_token: bool, longest: int) -> torch.Tensor:
    """S_t = decay_h S_(t-1) + k_t v_t^T and o_t = S_t^T q_t for every sequence's rows of the step, from and into `state`
    [slots + 1, heads, dim, vdim] (float32). q, k [rows, heads * dim] and v [rows, heads * vdim] are views of the step's
    element type; decay float32 [heads]. `one_token`: every sequence of the step brings one token (decoding); `longest`:
    the most tokens that a sequence brings. Returns the read-out, float32 [rows, heads * vdim]."""
    if not one_token and not chunks_fit(q, k, v, dim, vdim, longest):
        return scalar_recurrence.scalar_recurrence(k, q, v, None, state, heads=heads, k_heads=heads, q_heads=heads, dim=dim,
                                                   vdim=vdim, tables=tables, seqs=seqs, decay=decay)
    ops._need_cuda(q, k, v, decay, state)
    rows = v.shape[0]
    for tensor, width, what in ((k, heads * dim, "keys"), (q, heads * dim, "queries"), (v, heads * vdim, "values")):
        _rows_view(tensor, "linear attention")
        if tensor.shape != (rows, width) or tensor.dtype != v.dtype:
            raise invalid_argument(f"linear attention: the {what} have the wrong shape or type")
    _float_tensor(decay, (heads,), "the decays")
    if state.dtype != torch.float32 or tuple(state.shape[1:]) != (heads, dim, vdim) or not state.is_contiguous():
        raise invalid_argument("linear attention: the state is float32 [slots, heads, dim, vdim]")
    out = torch.empty((rows, heads * vdim), dtype=torch.float32, device=v.device)
    if not one_token:
        for head0, here, sums, before, lib in _head_groups(rows, seqs, heads, dim, vdim, v.device, False):
            args = LinearChunksArgs(
                q.data_ptr(), q.stride(0), k.data_ptr(), k.stride(0), v.data_ptr(), v.stride(0), decay.data_ptr(),
                state.data_ptr(), out.data_ptr(), sums, before,
                tables.row_seq.data_ptr(), tables.seq_slot.data_ptr(), tables.seq_row0.data_ptr(),
                tables.seq_len.data_ptr(), seqs, heads, head0, here, -(-longest // CHUNK))
            _check(lib.kidi_linear_chunks(ctypes.byref(args), ops._stream()), "linear_attention[chunks]", 3)
        return out
    args = LinearStepArgs(q.data_ptr(), q.stride(0), k.data_ptr(), k.stride(0), v.data_ptr(), v.stride(0), decay.data_ptr(),
                          state.data_ptr(), out.data_ptr(), tables.row_seq.data_ptr(), tables.seq_slot.data_ptr(),
                          tables.seq_row0.data_ptr(), seqs, heads, dim, vdim)
    _check(library().kidi_linear_step(ctypes.byref(args), dtype_code(v.dtype), ops._stream()), "linear_attention[one token]")
    return out


FINISH_SPANS = 8                        # blocks of 32 columns that finish a head together in the one-token kernel


def retention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, gate: torch.Tensor, decay: torch.Tensor,
              state: torch.Tensor, out: torch.Tensor, *, heads: int, dim: int, vdim: int, tables, seqs: int, one_token: bool,
              longest: int, cos: Optional[torch.Tensor], sin: Optional[torch.Tensor], rotary_dim: int, key_scale: float,
              eps: float, silu: bool) -> torch.Tensor:
    """`linear_attention` with queries and keys that turn by position (`cos`, `sin` float32 [positions, rotary_dim / 2]: the
    halves of a head's first rotary_dim entries are the pairs; None: they stay) and keys times `key_scale`, both in 32-bit on
    the way into the recurrence, and with each head finished: out = read / rms(read) * silu(gate) (or its sigmoid); gate and
    out [rows, heads * vdim], of the step's element type. One kernel for single tokens, the chunked form (which finishes in
    its last kernel) for prompts, the scan over 32-bit queries, keys and values else."""
    ops._need_cuda(q, k, v, gate, decay, state, out, cos, sin)
    rows, rotary_dim = v.shape[0], int(rotary_dim) if cos is not None else 0
    for tensor, width, what in ((k, heads * dim, "keys"), (q, heads * dim, "queries"), (v, heads * vdim, "values"),
                                (gate, heads * vdim, "gate"), (out, heads * vdim, "result")):
        _rows_view(tensor, "retention")
        if tensor.shape != (rows, width) or tensor.dtype != v.dtype:
            raise invalid_argument(f"retention: the {what} have the wrong shape or type")
    _float_tensor(decay, (heads,), "the decays")
    if state.dtype != torch.float32 or tuple(state.shape[1:]) != (heads, dim, vdim) or not state.is_contiguous():
        raise invalid_argument("retention: the state is float32 [slots, heads, dim, vdim]")
    if cos is not None:
        if sin is None or cos.dtype != torch.float32 or sin.dtype != torch.float32 or cos.shape != sin.shape or cos.dim() != 2 \
                or cos.shape[1] * 2 != rotary_dim or rotary_dim > dim or not cos.is_contiguous() or not sin.is_contiguous():
            raise invalid_argument("retention: the rotation tables are float32 [positions, rotary_dim / 2]")
    rotation = dict(cos_table=cos.data_ptr() if cos is not None else 0, sin_table=sin.data_ptr() if cos is not None else 0,
                    row_pos=tables.row_pos.data_ptr(), rotary_dim=rotary_dim, key_scale=float(key_scale))
    finish = dict(gate=gate.data_ptr(), ldg=gate.stride(0), finished=out.data_ptr(), ldf=out.stride(0), eps=float(eps),
                  gate_silu=int(silu))
    operands = (q.data_ptr(), q.stride(0), k.data_ptr(), k.stride(0), v.data_ptr(), v.stride(0), decay.data_ptr(),
                state.data_ptr())
    if one_token:
        fused = vdim <= 32 * FINISH_SPANS
        read = None if fused else torch.empty((rows, heads * vdim), dtype=torch.float32, device=v.device)
        args = LinearStepArgs(*operands, read.data_ptr() if read is not None else 0, tables.row_seq.data_ptr(),
                              tables.seq_slot.data_ptr(), tables.seq_row0.data_ptr(), seqs, heads, dim, vdim, **rotation,
                              **(finish if fused else {}))
        _check(library().kidi_linear_step(ctypes.byref(args), dtype_code(v.dtype), ops._stream()),
               "retention[one token]" if fused else "linear_attention[one token]")
        return out if fused else head_norm_gate(read, None, gate, heads, eps, 1.0, silu, out)
    if wide_chunks_fit(q, k, v, dim, vdim, longest) and gate.stride(0) % 2 == 0 and out.stride(0) % 2 == 0 \
            and gate.data_ptr() % 4 == 0 and out.data_ptr() % 4 == 0:
        for head0, here, sums, before, lib in _head_groups(rows, seqs, heads, dim, vdim, v.device, True):
            args = LinearChunksArgs(*operands, 0, sums, before, tables.row_seq.data_ptr(), tables.seq_slot.data_ptr(),
                                    tables.seq_row0.data_ptr(), tables.seq_len.data_ptr(), seqs, heads, head0, here,
                                    -(-longest // CHUNK), **rotation, **finish)
            _check(lib.kidi_linear_chunks(ctypes.byref(args), ops._stream()), "retention[chunks]", 3)
        return out
    wide = torch.empty((rows, heads * (2 * dim + vdim)), dtype=torch.float32, device=v.device)
    _check(library().kidi_rotate_heads(
        q.data_ptr(), q.stride(0), k.data_ptr(), k.stride(0), v.data_ptr(), v.stride(0), dtype_code(v.dtype), wide.data_ptr(),
        rotation["cos_table"], rotation["sin_table"], rotation["row_pos"], rotary_dim, float(key_scale), rows, heads, dim, vdim,
        ops._stream()), "rotate_heads")
    qk = heads * dim
    read = scalar_recurrence.scalar_recurrence(wide[:, qk:2 * qk], wide[:, :qk], wide[:, 2 * qk:], None, state, heads=heads,
                                               k_heads=heads, q_heads=heads, dim=dim, vdim=vdim, tables=tables, seqs=seqs,
                                               decay=decay)
    return head_norm_gate(read, None, gate, heads, eps, 1.0, silu, out)


def _head_groups(rows: int, seqs: int, heads: int, dim: int, vdim: int, device, wide: bool):
    """(first head, heads, address of the sums, address of the states before the chunks, library) for every launch of the
    chunked form: the heads of a step in groups that need at most SCRATCH_FLOATS of scratch memory, which they share."""
    lib = chunk_library(dim, vdim, wide)
    group = heads
    while group > 1 and lib.kidi_linear_chunks_scratch(rows, seqs, group) > SCRATCH_FLOATS:
        group = -(-group // 2)
    scratch = torch.empty(lib.kidi_linear_chunks_scratch(rows, seqs, group), dtype=torch.float32, device=device)
    for head0 in range(0, heads, group):
        here = min(group, heads - head0)
        sums = (rows // CHUNK + seqs + 1) * here * dim * vdim        # floats of the sums; the states follow them
        yield head0, here, scratch.data_ptr(), scratch.data_ptr() + 4 * sums, lib


def head_norm_gate(read: torch.Tensor, weight: Optional[torch.Tensor], gate: torch.Tensor, heads: int, eps: float,
                   factor: float, silu: bool, out: torch.Tensor) -> torch.Tensor:
    """out = read / rms(read) * weight * silu(gate) * factor (or sigmoid(gate)), the root mean square over each of `heads`
    equal parts of a row; read float32 [rows, width], weight float32 [width] or None, gate and out views of the step's
    element type whose rows are contiguous."""
    ops._need_cuda(read, weight, gate, out)
    rows, width = read.shape
    _float_tensor(read, (rows, width), "the read-out")
    if weight is not None:
        _float_tensor(weight, (width,), "the norm weight")
    _rows_view(gate, "head gate")
    _rows_view(out, "head gate")
    if width % heads or gate.shape != (rows, width) or out.shape != (rows, width) or gate.dtype != out.dtype:
        raise invalid_argument("head gate: the gate or the result has the wrong shape or type")
    _check(library().kidi_head_norm_gate(read.data_ptr(), weight.data_ptr() if weight is not None else 0, gate.data_ptr(),
                                         gate.stride(0), dtype_code(gate.dtype), out.data_ptr(), out.stride(0), rows, heads,
                                         width // heads, float(eps), float(factor), int(silu), ops._stream()),
           "head_norm_gate")
    return out


def normed_gate(read: torch.Tensor, weight: torch.Tensor, gate: torch.Tensor, eps: float, factor: float,
                out: torch.Tensor) -> torch.Tensor:
    """out = read / rms(read) * weight * sigmoid(gate) * factor over each row; read float32 [rows, width], gate and out
    views of the step's element type whose rows are contiguous."""
    ops._need_cuda(read, weight, gate, out)
    rows, width = read.shape
    _float_tensor(read, (rows, width), "the read-out")
    _float_tensor(weight, (width,), "the norm weight")
    _rows_view(gate, "normed gate")
    _rows_view(out, "normed gate")
    if gate.shape != (rows, width) or out.shape != (rows, width) or gate.dtype != out.dtype:
        raise invalid_argument("normed gate: the gate or the result has the wrong shape or type")
    _check(library().kidi_normed_gate(read.data_ptr(), weight.data_ptr(), gate.data_ptr(), gate.stride(0),
                                      dtype_code(gate.dtype), out.data_ptr(), out.stride(0), rows, width, float(eps),
                                      float(factor), ops._stream()), "normed_gate")
    return out


def silu_columns(x: torch.Tensor, begin: int, end: int) -> torch.Tensor:
    """x[:, begin:end] <- silu of itself, in place (32-bit arithmetic)."""
    ops._need_cuda(x)
    _rows_view(x, "silu columns")
    if not 0 <= begin <= end <= x.shape[1]:
        raise invalid_argument("silu columns: the range lies outside the matrix")
    _check(library().kidi_silu_columns(x.data_ptr(), x.stride(0), dtype_code(x.dtype), x.shape[0], int(begin),
                                       int(end - begin), ops._stream()), "silu_columns")
    return x
