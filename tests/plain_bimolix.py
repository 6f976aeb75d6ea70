"""Bimolix, plainly: whole sequences, no cache, one function per mechanism, float64 or float32 torch on the CPU.

This file shares no code with the package. It takes the config.json dictionary and a dictionary of tensors under
the checkpoint's names, and returns logits [tokens, vocab] (and, if asked, the stream after every layer).

Notation: T tokens, D width, H query heads, G key/value heads, d the width of a query or key head, e the width of a
value head. A linear weight W is stored [out, in]; `lin(W, x)` is x W^T.
"""
from __future__ import annotations

import math
from typing import List, Mapping, Optional

import torch


def lin(weight: torch.Tensor, x: torch.Tensor, bias: Optional[torch.Tensor] = None) -> torch.Tensor:
    y = x @ weight.to(x.dtype).t()
    return y if bias is None else y + bias.to(x.dtype)


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def by_rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    """The last axis divided by its root mean square, eps under the root."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def stream_norm(x: torch.Tensor, weight: torch.Tensor, eps: float) -> torch.Tensor:
    """The norm of the residual stream: its weight is stored around zero."""
    return by_rms(x, eps) * (1.0 + weight.to(x.dtype))


# ------------------------------------------------------------------------------------------------- retention
def rotate(x: torch.Tensor, dims: int, base: float, first: int = 0) -> torch.Tensor:
    """x [T, heads, d]; entries i and i + dims/2 of a head turn by p base^(-2i/dims) at position p, i < dims/2; the entries
    from `dims` on stay."""
    T, half = x.shape[0], dims // 2
    angle = torch.arange(first, first + T, dtype=torch.float64)[:, None] \
        * (float(base) ** (-2.0 * torch.arange(half, dtype=torch.float64) / dims))[None]
    cos, sin = torch.cos(angle).to(x.dtype)[:, None], torch.sin(angle).to(x.dtype)[:, None]
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * cos - v * sin, v * cos + u * sin, x[..., dims:]], -1)


def fixed_decay_recurrence(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, decay, state=None) -> torch.Tensor:
    """q, k [T, H, d], v [T, H, e], decay [H] numbers -> [T, H, e]; token by token, from a zero state (or from
    `state` [H, d, e], which is changed in place)."""
    T, H, d = q.shape
    out = torch.zeros(T, H, v.shape[-1], dtype=q.dtype)
    S = torch.zeros(H, d, v.shape[-1], dtype=q.dtype) if state is None else state
    keep = torch.tensor([float(value) for value in decay], dtype=q.dtype)[:, None, None]
    for t in range(T):
        S.mul_(keep).add_(k[t, :, :, None] * v[t, :, None, :])
        out[t] = (S * q[t, :, :, None]).sum(1)
    return out


def retention(h: torch.Tensor, w: Mapping[str, torch.Tensor], prefix: str, mixer: Mapping, eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, d, e = int(mixer["heads"]), int(mixer["dim"]), int(mixer["vdim"])
    dims, base = int(mixer["rot"]["dims"]), float(mixer["rot"]["base"])
    q = rotate(lin(w[prefix + "q"], h).reshape(T, H, d), dims, base)
    k = rotate(lin(w[prefix + "k"], h).reshape(T, H, d), dims, base) * d ** -0.5
    v = lin(w[prefix + "v"], h).reshape(T, H, e)
    o = by_rms(fixed_decay_recurrence(q, k, v, mixer["decay"]), eps).reshape(T, H * e)          # head by head
    return lin(w[prefix + "o"], o * silu(lin(w[prefix + "g"], h)))


# ------------------------------------------------------------------------------------------------- attention
def same_chunk(T: int, size: Optional[int]) -> torch.Tensor:
    """[T, T] boolean: query i sees key j when j <= i and both lie in one run of `size` positions counted from 0."""
    i = torch.arange(T)[:, None]
    j = torch.arange(T)[None, :]
    seen = j <= i
    if size is not None:
        seen = seen & (i // int(size) == j // int(size))
    return seen


def distance_bucket(n: int, rows: int, reach: int) -> int:
    """Which of `rows` numbers a key n positions back is given: the first half of them one position each, the second half
    spread over the logarithm of the distance up to `reach`, the last one for everything beyond."""
    half = rows // 2
    if n < half:
        return n
    if reach <= half:
        return rows - 1
    place = math.log(n / half) / math.log(reach / half) * (rows - half)
    if abs(place - round(place)) < 1e-9:            # an exact power, whatever the logarithms rounded to
        place = round(place)
    return min(rows - 1, half + math.floor(place))


def distance_bias(T: int, table: torch.Tensor, reach: int) -> torch.Tensor:
    """[H, T, T]: what is added to the score of query i and key j <= i."""
    by_distance = table[[distance_bucket(n, table.shape[0], reach) for n in range(T)]]             # [T, H]
    back = (torch.arange(T)[:, None] - torch.arange(T)[None, :]).clamp(min=0)
    return by_distance[back].permute(2, 0, 1)


def softmax_with_one(scores: torch.Tensor, seen: torch.Tensor) -> torch.Tensor:
    """exp(s) / (1 + sum of exp(s)) over the keys that are seen."""
    scores = scores.masked_fill(~seen, -math.inf)
    top = scores.amax(-1, keepdim=True).clamp(min=0.0)                  # the one is a key whose score is zero
    power = torch.exp(scores - top)
    return power / (power.sum(-1, keepdim=True) + torch.exp(-top))


def attention(h: torch.Tensor, w: Mapping[str, torch.Tensor], prefix: str, mixer: Mapping, eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, G, d = int(mixer["heads"]), int(mixer["kv_heads"]), int(mixer["dim"])
    q = lin(w[prefix + "q"], h, w[prefix + "q.b"]).reshape(T, H, d)
    v = lin(w[prefix + "k"], h, w[prefix + "k.b"]).reshape(T, G, d)     # a value is its key before the norm
    q = by_rms(q, eps) * w[prefix + "q.norm"].to(h.dtype)
    k = by_rms(v, eps) * w[prefix + "k.norm"].to(h.dtype)
    seen = same_chunk(T, (mixer.get("mask") or {}).get("size"))
    bias = distance_bias(T, w[prefix + "rel"].to(h.dtype), int(mixer["bias_max"]))
    heads = []
    for head in range(H):
        g = head // (H // G)
        scores = (q[:, head] @ k[:, g].t()) * float(mixer["scale"]) + bias[head]
        heads.append(softmax_with_one(scores, seen) @ v[:, g])
    return lin(w[prefix + "o"], torch.cat(heads, -1) * torch.sigmoid(lin(w[prefix + "g"], h)))


# ------------------------------------------------------------------------------------------------- feed-forward
def gated(h: torch.Tensor, w: Mapping[str, torch.Tensor], prefix: str) -> torch.Tensor:
    return lin(w[prefix + "down"], silu(lin(w[prefix + "gate"], h)) * lin(w[prefix + "up"], h))


def bounded_expert(h: torch.Tensor, w: Mapping[str, torch.Tensor], prefix: str, limit: float) -> torch.Tensor:
    g = lin(w[prefix + "gate"], h).clamp(max=limit)
    u = lin(w[prefix + "up"], h).clamp(min=-limit, max=limit)
    return lin(w[prefix + "down"], g * torch.sigmoid(1.702 * g) * (u + 1.0))


def router_choice(choice: torch.Tensor, top: int, groups: int, keep: int) -> torch.Tensor:
    """The `top` largest of choice [experts] among the experts of the `keep` groups whose two largest add up to most."""
    per = choice.shape[0] // groups
    score = torch.topk(choice.reshape(groups, per), min(2, per), dim=-1).values.sum(-1)
    kept = torch.topk(score, keep).indices
    open_ = torch.full_like(choice, -math.inf).reshape(groups, per)
    open_[kept] = choice.reshape(groups, per)[kept]
    return torch.topk(open_.reshape(-1), top).indices


def chosen_or_given(choice, top, groups, keep, given, margin):
    """This one's own choice, or another implementation's (`given` [top]) where it is a close call: where it becomes this
    one's own once the given experts' scores are raised by `margin`, and the others lowered by it."""
    chosen = router_choice(choice, top, groups, keep)
    if given is not None and sorted(given.tolist()) != sorted(chosen.tolist()):
        tilted = choice - margin
        tilted[given.long()] = choice[given.long()] + margin
        if sorted(router_choice(tilted, top, groups, keep).tolist()) == sorted(given.tolist()):
            return given.long()
    return chosen


def routed(h: torch.Tensor, w: Mapping[str, torch.Tensor], prefix: str, mlp: Mapping,
           given: Optional[torch.Tensor] = None, margin: float = 0.0) -> torch.Tensor:
    router = mlp["router"]
    groups = router.get("groups") or {"count": 1, "keep": 1}
    scores = torch.sigmoid(lin(w[prefix + "router"], h))
    choice = scores + w[prefix + "correction"].to(h.dtype)
    share = torch.zeros(h.shape[0], int(router["experts"]), dtype=h.dtype)          # of every expert in every token
    for t in range(h.shape[0]):
        chosen = chosen_or_given(choice[t], int(router["top"]), int(groups["count"]), int(groups["keep"]),
                                 given[t] if given is not None else None, margin)
        share[t, chosen] = scores[t, chosen] / (scores[t, chosen].sum() + 1e-20) * float(router.get("scale", 1.0))
    out = torch.zeros_like(h)
    for index in range(share.shape[1]):
        users = (share[:, index] != 0).nonzero().flatten()
        out[users] += share[users, index, None] * bounded_expert(h[users], w, f"{prefix}e{index}.", float(mlp["expert"]["limit"]))
    shared = mlp.get("shared")
    if shared:
        out = out + torch.sigmoid(lin(w[prefix + "shared.sg"], h)) \
            * bounded_expert(h, w, prefix + "shared.", float(shared["limit"]))
    return out


# ------------------------------------------------------------------------------------------------- model
MIXERS = {"retention": retention, "attention": attention}


def forward(config: Mapping, w: Mapping[str, torch.Tensor], tokens, dtype=torch.float64,
            streams: Optional[List[torch.Tensor]] = None, choices: Optional[List[torch.Tensor]] = None,
            margin: float = 0.0) -> torch.Tensor:
    """`choices`: for every routed layer that is run, in order, the experts [T, top] that another implementation chose
    (see `chosen_or_given`)."""
    ids = torch.as_tensor(list(tokens), dtype=torch.long)
    w = {name: (tensor.to(dtype) if tensor.is_floating_point() else tensor) for name, tensor in w.items()}
    eps = float(config["norm"]["eps"])
    x = stream_norm(w["embed"][ids], w["embed.norm"], eps)
    routed_layers = 0
    for index, layer in enumerate(config["layers"]):
        source = index
        while config["layers"][source].get("weights_of") is not None:
            source = int(config["layers"][source]["weights_of"])
        prefix = f"l{source}."
        x = x + MIXERS[layer["type"]](stream_norm(x, w[prefix + "norm1"], eps), w, prefix + "mix.", layer["mixer"], eps)
        mlp = layer.get("mlp")
        if mlp is not None:
            h = stream_norm(x, w[prefix + "norm2"], eps)
            if mlp["kind"] == "dense":
                x = x + gated(h, w, prefix + "mlp.")
            else:
                given = choices[routed_layers] if choices is not None else None
                routed_layers += 1
                x = x + routed(h, w, prefix + "mlp.", mlp, given, margin)
        if streams is not None:
            streams.append(x.clone())
    return lin(w["head"], stream_norm(x, w["final.norm"], eps))
