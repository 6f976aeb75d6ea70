"""Dibesun, plainly: whole sequences, no cache, one function per mechanism, float64 or float32 torch on the CPU.

This file shares no code with the package. It takes the config.json dictionary and a dictionary of tensors under
the checkpoint's names, and returns logits [tokens, vocab] (and, if asked, the stream after every layer).

Notation: T tokens, D width, H query heads, G key/value heads, d the width of a query or key head, e the width of a
value head. A linear weight W is stored [out, in]; `lin(W, x)` is x W^T.
"""
from __future__ import annotations

from typing import List, Mapping, Optional

import torch


def lin(weight: torch.Tensor, x: torch.Tensor) -> torch.Tensor:
    return x @ weight.to(x.dtype).t()


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def grouped_rms(x: torch.Tensor, weight: torch.Tensor, eps: float, groups: int = 1) -> torch.Tensor:
    """Each of `groups` equal runs of the last axis divided by its own root mean square (eps under the root), then
    the whole multiplied by the weight."""
    parts = x.reshape(*x.shape[:-1], groups, x.shape[-1] // groups)
    parts = parts / torch.sqrt((parts * parts).mean(-1, keepdim=True) + eps)
    return parts.reshape(x.shape) * weight.to(x.dtype)


# ------------------------------------------------------------------------------------------------- attention
def same_chunk(T: int, size: Optional[int]) -> torch.Tensor:
    """[T, T] boolean: query i sees key j when j <= i and both lie in one run of `size` positions counted from 0."""
    i = torch.arange(T)[:, None]
    j = torch.arange(T)[None, :]
    seen = j <= i
    if size is not None:
        seen = seen & (i // int(size) == j // int(size))
    return seen


def sigmoid_weights(scores: torch.Tensor, seen: torch.Tensor, bias) -> torch.Tensor:
    """The weight of a key that is seen is sigmoid(score + bias), of any other key zero; nothing is normalised."""
    return torch.sigmoid(scores + bias) * seen.to(scores.dtype)


def bounded(scores: torch.Tensor, cap: Optional[float]) -> torch.Tensor:
    return cap * torch.tanh(scores / cap) if cap else scores


def sigmoid_attention(h: torch.Tensor, w: Mapping[str, torch.Tensor], prefix: str, mixer: Mapping, eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, G, d, e = int(mixer["heads"]), int(mixer["kv_heads"]), int(mixer["dim"]), int(mixer["vdim"])
    q = grouped_rms(lin(w[prefix + "q"], h), w[prefix + "q.norm"], eps).reshape(T, H, d)    # over all heads at once
    k = grouped_rms(lin(w[prefix + "k"], h), w[prefix + "k.norm"], eps).reshape(T, G, d)
    v = lin(w[prefix + "v"], h).reshape(T, G, e)
    seen = same_chunk(T, (mixer.get("mask") or {}).get("size"))
    heads = []
    for head in range(H):
        g = head // (H // G)
        scores = bounded((q[:, head] @ k[:, g].t()) * float(mixer["scale"]), mixer.get("softcap"))
        heads.append(sigmoid_weights(scores, seen, w[prefix + "pb"][head].to(h.dtype)) @ v[:, g])
    return lin(w[prefix + "o"], torch.cat(heads, -1))


# ------------------------------------------------------------------------------------------------- recurrence
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


def linear_attention(h: torch.Tensor, w: Mapping[str, torch.Tensor], prefix: str, mixer: Mapping, eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, d, e = int(mixer["heads"]), int(mixer["dim"]), int(mixer["vdim"])
    q = silu(lin(w[prefix + "q"], h)).reshape(T, H, d)
    k = silu(lin(w[prefix + "k"], h)).reshape(T, H, d)
    v = silu(lin(w[prefix + "v"], h)).reshape(T, H, e)
    o = fixed_decay_recurrence(q, k, v, mixer["decay"]).reshape(T, H * e)
    o = grouped_rms(o, w[prefix + "norm"], eps) * torch.sigmoid(lin(w[prefix + "g"], h))
    return lin(w[prefix + "o"], o)


def two_mixers(h: torch.Tensor, w: Mapping[str, torch.Tensor], prefix: str, mixer: Mapping, eps: float) -> torch.Tensor:
    return float(mixer["left_scale"]) * sigmoid_attention(h, w, prefix + "left.", mixer["left"], eps) \
        + float(mixer["right_scale"]) * linear_attention(h, w, prefix + "right.", mixer["right"], eps)


# ------------------------------------------------------------------------------------------------- feed-forward
def gated(h: torch.Tensor, w: Mapping[str, torch.Tensor], prefix: str) -> torch.Tensor:
    return lin(w[prefix + "down"], silu(lin(w[prefix + "gate"], h)) * lin(w[prefix + "up"], h))


def router_choice(z: torch.Tensor, top: int, given: Optional[torch.Tensor] = None, margin: float = 0.0) -> torch.Tensor:
    """The `top` largest of z [experts]. `given` [top]: another implementation's choice, taken instead if it is this
    one's own once the given logits are raised and the others lowered by `margin` (a close call)."""
    chosen = torch.topk(z, top).indices
    if given is not None and sorted(given.tolist()) != sorted(chosen.tolist()):
        tilted = z - margin
        tilted[given.long()] = z[given.long()] + margin
        if sorted(torch.topk(tilted, top).indices.tolist()) == sorted(given.tolist()):
            return given.long()
    return chosen


def routed(h: torch.Tensor, w: Mapping[str, torch.Tensor], prefix: str, mlp: Mapping,
           given: Optional[torch.Tensor] = None, margin: float = 0.0) -> torch.Tensor:
    top = int(mlp["router"]["top"])
    z = lin(w[prefix + "router"], h) + w[prefix + "router.b"].to(h.dtype)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        chosen = router_choice(z[t], top, given[t] if given is not None else None, margin)
        weights = torch.softmax(z[t, chosen], -1)                  # over the chosen logits only
        for weight, index in zip(weights, chosen.tolist()):
            out[t] += weight * gated(h[t:t + 1], w, f"{prefix}e{index}.")[0]
    if mlp.get("shared"):
        out = out + gated(h, w, prefix + "shared.")
    return out


# ------------------------------------------------------------------------------------------------- model
def forward(config: Mapping, w: Mapping[str, torch.Tensor], tokens, dtype=torch.float64,
            streams: Optional[List[torch.Tensor]] = None, choices: Optional[List[torch.Tensor]] = None,
            margin: float = 0.0) -> torch.Tensor:
    """`choices`: for every routed layer, in order, the experts [T, top] that another implementation chose (see
    `router_choice`)."""
    ids = torch.as_tensor(list(tokens), dtype=torch.long)
    w = {name: (tensor.to(dtype) if tensor.is_floating_point() else tensor) for name, tensor in w.items()}
    eps, groups = float(config["norm"]["eps"]), int(config["norm"]["groups"])
    x = w["embed"][ids] * float(config["embedding"]["scale"])
    routed_layers = 0
    for index, layer in enumerate(config["layers"]):
        prefix = f"l{index}."
        x = x + grouped_rms(two_mixers(x, w, prefix + "mix.", layer["mixer"], eps), w[prefix + "norm1"], eps, groups)
        mlp = layer.get("mlp")
        if mlp is not None:
            if mlp["kind"] == "dense":
                y = gated(x, w, prefix + "mlp.")
            else:
                given = choices[routed_layers] if choices is not None else None
                routed_layers += 1
                y = routed(x, w, prefix + "mlp.", mlp, given, margin)
            x = x + grouped_rms(y, w[prefix + "norm2"], eps, groups)
        if streams is not None:
            streams.append(x.clone())
    return lin(w["embed"], grouped_rms(x, w["final.norm"], eps, groups))
