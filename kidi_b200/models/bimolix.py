"""Bimolix as a `ModelSpec`.

A decoder-only pre-norm stack: token embeddings that pass a norm of their own, layers that are one of two mixers and a
feed-forward (or none), a final norm and a head of its own. Every norm of the stream is an RMS norm whose weight is stored
around zero.

* retention: linear attention with one fixed decay per head; queries and keys are rotated (keys also scaled), every head is
  divided by its own root mean square, and the whole multiplied by the SiLU of a gate;
* attention: grouped queries over runs of positions (a query sees the earlier keys of its own run) without rotation; a
  value is its key before the key norm; a learned number per head and bucket of distance is added to a score, a one to the
  softmax's denominator, and the heads are multiplied by the sigmoid of a gate.

A feed-forward is a dense SiLU-gated one or routed experts with bounded gates: a sigmoid router with a correction that only
the choice sees, groups ranked by their two best experts, scaled weights, and an optional shared expert under a gate of one
number a token. Layers may run with another layer's tensors (and a cache of their own): they are entries of the schedule.

Tensor names: `embed`, `embed.norm`, `final.norm`, `head`, and per layer `l<i>.norm1`, `l<i>.norm2`, `l<i>.mix.{q,k,v,g,o}`
(retention) or `l<i>.mix.{q,q.b,k,k.b,q.norm,k.norm,rel,g,o}` (attention), `l<i>.mlp.{gate,up,down}` or
`l<i>.mlp.{router,correction}`, `l<i>.mlp.{e<j>,shared}.{gate,up,down}`, `l<i>.mlp.shared.sg`. The number of distance buckets is
the height of `rel`.

This file maps a `BimolixConfig` to parts and their parameters; nothing here computes.
"""
from __future__ import annotations

from ..config.bimolix import ATTENTION, BimolixConfig
from ..parts.spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry
from ..registry import register_architecture

RENORMALISE_EPS = 1e-20
GATE_SLOPE = 1.702                  # of the experts' bounded gates


def build_spec(config: BimolixConfig) -> ModelSpec:
    hidden, eps = config.width, config.norm_eps
    norm = lambda name, prefix="": PartSpec("rms_norm", {"size": hidden, "eps": eps, "weight_offset": 1.0, "fold": True,
                                                         "weight_name": name}, prefix)
    positions, layers, place = {}, [], {}
    for index, layer in enumerate(config.layers):
        if config.owner(index) != index:
            continue
        prefix, mixer, mlp = f"l{index}.", layer.mixer, layer.mlp
        if mixer.kind == ATTENTION:
            part = PartSpec("attention", {
                "hidden_size": hidden, "num_heads": mixer.heads, "num_kv_heads": mixer.kv_heads, "head_dim": mixer.dim,
                "scale": mixer.scale, "position": None, "chunk": mixer.chunk, "values_from_keys": True, "qkv_bias": True,
                "qk_norm": True, "qk_norm_eps": eps, "distance_bias_reach": mixer.bias_max, "sink_score": 0.0,
                "output_gate": True, "q_name": "q", "k_name": "k", "q_bias_name": "q.b", "k_bias_name": "k.b",
                "q_norm_name": "q.norm", "k_norm_name": "k.norm", "distance_bias_name": "rel", "gate_name": "g",
                "o_name": "o"}, prefix + "mix.")
        else:
            rotation = None
            if mixer.rot_dims:
                rotation = f"rotary {mixer.dim} {mixer.rot_dims} {mixer.rot_base!r}"
                positions[rotation] = PartSpec("rotary", {
                    "head_dim": mixer.dim, "rotary_dim": mixer.rot_dims, "theta": mixer.rot_base, "angles64": True,
                    "max_positions": config.max_positions})
            part = PartSpec("lightning_attention", {
                "hidden_size": hidden, "num_heads": mixer.heads, "dim": mixer.dim, "vdim": mixer.vdim,
                "decay": list(mixer.decay), "eps": eps, "activation": None, "position": rotation,
                "key_scale": mixer.dim ** -0.5, "norm_scope": "head", "norm_weight": False, "gate_activation": "silu"},
                prefix + "mix.")
        parts = {"input_norm": norm("norm1", prefix), "mixer": part}
        if mlp is not None:
            parts["post_norm"] = norm("norm2", prefix)
            if mlp.experts is None:
                parts["feed_forward"] = PartSpec("gated_mlp", {
                    "hidden_size": hidden, "intermediate_size": mlp.ff, "gate_name": "gate", "up_name": "up",
                    "down_name": "down"}, prefix + "mlp.")
            else:
                parts["feed_forward"] = PartSpec("routed_experts", {
                    "hidden_size": hidden, "expert_size": mlp.ff, "experts": mlp.experts, "top": mlp.top,
                    "score": "sigmoid", "renormalise": True, "renormalise_eps": RENORMALISE_EPS, "weight_on": "output",
                    "correction_name": "correction", "groups": mlp.groups, "keep_groups": mlp.keep_groups,
                    "group_score": "two_largest", "weight_scale": mlp.router_scale, "activation": "bounded_swish",
                    "limit": mlp.limit, "alpha": GATE_SLOPE, "up_shift": 1.0, "shared_size": mlp.shared_ff,
                    "shared_limit": mlp.shared_limit, "shared_gate_name": "sg"}, prefix + "mlp.")
        place[index] = len(layers)
        layers.append(LayerSpec(arrangement=PartSpec("pre_norm"), parts=parts))
    return ModelSpec(
        architecture=config.architecture,
        vocab_size=config.vocab,
        hidden_size=hidden,
        max_positions=config.max_positions,
        embedding=PartSpec("token_embedding", {"vocab_size": config.vocab, "hidden_size": hidden, "name": "embed"}, ""),
        embedding_norm=norm("embed.norm"),
        positions=positions,
        layers=tuple(layers),
        schedule=tuple(ScheduleEntry(place[config.owner(index)]) for index in range(len(config.layers))),
        final_norm=norm("final.norm"),
        head=PartSpec("linear_head", {"hidden_size": hidden, "vocab_size": config.vocab, "name": "head"}, ""),
        eos_token_ids=config.eos_token_ids,
    )


register_architecture("Bimolix", BimolixConfig, build_spec)
