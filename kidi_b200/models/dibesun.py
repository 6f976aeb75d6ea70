"""Dibesun as a `ModelSpec`.

A decoder-only stack: token embeddings times a number; every layer adds to the stream the normed result of a mixer and,
where it has one, of a feed-forward, both of which read the stream itself (the `output_norm` arrangement; the norms are
RMS norms in equal parts); a final norm of the same kind and the embedding table as head. A mixer is two side by side on
one input, added with a weight each:

* left: grouped-query attention without rotation over runs of positions (a query sees the earlier keys of its own run),
  queries and keys RMS-normed over their whole projections, bounded scores, and the sigmoid of score plus a number per
  head as a key's weight, normalised over nothing;
* right: linear attention with one fixed decay per head, SiLU on q, k and v, a norm over all heads and a sigmoid gate.

A feed-forward is a dense SiLU-gated one or routed SiLU-gated experts (a router with a bias, a softmax over the chosen
logits) with an optional shared expert.

Tensor names: `embed`, `final.norm`, and per layer `l<i>.norm1`, `l<i>.norm2`,
`l<i>.mix.left.{q,k,v,o,q.norm,k.norm,pb}`, `l<i>.mix.right.{q,k,v,g,o,norm}`, `l<i>.mlp.{gate,up,down}` or
`l<i>.mlp.{router,router.b}`, `l<i>.mlp.{e<j>,shared}.{gate,up,down}`.

This file maps a `DibesunConfig` to parts and their parameters; nothing here computes.
"""
from __future__ import annotations

from ..config.dibesun import DibesunConfig
from ..parts.spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry
from ..registry import register_architecture


def build_spec(config: DibesunConfig) -> ModelSpec:
    hidden, eps = config.width, config.norm_eps
    norm = lambda name, prefix="": PartSpec("rms_norm", {"size": hidden, "eps": eps, "groups": config.norm_groups,
                                                         "weight_name": name}, prefix)
    layers = []
    for index, layer in enumerate(config.layers):
        prefix = f"l{index}."
        left, right, mlp = layer.left, layer.right, layer.mlp
        attention = PartSpec("attention", {
            "hidden_size": hidden, "num_heads": left.heads, "num_kv_heads": left.kv_heads, "head_dim": left.dim,
            "value_dim": left.vdim, "scale": left.scale, "position": None, "score_softcap": left.softcap,
            "chunk": left.chunk, "weights": "sigmoid", "weight_bias_name": "pb", "qk_norm": True,
            "qk_norm_scope": "rows", "qk_norm_eps": eps, "q_norm_name": "q.norm", "k_norm_name": "k.norm",
            "q_name": "q", "k_name": "k", "v_name": "v", "o_name": "o"}, prefix + "mix.left.")
        lightning = PartSpec("lightning_attention", {
            "hidden_size": hidden, "num_heads": right.heads, "dim": right.dim, "vdim": right.vdim,
            "decay": list(right.decay), "eps": eps}, prefix + "mix.right.")
        parts = {"mixer": PartSpec("parallel_mixers", {
                     "hidden_size": hidden, "left": attention, "right": lightning, "combine": "plain",
                     "share_left": layer.left_scale, "share_right": layer.right_scale}, prefix + "mix."),
                 "mixer_out_norm": norm("norm1", prefix)}
        if mlp is not None:
            parts["feed_forward_out_norm"] = norm("norm2", prefix)
            if mlp.experts is None:
                parts["feed_forward"] = PartSpec("gated_mlp", {
                    "hidden_size": hidden, "intermediate_size": mlp.ff, "gate_name": "gate", "up_name": "up",
                    "down_name": "down"}, prefix + "mlp.")
            else:
                parts["feed_forward"] = PartSpec("routed_experts", {
                    "hidden_size": hidden, "expert_size": mlp.ff, "experts": mlp.experts, "top": mlp.top,
                    "score": "softmax", "renormalise": True, "weight_on": "output", "router_bias_name": "router.b",
                    "shared_size": mlp.shared_ff}, prefix + "mlp.")
        layers.append(LayerSpec(arrangement=PartSpec("output_norm"), parts=parts))
    return ModelSpec(
        architecture=config.architecture,
        vocab_size=config.vocab,
        hidden_size=hidden,
        max_positions=config.max_positions,
        embedding=PartSpec("token_embedding", {"vocab_size": config.vocab, "hidden_size": hidden, "name": "embed",
                                               "scale": config.embedding_scale}, ""),
        positions={},
        layers=tuple(layers),
        schedule=tuple(ScheduleEntry(index) for index in range(len(layers))),
        final_norm=norm("final.norm"),
        head=PartSpec("linear_head", {"hidden_size": hidden, "vocab_size": config.vocab, "name": "head",
                                      "tied_to": "embed"}, ""),
        eos_token_ids=config.eos_token_ids,
    )


register_architecture("Dibesun", DibesunConfig, build_spec)
