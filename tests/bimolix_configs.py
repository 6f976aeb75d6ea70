"""Small Bimolix configurations and random weights for them, made by the tests themselves.

The configurations differ in every size and constant: one to twenty query heads a key/value head, head widths that the
tensor-core kernels take and that they do not, chunks shorter and longer than a cache page, of exactly a page, of one
position and none, distance buckets from 2 to 40 that reach less and further than a chunk, score scales of any size, retention
with more and fewer heads than the attention beside it, whole and partly rotated heads (and unrotated ones), values wider and
narrower than keys, decays from 0 to 1, dense and routed feed-forwards and none, groups of one expert and of many, one expert
a token to all of them, limits that bind and limits that do not, shared experts or none, layers that run with another layer's
tensors, widths that are no multiples of 8 (or of 4).
(A retention head's read-out is divided by its own size: where it nearly vanishes, as with a first token whose q . k is near
zero, or any such token of a head with a decay of 0, its sign rests on rounding. The whole models therefore have an eps that
is felt there; those of one layer have a small one.)
`tensors(config, seed)` draws every tensor under its checkpoint name.
"""
import torch


def retention(heads, dim, vdim, decay=None, rot=None, base=10000.0):
    return {"heads": heads, "dim": dim, "vdim": vdim, "rot": {"base": base, "dims": dim if rot is None else rot},
            "decay": list(decay) if decay else [1.0 - 2.0 ** (-1.0 - 1.5 * index) for index in range(heads)]}


def attention(heads, kv_heads, dim, scale, bias_max, chunk=None):
    mixer = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale, "bias_max": bias_max}
    if chunk is not None:
        mixer["mask"] = {"size": chunk}
    return mixer


def dense(ff):
    return {"kind": "dense", "ff": ff}


def routed(experts, top, ff, limit=2.0, scale=1.0, groups=None, shared=None, shared_limit=1.5):
    router = {"experts": experts, "top": top, "scale": scale}
    if groups is not None:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    mlp = {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": router}
    if shared is not None:
        mlp["shared"] = {"ff": shared, "limit": shared_limit}
    return mlp


def layer(mixer, mlp=None, weights_of=None):
    one = {"type": "retention" if "decay" in mixer else "attention", "mixer": mixer, "mlp": mlp}
    if weights_of is not None:
        one["weights_of"] = weights_of
    return one


def again(layers, index):
    """A layer that runs with the tensors of `layers[index]`."""
    return dict(layers[index], weights_of=index)


def model(vocab, width, eps, layers, positions=None):
    config = {"architecture": "Bimolix", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}
    if positions is not None:
        config["max_positions"] = positions
    return config


# every kind of layer and feed-forward; shared tensors of both mixers, one of them shared twice
_A = [layer(retention(3, 8, 12), dense(48)),
      layer(attention(4, 2, 16, 0.3, 30, chunk=40), routed(6, 2, 24, groups=(3, 2), scale=2.0, shared=40)),
      layer(attention(6, 1, 8, 0.4, 100, chunk=64), None),
      layer(retention(2, 16, 8, (0.0, 1.0), rot=6, base=300.0), routed(8, 3, 16, limit=0.7))]
SMALL_A = model(97, 64, 0.1, _A + [again(_A, 1), again(_A, 0), dict(_A[0], weights_of=5),
                                    layer(attention(2, 2, 24, 0.25, 70, chunk=150), dense(40))], positions=700)

# widths that no kernel takes in pieces of several elements; chunks of one position and of three; as many experts a token as
# there are; twenty query heads to a key/value head; heads that are not rotated
_B = [layer(attention(2, 1, 10, 0.3, 17, chunk=1), routed(4, 4, 22, shared=18, shared_limit=0.5)),
      layer(retention(3, 7, 5, rot=2), dense(30)),
      layer(attention(20, 1, 6, 0.5, 40, chunk=45), routed(3, 2, 12, groups=(3, 2))),
      layer(retention(2, 5, 9, (0.5, 0.9375), rot=0), None),
      layer(attention(3, 3, 10, 0.3, 25, chunk=3), dense(26))]
ODD = model(71, 50, 0.02, _B + [again(_B, 3)], positions=600)

# widths that the tensor-core kernels take: heads of 64 and 128 in groups of 1, 2 and 4, of 48 in a group of 3, a group of
# twelve heads (decoding's wider form), no chunks, retention with heads that the chunked form takes and with heads that it
# does not; chunks whose edge falls inside a tile
_C = [layer(retention(4, 32, 64), dense(256)),
      layer(attention(8, 2, 64, 0.15, 90, chunk=150), routed(8, 2, 64, groups=(4, 3), scale=1.7, shared=96)),
      layer(retention(2, 128, 128, (0.9, 0.999), base=1e6), routed(6, 2, 72)),
      layer(attention(2, 1, 128, 0.1, 400, chunk=200), dense(128)),
      layer(retention(3, 48, 16, rot=20), None),
      layer(attention(3, 1, 48, 0.15, 60, chunk=100), routed(12, 4, 40, groups=(2, 1), shared=64)),
      layer(retention(2, 24, 40), dense(96)),
      layer(attention(12, 1, 32, 0.2, 33), dense(128))]
WIDE = model(211, 240, 0.03, _C + [again(_C, 3), again(_C, 0)], positions=1400)

ALL = {"small_a": SMALL_A, "odd": ODD, "wide": WIDE}


def buckets(index):
    """How many distance buckets the attention layer `index` of these models has (its tensor says so, no configuration)."""
    return (32, 8, 2, 40, 16, 12, 20, 24)[index % 8]


def single(one, vocab=67, width=48, eps=1e-5, positions=900):
    """A model of one layer (a mechanism alone)."""
    return model(vocab, width, eps, [one], positions=positions)


def tensors(config, seed, logits=4.0, sharp=1.0, bias=1.5):
    """Every tensor of a model of `config`, bfloat16, under its checkpoint name. `logits` is about the standard
    deviation of the logits; `sharp` multiplies the weights of the query norms (sharper scores), `bias` is the standard
    deviation of the distance biases."""
    generator = torch.Generator().manual_seed(seed)
    width, vocab = config["width"], config["vocab"]

    def normal(*shape, std=1.0, mean=0.0):
        return (torch.randn(*shape, generator=generator) * std + mean).to(torch.bfloat16)

    def matrix(out, inner, gain=1.0):
        return normal(out, inner, std=gain / inner ** 0.5)

    def expert(p, ff):
        out[p + "gate"], out[p + "up"], out[p + "down"] = matrix(ff, width, 1.0), matrix(ff, width, 1.0), matrix(width, ff)

    out = {"embed": normal(vocab, width), "embed.norm": normal(width, std=0.2), "final.norm": normal(width, std=0.2),
           "head": matrix(vocab, width, logits)}
    for i, one in enumerate(config["layers"]):
        if one.get("weights_of") is not None:
            continue
        p, mixer, mlp = f"l{i}.", one["mixer"], one["mlp"]
        m, heads, dim = p + "mix.", mixer["heads"], mixer["dim"]
        out[p + "norm1"] = normal(width, std=0.2)
        out[m + "q"] = matrix(heads * dim, width, 1.2)
        if one["type"] == "retention":
            values = heads * mixer["vdim"]
            out[m + "k"], out[m + "v"] = matrix(heads * dim, width, 1.2), matrix(values, width, 1.2)
            out[m + "g"], out[m + "o"] = matrix(values, width, 1.5), matrix(width, values)
        else:
            keys = mixer["kv_heads"] * dim
            out[m + "k"] = matrix(keys, width)
            out[m + "q.b"], out[m + "k.b"] = normal(heads * dim, std=0.4), normal(keys, std=0.4)
            out[m + "q.norm"] = normal(dim, std=0.3 * sharp, mean=1.5 * sharp)
            out[m + "k.norm"] = normal(dim, std=0.3, mean=1.0)
            out[m + "rel"] = normal(buckets(i), heads, std=bias)
            out[m + "g"], out[m + "o"] = matrix(heads * dim, width, 1.5), matrix(width, heads * dim, 1.5)
        if mlp is None:
            continue
        out[p + "norm2"] = normal(width, std=0.2)
        if mlp["kind"] == "dense":
            expert(p + "mlp.", mlp["ff"])
            continue
        router = mlp["router"]
        out[p + "mlp.router"] = matrix(router["experts"], width, 2.0)
        out[p + "mlp.correction"] = normal(router["experts"], std=0.3)
        for e in range(router["experts"]):
            expert(f"{p}mlp.e{e}.", mlp["expert"]["ff"])
        if mlp.get("shared"):
            expert(p + "mlp.shared.", mlp["shared"]["ff"])
            out[p + "mlp.shared.sg"] = matrix(1, width, 1.5)
    return out
