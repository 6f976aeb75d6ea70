"""Small Dibesun configurations and random weights for them, made by the tests themselves.

The configurations differ in every size and constant: one to twelve query heads a key/value head, key and value widths
that are equal, smaller and larger than one another, chunks shorter and longer than a cache page, of exactly a page, of
one position and none, bounded scores and scores as they are, linear attention with more and fewer heads than the
attention beside it, decays from 0 to 1, dense feed-forwards, routed ones with and without a shared expert and none, norms
in one to five parts, shares of any size and sign, widths that are no multiples of 8 (or of 4).
(A first token's read-out is (q . k) v divided by the size of all heads together: with a single head and q . k near zero
rounding decides its sign. Layers of few small heads therefore do not stand before a router here.)
`tensors(config, seed)` draws every tensor under its checkpoint name.
"""
import torch


def attention(heads, kv_heads, dim, vdim, scale, chunk=None, softcap=None):
    mixer = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if chunk is not None:
        mixer["mask"] = {"size": chunk}
    if softcap is not None:
        mixer["softcap"] = softcap
    return mixer


def linear(heads, dim, vdim, decay=None):
    return {"heads": heads, "dim": dim, "vdim": vdim,
            "decay": list(decay) if decay else [1.0 - 2.0 ** (-1.0 - 1.5 * index) for index in range(heads)]}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def routed(experts, top, ff, shared=None):
    mlp = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared is not None:
        mlp["shared"] = {"ff": shared}
    return mlp


def layer(left, right, mlp=None, left_scale=0.7, right_scale=0.9):
    return {"type": "parallel", "mixer": {"left": left, "right": right, "left_scale": left_scale,
                                          "right_scale": right_scale}, "mlp": mlp}


def model(vocab, width, eps, groups, embedding, layers, positions=None):
    config = {"architecture": "Dibesun", "vocab": vocab, "width": width, "norm": {"eps": eps, "groups": groups},
              "embedding": {"scale": embedding}, "layers": layers}
    if positions is not None:
        config["max_positions"] = positions
    return config


# every kind of feed-forward; values wider and narrower than keys; chunks shorter than a page, of a page and longer
SMALL_A = model(97, 64, 1e-5, 4, 3.0, [
    layer(attention(4, 2, 16, 24, 0.3, chunk=40, softcap=20.0), linear(3, 8, 12), dense(48)),
    layer(attention(6, 1, 8, 8, 0.4, chunk=64, softcap=6.0), linear(2, 16, 16, (0.0, 1.0)), routed(6, 2, 24, shared=40),
          left_scale=1.0, right_scale=-0.5),
    layer(attention(2, 2, 24, 8, 0.25, chunk=150), linear(4, 12, 20), None, left_scale=1.3, right_scale=1.0),
    layer(attention(3, 3, 16, 16, 0.2, softcap=9.0), linear(1, 20, 8, (0.97,)), routed(5, 3, 16), right_scale=0.4),
], positions=700)

# one part, no scale on the embedding to speak of; chunks of one position and of three; as many experts a token as there
# are; widths that no kernel takes in pieces of several elements
ODD = model(71, 50, 3e-6, 1, 1.0, [
    layer(attention(2, 1, 10, 6, 0.3, chunk=1, softcap=12.0), linear(3, 7, 5), routed(4, 4, 22, shared=18)),
    layer(attention(3, 1, 6, 10, 0.3, chunk=3), linear(2, 5, 9, (0.5, 0.9375)), dense(30), left_scale=0.9),
    layer(attention(5, 5, 4, 4, 0.5, chunk=45, softcap=4.0), linear(4, 6, 6), routed(3, 2, 12)),
], positions=600)

# widths that the tensor-core kernels take: heads of 64 and 128 in groups of 1, 2 and 4, of 48 in a group of 3, a group of
# twelve heads (decoding's wider form), linear attention with heads that the chunked form takes and with heads that it
# does not; chunks whose edge falls inside a tile
WIDE = model(211, 240, 1e-5, 5, 4.0, [
    layer(attention(8, 2, 64, 64, 0.15, chunk=150, softcap=25.0), linear(4, 32, 64), dense(256)),
    layer(attention(2, 1, 128, 128, 0.1, chunk=200, softcap=30.0), linear(2, 128, 128), routed(8, 2, 64, shared=96)),
    layer(attention(3, 1, 48, 48, 0.15, chunk=100), linear(3, 48, 16), routed(6, 2, 72)),
    layer(attention(12, 1, 32, 32, 0.2, softcap=15.0), linear(2, 24, 40), dense(128)),
    layer(attention(4, 4, 64, 64, 0.15), linear(5, 16, 48), None),
], positions=1400)

ALL = {"small_a": SMALL_A, "odd": ODD, "wide": WIDE}


def single(one, vocab=67, width=48, eps=1e-5, groups=3, embedding=2.0, positions=900):
    """A model of one layer (a mechanism alone)."""
    return model(vocab, width, eps, groups, embedding, [one], positions=positions)


def tensors(config, seed, logits=4.0, sharp=1.0):
    """Every tensor of a model of `config`, bfloat16, under its checkpoint name. `logits` is about the standard
    deviation of the logits; `sharp` multiplies the weights of the query norms (sharper scores)."""
    generator = torch.Generator().manual_seed(seed)
    width, vocab = config["width"], config["vocab"]

    def normal(*shape, std=1.0, mean=0.0):
        return (torch.randn(*shape, generator=generator) * std + mean).to(torch.bfloat16)

    def matrix(out, inner, gain=1.0):
        return normal(out, inner, std=gain / inner ** 0.5)

    def expert(p, ff):
        out[p + "gate"], out[p + "up"], out[p + "down"] = matrix(ff, width, 1.0), matrix(ff, width, 1.0), matrix(width, ff)

    # the table is also the head: rows of the length that gives logits of the asked size; the embedding scale restores
    # about 1 for the stream
    out = {"embed": normal(vocab, width, std=logits / width ** 0.5), "final.norm": normal(width, std=0.2, mean=1.0)}
    for i, one in enumerate(config["layers"]):
        p, left, right = f"l{i}.", one["mixer"]["left"], one["mixer"]["right"]
        q, r = p + "mix.left.", p + "mix.right."
        queries, keys = left["heads"] * left["dim"], left["kv_heads"] * left["dim"]
        out[q + "q"], out[q + "k"] = matrix(queries, width), matrix(keys, width)
        out[q + "v"] = matrix(left["kv_heads"] * left["vdim"], width)
        out[q + "q.norm"] = normal(queries, std=0.3 * sharp, mean=1.5 * sharp)
        out[q + "k.norm"] = normal(keys, std=0.3, mean=1.0)
        out[q + "pb"] = normal(left["heads"], std=1.0, mean=-3.0)
        out[q + "o"] = matrix(width, left["heads"] * left["vdim"])
        for name in "qk":
            out[r + name] = matrix(right["heads"] * right["dim"], width, 1.2)
        values = right["heads"] * right["vdim"]
        out[r + "v"], out[r + "g"], out[r + "o"] = matrix(values, width, 1.2), matrix(values, width, 2.0), matrix(width, values, 2.0)
        out[r + "norm"] = normal(values, std=0.2, mean=1.0)
        out[p + "norm1"] = normal(width, std=0.2, mean=1.0)
        mlp = one["mlp"]
        if mlp is None:
            continue
        out[p + "norm2"] = normal(width, std=0.2, mean=1.0)
        if mlp["kind"] == "dense":
            expert(p + "mlp.", mlp["ff"])
            continue
        router = mlp["router"]
        out[p + "mlp.router"] = matrix(router["experts"], width, 3.0)
        out[p + "mlp.router.b"] = normal(router["experts"], std=1.0)
        for e in range(router["experts"]):
            expert(f"{p}mlp.e{e}.", mlp["expert"]["ff"])
        if mlp.get("shared"):
            expert(p + "mlp.shared.", mlp["shared"]["ff"])
    return out
