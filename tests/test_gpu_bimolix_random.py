"""Random Bimolix configurations (sizes that are no round numbers, one to twenty heads a key/value head, head widths with and
without the tensor-core kernels' multiples of 16, chunks from 1 to 300 tokens or none, any number of distance buckets, retention
of any widths with any even part of a head rotated, decays from 0 to 1, dense, routed and absent feed-forwards with one expert
a token to all of them in any equal groups, limits of any size, shared experts or none, layers that run with another layer's
tensors) through the engine in both precisions against the plain implementation: a prompt in two portions, then eight tokens
decoded one by one. Two of the draws run prompts of more than 1,024 tokens, so that the products of prompts take their
tensor-memory kernel at these sizes."""
import numpy as np
import pytest
import torch

import bimolix_configs as configs
import plain_bimolix

pytestmark = pytest.mark.gpu

DRAWS = 14


def draw(seed):
    rng = np.random.default_rng(8300 + seed)
    pick = lambda values: int(rng.choice(values))
    width = pick([n for n in range(40, 220) if n % 8 == 0 or rng.random() < 0.05])

    def feed_forward():
        kind = rng.random()
        if kind < 0.15:
            return None
        if kind < 0.45:
            return configs.dense(pick([24, 40, 100, 160]))
        groups = pick([1, 1, 2, 3, 4])
        experts = groups * pick([1, 2, 3, 4])
        keep = pick(range(1, groups + 1))
        top = pick(range(1, min(8, keep * (experts // groups)) + 1))
        return configs.routed(experts, top, pick([8, 24, 40, 64]), limit=float(rng.choice([0.4, 1.0, 7.0])),
                              scale=float(rng.choice([0.5, 1.0, 2.5])), groups=(groups, keep) if (groups, keep) != (1, 1) else None,
                              shared=pick([8, 24, 40, 72]) if rng.random() < 0.6 else None, shared_limit=float(rng.choice([0.3, 2.0])))

    layers = []
    for index in range(pick([2, 3, 4, 5, 6])):
        if layers and rng.random() < 0.25:
            layers.append(configs.again(layers, pick([i for i, layer in enumerate(layers) if "weights_of" not in layer])))
            continue
        if rng.random() < 0.5:
            kv_heads = pick([1, 1, 2, 3])
            dim = pick([16, 32, 48, 64, 128]) if rng.random() < 0.7 else pick([4, 6, 10, 20, 24, 40])
            mixer = configs.attention(kv_heads * pick([1, 2, 3, 4, 12, 20]), kv_heads, dim, float(rng.uniform(0.5, 1.5)) * dim ** -0.5,
                                      pick([33, 64, 120, 500]), chunk=pick([1, 3, 17, 63, 64, 65, 100, 128, 300]) if rng.random() < 0.8 else None)
        else:
            heads = pick([2, 3, 5, 8])
            pairs = [(16, 16), (16, 48), (32, 64), (48, 16), (64, 64), (80, 32)]       # the chunked form's, and others
            dim, vdim = pairs[pick(range(6))] if rng.random() < 0.6 else (pick([8, 12, 20, 33]), pick([8, 12, 33]))
            mixer = configs.retention(heads, dim, vdim, rot=2 * pick(range(0, dim // 2 + 1)), base=float(rng.choice([100.0, 1e4, 1e6])),
                                      decay=[float(x) for x in rng.choice([0.0, 0.4, 0.8, 0.95, 0.99, 0.999, 1.0], size=heads)])
        layers.append(configs.layer(mixer, feed_forward()))
    return configs.model(pick(range(61, 400)), width, float(rng.choice([0.02, 0.05, 0.2])), layers, positions=1536)


# In bfloat16 a router's choice between experts whose logits lie closer together than the rounding of its input may fall
# the other way, and the recurrences and attention carry the difference to every later token. The plain model therefore
# takes the engine's choice at such a token, but only if moving the logits by this much towards it makes it the plain
# model's own choice; any other difference of choices stays a difference of logits.
CLOSE_CALL = 0.12


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("seed", range(DRAWS))
def test_random_configuration(seed, dtype, record_property, monkeypatch):
    from kidi_b200 import Engine, StepBatch
    from kidi_b200.kernels import routed
    config = draw(seed)
    tensors = configs.tensors(config, 50 + seed)
    length = 1100 if seed in (2, 5) else 60 + 31 * seed
    tokens = np.random.default_rng(seed).integers(0, config["vocab"], size=length + 8).tolist()
    calls, route = [], routed.route

    def recorded(x, *args, **kwargs):
        chosen, weight = route(x, *args, **kwargs)
        calls.append(chosen.clone())
        return chosen, weight

    monkeypatch.setattr(routed, "route", recorded)
    engine = Engine.from_config(config, tensors=tensors, dtype=dtype, max_tokens=4096)
    slot = engine.acquire()
    cut = length // 3
    rows = [engine.step(StepBatch([slot], [tokens[:cut]], [list(range(cut))])).double().cpu(),
            engine.step(StepBatch([slot], [tokens[cut:length]], [list(range(length - cut))])).double().cpu()]
    rows += [engine.step(StepBatch([slot], [[token]], None)).double().cpu() for token in tokens[length:]]
    engine.release(slot)
    engine.check_device_errors()
    got = torch.cat(rows)
    assert torch.isfinite(got).all()
    choices = None
    if dtype == "bfloat16":
        runs = sum((layer["mlp"] or {}).get("kind") == "moe" for layer in config["layers"])
        assert len(calls) == runs * len(rows)
        choices = [torch.cat([calls[step * runs + run].cpu() for step in range(len(rows))]) for run in range(runs)]
    want = plain_bimolix.forward(config, tensors, tokens, dtype=torch.float64, choices=choices, margin=CLOSE_CALL)
    largest = float((got - want).abs().max() / want.abs().max())
    mean = float((got - want).pow(2).mean().sqrt() / want.pow(2).mean().sqrt())
    record_property("largest and mean relative difference", (largest, mean))
    assert largest < (4e-5 if dtype == "float32" else 0.15) and mean < (1e-5 if dtype == "float32" else 0.04), \
        (config, largest, mean)
