"""Random Dibesun configurations (sizes that are no round numbers, one to twelve heads a key/value head, key and value
widths with and without the tensor-core kernels' multiples of 16, chunks from 1 to 300 tokens or none, bounded scores or
not, linear attention of any widths, decays from 0 to 1, dense, routed and absent feed-forwards with one expert a token to
all of them, shared experts or none, norms in any number of parts, shares of any size and sign) through the engine in both
precisions against the plain implementation: a prompt in two portions, then eight tokens decoded one by one. Two of the
draws run prompts of more than 1,024 tokens, so that the products of prompts take their tensor-memory kernel at these
sizes."""
import numpy as np
import pytest
import torch

import dibesun_configs as configs
import plain_dibesun

pytestmark = pytest.mark.gpu

DRAWS = 14


def draw(seed):
    rng = np.random.default_rng(7100 + seed)
    pick = lambda values: int(rng.choice(values))
    groups = pick([1, 1, 2, 3, 4, 6])
    width = groups * pick([n for n in range(8, 200) if 40 <= n * groups <= 220 and (n * groups % 8 == 0 or rng.random() < 0.2)])

    def feed_forward():
        kind = rng.random()
        if kind < 0.15:
            return None
        if kind < 0.45:
            return configs.dense(pick([24, 40, 100, 160]))
        experts = pick([2, 3, 4, 6, 9, 16])
        return configs.routed(experts, pick(range(1, min(8, experts) + 1)), pick([8, 24, 40, 64]),
                              shared=pick([8, 24, 40, 72]) if rng.random() < 0.6 else None)

    layers = []
    for _ in range(pick([1, 2, 3, 3, 4, 5])):
        kv_heads = pick([1, 1, 2, 3])
        if rng.random() < 0.6:
            dim = pick([16, 32, 48, 64, 128])
            vdim = dim if rng.random() < 0.7 else pick([16, 32, 64])
        else:
            dim, vdim = pick([4, 6, 10, 20, 24, 40]), pick([4, 8, 12, 24, 36])
        left = configs.attention(kv_heads * pick([1, 2, 3, 4, 12]), kv_heads, dim, vdim, float(rng.uniform(0.5, 1.5)) * dim ** -0.5,
                                 chunk=pick([1, 3, 17, 63, 64, 65, 100, 128, 300]) if rng.random() < 0.8 else None,
                                 softcap=float(rng.choice([3.0, 10.0, 30.0, 50.0])) if rng.random() < 0.8 else None)
        heads = pick([1, 2, 3, 5, 8])
        right = configs.linear(heads, *((pick([16, 32, 48, 64]), pick([16, 32, 48, 80])) if rng.random() < 0.6
                                        else (pick([4, 7, 12, 20]), pick([5, 8, 12, 33]))),
                               decay=[float(x) for x in rng.choice([0.0, 0.4, 0.8, 0.95, 0.99, 0.999, 1.0], size=heads)])
        layers.append(configs.layer(left, right, feed_forward(), left_scale=float(rng.uniform(0.3, 1.5)),
                                    right_scale=float(rng.choice([-0.7, 0.4, 1.0, 1.3]))))
    return configs.model(pick(range(61, 400)), width, float(rng.choice([1e-6, 1e-5, 3e-5])), groups,
                         float(rng.choice([1.0, 2.0, 5.5])), layers, positions=1536)


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
    want = plain_dibesun.forward(config, tensors, tokens, dtype=torch.float64, choices=choices, margin=CLOSE_CALL)
    largest = float((got - want).abs().max() / want.abs().max())
    mean = float((got - want).pow(2).mean().sqrt() / want.pow(2).mean().sqrt())
    record_property("largest and mean relative difference", (largest, mean))
    assert largest < (4e-5 if dtype == "float32" else 0.15) and mean < (1e-5 if dtype == "float32" else 0.04), \
        (config, largest, mean)
