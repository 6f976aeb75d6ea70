"""Bimolix without a GPU: its typed configuration, the registry, the tensors its parts declare, distance buckets, a random
model folder through the command line, and the plain implementation's mechanisms against closed forms worked out by hand."""
import copy
import json
import math

import pytest
import torch

import bimolix_configs as configs
import plain_bimolix as plain


def test_the_configuration_round_trips_and_is_chosen_by_its_name():
    from kidi_b200.config.bimolix import BimolixConfig
    from kidi_b200.registry import registered_architectures, resolve_architecture
    assert "Bimolix" in registered_architectures()
    for config in configs.ALL.values():
        assert resolve_architecture(config).config_type is BimolixConfig
        typed = BimolixConfig.from_dict(config)
        assert typed.to_dict() == config
        assert BimolixConfig.from_dict(typed.to_dict()) == typed
    typed = BimolixConfig.from_dict(configs.SMALL_A)
    first, second, third, fourth = typed.layers[:4]
    assert (first.mixer.kind, first.mixer.rot_dims, first.mlp.ff, first.mlp.experts) == ("retention", 8, 48, None)
    assert (second.mixer.kv_heads, second.mixer.chunk, second.mixer.bias_max, second.mlp.groups, second.mlp.keep_groups) == (2, 40, 30, 3, 2)
    assert (second.mlp.router_scale, second.mlp.shared_ff, second.mlp.shared_limit, second.mlp.limit) == (2.0, 40, 1.5, 2.0)
    assert third.mlp is None and fourth.mixer.decay == (0.0, 1.0) and fourth.mlp.shared_ff is None and fourth.mlp.groups == 1
    assert [typed.owner(index) for index in range(8)] == [0, 1, 2, 3, 1, 0, 0, 7]
    bare = copy.deepcopy(configs.ODD)
    del bare["layers"][0]["mlp"]["router"]["scale"]
    assert BimolixConfig.from_dict(bare) == BimolixConfig.from_dict(configs.ODD)       # a scale of one
    assert BimolixConfig.from_dict(configs.WIDE).layers[7].mixer.chunk is None


@pytest.mark.parametrize("change,message", [
    (lambda c: c.pop("norm"), "norm"),
    (lambda c: c["norm"].pop("eps"), "eps"),
    (lambda c: c.pop("width"), "width"),
    (lambda c: c.update(vocab="many"), "vocab"),
    (lambda c: c["layers"][0].update(type="serial"), "not supported"),
    (lambda c: c["layers"][0].pop("mixer"), "mixer"),
    (lambda c: c["layers"][0]["mixer"].pop("rot"), "rot"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=3), "rot.dims"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=10), "rot.dims"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(base=0.0), "rot.base"),
    (lambda c: c["layers"][0]["mixer"].update(decay=[0.5, 0.5]), "decay"),
    (lambda c: c["layers"][0]["mixer"].update(decay=[0.5, 0.5, 1.5]), "decay"),
    (lambda c: c["layers"][1]["mixer"].update(vdim=24), "vdim"),
    (lambda c: c["layers"][1]["mixer"].update(heads=3), "multiple"),
    (lambda c: c["layers"][1]["mixer"].pop("bias_max"), "bias_max"),
    (lambda c: c["layers"][1]["mixer"]["mask"].update(size=0), "mask.size"),
    (lambda c: c["layers"][0]["mlp"].update(kind="sparse"), "not supported"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=7), "router.top"),
    (lambda c: c["layers"][1]["mlp"]["router"]["groups"].update(count=4), "router.groups"),
    (lambda c: c["layers"][1]["mlp"]["router"]["groups"].update(keep=4), "router.groups"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=5), "kept groups"),
    (lambda c: c["layers"][1]["mlp"].pop("expert"), "expert"),
    (lambda c: c["layers"][1]["mlp"]["expert"].pop("limit"), "limit"),
    (lambda c: c["layers"][1]["mlp"]["shared"].update(limit=0.0), "limit"),
    (lambda c: c["layers"][1]["mlp"]["shared"].update(ff=0), "widths"),
    (lambda c: c["layers"][4].update(weights_of=4), "weights_of"),
    (lambda c: c["layers"][4].update(weights_of=9), "weights_of"),
    (lambda c: c["layers"][4].update(weights_of=2), "described as"),
])
def test_refused_configurations(change, message):
    from kidi_b200.config.bimolix import BimolixConfig
    from kidi_b200.errors import KidiError
    config = copy.deepcopy(configs.SMALL_A)
    change(config)
    with pytest.raises(KidiError) as caught:
        BimolixConfig.from_dict(config)
    assert message in str(caught.value)


def test_declared_tensors_are_the_checkpoint_names():
    from kidi_b200.engine.model import declared_parameters
    from kidi_b200.registry import spec_from_config
    for config in configs.ALL.values():
        _, _, spec = spec_from_config(config)
        declared = {}
        for prefix, parameter in declared_parameters(spec):
            for name, shape in (parameter.sources or ((parameter.name, parameter.shape),)):
                declared[prefix + name] = tuple(shape)
            if parameter.open_axes:
                assert parameter.name == "rel" and parameter.open_axes == (0,)
        given = {name: tuple(tensor.shape) for name, tensor in configs.tensors(config, 1).items()}
        assert declared.keys() == given.keys()
        for name, shape in given.items():             # the number of buckets is the checkpoint's choice
            assert declared[name][1:] == shape[1:] and (name.endswith(".rel") or declared[name] == shape)
        assert len(spec.layers) == sum("weights_of" not in layer for layer in config["layers"])
        assert len(spec.schedule) == len(config["layers"])


def test_an_open_axis_takes_what_the_checkpoint_holds():
    from kidi_b200.errors import KidiError
    from kidi_b200.parts.spec import ParamSpec
    from kidi_b200.weights.loader import TensorDict, bind_parameters
    bind = lambda shape: bind_parameters([("", ParamSpec("rel", (32, 6), open_axes=(0,)))], TensorDict({"rel": torch.zeros(shape)}),
                                         engine_dtype=torch.float32, device=torch.device("cpu"))
    assert bind((7, 6))["rel"].shape == (7, 6)
    for shape in ((7, 5), (0, 6), (32, 6, 1)):
        with pytest.raises(KidiError, match="rel"):
            bind(shape)


def test_what_the_cache_is_asked_for():
    """One row a token and key/value head (no values), of a chunk's length at most, and a 32-bit state per head; a layer that
    runs with another's tensors asks for its own."""
    from kidi_b200.cache.sequence_cache import KVRequest, SequenceCache, StateRequest
    from kidi_b200.engine.model import CausalLM
    from kidi_b200.registry import spec_from_config
    model = CausalLM(spec_from_config(configs.SMALL_A)[2], torch.bfloat16, torch.device("cpu"))
    requests = model.cache_requests()
    assert len(requests) == 8 and requests[0] == [StateRequest((3, 8, 12), torch.float32)] == requests[5] == requests[6]
    assert requests[1] == [KVRequest(2, 16, 40, value_dim=0)] == requests[4]
    wide = CausalLM(spec_from_config(configs.WIDE)[2], torch.bfloat16, torch.device("cpu"))
    assert wide.cache_requests()[7] == [KVRequest(1, 32, None, value_dim=0)]
    cache = SequenceCache(requests, max_tokens=256, max_positions=700, dtype=torch.bfloat16, device=torch.device("cpu"))
    views = [cache.views(entry)[0] for entry in (1, 4)]
    assert views[0].keys.data_ptr() != views[1].keys.data_ptr() and views[0].values.shape[-1] == 0
    states = [cache.views(entry)[0] for entry in (0, 5, 6)]
    assert len({state.data_ptr() for state in states}) == 3


@pytest.mark.parametrize("buckets,reach", [(32, 120), (32, 128), (8, 256), (2, 9), (3, 50), (40, 21), (16, 4096), (1, 5)])
def test_distance_buckets(buckets, reach):
    """Against the definition in exact arithmetic: floor(ln(n / h) / ln(r / h) (B - h)) >= m as (n / h)^(B - h) >= (r / h)^m
    in whole numbers, so that exact powers fall where they belong."""
    from kidi_b200.parts.position import distance_buckets
    half, count = buckets // 2, min(2 * reach + 3, 2000)
    got = distance_buckets(count, buckets, reach).tolist()

    def exact(n):
        if n < half or half == 0:
            return min(n, buckets - 1) if half else 0
        rest, m = buckets - half, 0
        # (n / half)^rest >= (reach / half)^m, i.e. n^rest half^m >= reach^m half^rest
        while half + m < buckets - 1 and n ** rest * half ** (m + 1) >= reach ** (m + 1) * half ** rest:
            m += 1
        return half + m

    assert got == [exact(n) for n in range(count)]
    if half:
        assert got == [plain.distance_bucket(n, buckets, reach) for n in range(count)]
        # a reach within the first half: what lies beyond that half has the last bucket
        assert distance_buckets(half + 5, buckets, half).tolist() == list(range(half)) + [buckets - 1] * 5


def test_a_random_model_folder_through_the_command_line(tmp_path, capsys):
    import kidi_b200
    from kidi_b200.weights.loader import Checkpoint
    (tmp_path / "config.json").write_text(json.dumps(configs.SMALL_A))
    assert kidi_b200.main(["random-model", "--config", str(tmp_path / "config.json"), "-o", str(tmp_path / "model"),
                           "--seed", "3"]) == 0, capsys.readouterr().err
    held = Checkpoint(str(tmp_path / "model"))
    assert held.shape("l1.mlp.e5.down") == (64, 24) and held.shape("l1.mlp.shared.sg") == (1, 64)
    assert held.shape("l1.mix.q.norm") == (16,) and held.shape("l1.mix.k.b") == (32,) and held.shape("l1.mix.rel") == (32, 4)
    assert held.shape("l1.mlp.correction") == (6,) and "l2.norm2" not in held and held.shape("head") == (97, 64)
    assert "l4.norm1" not in held and "l1.mix.v" not in held and held.shape("l3.mix.v") == (16, 64)
    held.close()
    assert kidi_b200.main(["inspect", "-m", str(tmp_path / "model")]) == 0
    shown = capsys.readouterr().out
    assert "Bimolix" in shown and "layers: 5 (run order: 8 entries)" in shown


# ------------------------------------------------------------------ the plain mechanisms against closed forms
def test_the_plain_norm_adds_one_to_its_weight():
    x = torch.tensor([[3.0, -1.0]], dtype=torch.float64)                  # mean square 5
    want = torch.tensor([[3.0 / 3.0 * 1.5, -1.0 / 3.0 * 0.0]], dtype=torch.float64)
    assert torch.allclose(plain.stream_norm(x, torch.tensor([0.5, -1.0]), 4.0), want)


def test_the_plain_rotation():
    """Pairs are half the rotated width apart; position 0 stays; entries behind the rotated ones stay; a turn by base^0 = 1
    radian a position for the first pair, base^(-1/2) for the second of two."""
    x = torch.tensor([1.0, 0.0, 0.0, 2.0, 9.0], dtype=torch.float64).repeat(3, 1, 1)
    got = plain.rotate(x, 4, 100.0)
    assert torch.equal(got[0], x[0]) and torch.equal(got[:, 0, 4], x[:, 0, 4])
    for p in (1, 2):
        want = [math.cos(p), -2.0 * math.sin(0.1 * p), math.sin(p), 2.0 * math.cos(0.1 * p)]
        assert torch.allclose(got[p, 0, :4], torch.tensor(want, dtype=torch.float64))
    assert torch.allclose(plain.rotate(x, 4, 100.0, first=7)[0, 0, 0], torch.tensor(math.cos(7.0), dtype=torch.float64))


def test_the_plain_recurrence_forgets_by_its_decay():
    one = torch.ones(3, 1, 1, dtype=torch.float64)
    v = torch.tensor([1.0, 10.0, 100.0], dtype=torch.float64).reshape(3, 1, 1)
    assert plain.fixed_decay_recurrence(one, one, v, [0.5]).flatten().tolist() == [1.0, 10.5, 105.25]
    assert plain.fixed_decay_recurrence(one, one, v, [0.0]).flatten().tolist() == [1.0, 10.0, 100.0]


def test_the_plain_chunks_sink_and_distance_bias():
    seen = plain.same_chunk(7, 3)
    assert [row.nonzero().flatten().tolist() for row in seen] == [[0], [0, 1], [0, 1, 2], [3], [3, 4], [3, 4, 5], [6]]
    weights = plain.softmax_with_one(torch.tensor([[math.log(2.0), math.log(3.0), 50.0]], dtype=torch.float64),
                                     torch.tensor([[True, True, False]]))
    assert torch.allclose(weights, torch.tensor([[2.0 / 6.0, 3.0 / 6.0, 0.0]], dtype=torch.float64))
    low = plain.softmax_with_one(torch.full((1, 1), -800.0, dtype=torch.float64), torch.ones(1, 1, dtype=torch.bool))
    assert float(low) == 0.0                                                # the one takes nearly everything
    # eight buckets that reach 64: four distances by themselves, then 4 ln(n / 4) / ln(16) rounded down: 4-7, 8-15, 16-31, 32-
    assert [plain.distance_bucket(n, 8, 64) for n in (0, 3, 4, 7, 8, 15, 16, 31, 32, 63, 64, 900)] == \
        [0, 3, 4, 4, 5, 5, 6, 6, 7, 7, 7, 7]
    table = torch.arange(16, dtype=torch.float64).reshape(8, 2)
    bias = plain.distance_bias(10, table, 64)
    assert bias[1, 9, 1].item() == 11.0 and bias[0, 9, 9].item() == 0.0 and bias[1, 5, 3].item() == 5.0


def test_the_plain_router_ranks_groups_by_two_and_weighs_without_the_correction():
    # groups (0, 1), (2, 3), (4, 5): one best expert alone does not carry its group
    choice = torch.tensor([0.9, -2.0, 0.5, 0.4, 0.3, 0.2], dtype=torch.float64)
    assert sorted(plain.router_choice(choice, 2, 3, 1).tolist()) == [2, 3]
    assert sorted(plain.router_choice(choice, 3, 3, 2).tolist()) == [2, 3, 4]
    assert sorted(plain.router_choice(-choice - 1.0, 3, 3, 2).tolist()) == [1, 4, 5]    # negative scores: closed is not zero
    assert sorted(plain.router_choice(choice, 2, 6, 2).tolist()) == [0, 2]              # groups of one
    eye = torch.eye(2, dtype=torch.float64)
    w = {"router": torch.tensor([[1.0, 0.0], [0.0, 1.0], [1.0, 1.0]], dtype=torch.float64),
         "correction": torch.tensor([0.0, 5.0, 0.0], dtype=torch.float64)}
    for e in range(3):
        w.update({f"e{e}.gate": eye, f"e{e}.up": eye, f"e{e}.down": (e + 1.0) * eye})
    h = torch.tensor([[0.4, -3.0]], dtype=torch.float64)
    mlp = {"expert": {"limit": 1.0}, "router": {"experts": 3, "top": 2, "scale": 2.0}}
    s = torch.sigmoid(torch.tensor([0.4, -3.0, -2.6], dtype=torch.float64))             # expert 1 by its correction, then 0
    y = torch.tensor([0.4 * torch.sigmoid(torch.tensor(1.702 * 0.4)) * 1.4, 0.0], dtype=torch.float64)   # -3: u = -1
    weights = s[[1, 0]] / s[[1, 0]].sum() * 2.0
    assert torch.allclose(plain.routed(h, w, "", mlp)[0], weights[0] * 2.0 * y + weights[1] * y, atol=1e-7)
    # a gate above the limit is held, one below minus the limit is not
    out = plain.bounded_expert(torch.tensor([[3.0, -3.0]], dtype=torch.float64), {"gate": eye, "up": -eye, "down": eye}, "", 1.0)
    sig = lambda z: 1.0 / (1.0 + math.exp(-z))
    assert torch.allclose(out, torch.tensor([[0.0, -3.0 * sig(-5.106) * 2.0]], dtype=torch.float64))
