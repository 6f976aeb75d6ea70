"""Dibesun without a GPU: its typed configuration, the registry, the tensors its parts declare, a random model folder
through the command line, and the plain implementation's mechanisms against closed forms worked out by hand."""
import copy
import json
import math

import pytest
import torch

import dibesun_configs as configs
import plain_dibesun as plain


def test_the_configuration_round_trips_and_is_chosen_by_its_name():
    from kidi_b200.config.dibesun import DibesunConfig
    from kidi_b200.registry import registered_architectures, resolve_architecture
    assert "Dibesun" in registered_architectures()
    for config in configs.ALL.values():
        assert resolve_architecture(config).config_type is DibesunConfig
        typed = DibesunConfig.from_dict(config)
        assert typed.to_dict() == config
        assert DibesunConfig.from_dict(typed.to_dict()) == typed
    typed = DibesunConfig.from_dict(configs.SMALL_A)
    first, second, third = typed.layers[:3]
    assert (first.left.heads, first.left.kv_heads, first.left.dim, first.left.vdim, first.left.chunk) == (4, 2, 16, 24, 40)
    assert (first.mlp.ff, first.mlp.experts) == (48, None)
    assert (second.right_scale, second.right.decay, second.mlp.top, second.mlp.shared_ff) == (-0.5, (0.0, 1.0), 2, 40)
    assert third.left.softcap is None and third.mlp is None
    assert typed.layers[3].left.chunk is None and typed.layers[3].mlp.shared_ff is None
    assert (typed.norm_groups, typed.embedding_scale) == (4, 3.0)
    bare = copy.deepcopy(configs.ODD)
    del bare["embedding"], bare["norm"]["groups"]
    assert DibesunConfig.from_dict(bare) == DibesunConfig.from_dict(configs.ODD)       # one part, a scale of one


@pytest.mark.parametrize("change,message", [
    (lambda c: c.pop("norm"), "norm"),
    (lambda c: c["norm"].pop("eps"), "eps"),
    (lambda c: c["norm"].update(groups=3), "norm.groups"),
    (lambda c: c.pop("width"), "width"),
    (lambda c: c.update(vocab="many"), "vocab"),
    (lambda c: c["layers"][0].update(type="serial"), "not supported"),
    (lambda c: c["layers"][0]["mixer"].pop("left"), "left"),
    (lambda c: c["layers"][0]["mixer"].pop("right_scale"), "right_scale"),
    (lambda c: c["layers"][0]["mixer"]["left"].pop("vdim"), "vdim"),
    (lambda c: c["layers"][0]["mixer"]["left"].update(heads=3), "multiple"),
    (lambda c: c["layers"][0]["mixer"]["left"]["mask"].update(size=0), "mask.size"),
    (lambda c: c["layers"][0]["mixer"]["left"].update(softcap=-1.0), "softcap"),
    (lambda c: c["layers"][0]["mixer"]["right"].pop("decay"), "decay"),
    (lambda c: c["layers"][0]["mixer"]["right"].update(decay=[0.5, 0.5]), "decay"),
    (lambda c: c["layers"][0]["mixer"]["right"].update(decay=[0.5, 0.5, 1.5]), "decay"),
    (lambda c: c["layers"][0]["mlp"].update(kind="sparse"), "not supported"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=7), "router.top"),
    (lambda c: c["layers"][1]["mlp"].pop("expert"), "expert"),
    (lambda c: c["layers"][1]["mlp"]["shared"].update(ff=0), "widths"),
])
def test_refused_configurations(change, message):
    from kidi_b200.config.dibesun import DibesunConfig
    from kidi_b200.errors import KidiError
    config = copy.deepcopy(configs.SMALL_A)
    change(config)
    with pytest.raises(KidiError) as caught:
        DibesunConfig.from_dict(config)
    assert message in str(caught.value)


def test_declared_tensors_are_the_checkpoint_names():
    from kidi_b200.engine.model import declared_parameters
    from kidi_b200.registry import spec_from_config
    for config in configs.ALL.values():
        _, _, spec = spec_from_config(config)
        declared, tied = {}, []
        for prefix, parameter in declared_parameters(spec):
            if parameter.alias_of is not None:
                tied.append((prefix + parameter.name, parameter.alias_of))
                continue
            for name, shape in (parameter.sources or ((parameter.name, parameter.shape),)):
                declared[prefix + name] = tuple(shape)
        assert declared == {name: tuple(tensor.shape) for name, tensor in configs.tensors(config, 1).items()}
        assert tied == [("head", "embed")]                       # the head is the embedding table
    assert "feed_forward" not in spec_from_config(configs.SMALL_A)[2].layers[2].parts


def test_what_the_cache_is_asked_for():
    """Keys and values of a chunk's length at most, and a 32-bit state per head."""
    from kidi_b200.cache.sequence_cache import KVRequest, StateRequest
    from kidi_b200.engine.model import CausalLM
    from kidi_b200.registry import spec_from_config
    model = CausalLM(spec_from_config(configs.SMALL_A)[2], torch.bfloat16, torch.device("cpu"))
    assert model.cache_requests()[0] == [KVRequest(2, 16, 40, value_dim=24), StateRequest((3, 8, 12), torch.float32)]
    assert model.cache_requests()[3] == [KVRequest(3, 16, None), StateRequest((1, 20, 8), torch.float32)]


def test_a_random_model_folder_through_the_command_line(tmp_path, capsys):
    import kidi_b200
    from kidi_b200.weights.loader import Checkpoint
    (tmp_path / "config.json").write_text(json.dumps(configs.SMALL_A))
    assert kidi_b200.main(["random-model", "--config", str(tmp_path / "config.json"), "-o", str(tmp_path / "model"),
                           "--seed", "3"]) == 0, capsys.readouterr().err
    held = Checkpoint(str(tmp_path / "model"))
    assert held.shape("l1.mlp.e5.down") == (64, 24) and held.shape("l1.mlp.shared.up") == (40, 64)
    assert held.shape("l0.mix.left.q.norm") == (64,) and held.shape("l0.mix.left.pb") == (4,)
    assert held.shape("l1.mlp.router.b") == (6,) and "l2.norm2" not in held and "head" not in held
    held.close()
    assert kidi_b200.main(["inspect", "-m", str(tmp_path / "model")]) == 0
    assert "Dibesun" in capsys.readouterr().out


# ------------------------------------------------------------------ the plain mechanisms against closed forms
def test_the_plain_norm_in_parts():
    x = torch.tensor([[3.0, 4.0, 0.0, 2.0]], dtype=torch.float64)
    weight = torch.tensor([1.0, 2.0, 0.5, -1.0], dtype=torch.float64)
    # mean squares of the parts: 12.5 and 2
    want = torch.tensor([[3.0 / 4.0, 2.0 * 4.0 / 4.0, 0.0, -2.0 / math.sqrt(5.5)]], dtype=torch.float64)
    assert torch.allclose(plain.grouped_rms(x, weight, 3.5, 2), want)
    assert torch.allclose(plain.grouped_rms(x, weight, 1.75, 1), x / 3.0 * weight)          # mean square 7.25


def test_the_plain_chunks_and_weights():
    seen = plain.same_chunk(7, 3)
    assert seen[5].tolist() == [False, False, False, True, True, True, False]
    assert seen[3].tolist() == [False, False, False, True, False, False, False]
    assert seen[6].tolist() == [False] * 6 + [True]
    assert torch.equal(plain.same_chunk(5, None), torch.ones(5, 5).tril().bool())
    assert torch.equal(plain.same_chunk(4, 1), torch.eye(4).bool())
    scores = torch.tensor([[0.0, math.log(3.0), 9.0]], dtype=torch.float64)
    weights = plain.sigmoid_weights(scores, torch.tensor([[True, True, False]]), 0.0)
    assert torch.allclose(weights, torch.tensor([[0.5, 0.75, 0.0]], dtype=torch.float64))   # not normalised
    assert abs(float(plain.sigmoid_weights(scores, torch.ones(1, 3).bool(), math.log(2.0))[0, 0]) - 2.0 / 3.0) < 1e-12
    assert torch.equal(plain.bounded(scores, None), scores)
    assert abs(float(plain.bounded(torch.tensor(3.0, dtype=torch.float64), 2.0)) - 2.0 * math.tanh(1.5)) < 1e-12


def test_the_plain_recurrence_is_a_decayed_sum():
    generator = torch.Generator().manual_seed(1)
    q, k = (torch.randn(5, 2, 3, generator=generator, dtype=torch.float64) for _ in range(2))
    v = torch.randn(5, 2, 4, generator=generator, dtype=torch.float64)
    decay = [0.5, 0.0]
    out = plain.fixed_decay_recurrence(q, k, v, decay)
    for head in range(2):
        for t in range(5):
            want = sum((decay[head] ** (t - j)) * float(q[t, head] @ k[j, head]) * v[j, head] for j in range(t + 1))
            assert torch.allclose(out[t, head], want)
    state = torch.ones(2, 3, 4, dtype=torch.float64)                    # a state that is carried in
    first = plain.fixed_decay_recurrence(q[:1], k[:1], v[:1], decay, state)
    assert torch.allclose(first[0, 0], out[0, 0] + 0.5 * q[0, 0].sum()) and torch.allclose(first[0, 1], out[0, 1])


def test_the_plain_router_takes_the_bias_into_choice_and_weights():
    generator = torch.Generator().manual_seed(4)
    w = {"router": torch.tensor([[2.0], [1.0], [0.0]], dtype=torch.float64),
         "router.b": torch.tensor([-1.5, 0.0, 0.6], dtype=torch.float64)}            # logits of h = 1: 0.5, 1, 0.6
    for name in ("e0", "e1", "e2", "shared"):
        for kind, shape in (("gate", (4, 1)), ("up", (4, 1)), ("down", (1, 4))):
            w[f"{name}.{kind}"] = torch.randn(*shape, generator=generator, dtype=torch.float64)
    h = torch.ones(1, 1, dtype=torch.float64)
    got = plain.routed(h, w, "", {"router": {"experts": 3, "top": 2}, "shared": {"ff": 4}})
    first = 1.0 / (1.0 + math.exp(-0.4))                                             # experts 1 and 2, 1 before 0.6
    want = first * plain.gated(h, w, "e1.") + (1.0 - first) * plain.gated(h, w, "e2.") + plain.gated(h, w, "shared.")
    assert torch.allclose(got, want)
    z = torch.tensor([0.5, 1.0, 0.6], dtype=torch.float64)
    assert plain.router_choice(z, 2, torch.tensor([0, 1]), margin=0.1).tolist() == [0, 1]    # a close call is taken over
    assert sorted(plain.router_choice(z, 2, torch.tensor([0, 1]), margin=0.01).tolist()) == [1, 2]


def test_the_plain_layer_norms_what_its_sublayers_return():
    """With zero norm weights the stream stays the scaled embedding; the head is the table without the scale."""
    config = configs.SMALL_A
    tensors = configs.tensors(config, 2)
    for name in tensors:
        if name.endswith("norm1") or name.endswith("norm2"):
            tensors[name] = torch.zeros_like(tensors[name])
    streams, tokens = [], [3, 9, 27]
    logits = plain.forward(config, tensors, tokens, streams=streams)
    x = 3.0 * tensors["embed"].double()[tokens]
    assert len(streams) == 4 and all(torch.allclose(stream, x) for stream in streams)
    want = plain.grouped_rms(x, tensors["final.norm"], 1e-5, 4) @ tensors["embed"].double().t()
    assert torch.allclose(logits, want)
